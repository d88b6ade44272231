// Window + pooled-block attention of a prompt portion on tensor cores (bf16): one CTA per eight queries, all heads.
//
// The weights of all heads of a (query, key) pair meet in the mix across heads, so they have to be in one CTA,
// normalised, before the mix. Pass 1 computes every head's softmax statistics, pass 2 the scores again and from
// them normalised weights, the mix and the product with the values. Scores and outputs are computed transposed
// (keys or value columns as the 16 rows of an MMA tile, the eight queries as its columns), which keeps the
// output accumulators of 32 heads x 128 columns in the registers of eight warps. Weights enter the mix as two
// bf16 numbers each (16 bits); after it they are rounded once for the product with the values.
//
// A warp owns HPW query heads of one kv head; with few heads, several warps share a head and take every KS-th
// key tile. Key rows go straight from L2 to registers, value rows through shared memory because their
// fragments need the transposing load.

#include <algorithm>

#include "window_pool.cuh"

namespace leankv {
namespace {

constexpr int kWarps = 8;
constexpr int kThreads = 32 * kWarps;
constexpr int kQ = 8;           // queries per CTA
constexpr int kMaxNb = 4;       // blocks of 32 dimensions

struct TileParams {
    leankv_window_pool_t a;
    const bf16* q;
    bf16* out;
    int out_ld, rows, start;
    float out_scale;
    int hs, ks;                 // head slots, key splits
    int nb;                     // 32-blocks of dim_pad, the last may be half
    int off_p, off_pm, off_v, off_t, off_stat, p_row, p_key, pm_q, pm_h, v_row;      // bytes, words for pm_*
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// HPW query heads per warp, NB blocks of 32 dimensions and DVT tiles of 16 value columns; EXACT: the sizes are
// those, otherwise at most those.
template <int HPW, int NB, int DVT, bool EXACT>
__global__ void __launch_bounds__(kThreads, 1) window_pool_tile_kernel(const __grid_constant__ TileParams p) {
    extern __shared__ __align__(128) unsigned char smem[];
    pdl_begin();
    const leankv_window_pool_t& a = p.a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int H = a.heads, G = a.kv_heads, rep = H / G, KS = p.ks;
    const int dp = EXACT ? NB * 32 : a.dim_pad, vp = EXACT ? DVT * 16 : a.vdim_pad, nb = EXACT ? NB : p.nb;
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kQ;           // the longest rows first
    const int nq = min(kQ, p.rows - q0), i0 = p.start + q0, iL = i0 + nq - 1;
    const VisibleKeys first(i0, a.size, a.pool), last(iL, a.size, a.pool);
    const int tok0 = first.w0, ntok = iL - tok0 + 1, TB = (last.n_blk + 15) / 16, NT = TB + (ntok + 15) / 16;
    const int hslot = warp % p.hs, ks = warp / p.hs, h0 = hslot * HPW, kv = h0 / rep;
    const bool worker = ks < KS;
    const float c = a.scale * 1.4426950408889634f;

    // queries in fragment order: [head][block][lane] 16 bytes (query lane / 4, dimensions 8 (lane % 4) ..)
    for (int e = tid; e < H * nb * 32; e += kThreads) {
        const int l = e & 31, b = (e >> 5) % nb, h = (e >> 5) / nb, d = b * 32 + (l & 3) * 8;
        const int row = min(q0 + (l >> 2), p.rows - 1);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (d < dp) v = *reinterpret_cast<const uint4*>(p.q + ((size_t)row * H + h) * dp + d);
        reinterpret_cast<uint4*>(smem)[e] = v;
    }
    // mixing matrix in fragment order, high then low parts: [row tile][column tile][2][lane] 16 bytes; lane t holds
    // input heads 4 t .. 4 t + 3 of the column tile
    const int MT = (H + 15) / 16;
    for (int e = tid; e < MT * MT * 32; e += kThreads) {
        const int l = e & 31, kt = (e >> 5) % MT, mt = (e >> 5) / MT;
        const int r = mt * 16 + (l >> 2), col = kt * 16 + (l & 3) * 4;
        auto at = [&](int h, int x) {
            if (h >= H || x >= H) return 0.f;
            return a.talk != nullptr ? __ldg(a.talk + h * H + x) : (h == x ? 1.f : 0.f);
        };
        uint32_t hi[4], lo[4];
        split_bf16(at(r, col), at(r, col + 1), hi[0], lo[0]);
        split_bf16(at(r + 8, col), at(r + 8, col + 1), hi[1], lo[1]);
        split_bf16(at(r, col + 2), at(r, col + 3), hi[2], lo[2]);
        split_bf16(at(r + 8, col + 2), at(r + 8, col + 3), hi[3], lo[3]);
        uint4* dst = reinterpret_cast<uint4*>(smem + p.off_t) + (e >> 5) * 64 + l;
        dst[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        dst[32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    // weights of padding heads stay zero
    for (int e = tid; e < (p.off_pm - p.off_p) / 4; e += kThreads) reinterpret_cast<uint32_t*>(smem + p.off_p)[e] = 0;
    __syncthreads();

    // this thread's two queries
    int iq[2], w0q[2], nbq[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        iq[x] = i0 + min(2 * t + x, nq - 1);
        const VisibleKeys v(iq[x], a.size, a.pool);
        w0q[x] = v.w0;
        nbq[x] = v.n_blk;
    }
    const bf16* k_ring = static_cast<const bf16*>(a.k_ring);
    const bf16* k_pool = static_cast<const bf16*>(a.k_pool);

    // row of a tile's key r (clamped to the keys that exist): index into the pooled blocks or the ring
    struct TileRows { bool pooled; int n, slot0; };
    const int ring0 = tok0 % a.ring;
    auto rows_of = [&](int tile) {
        TileRows tr;
        tile = min(tile, NT - 1);
        tr.pooled = tile < TB;
        const int base = (tr.pooled ? tile : tile - TB) * 16;
        tr.n = (tr.pooled ? last.n_blk : ntok) - base - 1;
        tr.slot0 = tr.pooled ? base : ring0 + base;              // the tokens of a portion fit into the ring once
        return tr;
    };
    auto index_of = [&](const TileRows& tr, int r) {
        int s = tr.slot0 + min(r, tr.n);
        if (!tr.pooled && s >= a.ring) s -= a.ring;
        return s;
    };
    struct Keys { uint4 x0[NB], x1[NB]; };
    const size_t k_stride = (size_t)G * dp;
    auto load_keys = [&](int tile, Keys& k) {
        const TileRows tr = rows_of(tile);
        const bf16* src = (tr.pooled ? k_pool : k_ring) + (size_t)kv * dp + t * 8;
        const bf16* r0 = src + index_of(tr, g) * k_stride;
        const bf16* r1 = src + index_of(tr, g + 8) * k_stride;
#pragma unroll
        for (int b = 0; b < NB; ++b)
            if (b < nb) {
                const bool on = b * 32 + t * 8 < dp;
                k.x0[b] = on ? *reinterpret_cast<const uint4*>(r0 + b * 32) : make_uint4(0, 0, 0, 0);
                k.x1[b] = on ? *reinterpret_cast<const uint4*>(r1 + b * 32) : make_uint4(0, 0, 0, 0);
            }
    };
    const uint4* q_frag = reinterpret_cast<const uint4*>(smem) + h0 * nb * 32 + lane;
    float s[HPW][4];
    auto score = [&](int tile, const Keys& k) {        // -inf where the query does not see the key
#pragma unroll
        for (int h = 0; h < HPW; ++h)
#pragma unroll
            for (int x = 0; x < 4; ++x) s[h][x] = 0.f;
        float s2[4] = {};          // with one head, a second accumulator halves the chain of dependent products
#pragma unroll
        for (int b = 0; b < NB; ++b)
            if (b < nb) {
                uint4 y[HPW];
#pragma unroll
                for (int h = 0; h < HPW; ++h) y[h] = q_frag[(h * nb + b) * 32];
#pragma unroll
                for (int h = 0; h < HPW; ++h) mma_bf16(s[h], k.x0[b].x, k.x1[b].x, k.x0[b].y, k.x1[b].y, y[h].x, y[h].y);
#pragma unroll
                for (int h = 0; h < HPW; ++h)
                    mma_bf16(HPW == 1 ? s2 : s[h], k.x0[b].z, k.x1[b].z, k.x0[b].w, k.x1[b].w, y[h].z, y[h].w);
            }
        if (HPW == 1)
#pragma unroll
            for (int x = 0; x < 4; ++x) s[0][x] += s2[x];
        const bool pooled = tile < TB;
        const int base = pooled ? tile * 16 : tok0 + (tile - TB) * 16;
        const bool all = tile < NT && (pooled ? base + 15 < first.n_blk : base >= last.w0 && base + 15 <= i0);
        if (!all) {
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int at = base + g + (x < 2 ? 0 : 8), qx = x & 1;
                const bool see = tile < NT && (pooled ? at < nbq[qx] : at >= w0q[qx] && at <= iq[qx]);
#pragma unroll
                for (int h = 0; h < HPW; ++h) s[h][x] = see ? s[h][x] : -INFINITY;
            }
        }
    };

    // ---- pass 1: log2 of the softmax denominators ----
    float lse[HPW][2];
    {
        // m: a reference exponent per (head, query) and lane, raised only when a score exceeds it by kSlack: the
        // exponentials stay below 2^kSlack and most tiles need no rescaling
        constexpr float kSlack = 12.f;
        float m[HPW][2], l[HPW][2];
#pragma unroll
        for (int h = 0; h < HPW; ++h) m[h][0] = m[h][1] = -1e30f, l[h][0] = l[h][1] = 0.f;
        auto count = [&]() {
            bool raise = false;
#pragma unroll
            for (int h = 0; h < HPW; ++h)
#pragma unroll
                for (int x = 0; x < 2; ++x) raise = raise || fmaxf(s[h][x], s[h][x + 2]) * c > m[h][x] + kSlack;
            if (__any_sync(0xffffffffu, raise)) {
#pragma unroll
                for (int h = 0; h < HPW; ++h)
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const float mn = fmaxf(m[h][x], fmaxf(s[h][x], s[h][x + 2]) * c);
                        l[h][x] *= ex2(m[h][x] - mn);
                        m[h][x] = mn;
                    }
            }
#pragma unroll
            for (int h = 0; h < HPW; ++h)
#pragma unroll
                for (int x = 0; x < 4; ++x) l[h][x & 1] += ex2(fmaf(s[h][x], c, -m[h][x & 1]));
        };
        if (worker) {
            Keys ka, kb;
            load_keys(ks, ka);
            load_keys(ks + KS, kb);
#pragma unroll 1
            for (int tile = ks; tile < NT; tile += 2 * KS) {
                score(tile, ka);
                load_keys(tile + 2 * KS, ka);
                count();
                if (tile + KS < NT) {
                    score(tile + KS, kb);
                    load_keys(tile + 3 * KS, kb);
                    count();
                }
            }
        }
        float* stat = reinterpret_cast<float*>(smem + p.off_stat);       // [KS][H][8][2]
#pragma unroll
        for (int h = 0; h < HPW; ++h)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
#pragma unroll
                for (int o = 4; o < 32; o *= 2) {
                    const float mo = __shfl_xor_sync(0xffffffffu, m[h][x], o), lo = __shfl_xor_sync(0xffffffffu, l[h][x], o);
                    const float mn = fmaxf(m[h][x], mo);
                    l[h][x] = l[h][x] * ex2(m[h][x] - mn) + lo * ex2(mo - mn);
                    m[h][x] = mn;
                }
                if (worker && g == 0) {
                    float* d = stat + (((size_t)ks * H + h0 + h) * kQ + 2 * t + x) * 2;
                    d[0] = m[h][x];
                    d[1] = l[h][x];
                }
            }
        __syncthreads();
        if (worker) {
#pragma unroll
            for (int h = 0; h < HPW; ++h)
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const float* d = stat + ((size_t)(h0 + h) * kQ + 2 * t + x) * 2;
                    float mm = -1e30f, ll = 0.f;
                    for (int k = 0; k < KS; ++k) mm = fmaxf(mm, d[(size_t)k * H * kQ * 2]);
                    for (int k = 0; k < KS; ++k)
                        ll += d[(size_t)k * H * kQ * 2 + 1] * ex2(d[(size_t)k * H * kQ * 2] - mm);
                    lse[h][x] = mm + log2f(ll);
                }
        }
    }

    // ---- pass 2 ----
    float o[HPW][DVT][4];
#pragma unroll
    for (int h = 0; h < HPW; ++h)
#pragma unroll
        for (int m = 0; m < DVT; ++m)
#pragma unroll
            for (int x = 0; x < 4; ++x) o[h][m][x] = 0.f;
    const int dvt = vp / 16;
    // value rows of a (key split, kv head) are shared by the warps of that head's queries, in two buffers
    const int sharers = rep / HPW, v_buf = 16 * p.v_row, v_half = KS * G * v_buf;
    const uint32_t vaddr = (uint32_t)__cvta_generic_to_shared(smem + p.off_v) + (ks * G + kv) * v_buf;
    uint32_t* pm = reinterpret_cast<uint32_t*>(smem + p.off_pm);
    Keys keys;
    if (worker) load_keys(ks, keys);
    const int v_per = vp / 8, v_id = hslot % sharers * 32 + lane, v_r0 = v_id / v_per, v_c0 = v_id % v_per;
    const int v_dr = sharers * 32 / v_per, v_dc = sharers * 32 % v_per;
    const size_t v_stride = (size_t)G * vp;
#pragma unroll 1
    for (int base = 0, half = 0; base < NT; base += KS, half ^= 1) {
        const int tile = base + ks;
        const uint32_t v_now = vaddr + half * v_half;
        if (worker) {
            {       // this tile's values start their way
                const TileRows tr = rows_of(tile);
                const bf16* src = static_cast<const bf16*>(tr.pooled ? a.v_pool : a.v_ring) + (size_t)kv * vp;
                int r = v_r0, ch = v_c0;
                while (r < 16) {
                    const bf16* from = src + index_of(tr, r) * v_stride + ch * 8;
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(v_now + r * p.v_row + ch * 16), "l"(from)
                                 : "memory");
                    r += v_dr;
                    ch += v_dc;
                    if (ch >= v_per) { ch -= v_per; ++r; }
                }
                asm volatile("cp.async.commit_group;" ::: "memory");
            }
            score(tile, keys);
            if (base + KS < NT) load_keys(tile + KS, keys);
            // normalised weights as high + low bf16: [key][query][head / 4] {4 high, 4 low}
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                float w[HPW];
#pragma unroll
                for (int h = 0; h < HPW; ++h) w[h] = ex2(fmaf(s[h][x], c, -lse[h][x & 1]));
                const int key = ks * 16 + g + (x < 2 ? 0 : 8), qq = 2 * t + (x & 1);
                unsigned char* dst = smem + p.off_p + key * p.p_key + qq * p.p_row + (h0 >> 2) * 16;
                if constexpr (HPW == 4) {
                    uint4 v;
                    split_bf16(w[0], w[1], v.x, v.z);
                    split_bf16(w[2], w[3], v.y, v.w);
                    *reinterpret_cast<uint4*>(dst) = v;
                } else if constexpr (HPW == 2) {
                    uint32_t hi, lo;
                    split_bf16(w[0], w[1], hi, lo);
                    *reinterpret_cast<uint32_t*>(dst + (h0 & 2) * 2) = hi;
                    *reinterpret_cast<uint32_t*>(dst + 8 + (h0 & 2) * 2) = lo;
                } else {
#pragma unroll
                    for (int h = 0; h < HPW; ++h) {
                        const int hh = h0 + h;
                        unsigned char* d = smem + p.off_p + key * p.p_key + qq * p.p_row + (hh >> 2) * 16 + (hh & 3) * 2;
                        const bf16 hi = from_f32<bf16>(w[h]);
                        *reinterpret_cast<bf16*>(d) = hi;
                        *reinterpret_cast<bf16*>(d + 8) = from_f32<bf16>(w[h] - to_f32(hi));
                    }
                }
            }
        }
        __syncthreads();
        // mix across heads, two keys and 16 output heads at a time: [head][query][key] bf16
        for (int e = warp; e < 8 * KS * MT; e += kWarps) {
            const int pair = e / MT, mt = e - pair * MT;
            const unsigned char* src = smem + p.off_p + (size_t)pair * 2 * p.p_key + g * p.p_row + t * 16;
            float d0[2][4] = {}, d1[2][4] = {};
#pragma unroll 2
            for (int kt = 0; kt < MT; ++kt) {
                const uint4* tf = reinterpret_cast<const uint4*>(smem + p.off_t) + (mt * MT + kt) * 64 + lane;
                const uint4 ah = tf[0], al = tf[32];
                const uint4 b0 = *reinterpret_cast<const uint4*>(src + kt * 64);
                const uint4 b1 = *reinterpret_cast<const uint4*>(src + p.p_key + kt * 64);
                mma_bf16(d0[0], ah.x, ah.y, ah.z, ah.w, b0.x, b0.y);
                mma_bf16(d1[0], ah.x, ah.y, ah.z, ah.w, b1.x, b1.y);
                mma_bf16(d0[1], ah.x, ah.y, ah.z, ah.w, b0.z, b0.w);
                mma_bf16(d1[1], ah.x, ah.y, ah.z, ah.w, b1.z, b1.w);
                mma_bf16(d0[1], al.x, al.y, al.z, al.w, b0.x, b0.y);
                mma_bf16(d1[1], al.x, al.y, al.z, al.w, b1.x, b1.y);
            }
            uint32_t* dst = pm + (mt * 16 + g) * p.pm_h + 2 * t * p.pm_q + pair;
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (mt * 16 + g + (x < 2 ? 0 : 8) < H)
                    dst[(x < 2 ? 0 : 8) * p.pm_h + (x & 1) * p.pm_q] =
                        pack_bf16(d0[0][x] + d0[1][x], d1[0][x] + d1[1][x]);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (worker) {
            uint32_t b[HPW][2];
#pragma unroll
            for (int h = 0; h < HPW; ++h) {
                const uint32_t* w = pm + (h0 + h) * p.pm_h + g * p.pm_q + ks * 8 + t;
                b[h][0] = w[0];
                b[h][1] = w[4];
            }
            const int mi = lane >> 3, r = (lane & 7) + (mi >= 2 ? 8 : 0);
            const uint32_t from = v_now + r * p.v_row + (mi & 1) * 16;
#pragma unroll
            for (int m = 0; m < DVT; ++m)
                if (m < dvt) {
                    uint32_t a0, a1, a2, a3;
                    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                                 : "=r"(a0), "=r"(a1), "=r"(a2), "=r"(a3)
                                 : "r"(from + m * 32));
#pragma unroll
                    for (int h = 0; h < HPW; ++h) mma_bf16(o[h][m], a0, a1, a2, a3, b[h][0], b[h][1]);
                }
        }
    }

    // ---- outputs: sum over the key splits, through the value buffers' space ----
    if (KS > 1) {
        float* red = reinterpret_cast<float*>(smem + p.off_v);           // [head][vp][8 queries]
        for (int k = 1; k < KS; ++k) {
            __syncthreads();
            if (ks == k) {
#pragma unroll
                for (int h = 0; h < HPW; ++h)
#pragma unroll
                    for (int m = 0; m < DVT; ++m)
                        if (m < dvt)
#pragma unroll
                            for (int x = 0; x < 4; ++x)
                                red[((h0 + h) * vp + m * 16 + g + (x < 2 ? 0 : 8)) * kQ + 2 * t + (x & 1)] = o[h][m][x];
            }
            __syncthreads();
            if (ks == 0) {
#pragma unroll
                for (int h = 0; h < HPW; ++h)
#pragma unroll
                    for (int m = 0; m < DVT; ++m)
                        if (m < dvt)
#pragma unroll
                            for (int x = 0; x < 4; ++x)
                                o[h][m][x] += red[((h0 + h) * vp + m * 16 + g + (x < 2 ? 0 : 8)) * kQ + 2 * t + (x & 1)];
            }
        }
    }
    if (ks == 0) {
#pragma unroll
        for (int h = 0; h < HPW; ++h)
#pragma unroll
            for (int m = 0; m < DVT; ++m)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int d = m * 16 + g + (x < 2 ? 0 : 8), qq = 2 * t + (x & 1);
                    if (d < a.vdim && qq < nq)
                        p.out[(size_t)(q0 + qq) * p.out_ld + (h0 + h) * a.vdim + d] = from_f32<bf16>(o[h][m][x] * p.out_scale);
                }
    }
}

template <int HPW, int NB, int DVT, bool EXACT>
int launch(const TileParams& p, size_t smem, cudaStream_t st) {
    auto kernel = window_pool_tile_kernel<HPW, NB, DVT, EXACT>;
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    LEANKV_CUDA_TRY(launch_kernel(kernel, dim3((p.rows + kQ - 1) / kQ), dim3(kThreads), smem, st, p));
    return LEANKV_OK;
}

template <int HPW>
int launch_sizes(const TileParams& p, size_t smem, cudaStream_t st) {
    const int dp = p.a.dim_pad, vp = p.a.vdim_pad;
    if (dp == 64 && vp == 64) return launch<HPW, 2, 4, true>(p, smem, st);
    if (dp == 128 && vp == 128) return launch<HPW, 4, 8, true>(p, smem, st);
    return launch<HPW, 4, 8, false>(p, smem, st);
}

}  // namespace

int window_pool_tile_attend(const leankv_window_pool_t& a, const void* q, void* out, int out_ld, float out_scale, int rows,
                            int start, cudaStream_t st) {
    const int rep = a.heads / a.kv_heads;
    if (a.dtype != LEANKV_DT_BF16 || a.dim_pad > 32 * kMaxNb || a.vdim_pad > 128) return LEANKV_EUNSUPPORTED;
    // the most heads per warp: fewer warps read the same key and value rows, and more key tiles go in parallel
    int hpw = 4;
    while (hpw > 1 && rep % hpw != 0) --hpw;
    if (a.heads / hpw > kWarps) return LEANKV_EUNSUPPORTED;
    TileParams p{};
    p.a = a;
    p.q = static_cast<const bf16*>(q);
    p.out = static_cast<bf16*>(out);
    p.out_ld = out_ld;
    p.out_scale = out_scale;
    p.rows = rows;
    p.start = start;
    p.hs = a.heads / hpw;
    p.ks = kWarps / p.hs;
    p.nb = (a.dim_pad + 31) / 32;
    const int hp = (a.heads + 15) / 16 * 16, mt = hp / 16;
    p.p_row = hp * 4 + 16;              // fragment rows a few banks apart
    p.p_key = kQ * p.p_row + 16;
    p.pm_q = 8 * p.ks + 4;
    p.pm_h = kQ * p.pm_q + 1;
    p.v_row = a.vdim_pad * 2 + 16;
    int at = a.heads * p.nb * 512;
    const auto take = [&](int bytes) { const int o = at; at += (bytes + 127) / 128 * 128; return o; };
    p.off_t = take(mt * mt * 1024);
    p.off_stat = take(p.ks * a.heads * kQ * 8);
    p.off_p = take(16 * p.ks * p.p_key);
    p.off_pm = take(a.heads * p.pm_h * 4);
    p.off_v = take(std::max(2 * p.ks * a.kv_heads * 16 * p.v_row, p.ks > 1 ? a.heads * a.vdim_pad * kQ * 4 : 0));
    if (at > 227 * 1024) return LEANKV_EUNSUPPORTED;
    switch (hpw) {
        case 1: return launch_sizes<1>(p, at, st);
        case 2: return launch_sizes<2>(p, at, st);
        case 3: return launch_sizes<3>(p, at, st);
        default: return launch_sizes<4>(p, at, st);
    }
}

}  // namespace leankv
