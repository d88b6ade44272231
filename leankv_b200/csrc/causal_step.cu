// One decode step of causal attention over a ring of keys, split over the keys. A CTA takes up to 16 query heads of one
// kv head and a range of 64-key tiles: the rows of a tile come by bulk copies through a few stages, so several
// tiles are in flight while one is computed, and the first ones are on their way before the launch ahead has
// finished. The last CTA of a head block to finish merges the partial outputs (in split order) and gates them.
//
// bf16: scores and outputs on tensor cores (16 heads x 8 keys, 16 heads x 8 columns). Queries and softmax weights enter
// as two bf16 numbers each, so a 32-bit query meets the stored keys exactly. fp32: the same walk on FMA units.

#include <algorithm>

#include "causal_attn.cuh"
#include "decode_frame.cuh"
#include "umma.cuh"

namespace leankv {
namespace {

constexpr int kWarps = 8;
constexpr int kThreads = 32 * kWarps;
constexpr int kHeads = 16;                // query heads of a CTA
constexpr int kMaxStages = 4;
constexpr int kMaxCols = 1024;            // value columns
constexpr int kMaxPairs = 512;            // rotated pairs

template <typename T> constexpr int kTileOf = sizeof(T) == 2 ? 64 : 32;      // keys of a tile

// Shared-memory plan in bytes. Row lengths are 16 bytes past a multiple of 128, so that the eight rows of a matrix
// fragment fall into different banks.
struct StepPlan {
    int k_row, v_row, stages, stage_bytes;             // bytes of a key row (own part, then shared), of a value row
    int q, q_row, s, p, stat, trig, fresh, stage, total;
    __host__ __device__ static constexpr int row(int bytes) { return (bytes + 127) / 128 * 128 + 16; }
    __host__ __device__ StepPlan(const leankv_causal_attn_t& a, int tile, int limit) {
        const int es = a.dtype == LEANKV_DT_BF16 ? 2 : 4, kd = a.dim_pad + a.shared_pad;
        k_row = row(kd * es);
        v_row = a.v != nullptr ? row(a.vdim_pad * es) : 0;
        int o = 0;
        const auto take = [&](int n) { const int at = o; o += (n + 127) / 128 * 128; return at; };
        q_row = es == 2 ? k_row : kd * 4;
        q = take(kHeads * q_row * (es == 2 ? 2 : 1));   // high parts, then low parts
        s = take(kHeads * (tile + 4) * 4);
        p = take(kHeads * row(tile * 2) * 2);
        stat = take(kHeads * 4 * 4);                    // maximum, sum, rescale factor
        trig = take(kMaxPairs * 8);
        fresh = take(k_row + v_row);
        stage = o;
        stage_bytes = (tile * (k_row + v_row) + 127) / 128 * 128;
        stages = (limit - o) / stage_bytes;
        if (stages > kMaxStages) stages = kMaxStages;
        total = o + stages * stage_bytes;
    }
};

struct StepArgs {
    leankv_causal_attn_t a;
    leankv_causal_step_t s;
    int blocks, splits, limit;            // head blocks per kv head, splits, shared memory
    float* part;                          // [kv head][block][split][kHeads][vdim_pad]
    float* ml;                            // [kv head][block][split][kHeads][2]
    unsigned* tickets;                    // [kv head][block]
};

__device__ __forceinline__ void bulk_row(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
                 "r"(bytes), "r"(bar)
                 : "memory");
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}

// NP: 16-column pieces of the values that a warp accumulates at most (bf16).
template <typename T, int NP>
__global__ void __launch_bounds__(kThreads, NP <= 1 ? 2 : 1) causal_step_kernel(const __grid_constant__ StepArgs p) {
    extern __shared__ __align__(128) unsigned char sm[];
    __shared__ __align__(8) uint64_t s_bar[kMaxStages];
    __shared__ float s_tmp[32];
    __shared__ int s_last;
    constexpr bool HALF = sizeof(T) == 2;
    constexpr int KT = kTileOf<T>;
    const leankv_causal_attn_t& a = p.a;
    const StepPlan pl(a, KT, p.limit);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = blockIdx.y / p.blocks, hb = blockIdx.y % p.blocks, rep = a.heads / a.kv_heads;
    const int h0 = g * rep + hb * kHeads, nh = min(kHeads, rep - hb * kHeads);
    const int i = p.s.state[kPos], lo = first_visible(i, a.size), n = i + 1 - lo, tiles = (n + KT - 1) / KT;
    const int active = min(p.splits, tiles), split = blockIdx.x;
    if (split >= active) {
        pdl_begin();
        return;
    }
    const int j0 = (int)((long long)tiles * split / active), j1 = (int)((long long)tiles * (split + 1) / active);
    const int kd = a.dim_pad + a.shared_pad;
    const T* K = static_cast<const T*>(a.k);
    const T* V = static_cast<const T*>(a.v);
    const T* S = static_cast<const T*>(a.shared);
    auto bar = [&](int s) { return umma::smem_addr(&s_bar[s]); };
    if (tid < pl.stages) umma::bar_init_n(bar(tid), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    __syncthreads();

    // tile j into its stage; the position of this step is not in the ring yet
    auto fetch = [&](int j) {                             // warp 0
        const int st = (j - j0) % pl.stages, first = lo + j * KT, cnt = min(KT, i - first);       // rows that are in the ring
        const uint32_t row_bytes = (uint32_t)(kd + (V != nullptr ? a.vdim_pad : 0)) * sizeof(T);
        if (lane == 0)
            asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar(st)), "r"((uint32_t)max(cnt, 0) * row_bytes)
                         : "memory");
        __syncwarp();
        const uint32_t kb = umma::smem_addr(sm + pl.stage + st * pl.stage_bytes), vb = kb + KT * pl.k_row;
        for (int r = lane; r < cnt; r += 32) {
            const size_t slot = ring_slot(first + r, a.k_base, a.k_ring);
            bulk_row(kb + r * pl.k_row, K + (slot * a.kv_heads + g) * a.dim_pad, a.dim_pad * sizeof(T), bar(st));
            if (a.shared_dim > 0)
                bulk_row(kb + r * pl.k_row + a.dim_pad * sizeof(T), S + (size_t)ring_slot(first + r, 0, a.s_ring) * a.shared_pad,
                         a.shared_pad * sizeof(T), bar(st));
            if (V != nullptr)
                bulk_row(vb + r * pl.v_row, V + (slot * a.kv_heads + g) * a.vdim_pad, a.vdim_pad * sizeof(T), bar(st));
        }
    };
    int issued = j0;
    for (; issued < j1 && issued < j0 + pl.stages; ++issued)
        if (warp == 0) fetch(issued);
    float* s_sin = reinterpret_cast<float*>(sm + pl.trig);
    float* s_cos = s_sin + kMaxPairs;
    for (int x = tid; x < max(p.s.rot_own, p.s.rot_shared) / 2; x += kThreads)
        sincosf((float)i * __ldg(p.s.rate + x), &s_sin[x], &s_cos[x]);
    pdl_begin();
    __syncthreads();

    // ---- queries, and the new key / value row ----
    const float c = a.scale * 1.4426950408889634f;        // scores in units of log2
    auto pair_at = [&](const float* x, int d, int dim, int rot) {
        float2 v = make_float2(d < dim ? ld_cg_f32(x + d) : 0.f, d + 1 < dim ? ld_cg_f32(x + d + 1) : 0.f);
        return d < rot ? turn(v.x, v.y, s_sin[d >> 1], s_cos[d >> 1]) : v;
    };
    for (int e = tid; e < kHeads * (kd / 2); e += kThreads) {
        const int h = e / (kd / 2), d = (e - h * (kd / 2)) * 2;
        float2 v = make_float2(0.f, 0.f);
        if (h < nh)
            v = d < a.dim_pad ? pair_at(p.s.q + (size_t)(h0 + h) * p.s.q_stride, d, a.dim, p.s.rot_own)
                              : pair_at(p.s.q_shared + (size_t)(h0 + h) * p.s.qs_stride, d - a.dim_pad, a.shared_dim, p.s.rot_shared);
        if constexpr (HALF) {
            uint32_t hi, low;
            split_bf16(v.x, v.y, hi, low);
            *reinterpret_cast<uint32_t*>(sm + pl.q + h * pl.q_row + d * 2) = hi;
            *reinterpret_cast<uint32_t*>(sm + pl.q + (kHeads + h) * pl.q_row + d * 2) = low;
        } else {
            *reinterpret_cast<float2*>(sm + pl.q + h * pl.q_row + d * 4) = v;
        }
    }
    const bool newest = j1 == tiles;                      // this CTA's range ends with the new position
    T* fresh = reinterpret_cast<T*>(sm + pl.fresh);
    if (newest) {
        float f = 1.f;
        const float* kn = p.s.k_new + (size_t)g * a.dim;
        if (p.s.k_gain != nullptr) {
            float ss = 0.f;
            for (int d = tid; d < a.dim; d += kThreads) {
                const float v = ld_cg_f32(kn + d);
                ss = fmaf(v, v, ss);
            }
            f = 1.f / sqrtf(cta_sum(ss, s_tmp) / (float)a.dim + p.s.eps);
        }
        const size_t slot = ring_slot(i, a.k_base, a.k_ring);
        T* k_out = static_cast<T*>(a.k) + (slot * a.kv_heads + g) * a.dim_pad;
        T* s_out = a.shared_dim > 0 ? static_cast<T*>(a.shared) + (size_t)ring_slot(i, 0, a.s_ring) * a.shared_pad : nullptr;
        for (int e = tid; e < kd / 2; e += kThreads) {
            const int d = e * 2;
            const bool own = d < a.dim_pad;
            float2 v;
            if (own && p.s.k_gain != nullptr)
                v = make_float2(d < a.dim ? ld_cg_f32(kn + d) * f * __ldg(p.s.k_gain + d) : 0.f,
                                d + 1 < a.dim ? ld_cg_f32(kn + d + 1) * f * __ldg(p.s.k_gain + d + 1) : 0.f);
            else
                v = own ? pair_at(kn, d, a.dim, p.s.rot_own) : pair_at(p.s.shared_new, d - a.dim_pad, a.shared_dim, p.s.rot_shared);
            fresh[d] = from_f32<T>(v.x);
            fresh[d + 1] = from_f32<T>(v.y);
            if (hb == 0) {
                T* to = own ? k_out + d : s_out + d - a.dim_pad;
                to[0] = from_f32<T>(v.x);
                to[1] = from_f32<T>(v.y);
            }
        }
        if (V != nullptr) {
            T* fv = reinterpret_cast<T*>(sm + pl.fresh + pl.k_row);
            T* v_out = static_cast<T*>(a.v) + (slot * a.kv_heads + g) * a.vdim_pad;
            for (int d = tid; d < a.vdim_pad; d += kThreads) {
                const T v = from_f32<T>(d < a.vdim ? ld_cg_f32(p.s.v_new + (size_t)g * a.vdim + d) : 0.f);
                fv[d] = v;
                if (hb == 0) v_out[d] = v;
            }
        }
    }
    float* stat = reinterpret_cast<float*>(sm + pl.stat);
    if (tid < kHeads) {
        stat[tid] = -1e30f;
        stat[kHeads + tid] = 0.f;
    }
    __syncthreads();

    // ---- the tiles ----
    float* s_s = reinterpret_cast<float*>(sm + pl.s);
    constexpr int SLD = KT + 4;
    constexpr int kColsOfThread = kMaxCols / kThreads;              // columns of a thread (fp32)
    float o[HALF ? NP : 1][2][4], of[HALF ? 1 : kColsOfThread][kHeads];
    if constexpr (HALF) {
#pragma unroll
        for (int x = 0; x < NP; ++x)
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int z = 0; z < 4; ++z) o[x][y][z] = 0.f;
    } else {
#pragma unroll
        for (int x = 0; x < kColsOfThread; ++x)
#pragma unroll
            for (int h = 0; h < kHeads; ++h) of[x][h] = 0.f;
    }
    bool ok = true;
    for (int j = j0; j < j1; ++j) {
        const int st = (j - j0) % pl.stages, round = (j - j0) / pl.stages, first = lo + j * KT, cnt = min(KT, i + 1 - first);
        unsigned char* kt = sm + pl.stage + st * pl.stage_bytes;
        unsigned char* vt = V != nullptr ? kt + KT * pl.k_row : kt;
        const int v_row = V != nullptr ? pl.v_row : pl.k_row;
        ok = ok && umma::bar_wait(bar(st), round & 1);
        if (j == tiles - 1) {                             // the new row, and zeros behind it
            const int words = (KT - cnt + 1) * (pl.k_row / 4), words_v = V != nullptr ? (KT - cnt + 1) * (pl.v_row / 4) : 0;
            for (int e = tid; e < words; e += kThreads)
                reinterpret_cast<uint32_t*>(kt + (cnt - 1) * pl.k_row)[e] =
                    e < pl.k_row / 4 && e * 4 < kd * (int)sizeof(T) ? reinterpret_cast<const uint32_t*>(fresh)[e] : 0u;
            for (int e = tid; e < words_v; e += kThreads)
                reinterpret_cast<uint32_t*>(vt + (cnt - 1) * pl.v_row)[e] =
                    e < pl.v_row / 4 && e * 4 < a.vdim_pad * (int)sizeof(T)
                        ? reinterpret_cast<const uint32_t*>(sm + pl.fresh + pl.k_row)[e]
                        : 0u;
            __syncthreads();
        }
        // scores
        if constexpr (HALF) {
            float acc[4] = {0.f, 0.f, 0.f, 0.f}, acc2[4] = {0.f, 0.f, 0.f, 0.f};
            const uint32_t qa = umma::smem_addr(sm + pl.q) + (lane & 15) * pl.q_row + (lane >> 4) * 16;
            const uint32_t ka = umma::smem_addr(kt) + (warp * 8 + (lane & 7)) * pl.k_row + (lane >> 3) * 16;
            for (int d = 0; d < kd; d += 32) {
                uint32_t b[4], qh[4], ql[4];
                const bool two = d + 16 < kd;             // the last block may hold 16 dimensions
                ldmatrix4(b, ka + (two || lane < 16 ? d * 2 : d * 2 - 32));
                ldmatrix4(qh, qa + d * 2);
                ldmatrix4(ql, qa + kHeads * pl.q_row + d * 2);
                mma_bf16(acc, qh[0], qh[1], qh[2], qh[3], b[0], b[1]);
                mma_bf16(acc2, ql[0], ql[1], ql[2], ql[3], b[0], b[1]);
                if (two) {
                    ldmatrix4(qh, qa + d * 2 + 32);
                    ldmatrix4(ql, qa + kHeads * pl.q_row + d * 2 + 32);
                    mma_bf16(acc, qh[0], qh[1], qh[2], qh[3], b[2], b[3]);
                    mma_bf16(acc2, ql[0], ql[1], ql[2], ql[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int h = (lane >> 2) + (x < 2 ? 0 : 8), k = warp * 8 + (lane & 3) * 2 + (x & 1);
                s_s[h * SLD + k] = k < cnt ? (acc[x] + acc2[x]) * c : -INFINITY;
            }
        } else {
            for (int k = warp; k < KT; k += kWarps) {
                const float* row = reinterpret_cast<const float*>(kt + k * pl.k_row);
                for (int h = 0; h < nh; ++h) {
                    const float* q = reinterpret_cast<const float*>(sm + pl.q + h * pl.q_row);
                    float t = 0.f;
                    if (k < cnt)
                        for (int d = lane; d < kd; d += 32) t = fmaf(q[d], row[d], t);
                    t = warp_sum(t);
                    if (lane == 0) s_s[h * SLD + k] = k < cnt ? t * c : -INFINITY;
                }
            }
        }
        __syncthreads();
        // softmax: a warp two heads
#pragma unroll
        for (int x = 0; x < kHeads / kWarps; ++x) {
            const int h = warp * (kHeads / kWarps) + x;
            if (h >= nh) continue;
            float v[KT / 32], best = stat[h], l = 0.f;
#pragma unroll
            for (int y = 0; y < KT / 32; ++y) {
                v[y] = s_s[h * SLD + lane * (KT / 32) + y];
                best = fmaxf(best, v[y]);
            }
            best = warp_max(best);
            const float f = exp2f(stat[h] - best);
#pragma unroll
            for (int y = 0; y < KT / 32; ++y) {
                v[y] = exp2f(v[y] - best);
                l += v[y];
            }
            l = warp_sum(l);
            if constexpr (HALF) {
                uint32_t hi, low;
                split_bf16(v[0], v[KT / 32 - 1], hi, low);
                *reinterpret_cast<uint32_t*>(sm + pl.p + h * StepPlan::row(KT * 2) + lane * 4) = hi;
                *reinterpret_cast<uint32_t*>(sm + pl.p + (kHeads + h) * StepPlan::row(KT * 2) + lane * 4) = low;
            } else {
                s_s[h * SLD + lane] = v[0];
            }
            __syncwarp();
            if (lane == 0) {
                stat[h] = best;
                stat[kHeads + h] = stat[kHeads + h] * f + l;
                stat[2 * kHeads + h] = f;
            }
        }
        __syncthreads();
        // outputs
        if constexpr (HALF) {
            constexpr int PROW = StepPlan::row(KT * 2);
            const float f0 = stat[2 * kHeads + (lane >> 2)], f1 = stat[2 * kHeads + (lane >> 2) + 8];
            const uint32_t pa = umma::smem_addr(sm + pl.p) + (lane & 15) * PROW + (lane >> 4) * 16;
            uint32_t wh[KT / 16][4], wl[KT / 16][4];
#pragma unroll
            for (int k = 0; k < KT / 16; ++k) {
                ldmatrix4(wh[k], pa + k * 32);
                ldmatrix4(wl[k], pa + kHeads * PROW + k * 32);
            }
#pragma unroll
            for (int x = 0; x < NP; ++x) {
                const int col = (warp + x * kWarps) * 16;
                if (col >= a.vdim_pad) break;
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    o[x][y][0] *= f0; o[x][y][1] *= f0;
                    o[x][y][2] *= f1; o[x][y][3] *= f1;
                }
                const uint32_t va = umma::smem_addr(vt) + (lane & 15) * v_row + col * 2 + (lane >> 4) * 16;
#pragma unroll
                for (int k = 0; k < KT / 16; ++k) {
                    uint32_t b[4];                        // keys 0-7, 8-15 of columns 0-7, then of columns 8-15
                    ldmatrix4_t(b, va + k * 16 * v_row);
                    mma_bf16(o[x][0], wh[k][0], wh[k][1], wh[k][2], wh[k][3], b[0], b[1]);
                    mma_bf16(o[x][1], wh[k][0], wh[k][1], wh[k][2], wh[k][3], b[2], b[3]);
                    mma_bf16(o[x][0], wl[k][0], wl[k][1], wl[k][2], wl[k][3], b[0], b[1]);
                    mma_bf16(o[x][1], wl[k][0], wl[k][1], wl[k][2], wl[k][3], b[2], b[3]);
                }
            }
        } else {
#pragma unroll
            for (int x = 0; x < kColsOfThread; ++x) {
                const int d = tid + x * kThreads;
                if (d >= a.vdim_pad) break;
#pragma unroll
                for (int h = 0; h < kHeads; ++h)
                    if (h < nh) of[x][h] *= stat[2 * kHeads + h];
                for (int k = 0; k < cnt; ++k) {
                    const float v = reinterpret_cast<const float*>(vt + k * v_row)[d];
#pragma unroll
                    for (int h = 0; h < kHeads; ++h)
                        if (h < nh) of[x][h] = fmaf(s_s[h * SLD + k], v, of[x][h]);
                }
            }
        }
        __syncthreads();
        if (issued < j1) {                                // this stage is free again
            if (warp == 0) {
                umma::fence_operands();
                fetch(issued);
            }
            ++issued;
        }
    }
    if (!ok && p.s.status != nullptr && tid == 0) *p.s.status = 1;

    // ---- partial results, merged by the last CTA of the head block ----
    const int gb = blockIdx.y;
    auto finish = [&](int h, int d, float v) {            // v: normalised
        const int at = (h0 + h) * a.vdim + d;
        if (p.s.gate != nullptr) v *= sigmoid_f32(ld_cg_f32(p.s.gate + at));
        p.s.out[at] = v;
    };
    float* part = p.part + ((size_t)gb * p.splits + split) * kHeads * a.vdim_pad;
    auto put = [&](int h, int d, float v) {
        if (h >= nh || d >= a.vdim) return;
        if (active == 1) finish(h, d, v / stat[kHeads + h]);
        else part[h * a.vdim_pad + d] = v;
    };
    if constexpr (HALF) {
#pragma unroll
        for (int x = 0; x < NP; ++x) {
            const int col = (warp + x * kWarps) * 16;
            if (col >= a.vdim_pad) break;
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int z = 0; z < 4; ++z) put((lane >> 2) + (z < 2 ? 0 : 8), col + y * 8 + (lane & 3) * 2 + (z & 1), o[x][y][z]);
        }
    } else {
#pragma unroll
        for (int x = 0; x < kColsOfThread; ++x) {
            const int d = tid + x * kThreads;
            if (d >= a.vdim_pad) break;
#pragma unroll
            for (int h = 0; h < kHeads; ++h) put(h, d, of[x][h]);
        }
    }
    if (active == 1) return;
    float* ml = p.ml + (size_t)gb * p.splits * kHeads * 2;
    if (tid < nh) {
        ml[(split * kHeads + tid) * 2] = stat[tid];
        ml[(split * kHeads + tid) * 2 + 1] = stat[kHeads + tid];
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(p.tickets + gb, 1u) == (unsigned)active - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) p.tickets[gb] = 0;
    float* factor = reinterpret_cast<float*>(sm + pl.q);            // [nh][active], room checked on the host
    for (int h = warp; h < nh; h += kWarps) {
        float best = -1e30f, l = 0.f;
        for (int s = lane; s < active; s += 32) best = fmaxf(best, __ldcg(ml + (s * kHeads + h) * 2));
        best = warp_max(best);
        for (int s = lane; s < active; s += 32) {
            const float f = exp2f(__ldcg(ml + (s * kHeads + h) * 2) - best);
            factor[h * active + s] = f;
            l += f * __ldcg(ml + (s * kHeads + h) * 2 + 1);
        }
        l = warp_sum(l);
        __syncwarp();
        for (int s = lane; s < active; s += 32) factor[h * active + s] /= l;
    }
    __syncthreads();
    const float* all = p.part + (size_t)gb * p.splits * kHeads * a.vdim_pad;
    const int v4 = a.vdim_pad / 4;
    for (int e = tid; e < nh * v4; e += kThreads) {
        const int h = e / v4, d = (e - h * v4) * 4;
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        const float* src = all + (size_t)h * a.vdim_pad + d;
#pragma unroll 8
        for (int s = 0; s < active; ++s) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * kHeads * a.vdim_pad));
            const float f = factor[h * active + s];
            t.x = fmaf(f, v.x, t.x); t.y = fmaf(f, v.y, t.y); t.z = fmaf(f, v.z, t.z); t.w = fmaf(f, v.w, t.w);
        }
        if (d < a.vdim) finish(h, d, t.x);
        if (d + 1 < a.vdim) finish(h, d + 1, t.y);
        if (d + 2 < a.vdim) finish(h, d + 2, t.z);
        if (d + 3 < a.vdim) finish(h, d + 3, t.w);
    }
}

struct Grid { int blocks, splits, limit; size_t part, ml, tickets, bytes; };

// Splits: enough CTAs to fill the device once (twice where two fit an SM), at most one per tile.
template <typename T>
int plan_grid(const leankv_causal_attn_t& a, int max_pos, Grid& gr) {
    constexpr int KT = kTileOf<T>;
    const int rep = a.heads / a.kv_heads;
    gr.blocks = (rep + kHeads - 1) / kHeads;
    gr.limit = 112 * 1024;                               // two CTAs per SM
    int per_sm = 2;
    if (StepPlan(a, KT, gr.limit).stages < 2) {
        gr.limit = 226 * 1024;
        per_sm = 1;
        if (StepPlan(a, KT, gr.limit).stages < 1) return LEANKV_ELIMIT;
    }
    const int tiles = (std::min(a.size, max_pos) + KT - 1) / KT;
    const StepPlan pl(a, KT, gr.limit);
    const int fit = (pl.stage + pl.stages * pl.stage_bytes) / (kHeads * 4);           // merge factors
    gr.splits = std::max(1, std::min({tiles, sm_count() * per_sm / (a.kv_heads * gr.blocks), fit}));
    const size_t groups = (size_t)a.kv_heads * gr.blocks;
    const auto take = [&](size_t n) { const size_t at = gr.bytes; gr.bytes += round_up(n, 256); return at; };
    gr.bytes = 0;
    gr.tickets = take(groups * 4);
    gr.ml = take(groups * gr.splits * kHeads * 2 * 4);
    gr.part = take(groups * gr.splits * kHeads * a.vdim_pad * 4);
    return LEANKV_OK;
}

int plan(const leankv_causal_attn_t& a, int max_pos, Grid& gr) {
    if (a.vdim_pad > kMaxCols) return LEANKV_ELIMIT;
    return a.dtype == LEANKV_DT_BF16 ? plan_grid<bf16>(a, max_pos, gr) : plan_grid<float>(a, max_pos, gr);
}

template <typename T, int NP>
int launch_step(const StepArgs& p, cudaStream_t st) {
    const size_t smem = StepPlan(p.a, kTileOf<T>, p.limit).total;
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(causal_step_kernel<T, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    LEANKV_CUDA_TRY(launch_kernel_ex(true, causal_step_kernel<T, NP>, dim3(p.splits, p.a.kv_heads * p.blocks), dim3(kThreads), smem, st, p));
    return LEANKV_OK;
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" size_t leankv_causal_step_workspace_bytes(const leankv_causal_attn_t* a, int max_pos) {
    Grid gr;
    return check_causal(a) || max_pos <= 0 || plan(*a, max_pos, gr) ? 0 : gr.bytes;
}

extern "C" int leankv_causal_step(const leankv_causal_attn_t* a, const leankv_causal_step_t* s, void* stream) {
    int rc = check_causal(a);
    if (rc) return rc;
    if (!s || !s->q || !s->k_new || !s->out || !s->state || s->max_pos <= 0 || (a->v && !s->v_new) ||
        (a->shared_dim > 0 && (!s->q_shared || !s->shared_new)) || s->rot_own < 0 || s->rot_own > a->dim || s->rot_own % 2 ||
        s->rot_shared < 0 || s->rot_shared > a->shared_dim || s->rot_shared % 2 ||
        ((s->rot_own > 0 || s->rot_shared > 0) && !s->rate) || (s->k_gain && (a->kv_heads != 1 || s->rot_own > 0)))
        return LEANKV_EINVAL;
    if (std::max(s->rot_own, s->rot_shared) > 2 * kMaxPairs) return LEANKV_EUNSUPPORTED;
    const int keys = std::min(a->size, s->max_pos);
    if (keys > a->k_ring || (a->shared_dim > 0 && keys > a->s_ring) || a->k_rows < a->k_ring) return LEANKV_ELIMIT;
    Grid gr;
    rc = plan(*a, s->max_pos, gr);
    if (rc) return rc;
    if (!s->ws || s->ws_bytes < gr.bytes) return LEANKV_EWORKSPACE;
    StepArgs p{};
    p.a = *a;
    p.s = *s;
    p.blocks = gr.blocks;
    p.splits = gr.splits;
    p.limit = gr.limit;
    char* ws = static_cast<char*>(s->ws);
    p.tickets = reinterpret_cast<unsigned*>(ws + gr.tickets);
    p.ml = reinterpret_cast<float*>(ws + gr.ml);
    p.part = reinterpret_cast<float*>(ws + gr.part);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a->dtype == LEANKV_DT_F32) return launch_step<float, 1>(p, st);
    if (a->vdim_pad <= 16 * kWarps) return launch_step<bf16, 1>(p, st);
    return a->vdim_pad <= 4 * 16 * kWarps ? launch_step<bf16, 4>(p, st) : launch_step<bf16, kMaxCols / 16 / kWarps>(p, st);
}
