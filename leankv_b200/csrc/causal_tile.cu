// Causal attention of a prompt portion on the fifth-generation tensor cores (bf16 operands, fp32 scores and
// weights). A CTA holds 128 rows, (token, query head) pairs of one kv head, and walks the 64-key tiles they see:
//
//   copy thread     Q once, then K and V tiles by TMA into swizzled shared memory, two buffers each
//   MMA thread      S = Q K^T into tensor memory, two buffers, a tile ahead of O += P V with P from tensor memory
//   128 row threads a thread a row: mask, running maximum, exponentials; P goes back over S as two bf16 numbers per
//                   weight (16 bits), so two products per V tile. At the end the rows leave through shared
//                   memory, a warp a row, so that the gate is read and the output written in whole lines.
//
// Two CTAs share an SM and fill each other's waits. O stays in tensor memory; it is rescaled only when a row's
// maximum grows by more than 2^kSlack. Tiles start at positions that are multiples of 64 and rings are
// multiples of 128 slots, so a tile never wraps.

#include <algorithm>

#include "causal_attn.cuh"
#include "tma.cuh"

namespace leankv {
namespace {

constexpr int kTile = 128;                       // rows of a CTA
constexpr int kKeys = 64;                        // keys of a tile
constexpr int kThreads = 192;
constexpr uint32_t kBlock = kTile * 128;         // 128 rows of 64 columns: 16 KB
constexpr uint32_t kKeyBlock = kKeys * 128;      // 64 keys of 64 columns: 8 KB
constexpr float kSlack = 8.f;

struct TileArgs {
    CUtensorMap q, k, shared, v;
    const float* gate;
    bf16* out;
    int32_t* status;
    int gate_ld, out_ld, rows, start, size, vec;
    int heads, rep, tq;                          // query heads, per kv head, tokens of a CTA
    int dim_pad, shared_pad, vdim, vdim_pad;
    int k_base, k_ring, s_ring, v_from_k;
    int nb1, nb2, nbv;                           // 64-column blocks
    uint32_t q_box, tmem_cols;
    float c;                                     // scale * log2(e)
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Two floats at a time.
struct Two { float x, y; };
__device__ __forceinline__ Two fma2(Two a, Two b, Two c) {
    Two d;
    asm("{\n\t.reg .b64 a, b, c, d;\n\t"
        "mov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tmov.b64 c, {%6, %7};\n\t"
        "fma.rn.f32x2 d, a, b, c;\n\tmov.b64 {%0, %1}, d;\n\t}"
        : "=f"(d.x), "=f"(d.y)
        : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
    return d;
}
__device__ __forceinline__ Two add2(Two a, Two b) {
    Two d;
    asm("{\n\t.reg .b64 a, b, d;\n\t"
        "mov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\t"
        "add.rn.f32x2 d, a, b;\n\tmov.b64 {%0, %1}, d;\n\t}"
        : "=f"(d.x), "=f"(d.y)
        : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

enum { kQ, kO, kKFull, kKFree = kKFull + 2, kVFull = kKFree + 2, kS = kVFull + 2, kP = kS + 2, kPV = kP + 2, kBars = kPV + 2 };

__global__ void __launch_bounds__(kThreads, 2) causal_tile_kernel(const __grid_constant__ TileArgs p) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ __align__(8) uint64_t s_bar[kBars];
    __shared__ uint32_t s_tmem;
    pdl_begin();
    const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
    const uint32_t base = (umma::smem_addr(raw) + 1023u) & ~1023u;
    const int nbk = p.nb1 + p.nb2;
    const uint32_t k_bytes = nbk * kKeyBlock, v_bytes = p.v_from_k ? k_bytes : p.nbv * kKeyBlock;      // of a buffer
    const uint32_t sq = base, sk = sq + nbk * kBlock, sv = p.v_from_k ? sk : sk + 2 * k_bytes;
    // barrier pairs: tile j uses b + (j & 1), in its phase j / 2
    auto bar = [&](int b) { return umma::smem_addr(&s_bar[b]); };
    auto wait = [&](int b, int j) { return umma::bar_wait(bar(b + (j & 1)), (j >> 1) & 1); };
    if (tid == 0)
        for (int b = 0; b < kBars; ++b) umma::bar_init_n(bar(b), b == kP || b == kP + 1 ? kTile : 1);
    if (warp == 4) umma::tmem_alloc_n(umma::smem_addr(&s_tmem), p.tmem_cols);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    umma::fence_before_sync();
    __syncthreads();
    umma::fence_after_sync();
    const uint32_t tmem = __shfl_sync(0xffffffffu, s_tmem, 0), tm_s = tmem, tm_o = tmem + kTile;

    const int g = blockIdx.y, q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * p.tq;      // the longest rows first
    const int nt = min(p.tq, p.rows - q0);
    const int lo = first_visible(p.start + q0, p.size), hi = p.start + q0 + nt - 1;
    const int t0 = lo / kKeys, n_tiles = hi / kKeys - t0 + 1;
    bool ok = true;

    if (tid == 128) {                                    // ---- copies ----
        tma::expect(bar(kQ), nbk * p.q_box);
        for (int b = 0; b < nbk; ++b)
            tma::load3(sq + b * kBlock, &p.q, b < p.nb1 ? b * 64 : p.dim_pad + (b - p.nb1) * 64, g * p.rep, q0, bar(kQ));
        int nk = 0, nv = 0;
        for (int j = 0; j < n_tiles; ++j) {
            const int at = (t0 + j) * kKeys, slot = ring_slot(at, p.k_base, p.k_ring), odd = j & 1;
            if (j > 1) ok = wait(p.v_from_k ? kPV : kKFree, j - 2);
            if (!ok) break;
            tma::expect(bar(kKFull + odd), k_bytes);
            for (int b = 0; b < p.nb1; ++b) tma::load3(sk + odd * k_bytes + b * kKeyBlock, &p.k, b * 64, g, slot, bar(kKFull + odd));
            for (int b = 0; b < p.nb2; ++b)
                tma::load3(sk + odd * k_bytes + (p.nb1 + b) * kKeyBlock, &p.shared, b * 64, 0, ring_slot(at, 0, p.s_ring),
                           bar(kKFull + odd));
            ++nk;
            if (p.v_from_k) continue;
            if (j > 1) ok = wait(kPV, j - 2);
            if (!ok) break;
            tma::expect(bar(kVFull + odd), v_bytes);
            for (int b = 0; b < p.nbv; ++b) tma::load3(sv + odd * v_bytes + b * kKeyBlock, &p.v, b * 64, g, slot, bar(kVFull + odd));
            ++nv;
        }
        if (!ok) {                                       // give up only once the copies in flight have landed
            umma::bar_wait(bar(kQ), 0);
            for (int j = max(nk - 2, 0); j < nk; ++j) wait(kKFull, j);
            for (int j = max(nv - 2, 0); j < nv; ++j) wait(kVFull, j);
        }
    } else if (warp == 5) {                              // ---- products: the whole warp waits, one lane issues ----
        constexpr uint32_t idesc_s = tma::idesc_bf16(kKeys, false);
        const uint32_t idesc_o = tma::idesc_bf16(p.vdim_pad, true);
        const uint64_t desc_q = tma::swizzled(sq, 16), desc_k = tma::swizzled(sk, 16), desc_v = tma::swizzled(sv, kKeyBlock);
        auto all = [&](bool done) { return __all_sync(0xffffffffu, done) != 0; };
        // a K = 16 step is 32 bytes further in the rows of a block; descriptors count in 16 bytes
        auto scores = [&](int j) {
            ok = all(wait(kKFull, j));
            if (!ok) return;
            umma::fence_after_sync();
            const uint32_t to = tm_s + (j & 1) * kKeys;
            uint64_t dq = desc_q, dk = desc_k + (j & 1) * (k_bytes >> 4);
            if (umma::elect()) {
                for (int b = 0; b < nbk; ++b, dq += kBlock >> 4, dk += kKeyBlock >> 4) {
                    const int steps = b < p.nb1 ? p.dim_pad / 16 - b * 4 : p.shared_pad / 16 - (b - p.nb1) * 4;
                    umma::mma_f16_n(to, dq, dk, idesc_s, b > 0);
#pragma unroll
                    for (int s = 1; s < 4; ++s)
                        if (s < steps) umma::mma_f16_n(to, dq + 2 * s, dk + 2 * s, idesc_s, 1);
                }
                umma::commit(bar(kS + (j & 1)));
                umma::commit(bar(kKFree + (j & 1)));
            }
            __syncwarp();
        };
        ok = all(umma::bar_wait(bar(kQ), 0));
        for (int j = 0; j < min(2, n_tiles) && ok; ++j) scores(j);
        for (int j = 0; j < n_tiles && ok; ++j) {
            if (!p.v_from_k) ok = all(wait(kVFull, j));
            ok = ok && all(wait(kP, j));
            if (!ok) break;
            umma::fence_after_sync();
            const uint64_t dv = desc_v + (j & 1) * (v_bytes >> 4);
            const uint32_t pa = tm_s + (j & 1) * kKeys;
            if (umma::elect()) {
#pragma unroll
                for (int s = 0; s < kKeys / 16; ++s) {   // 16 keys: high parts, then low parts
                    umma::mma_f16_ts(tm_o, pa + (s >> 1) * 32 + (s & 1) * 8, dv + s * (2048 >> 4), idesc_o, j > 0 || s > 0);
                    umma::mma_f16_ts(tm_o, pa + (s >> 1) * 32 + (s & 1) * 8 + 16, dv + s * (2048 >> 4), idesc_o, 1);
                }
                umma::commit(bar(kPV + (j & 1)));
            }
            __syncwarp();
            if (j + 2 < n_tiles) {                       // its scores go over these weights
                ok = all(wait(kPV, j));
                if (ok) scores(j + 2);
            }
        }
        if (umma::elect()) umma::commit(bar(kO));
        __syncwarp();
        if (!ok) umma::bar_wait(bar(kO), 0);
    } else if (tid < kTile) {                            // ---- rows ----
        const int row0 = warp * 32, used = p.rep * nt;
        const int r = min(tid, used - 1), t = q0 + r / p.rep, h = g * p.rep + r % p.rep, i = p.start + t;
        const long long out_at = (long long)t * p.out_ld + h * p.vdim, gate_at = (long long)t * p.gate_ld + h * p.vdim;
        if (p.gate != nullptr)                           // the row's gate into L2, for the end
            for (int d = 0; d < p.vdim; d += 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.gate + gate_at + d));
        const int see0 = first_visible(i, p.size);
        float m = -1e30f, l = 0.f;
        for (int j = 0; j < n_tiles; ++j) {
            ok = __all_sync(0xffffffffu, wait(kS, j));      // the warp stays together
            if (!ok) break;
            umma::fence_after_sync();
            const int at = (t0 + j) * kKeys;
            const uint32_t tm = tm_s + (j & 1) * kKeys;
            // this row's keys of the tile: from k0 to k1
            const int k0 = see0 - at, k1 = i - at;
            uint32_t s[2][32];
            umma::ld32_async(s[0], tm, row0, 0);
            umma::ld32_async(s[1], tm, row0, 32);
            umma::settle(s[0]);
            umma::settled(s[1]);
            if (__any_sync(0xffffffffu, k0 > 0 || k1 < kKeys - 1)) {
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int x = 0; x < 32; ++x)
                        if (c * 32 + x < k0 || c * 32 + x > k1) s[c][x] = 0xff800000u;      // -inf
            }
            float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int x = 0; x < 32; ++x) top[x & 3] = fmaxf(top[x & 3], __uint_as_float(s[c][x]));
            const float best = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3]));
            const bool raise = best * p.c > m + kSlack;
            if (__any_sync(0xffffffffu, raise)) {
                const float mn = raise ? best * p.c : m, f = ex2(m - mn);
                m = mn;
                l *= f;
                if (j > 0) {
                    ok = __all_sync(0xffffffffu, wait(kPV, j - 1));      // nothing is being added to the outputs
                    if (!ok) break;
                    umma::fence_after_sync();
#pragma unroll 1
                    for (int c = 0; c < p.vdim_pad; c += 32) {
                        uint32_t o[32];
                        umma::ld32(o, tm_o, row0, c);
#pragma unroll
                        for (int x = 0; x < 32; ++x) o[x] = __float_as_uint(__uint_as_float(o[x]) * f);
                        umma::st32(o, tm_o, row0, c);
                    }
                }
            }
            Two sum[2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                uint32_t ph[16], pl[16];
#pragma unroll
                for (int x = 0; x < 32; x += 2) {
                    Two w = fma2({__uint_as_float(s[c][x]), __uint_as_float(s[c][x + 1])}, {p.c, p.c}, {-m, -m});
                    w.x = ex2(w.x);
                    w.y = ex2(w.y);
                    sum[(x >> 1) & 1] = add2(sum[(x >> 1) & 1], w);
                    const uint32_t hi = pack_bf16(w.x, w.y);
                    const Two left = add2(w, {-__uint_as_float(hi << 16), -__uint_as_float(hi & 0xffff0000u)});
                    ph[x / 2] = hi;
                    pl[x / 2] = pack_bf16(left.x, left.y);
                }
                umma::st16_async(ph, tm, row0, c * 32);
                umma::st16_async(pl, tm, row0, c * 32 + 16);
            }
            l += (sum[0].x + sum[0].y) + (sum[1].x + sum[1].y);
            umma::stored();
            umma::fence_before_sync();
            umma::bar_arrive(bar(kP + (j & 1)));
        }
        if (ok) ok = __all_sync(0xffffffffu, umma::bar_wait(bar(kO), 0));
        umma::fence_after_sync();
        // normalised rows to shared memory (all copies and products are done); 16 bytes past a multiple of 128 apart
        const float inv = 1.f / l;
        const int ld = (p.vdim_pad + 31) / 32 * 32 + 4;
        float* rows = reinterpret_cast<float*>(raw + (base - umma::smem_addr(raw)));
#pragma unroll 1
        for (int c = 0; c < p.vdim_pad; c += 32) {
            uint32_t o[32];
            umma::ld32(o, tm_o, row0, c);
#pragma unroll
            for (int x = 0; x < 32; x += 4)
                *reinterpret_cast<float4*>(rows + tid * ld + c + x) =
                    make_float4(__uint_as_float(o[x]) * inv, __uint_as_float(o[x + 1]) * inv, __uint_as_float(o[x + 2]) * inv,
                                __uint_as_float(o[x + 3]) * inv);
        }
        __syncwarp();
        const int n_rows = ok ? min(32, used - row0) : 0;
        auto gated = [](float v, float z) { return __fdividef(v, 1.f + __expf(-z)); };
        if (p.vec) {
            constexpr int kAhead = 8;
#pragma unroll 1
            for (int r0 = 0; r0 < n_rows; r0 += kAhead) {
                bf16* to[kAhead];
                const float* from[kAhead];
#pragma unroll
                for (int x = 0; x < kAhead; ++x) {
                    to[x] = p.out + __shfl_sync(0xffffffffu, out_at, r0 + x);
                    from[x] = p.gate + __shfl_sync(0xffffffffu, gate_at, r0 + x);
                }
#pragma unroll 1
                for (int d = lane * 4; d < p.vdim; d += 128) {
                    float4 z[kAhead];
                    if (p.gate != nullptr)
#pragma unroll
                        for (int x = 0; x < kAhead; ++x) z[x] = *reinterpret_cast<const float4*>(from[x] + d);
#pragma unroll
                    for (int x = 0; x < kAhead; ++x) {
                        float4 v = *reinterpret_cast<const float4*>(rows + (row0 + r0 + x) * ld + d);
                        if (p.gate != nullptr)
                            v = make_float4(gated(v.x, z[x].x), gated(v.y, z[x].y), gated(v.z, z[x].z), gated(v.w, z[x].w));
                        if (r0 + x < n_rows) store4(to[x] + d, v);
                    }
                }
            }
        } else {
            for (int r = 0; r < n_rows; ++r) {
                bf16* to = p.out + __shfl_sync(0xffffffffu, out_at, r);
                const float* from = p.gate + __shfl_sync(0xffffffffu, gate_at, r);
                for (int d = lane; d < p.vdim; d += 32) {
                    const float v = rows[(row0 + r) * ld + d];
                    to[d] = from_f32<bf16>(p.gate != nullptr ? gated(v, from[d]) : v);
                }
            }
        }
    }
    if (!ok && p.status != nullptr) *p.status = 1;
    __syncwarp();
    umma::fence_before_sync();
    __syncthreads();
    if (warp == 4) {
        umma::fence_after_sync();
        umma::tmem_free_n(tmem, p.tmem_cols);
    }
}

}  // namespace

int causal_tile_attend(const leankv_causal_attn_t& a, const void* q, const float* gate, int gate_ld, void* out, int out_ld,
                       int rows, int start, int32_t* status, cudaStream_t st) {
    const int rep = a.heads / a.kv_heads;
    if (a.dtype != LEANKV_DT_BF16 || !(a.scale > 0.f) || rep > kTile || a.vdim_pad > 256 || a.kv_heads > 65535 || a.k_base % kTile ||
        a.k_ring % kTile || (a.shared_dim > 0 && a.s_ring % kTile))
        return LEANKV_EUNSUPPORTED;
    TileArgs p{};
    p.nb1 = (a.dim_pad + 63) / 64;
    p.nb2 = a.shared_dim > 0 ? (a.shared_pad + 63) / 64 : 0;
    p.nbv = (a.vdim_pad + 63) / 64;
    p.v_from_k = a.v == nullptr;
    size_t smem = (size_t)(2 * (p.nb1 + p.nb2) + (p.v_from_k ? 0 : p.nbv)) * kBlock;
    smem = std::max(smem, (size_t)kTile * ((a.vdim_pad + 31) / 32 * 32 + 4) * 4) + 1024;      // tiles, then the rows
    if (smem > 226 * 1024) return LEANKV_EUNSUPPORTED;
    p.tmem_cols = kTile + (a.vdim_pad + 31) / 32 * 32 <= 256 ? 256 : 512;
    if (p.tmem_cols == 512) smem = std::max(smem, (size_t)116 * 1024);       // tensor memory for one CTA per SM
    p.gate = gate;
    p.gate_ld = gate_ld;
    p.out = static_cast<bf16*>(out);
    p.out_ld = out_ld;
    p.status = status;
    p.vec = a.vdim % 4 == 0 && out_ld % 4 == 0 && aligned16(out) && (!gate || (gate_ld % 4 == 0 && aligned16(gate)));
    p.rows = rows;
    p.start = start;
    p.size = a.size;
    p.heads = a.heads;
    p.rep = rep;
    p.tq = kTile / rep;
    p.dim_pad = a.dim_pad;
    p.shared_pad = a.shared_dim > 0 ? a.shared_pad : 0;
    p.vdim = a.vdim;
    p.vdim_pad = a.vdim_pad;
    p.k_base = a.k_base;
    p.k_ring = a.k_ring;
    p.s_ring = a.s_ring;
    p.q_box = 128u * rep * p.tq;
    p.c = a.scale * 1.4426950408889634f;
    const cuuint64_t dq = a.dim_pad + p.shared_pad, G = a.kv_heads, H = a.heads;
    const auto map = [](CUtensorMap* m, const void* base, cuuint64_t d, cuuint64_t h, cuuint64_t n, cuuint32_t bh, cuuint32_t bn) {
        const cuuint64_t dims[3] = {d, h, n}, strides[2] = {d, d * h};
        const cuuint32_t box[3] = {(cuuint32_t)tma::kBoxCols, bh, bn};
        return tma::make_map(m, base, 3, dims, strides, box);
    };
    int rc = map(&p.q, q, dq, H, rows, rep, p.tq);
    if (!rc) rc = map(&p.k, a.k, a.dim_pad, G, a.k_rows, 1, kKeys);
    if (!rc && p.nb2) rc = map(&p.shared, a.shared, a.shared_pad, 1, a.s_ring, 1, kKeys);
    if (!rc && a.v) rc = map(&p.v, a.v, a.vdim_pad, G, a.k_rows, 1, kKeys);
    if (rc) return rc;
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(causal_tile_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    LEANKV_CUDA_TRY(launch_kernel(causal_tile_kernel, dim3((rows + p.tq - 1) / p.tq, a.kv_heads), dim3(kThreads), smem, st, p));
    return LEANKV_OK;
}

}  // namespace leankv
