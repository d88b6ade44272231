// One decode step of causal attention over a ring of keys, split over the keys. A CTA takes up to 16 query heads of one
// kv head and a range of key tiles, which come by asynchronous copies through a few stages; the first are on their
// way before the launch ahead has finished. The CTAs of a cluster merge their outputs through distributed
// shared memory, each a slice of the columns. A long sequence takes several clusters per head block: there the
// last cluster to finish a slice merges the clusters' results, in cluster order.
//
// Three ways to walk the tiles (Walk): up to 128 value columns, every warp for itself, 16 keys at a time, with scores
// and weights in registers; more columns, the CTA together on 64 keys, a warp a share of the columns; fp32, the same
// on FMA units. The first two use tensor cores (16 heads x 8 keys, 16 heads x 8 columns): queries and softmax weights
// enter as two bf16 numbers each, so a 32-bit query meets the stored keys exactly.

#include <algorithm>

#include <cooperative_groups.h>

#include "causal_attn.cuh"
#include "decode_frame.cuh"

namespace leankv {
namespace {

namespace cg = cooperative_groups;

constexpr int kHeads = 16;                // query heads of a CTA
constexpr int kMaxStages = 4;
constexpr int kMaxCols = 1024;            // value columns
constexpr int kMaxPairs = 512;            // rotated pairs
constexpr int kMaxCluster = 16;           // non-portable; 8 where the device does not place 16
constexpr int kTilesPerUnit = 4;          // a further cluster joins when a warp / CTA would have more tiles

enum class Walk { kWarps, kColumns, kFma };
constexpr int kWarpCols = 128;            // value columns of Walk::kWarps
__host__ __device__ constexpr int tile_of(Walk w) { return w == Walk::kWarps ? 16 : w == Walk::kColumns ? 64 : 32; }
__host__ __device__ constexpr int warps_of(Walk w) { return w == Walk::kWarps ? 4 : 8; }           // of a CTA
__host__ __device__ constexpr int units_of(Walk w) { return w == Walk::kWarps ? 4 : 1; }           // that take tiles, per CTA
template <Walk W> struct TypeOf { using T = bf16; };
template <> struct TypeOf<Walk::kFma> { using T = float; };

// Shared-memory plan in bytes. Row lengths are 16 bytes past a multiple of 128, so that the eight rows of a matrix
// fragment fall into different banks.
struct StepPlan {
    int k_row, v_row, stages, stage_bytes;             // bytes of a key row (own part, then shared), of a value row
    int q, q_row, s, p, stat, factor, trig, fresh, stage, total;
    __host__ __device__ static constexpr int row(int bytes) { return (bytes + 127) / 128 * 128 + 16; }
    StepPlan() = default;
    StepPlan(const leankv_causal_attn_t& a, Walk w, int limit) {
        const int es = a.dtype == LEANKV_DT_BF16 ? 2 : 4, kd = a.dim_pad + a.shared_pad, tile = tile_of(w);
        k_row = row(kd * es);
        v_row = a.v != nullptr ? row(a.vdim_pad * es) : 0;
        int o = 0;
        const auto take = [&](int n) { const int at = o; o += (n + 127) / 128 * 128; return at; };
        q_row = es == 2 ? k_row : kd * 4;
        q = take(kHeads * q_row * (es == 2 ? 2 : 1));   // high parts, then low parts
        s = take(w == Walk::kWarps ? warps_of(w) * kHeads * 8 : kHeads * (tile + 4) * 4);      // scores; maxima and sums of the warps
        p = take(w == Walk::kColumns ? kHeads * row(tile * 2) * 2 : 0);
        stat = take(kHeads * 4 * 4);                    // maximum, sum, rescale factor
        factor = take(kHeads * kMaxCluster * 4 + kHeads * 8);
        trig = take(kMaxPairs * 8);
        fresh = take(k_row + v_row);
        stage = o;
        stage_bytes = (tile * (k_row + v_row) + 127) / 128 * 128;                          // of a unit
        stages = std::min((limit - o) / (stage_bytes * units_of(w)), kMaxStages);
        const int out = kHeads * a.vdim_pad * 4;        // the outputs of a unit take its stages' place
        if (stages * stage_bytes < out) stages = 0;
        total = o + stages * stage_bytes * units_of(w);
    }
};

struct StepArgs {
    leankv_causal_attn_t a;
    leankv_causal_step_t s;
    StepPlan plan;
    int blocks, cluster, clusters;        // head blocks per kv head, CTAs of a cluster, clusters of a head block
    float* part;                          // [head block][cluster][kHeads][vdim_pad]
    float* ml;                            // [head block][cluster][rank][kHeads][2]
    unsigned* tickets;                    // [head block][rank]
};

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
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

// All but the `newer` youngest copy groups of this thread have landed.
__device__ __forceinline__ void wait_copies(int newer) {
    switch (newer) {
        case 0: asm volatile("cp.async.wait_group 0;" ::: "memory"); break;
        case 1: asm volatile("cp.async.wait_group 1;" ::: "memory"); break;
        case 2: asm volatile("cp.async.wait_group 2;" ::: "memory"); break;
        default: asm volatile("cp.async.wait_group 3;" ::: "memory"); break;
    }
}

// NP: 16-column pieces of the values that a warp accumulates at most (tensor cores).
template <Walk W, int NP>
__global__ void __launch_bounds__(32 * warps_of(W), W == Walk::kWarps ? 2 : 1) causal_step_kernel(const __grid_constant__ StepArgs p) {
    using T = typename TypeOf<W>::T;
    extern __shared__ __align__(128) unsigned char sm[];
    __shared__ float s_tmp[32];
    __shared__ int s_last;
    constexpr bool HALF = sizeof(T) == 2, WARPS = W == Walk::kWarps;
    constexpr int KT = tile_of(W), UNITS = units_of(W), kWarps = warps_of(W), kThreads = 32 * kWarps;
    const leankv_causal_attn_t& a = p.a;
    const StepPlan& pl = p.plan;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int gb = blockIdx.y, g = gb / p.blocks, hb = gb % p.blocks, rep = a.heads / a.kv_heads;
    const int h0 = g * rep + hb * kHeads, nh = min(kHeads, rep - hb * kHeads);
    const int C = p.cluster, rank = blockIdx.x % C, cluster = blockIdx.x / C;
    const int i = p.s.state[kPos], lo = first_visible(i, a.size), tiles = (i - lo) / KT + 1;
    const int active = max(1, min(p.clusters, (tiles + C * UNITS * kTilesPerUnit - 1) / (C * UNITS * kTilesPerUnit)));
    if (cluster >= active) {
        pdl_begin();
        return;
    }
    // tiles j0 .. j1 - 1 of this unit; the last unit has the last tile
    const unsigned unit = (cluster * C + rank) * UNITS + (WARPS ? warp : 0), n_units = active * C * UNITS;
    const int j0 = (int)((unsigned)tiles * unit / n_units), j1 = (int)((unsigned)tiles * (unit + 1) / n_units);
    const int kd = a.dim_pad + a.shared_pad;
    const T* K = static_cast<const T*>(a.k);
    const T* V = static_cast<const T*>(a.v);
    const T* S = static_cast<const T*>(a.shared);

    // tile j into its stage (a lane a 16-byte column, the rows in turn); the position of this step is not in the ring yet
    constexpr int E16 = 16 / (int)sizeof(T);
    const int c_own = a.dim_pad / E16, c_key = kd / E16, c_all = c_key + (V != nullptr ? a.vdim_pad / E16 : 0);
    unsigned char* stage0 = sm + pl.stage + (WARPS ? warp * pl.stages * pl.stage_bytes : 0);
    auto fetch = [&](int j) {
        if (j < j1) {
            const int first = lo + j * KT, cnt = min(KT, i - first), r0 = WARPS ? 0 : warp;
            const uint32_t kb = smem_addr(stage0 + (j - j0) % pl.stages * pl.stage_bytes);
            const int k_slot = ring_slot(first, a.k_base, a.k_ring), s_slot = a.shared_dim > 0 ? ring_slot(first, 0, a.s_ring) : 0;
            for (int c = lane; c < c_all; c += 32) {
                const T* src;
                int step, slot, ring, row;
                uint32_t dst = kb;
                if (c < c_own) {
                    src = K + (size_t)g * a.dim_pad + c * E16;
                    step = a.kv_heads * a.dim_pad, slot = k_slot, ring = a.k_ring, row = pl.k_row, dst += c * 16;
                } else if (c < c_key) {
                    src = S + (c - c_own) * E16;
                    step = a.shared_pad, slot = s_slot, ring = a.s_ring, row = pl.k_row, dst += c * 16;
                } else {
                    src = V + (size_t)g * a.vdim_pad + (c - c_key) * E16;
                    step = a.kv_heads * a.vdim_pad, slot = k_slot, ring = a.k_ring, row = pl.v_row;
                    dst += KT * pl.k_row + (c - c_key) * 16;
                }
                slot += r0;
                dst += r0 * row;
                for (int r = r0; r < cnt; r += WARPS ? 1 : kWarps) {
                    if (slot >= ring) slot -= ring;       // a window fits into the ring once
                    copy16(dst, src + (size_t)slot * step);
                    slot += WARPS ? 1 : kWarps;
                    dst += (WARPS ? 1 : kWarps) * row;
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int x = 0; x < pl.stages; ++x) fetch(j0 + x);
    float* s_sin = reinterpret_cast<float*>(sm + pl.trig);
    float* s_cos = s_sin + kMaxPairs;
    for (int x = tid; x < max(p.s.rot_own, p.s.rot_shared) / 2; x += kThreads)
        sincosf((float)i * __ldg(p.s.rate + x), &s_sin[x], &s_cos[x]);
    pdl_begin();
    __syncthreads();

    // ---- queries, and the new key / value row ----
    const float c = a.scale * 1.4426950408889634f;        // scores in units of log2
    auto pair_of = [&](const float* x, int d, int dim) {
        return make_float2(d < dim ? __ldcg(x + d) : 0.f, d + 1 < dim ? __ldcg(x + d + 1) : 0.f);
    };
    auto turned = [&](float2 v, int d, int rot) { return d < rot ? turn(v.x, v.y, s_sin[d >> 1], s_cos[d >> 1]) : v; };
    auto pair_at = [&](const float* x, int d, int dim, int rot) { return turned(pair_of(x, d, dim), d, rot); };
    constexpr int kBatch = 6;                             // loads in flight per thread
    for (int e0 = tid; e0 < kHeads * (kd / 2); e0 += kBatch * kThreads) {
        float2 in[kBatch];
#pragma unroll
        for (int x = 0; x < kBatch; ++x) {
            const int e = e0 + x * kThreads, h = e / (kd / 2), d = (e - h * (kd / 2)) * 2;
            in[x] = make_float2(0.f, 0.f);
            if (h < nh)
                in[x] = d < a.dim_pad ? pair_of(p.s.q + (size_t)(h0 + h) * p.s.q_stride, d, a.dim)
                                      : pair_of(p.s.q_shared + (size_t)(h0 + h) * p.s.qs_stride, d - a.dim_pad, a.shared_dim);
        }
#pragma unroll
        for (int x = 0; x < kBatch; ++x) {
            const int e = e0 + x * kThreads, h = e / (kd / 2), d = (e - h * (kd / 2)) * 2;
            if (h >= kHeads) break;
            const float2 v = d < a.dim_pad ? turned(in[x], d, p.s.rot_own) : turned(in[x], d - a.dim_pad, p.s.rot_shared);
            if constexpr (HALF) {
                uint32_t hi, low;
                split_bf16(v.x, v.y, hi, low);
                *reinterpret_cast<uint32_t*>(sm + pl.q + h * pl.q_row + d * 2) = hi;
                *reinterpret_cast<uint32_t*>(sm + pl.q + (kHeads + h) * pl.q_row + d * 2) = low;
            } else {
                *reinterpret_cast<float2*>(sm + pl.q + h * pl.q_row + d * 4) = v;
            }
        }
    }
    const bool newest = rank == C - 1 && cluster == active - 1;      // this CTA's range ends with the new position
    T* fresh = reinterpret_cast<T*>(sm + pl.fresh);
    if (newest) {
        float f = 1.f;
        const float* kn = p.s.k_new + (size_t)g * a.dim;
        if (p.s.k_gain != nullptr) {
            float ss = 0.f;
            for (int d = tid; d < a.dim; d += kThreads) {
                const float v = __ldcg(kn + d);
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
                v = make_float2(d < a.dim ? __ldcg(kn + d) * f * __ldg(p.s.k_gain + d) : 0.f,
                                d + 1 < a.dim ? __ldcg(kn + d + 1) * f * __ldg(p.s.k_gain + d + 1) : 0.f);
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
                const T v = from_f32<T>(d < a.vdim ? __ldcg(p.s.v_new + (size_t)g * a.vdim + d) : 0.f);
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
    // the new row into row cnt - 1 of the last tile, and zeros behind it
    auto put_new_row = [&](unsigned char* kt, unsigned char* vt, int cnt, int id, int ids) {
        const int words = (KT - cnt + 1) * (pl.k_row / 4), words_v = V != nullptr ? (KT - cnt + 1) * (pl.v_row / 4) : 0;
        for (int e = id; e < words; e += ids)
            reinterpret_cast<uint32_t*>(kt + (cnt - 1) * pl.k_row)[e] =
                e * 4 < kd * (int)sizeof(T) ? reinterpret_cast<const uint32_t*>(fresh)[e] : 0u;
        for (int e = id; e < words_v; e += ids)
            reinterpret_cast<uint32_t*>(vt + (cnt - 1) * pl.v_row)[e] =
                e * 4 < a.vdim_pad * (int)sizeof(T) ? reinterpret_cast<const uint32_t*>(sm + pl.fresh + pl.k_row)[e] : 0u;
    };
    const int v_row = V != nullptr ? pl.v_row : pl.k_row;
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
    if constexpr (WARPS) {
        float m[2] = {-1e30f, -1e30f}, l[2] = {0.f, 0.f};           // of heads lane / 4 and lane / 4 + 8
        for (int j = j0; j < j1; ++j) {
            const int cnt = min(KT, i + 1 - lo - j * KT);
            unsigned char* kt = stage0 + (j - j0) % pl.stages * pl.stage_bytes;
            unsigned char* vt = V != nullptr ? kt + KT * pl.k_row : kt;
            wait_copies(pl.stages - 1);
            if (j == tiles - 1) put_new_row(kt, vt, cnt, lane, 32);
            __syncwarp();
            float hi[2][4] = {}, low[2][4] = {};                    // keys 0-7, 8-15
            const uint32_t qa = smem_addr(sm + pl.q) + (lane & 15) * pl.q_row + (lane >> 4) * 16;
            const uint32_t ka = smem_addr(kt) + ((lane & 7) + (lane >> 4) * 8) * pl.k_row + ((lane >> 3) & 1) * 16;
#pragma unroll 4
            for (int d = 0; d < kd; d += 16) {
                uint32_t b[4], qh[4], ql[4];
                ldmatrix4(b, ka + d * 2);
                ldmatrix4(qh, qa + d * 2);
                ldmatrix4(ql, qa + kHeads * pl.q_row + d * 2);
                mma_bf16(hi[0], qh[0], qh[1], qh[2], qh[3], b[0], b[1]);
                mma_bf16(hi[1], qh[0], qh[1], qh[2], qh[3], b[2], b[3]);
                mma_bf16(low[0], ql[0], ql[1], ql[2], ql[3], b[0], b[1]);
                mma_bf16(low[1], ql[0], ql[1], ql[2], ql[3], b[2], b[3]);
            }
            float best[2] = {m[0], m[1]}, f[2];
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int k = y * 8 + (lane & 3) * 2 + (x & 1);
                    hi[y][x] = k < cnt ? (hi[y][x] + low[y][x]) * c : -INFINITY;
                    best[x >> 1] = fmaxf(best[x >> 1], hi[y][x]);
                }
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                best[x] = fmaxf(best[x], __shfl_xor_sync(0xffffffffu, best[x], 1));
                best[x] = fmaxf(best[x], __shfl_xor_sync(0xffffffffu, best[x], 2));
                f[x] = exp2f(m[x] - best[x]);
                m[x] = best[x];
                l[x] *= f[x];
            }
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    hi[y][x] = exp2f(hi[y][x] - m[x >> 1]);
                    l[x >> 1] += hi[y][x];
                }
            uint32_t wh[4], wl[4];                                  // the weights as an operand: 16 heads x 16 keys
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int x = 0; x < 2; ++x) split_bf16(hi[y][2 * x], hi[y][2 * x + 1], wh[2 * y + x], wl[2 * y + x]);
            const uint32_t va = smem_addr(vt) + (lane & 15) * v_row + (lane >> 4) * 16;
#pragma unroll
            for (int x = 0; x < NP; ++x) {
                if (x * 16 >= a.vdim_pad) break;
                uint32_t b[4];                            // keys 0-7, 8-15 of columns 0-7, then of columns 8-15
                ldmatrix4_t(b, va + x * 32);
#pragma unroll
                for (int y = 0; y < 2; ++y) {
#pragma unroll
                    for (int z = 0; z < 4; ++z) o[x][y][z] *= f[z >> 1];
                    mma_bf16(o[x][y], wh[0], wh[1], wh[2], wh[3], b[2 * y], b[2 * y + 1]);
                    mma_bf16(o[x][y], wl[0], wl[1], wl[2], wl[3], b[2 * y], b[2 * y + 1]);
                }
            }
            __syncwarp();
            fetch(j + pl.stages);                         // this stage is free again
        }
        wait_copies(0);
        // the warps' outputs, to the CTA's maximum, summed in the first warp's place
        float* s_m = s_s;                                 // [warp][maximum, sum][kHeads]
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
            l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
            if ((lane & 3) == 0) {
                s_m[warp * 2 * kHeads + (lane >> 2) + 8 * x] = m[x];
                s_m[(warp * 2 + 1) * kHeads + (lane >> 2) + 8 * x] = l[x];
            }
        }
        __syncthreads();
        float f[2], best[2] = {-1e30f, -1e30f}, sum[2] = {0.f, 0.f};
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float* at = s_m + (lane >> 2) + 8 * x;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) best[x] = fmaxf(best[x], at[w * 2 * kHeads]);
#pragma unroll
            for (int w = 0; w < kWarps; ++w) sum[x] = fmaf(exp2f(at[w * 2 * kHeads] - best[x]), at[(w * 2 + 1) * kHeads], sum[x]);
            f[x] = exp2f(m[x] - best[x]);
            if (warp == 0 && (lane & 3) == 0) {
                stat[(lane >> 2) + 8 * x] = best[x];
                stat[kHeads + (lane >> 2) + 8 * x] = sum[x];
            }
        }
        float* mine = reinterpret_cast<float*>(stage0);
#pragma unroll
        for (int x = 0; x < NP; ++x) {
            if (x * 16 >= a.vdim_pad) break;
#pragma unroll
            for (int y = 0; y < 2; ++y)
#pragma unroll
                for (int z = 0; z < 2; ++z)
                    *reinterpret_cast<float2*>(mine + ((lane >> 2) + z * 8) * a.vdim_pad + x * 16 + y * 8 + (lane & 3) * 2) =
                        make_float2(o[x][y][2 * z] * f[z], o[x][y][2 * z + 1] * f[z]);
        }
        __syncthreads();
        const int next = pl.stages * pl.stage_bytes / 16;
        float4* sum4 = reinterpret_cast<float4*>(sm + pl.stage);
        for (int e = tid; e < nh * a.vdim_pad / 4; e += kThreads) {
            float4 t = sum4[e];
#pragma unroll
            for (int w = 1; w < kWarps; ++w) {
                const float4 v = sum4[e + w * next];
                t.x += v.x; t.y += v.y; t.z += v.z; t.w += v.w;
            }
            sum4[e] = t;
        }
    } else {
        for (int j = j0; j < j1; ++j) {
            const int cnt = min(KT, i + 1 - lo - j * KT);
            unsigned char* kt = stage0 + (j - j0) % pl.stages * pl.stage_bytes;
            unsigned char* vt = V != nullptr ? kt + KT * pl.k_row : kt;
            wait_copies(pl.stages - 1);
            if (j == tiles - 1) put_new_row(kt, vt, cnt, tid, kThreads);
            __syncthreads();
            // scores
            if constexpr (HALF) {
                float acc[4] = {0.f, 0.f, 0.f, 0.f}, acc2[4] = {0.f, 0.f, 0.f, 0.f};
                const uint32_t qa = smem_addr(sm + pl.q) + (lane & 15) * pl.q_row + (lane >> 4) * 16;
                const uint32_t ka = smem_addr(kt) + (warp * 8 + (lane & 7)) * pl.k_row + (lane >> 3) * 16;
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
                const uint32_t pa = smem_addr(sm + pl.p) + (lane & 15) * PROW + (lane >> 4) * 16;
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
                    const uint32_t va = smem_addr(vt) + (lane & 15) * v_row + col * 2 + (lane >> 4) * 16;
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
            fetch(j + pl.stages);                             // this stage is free again
        }
        wait_copies(0);
        float* s_o = reinterpret_cast<float*>(sm + pl.stage);
        auto put = [&](int h, int d, float v) { s_o[h * a.vdim_pad + d] = v; };
        if constexpr (HALF) {
#pragma unroll
            for (int x = 0; x < NP; ++x) {
                const int col = (warp + x * kWarps) * 16;
                if (col >= a.vdim_pad) break;
#pragma unroll
                for (int y = 0; y < 2; ++y)
#pragma unroll
                    for (int z = 0; z < 2; ++z)
                        *reinterpret_cast<float2*>(s_o + ((lane >> 2) + z * 8) * a.vdim_pad + col + y * 8 + (lane & 3) * 2) =
                            make_float2(o[x][y][2 * z], o[x][y][2 * z + 1]);
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
    }

    // ---- merge: every CTA of the cluster has its outputs in shared memory and takes a slice of the columns ----
    float* s_o = reinterpret_cast<float*>(sm + pl.stage);             // [kHeads][vdim_pad]
    auto cl = cg::this_cluster();
    cl.sync();
    float* factor = reinterpret_cast<float*>(sm + pl.factor);         // [kHeads][C]: to the cluster's maximum
    float* top = factor + kHeads * kMaxCluster;                       // [kHeads] maximum, sum of the cluster
    for (int e = tid; e < kHeads * C; e += kThreads) {                // the C lanes of a head are neighbours, C 8 or 16
        const int h = e / C, r = e - h * C;
        const float* from = cl.map_shared_rank(stat, r);
        const float m = h < nh ? from[h] : -1e30f, l = h < nh ? from[kHeads + h] : 0.f;
        float best = m;
        for (int x = C / 2; x > 0; x /= 2) best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, x));
        const float f = exp2f(m - best);
        float sum = f * l;
        for (int x = C / 2; x > 0; x /= 2) sum += __shfl_xor_sync(0xffffffffu, sum, x);
        factor[h * C + r] = active == 1 ? f / sum : f;
        if (r == 0) {
            top[h] = best;
            top[kHeads + h] = sum;
        }
    }
    __syncthreads();
    const int v4 = a.vdim_pad / 4, e_lo = nh * v4 * rank / C, e_hi = nh * v4 * (rank + 1) / C;
    auto finish = [&](int e, float4 t) {
        const int h = e / v4, d = (e - h * v4) * 4, at = (h0 + h) * a.vdim + d;
        const float v[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
            if (d + x < a.vdim) p.s.out[at + x] = p.s.gate != nullptr ? v[x] * sigmoid_f32(__ldcg(p.s.gate + at + x)) : v[x];
    };
    float* part = p.part + (size_t)gb * p.clusters * kHeads * a.vdim_pad;
    for (int e = e_lo + tid; e < e_hi; e += kThreads) {
        const int h = e / v4;
        float4 v[kMaxCluster], t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int r = 0; r < kMaxCluster; ++r) v[r] = reinterpret_cast<const float4*>(cl.map_shared_rank(s_o, r < C ? r : 0))[e];
#pragma unroll
        for (int r = 0; r < kMaxCluster; ++r) {
            const float f = r < C ? factor[h * C + r] : 0.f;
            t.x = fmaf(f, v[r].x, t.x); t.y = fmaf(f, v[r].y, t.y); t.z = fmaf(f, v[r].z, t.z); t.w = fmaf(f, v[r].w, t.w);
        }
        if (active == 1) finish(e, t);
        else reinterpret_cast<float4*>(part + (size_t)cluster * kHeads * a.vdim_pad)[e] = t;
    }
    if (active > 1) {
        float* ml = p.ml + ((size_t)gb * p.clusters * C + rank) * kHeads * 2;
        const size_t ml_step = (size_t)C * kHeads * 2;
        if (tid < 2 * kHeads) ml[cluster * ml_step + tid] = top[tid];
        __threadfence();
        __syncthreads();
        unsigned* ticket = p.tickets + gb * C + rank;
        if (tid == 0) s_last = atomicAdd(ticket, 1u) == (unsigned)active - 1;
        __syncthreads();
        if (s_last) {
            __threadfence();
            if (tid == 0) *ticket = 0;
            for (int e = e_lo + tid; e < e_hi; e += kThreads) {
                const int h = e / v4;
                float best = -1e30f, l = 0.f;
                float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
                for (int x = 0; x < active; ++x) best = fmaxf(best, __ldcg(ml + x * ml_step + h));
#pragma unroll 4
                for (int x = 0; x < active; ++x) {
                    const float f = exp2f(__ldcg(ml + x * ml_step + h) - best);
                    const float4 v = __ldcg(reinterpret_cast<const float4*>(part + (size_t)x * kHeads * a.vdim_pad) + e);
                    l = fmaf(f, __ldcg(ml + x * ml_step + kHeads + h), l);
                    t.x = fmaf(f, v.x, t.x); t.y = fmaf(f, v.y, t.y); t.z = fmaf(f, v.z, t.z); t.w = fmaf(f, v.w, t.w);
                }
                finish(e, make_float4(t.x / l, t.y / l, t.z / l, t.w / l));
            }
        }
    }
    cl.sync();                                            // the other CTAs still read this one's shared memory
}

struct Grid {
    Walk walk;
    StepPlan plan;
    int blocks, clusters;
    size_t part, ml, tickets, bytes;
};

// Clusters of a head block: enough CTAs to fill the device, at most one per kTilesPerUnit tiles of each unit. Sized for
// clusters of 8; with 16 half as many are launched.
int plan_grid(const leankv_causal_attn_t& a, int max_pos, Grid& gr) {
    if (a.vdim_pad > kMaxCols) return LEANKV_ELIMIT;
    int limit = 112 * 1024, per_sm = 2;                  // two CTAs per SM for warps on their own
    gr.walk = a.dtype != LEANKV_DT_BF16 ? Walk::kFma : a.vdim_pad <= kWarpCols ? Walk::kWarps : Walk::kColumns;
    gr.plan = StepPlan(a, gr.walk, limit);
    if (gr.walk == Walk::kWarps && gr.plan.stages < 1) gr.walk = Walk::kColumns;
    if (gr.walk != Walk::kWarps) {
        per_sm = 1;
        limit = 226 * 1024;
        gr.plan = StepPlan(a, gr.walk, limit);
    }
    if (gr.plan.stages < 1) return LEANKV_ELIMIT;
    gr.blocks = (a.heads / a.kv_heads + kHeads - 1) / kHeads;
    const int keys = std::min(a.size, max_pos), per = 8 * units_of(gr.walk) * kTilesPerUnit * tile_of(gr.walk);
    const int groups = a.kv_heads * gr.blocks;
    gr.clusters = std::max(1, std::min((keys + per - 1) / per, sm_count() * per_sm / (8 * groups)));
    const auto take = [&](size_t n) { const size_t at = gr.bytes; gr.bytes += round_up(n, 256); return at; };
    gr.bytes = 0;
    gr.tickets = take((size_t)groups * kMaxCluster * 4);
    gr.ml = take((size_t)groups * gr.clusters * kMaxCluster * kHeads * 2 * 4);
    gr.part = take((size_t)groups * gr.clusters * kHeads * a.vdim_pad * 4);
    return LEANKV_OK;
}

template <Walk W, int NP>
int launch_step(StepArgs p, cudaStream_t st) {
    const size_t smem = p.plan.total;
    const dim3 block(32 * warps_of(W));
    const auto kernel = causal_step_kernel<W, NP>;
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    const int groups = p.a.kv_heads * p.blocks;
    for (const int clusters8 = p.clusters;;) {
        p.cluster = p.cluster == kMaxCluster ? 8 : kMaxCluster;
        p.clusters = p.cluster == 8 ? clusters8 : (clusters8 + 1) / 2;
        const dim3 grid(p.cluster * p.clusters, groups);
        if (p.cluster > 8) {                             // does a cluster of this size fit this device, often enough?
            cudaLaunchConfig_t cfg = {};
            cfg.gridDim = grid;
            cfg.blockDim = block;
            cfg.dynamicSmemBytes = smem;
            cudaLaunchAttribute attr[1];
            attr[0].id = cudaLaunchAttributeClusterDimension;
            attr[0].val.clusterDim.x = p.cluster;
            attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
            cfg.attrs = attr;
            cfg.numAttrs = 1;
            int fits = 0;
            if (cudaOccupancyMaxActiveClusters(&fits, kernel, &cfg) != cudaSuccess || fits < p.clusters * groups) {
                (void)cudaGetLastError();
                continue;
            }
        }
        LEANKV_CUDA_TRY(launch_cluster_kernel_ex(true, dim3(p.cluster), kernel, grid, block, smem, st, p));
        return LEANKV_OK;
    }
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" size_t leankv_causal_step_workspace_bytes(const leankv_causal_attn_t* a, int max_pos) {
    Grid gr;
    return check_causal(a) || max_pos <= 0 || plan_grid(*a, max_pos, gr) ? 0 : gr.bytes;
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
    rc = plan_grid(*a, s->max_pos, gr);
    if (rc) return rc;
    if (!s->ws || s->ws_bytes < gr.bytes) return LEANKV_EWORKSPACE;
    StepArgs p{};
    p.a = *a;
    p.s = *s;
    p.blocks = gr.blocks;
    p.clusters = gr.clusters;
    p.plan = gr.plan;
    char* ws = static_cast<char*>(s->ws);
    p.tickets = reinterpret_cast<unsigned*>(ws + gr.tickets);
    p.ml = reinterpret_cast<float*>(ws + gr.ml);
    p.part = reinterpret_cast<float*>(ws + gr.part);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    switch (gr.walk) {
        case Walk::kFma: return launch_step<Walk::kFma, 1>(p, st);
        case Walk::kWarps: return a->vdim_pad <= 64 ? launch_step<Walk::kWarps, 4>(p, st) : launch_step<Walk::kWarps, 8>(p, st);
        default: break;
    }
    if (a->vdim_pad <= 128) return launch_step<Walk::kColumns, 1>(p, st);
    return a->vdim_pad <= 512 ? launch_step<Walk::kColumns, 4>(p, st)
                                          : launch_step<Walk::kColumns, kMaxCols / 128>(p, st);
}
