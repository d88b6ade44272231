// One decode step of causal attention over a ring of keys, split over the keys. A CTA takes up to 8 query heads of one
// kv head and a range of key tiles, which come by asynchronous copies through a few stages; the first are on their
// way before the launch ahead has finished. Every CTA of a cluster owns a slice of the outputs and merges it: the
// others write their share of it into its shared memory, one cluster barrier later everything is there. A long
// sequence takes several clusters per head block: there the last cluster to finish a slice merges the clusters'
// results, in cluster order.
//
// Three ways to walk the tiles (Walk): up to 128 value columns, every warp for itself, 16 keys at a time, with scores
// and weights in registers; more columns, the CTA together on 64 keys, a warp a share of the columns; fp32, the same
// on FMA units. The first two use tensor cores (16 keys x 8 heads, 16 columns x 8 heads): queries and softmax weights
// enter as two bf16 numbers each, so a 32-bit query meets the stored keys exactly.

#include <algorithm>

#include <cooperative_groups.h>

#include "causal_attn.cuh"
#include "decode_frame.cuh"

namespace leankv {
namespace {

namespace cg = cooperative_groups;

constexpr int kHeads = 8;                 // query heads of a CTA
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
    int q, q_row, s, p, stat, trig, fresh, inbox, stage, total;
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
        s = take(w == Walk::kWarps ? warps_of(w) * kHeads * 8 : 2 * kHeads * (tile + 4) * 4);      // scores; maxima and sums of the warps
        p = take(w == Walk::kColumns ? kHeads * row(tile * 2) * 2 : 0);
        stat = take(kHeads * 4 * 4);                    // maximum, sum, rescale factor
        // from every CTA of the cluster: maxima and sums, its share of this CTA's slice of the outputs; merge factors
        inbox = take((kMaxCluster * 3 + 2) * kHeads * 4 +
                     (std::min(kHeads, a.heads / a.kv_heads) * (a.vdim_pad / 4) + kMaxCluster) * 16);
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

// Scores of 16 keys (rows at k, k_row bytes apart) with 8 heads (rows at q: high parts, then low parts), dimensions d0 ..
// d1: s[0], s[1] key lane / 4 with heads 2 (lane % 4) and the next one, s[2], s[3] key lane / 4 + 8.
__device__ __forceinline__ void tile_scores(float (&s)[4], uint32_t k, uint32_t q, int k_row, int d0, int d1) {
    const int lane = threadIdx.x & 31;
    float low[4] = {0.f, 0.f, 0.f, 0.f};
    s[0] = s[1] = s[2] = s[3] = 0.f;
    const uint32_t ka = k + (lane & 15) * k_row + (lane >> 4) * 16;
    const uint32_t qa = q + ((lane & 7) + (lane >> 4) * kHeads) * k_row + ((lane >> 3) & 1) * 16;
#pragma unroll 4
    for (int d = d0; d < d1; d += 16) {
        uint32_t x[4], y[4];
        ldmatrix4(x, ka + d * 2);
        ldmatrix4(y, qa + d * 2);
        mma_bf16(s, x[0], x[1], x[2], x[3], y[0], y[1]);
        mma_bf16(low, x[0], x[1], x[2], x[3], y[2], y[3]);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) s[x] += low[x];
}
// An 8 x 8 matrix of 16-bit numbers, two per lane, transposed.
__device__ __forceinline__ uint32_t transpose8(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
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
    const int C = p.cluster, rank = blockIdx.x % C, gb = blockIdx.x / C, cluster = blockIdx.y;      // idle clusters come last
    const int g = gb / p.blocks, hb = gb % p.blocks, rep = a.heads / a.kv_heads;
    const int h0 = g * rep + hb * kHeads, nh = min(kHeads, rep - hb * kHeads);
    const int i = p.s.state[kPos], lo = first_visible(i, a.size), tiles = (i - lo) / KT + 1;
    const int active = max(1, min(p.clusters, (tiles + C * UNITS * kTilesPerUnit - 1) / (C * UNITS * kTilesPerUnit)));
    if (cluster >= active) return;        // without waiting: the clusters that work do
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
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // this CTA runs: its inbox may be written
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
    constexpr int kBatch = 5;                             // loads in flight per thread
    float2 in[kBatch];
    auto load_queries = [&](int e0) {
#pragma unroll
        for (int x = 0; x < kBatch; ++x) {
            const int e = e0 + x * kThreads, h = e / (kd / 2), d = (e - h * (kd / 2)) * 2;
            in[x] = make_float2(0.f, 0.f);
            if (h < nh)
                in[x] = d < a.dim_pad ? pair_of(p.s.q + (size_t)(h0 + h) * p.s.q_stride, d, a.dim)
                                      : pair_of(p.s.q_shared + (size_t)(h0 + h) * p.s.qs_stride, d - a.dim_pad, a.shared_dim);
        }
    };
    auto put_queries = [&](int e0) {
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
    };
    load_queries(tid);
    // this CTA's slice of the outputs, and its gate
    const int v4 = a.vdim_pad / 4, slice = (nh * v4 + C - 1) / C, mine = rank * slice + tid;      // float4s
    const int n_mine = min(slice, nh * v4 - rank * slice);
    auto place_of = [&](int e, int& at) {                 // of float4 e: first element, elements that exist
        const int h = e / v4, d = (e - h * v4) * 4;
        at = (h0 + h) * a.vdim + d;
        return min(4, a.vdim - d);
    };
    float gate[4] = {1.f, 1.f, 1.f, 1.f};
    if (p.s.gate != nullptr && tid < n_mine) {
        int at;
        const int cnt = place_of(mine, at);
#pragma unroll
        for (int x = 0; x < 4; ++x)
            if (x < cnt) gate[x] = __ldcg(p.s.gate + at + x);
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
    put_queries(tid);
    for (int e0 = tid + kBatch * kThreads; e0 < kHeads * (kd / 2); e0 += kBatch * kThreads) {
        load_queries(e0);
        put_queries(e0);
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
    float o[HALF ? NP : 1][4], of[HALF ? 1 : kColsOfThread][kHeads];
    if constexpr (HALF) {
#pragma unroll
        for (int x = 0; x < NP; ++x)
#pragma unroll
            for (int z = 0; z < 4; ++z) o[x][z] = 0.f;
    } else {
#pragma unroll
        for (int x = 0; x < kColsOfThread; ++x)
#pragma unroll
            for (int h = 0; h < kHeads; ++h) of[x][h] = 0.f;
    }
    if constexpr (WARPS) {
        // a lane: keys lane / 4 and lane / 4 + 8, heads 2 (lane % 4) and the next one
        float m[2] = {-1e30f, -1e30f}, l[2] = {0.f, 0.f};
        for (int j = j0; j < j1; ++j) {
            const int cnt = min(KT, i + 1 - lo - j * KT);
            unsigned char* kt = stage0 + (j - j0) % pl.stages * pl.stage_bytes;
            unsigned char* vt = V != nullptr ? kt + KT * pl.k_row : kt;
            wait_copies(pl.stages - 1);
            if (j == tiles - 1) put_new_row(kt, vt, cnt, lane, 32);
            __syncwarp();
            float sc[4];
            tile_scores(sc, smem_addr(kt), smem_addr(sm + pl.q), pl.k_row, 0, kd);
            float f[2];
#pragma unroll
            for (int x = 0; x < 4; ++x) sc[x] = (lane >> 2) + (x < 2 ? 0 : 8) < cnt ? sc[x] * c : -INFINITY;
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                float best = fmaxf(m[x], fmaxf(sc[x], sc[x + 2]));
#pragma unroll
                for (int y = 4; y < 32; y *= 2) best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, y));
                f[x] = exp2f(m[x] - best);
                m[x] = best;
                sc[x] = exp2f(sc[x] - best);
                sc[x + 2] = exp2f(sc[x + 2] - best);
                l[x] = l[x] * f[x] + sc[x] + sc[x + 2];
            }
            uint32_t wh[2], wl[2];                                  // the weights as an operand: 16 keys x 8 heads
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                split_bf16(sc[2 * y], sc[2 * y + 1], wh[y], wl[y]);
                wh[y] = transpose8(wh[y]);
                wl[y] = transpose8(wl[y]);
            }
            const uint32_t va = smem_addr(vt) + ((lane & 7) + (lane >> 4) * 8) * v_row + ((lane >> 3) & 1) * 16;
#pragma unroll
            for (int x = 0; x < NP; ++x) {
                if (x * 16 >= a.vdim_pad) break;
                uint32_t b[4];                            // columns 0-7, 8-15 of keys 0-7, then of keys 8-15
                ldmatrix4_t(b, va + x * 32);
#pragma unroll
                for (int z = 0; z < 4; ++z) o[x][z] *= f[z & 1];
                mma_bf16(o[x], b[0], b[1], b[2], b[3], wh[0], wh[1]);
                mma_bf16(o[x], b[0], b[1], b[2], b[3], wl[0], wl[1]);
            }
            __syncwarp();
            fetch(j + pl.stages);                         // this stage is free again
        }
        wait_copies(0);
        // the warps' outputs, to the CTA's maximum
        float* s_m = s_s;                                 // [warp][maximum, sum][kHeads]
        const int hl = (lane & 3) * 2;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
#pragma unroll
            for (int y = 4; y < 32; y *= 2) l[x] += __shfl_xor_sync(0xffffffffu, l[x], y);
            if (lane < 4) {
                s_m[warp * 2 * kHeads + hl + x] = m[x];
                s_m[(warp * 2 + 1) * kHeads + hl + x] = l[x];
            }
        }
        __syncthreads();
        float* own = reinterpret_cast<float*>(stage0);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float* at = s_m + hl + x;
            float best = -1e30f, sum = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) best = fmaxf(best, at[w * 2 * kHeads]);
#pragma unroll
            for (int w = 0; w < kWarps; ++w) sum = fmaf(exp2f(at[w * 2 * kHeads] - best), at[(w * 2 + 1) * kHeads], sum);
            const float f = exp2f(m[x] - best);
            if (warp == 0 && lane < 4) {
                stat[hl + x] = best;
                stat[kHeads + hl + x] = sum;
            }
#pragma unroll
            for (int y = 0; y < NP; ++y) {
                if (y * 16 >= a.vdim_pad) break;
                float* to = own + (hl + x) * a.vdim_pad + y * 16 + (lane >> 2);
                to[0] = o[y][x] * f;
                to[8] = o[y][x + 2] * f;
            }
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
            if constexpr (HALF) {                         // a warp 16 keys and half of the dimensions
                const int half = (kd / 16 + 1) / 2 * 16, part = warp / (KT / 16), k0 = warp % (KT / 16) * 16;
                float sc[4];
                tile_scores(sc, smem_addr(kt) + k0 * pl.k_row, smem_addr(sm + pl.q), pl.k_row, part * half, part ? kd : half);
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int h = (lane & 3) * 2 + (x & 1), k = k0 + (lane >> 2) + (x < 2 ? 0 : 8);
                    s_s[(part * kHeads + h) * SLD + k] = k < cnt ? sc[x] * c : -INFINITY;
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
                    v[y] = s_s[h * SLD + lane * (KT / 32) + y] + (HALF ? s_s[(kHeads + h) * SLD + lane * (KT / 32) + y] : 0.f);
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
                const float f0 = stat[2 * kHeads + (lane & 3) * 2], f1 = stat[2 * kHeads + (lane & 3) * 2 + 1];
                uint32_t w[KT / 16][4];                   // 16 keys x 8 heads: high parts, low parts
                const uint32_t pa = smem_addr(sm + pl.p) + ((lane & 7) + (lane >> 4) * kHeads) * PROW + ((lane >> 3) & 1) * 16;
#pragma unroll
                for (int k = 0; k < KT / 16; ++k) ldmatrix4(w[k], pa + k * 32);
                const uint32_t va = smem_addr(vt) + ((lane & 7) + (lane >> 4) * 8) * v_row + ((lane >> 3) & 1) * 16;
#pragma unroll
                for (int x = 0; x < NP; ++x) {
                    const int col = (warp + x * kWarps) * 16;
                    if (col >= a.vdim_pad) break;
                    o[x][0] *= f0; o[x][1] *= f1;
                    o[x][2] *= f0; o[x][3] *= f1;
#pragma unroll
                    for (int k = 0; k < KT / 16; ++k) {
                        uint32_t b[4];                    // columns 0-7, 8-15 of keys 0-7, then of keys 8-15
                        ldmatrix4_t(b, va + k * 16 * v_row + col * 2);
                        mma_bf16(o[x], b[0], b[1], b[2], b[3], w[k][0], w[k][1]);
                        mma_bf16(o[x], b[0], b[1], b[2], b[3], w[k][2], w[k][3]);
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
        float* s_o = reinterpret_cast<float*>(sm + pl.stage);                  // [kHeads][vdim_pad]
        auto put = [&](int h, int d, float v) { s_o[h * a.vdim_pad + d] = v; };
        if constexpr (HALF) {
#pragma unroll
            for (int x = 0; x < NP; ++x) {
                const int col = (warp + x * kWarps) * 16;
                if (col >= a.vdim_pad) break;
#pragma unroll
                for (int z = 0; z < 4; ++z) put((lane & 3) * 2 + (z & 1), col + (lane >> 2) + (z < 2 ? 0 : 8), o[x][z]);
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

    // ---- merge: every CTA's outputs to the owners of their slices ----
    float* box_ml = reinterpret_cast<float*>(sm + pl.inbox);          // [rank][maximum, sum][kHeads]
    float* factor = box_ml + kMaxCluster * 2 * kHeads;                // [kHeads][C]
    float* top = factor + kMaxCluster * kHeads;                       // [maximum, sum][kHeads] of the cluster
    float4* box = reinterpret_cast<float4*>(top + 2 * kHeads);        // [rank][slice]
    auto cl = cg::this_cluster();
    __syncthreads();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    for (int e = tid; e < C * 2 * kHeads; e += kThreads) {
        const int r = e / (2 * kHeads), x = e - r * 2 * kHeads;
        cl.map_shared_rank(box_ml, r)[rank * 2 * kHeads + x] = stat[x];
    }
    {
        const float4* from = reinterpret_cast<const float4*>(sm + pl.stage);
        const int next = pl.stages * pl.stage_bytes / 16;
        for (int e = tid; e < nh * v4; e += kThreads) {
            float4 t = from[e];
#pragma unroll
            for (int w = 1; w < UNITS; ++w) {                         // the warps' sums
                const float4 v = from[e + w * next];
                t.x += v.x; t.y += v.y; t.z += v.z; t.w += v.w;
            }
            const int r = e / slice;
            cl.map_shared_rank(box, r)[rank * slice + e - r * slice] = t;
        }
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    for (int e = tid; e < kHeads * C; e += kThreads) {                // the C lanes of a head are neighbours, C 8 or 16
        const int h = e / C, r = e - h * C;
        const float m = h < nh ? box_ml[r * 2 * kHeads + h] : -1e30f, l = h < nh ? box_ml[(r * 2 + 1) * kHeads + h] : 0.f;
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
    auto finish = [&](int k, float4 t) {                              // float4 k of the slice
        int at;
        const int cnt = place_of(rank * slice + k, at);
        const float v[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
            if (x < cnt) {
                float g = 1.f;
                if (p.s.gate != nullptr) g = sigmoid_f32(k == tid ? gate[x] : __ldcg(p.s.gate + at + x));
                p.s.out[at + x] = v[x] * g;
            }
    };
    float4* part = reinterpret_cast<float4*>(p.part) + (size_t)gb * p.clusters * kHeads * v4 + rank * slice;
    for (int k = tid; k < n_mine; k += kThreads) {
        const int h = (rank * slice + k) / v4;
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int r = 0; r < C; ++r) {
            const float f = factor[h * C + r];
            const float4 v = box[r * slice + k];
            t.x = fmaf(f, v.x, t.x); t.y = fmaf(f, v.y, t.y); t.z = fmaf(f, v.z, t.z); t.w = fmaf(f, v.w, t.w);
        }
        if (active == 1) finish(k, t);
        else part[(size_t)cluster * kHeads * v4 + k] = t;
    }
    if (active == 1) return;
    float* ml = p.ml + ((size_t)gb * p.clusters * C + rank) * kHeads * 2;
    const size_t ml_step = (size_t)C * kHeads * 2;
    if (tid < 2 * kHeads) ml[cluster * ml_step + tid] = top[tid];
    __threadfence();
    __syncthreads();
    unsigned* ticket = p.tickets + gb * C + rank;
    if (tid == 0) s_last = atomicAdd(ticket, 1u) == (unsigned)active - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) *ticket = 0;
    for (int k = tid; k < n_mine; k += kThreads) {
        const int h = (rank * slice + k) / v4;
        float best = -1e30f, l = 0.f;
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int x = 0; x < active; ++x) best = fmaxf(best, __ldcg(ml + x * ml_step + h));
#pragma unroll 4
        for (int x = 0; x < active; ++x) {
            const float f = exp2f(__ldcg(ml + x * ml_step + h) - best);
            const float4 v = __ldcg(part + (size_t)x * kHeads * v4 + k);
            l = fmaf(f, __ldcg(ml + x * ml_step + kHeads + h), l);
            t.x = fmaf(f, v.x, t.x); t.y = fmaf(f, v.y, t.y); t.z = fmaf(f, v.z, t.z); t.w = fmaf(f, v.w, t.w);
        }
        finish(k, make_float4(t.x / l, t.y / l, t.z / l, t.w / l));
    }
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
        const dim3 grid(p.cluster * groups, p.clusters);
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
