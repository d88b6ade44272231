// Attention over a sliding window of tokens and, before it, one mean key / value per block of `pool` tokens,
// with an optional linear mix of the softmax weights across heads. Device code shared by the decode step and
// the per-row prompt kernel.
//
// Position i sees n_blk = max(0, (i - size + 1) / pool) pooled blocks (block b ends at b * pool + pool - 1 <=
// i - size) and the last min(size, i + 1) tokens. "Key j" below counts the blocks first, then the tokens.
#pragma once

#include <cooperative_groups.h>

#include "leankv_mixers.h"
#include "typed.cuh"

namespace leankv {

namespace cg = cooperative_groups;

struct VisibleKeys {
    int n_blk, w0, n;      // pooled blocks, first token of the window, keys in all
    __host__ __device__ VisibleKeys(int i, int size, int pool) {
        w0 = i - size + 1 > 0 ? i - size + 1 : 0;
        n_blk = w0 / pool;
        n = n_blk + i + 1 - w0;
    }
};

constexpr int kAttendHeads = 4;     // query heads a thread carries at once

// Shared-memory plan of attend_query (floats), `threads` per CTA, at most n_local keys per CTA.
struct AttendPlan {
    int q, knew, vnew, stat, out, part, talk, p, total;    // offsets; total in floats
    int ldp;               // row length of the weight buffers
    bool p_in_smem;
    __host__ __device__ AttendPlan(const leankv_window_pool_t& a, int threads, int n_local, int max_floats) {
        int o = 0;
        const auto take = [&](int n) { const int at = o; o += (n + 3) / 4 * 4; return at; };
        q = take(a.heads * a.dim_pad);
        knew = take(a.kv_heads * a.dim_pad);
        vnew = take(a.kv_heads * a.vdim_pad);
        stat = take(4 * a.heads);
        out = take(a.heads * a.vdim_pad);
        const int slots = a.kv_heads * (a.vdim_pad / 8);
        const int split = threads / slots > 1 ? threads / slots : 1;
        part = take(split > 1 ? split * a.kv_heads * kAttendHeads * a.vdim_pad : 0);
        talk = take(a.talk ? a.heads * ((a.heads + 7) / 8 * 8) : 0);
        ldp = (n_local + 3) / 4 * 4 + 1;
        const int need = 2 * a.heads * ldp;
        p_in_smem = o + need <= max_floats;
        p = take(p_in_smem ? need : 0);
        total = o;
    }
};

template <typename T>
__device__ __forceinline__ void key_row8(const T* row, int d, float (&v)[8]) {
    Raw8<T> r;
    load8(row + d, r);
    unpack8(r, v);
}

// Attention of position i over this CTA's share (rank of C) of its visible keys, everything in fp32.
// sm: shared memory laid out by `pl`; sm[pl.q] holds the normed queries times the score scale. If `fresh`, the key / value of
// position i come from sm[pl.knew] / sm[pl.vnew] instead of the ring (it may not be written yet).
// p_gmem: weight buffers (2 * heads * ldp floats of this CTA) when they do not fit into shared memory.
// Writes out[h * out_stride + d], d < vdim, times out_scale; with C > 1 the CTAs are a cluster and each
// writes its share of the elements.
template <typename T, typename O>
__device__ void attend_query(const leankv_window_pool_t& a, const AttendPlan& pl, float* sm, float* p_gmem, int i,
                             bool fresh, int rank, int C, O* out, float out_scale) {
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nt >> 5;
    const int H = a.heads, G = a.kv_heads, rep = H / G, dp = a.dim_pad, vp = a.vdim_pad, ldp = pl.ldp;
    const VisibleKeys vis(i, a.size, a.pool);
    const int j0 = (int)((long long)vis.n * rank / C), j1 = (int)((long long)vis.n * (rank + 1) / C), n = j1 - j0;
    const T* k_ring = static_cast<const T*>(a.k_ring);
    const T* v_ring = static_cast<const T*>(a.v_ring);
    const T* k_pool = static_cast<const T*>(a.k_pool);
    const T* v_pool = static_cast<const T*>(a.v_pool);
    float* p = pl.p_in_smem ? sm + pl.p : p_gmem;
    float* pm = a.talk ? p + H * ldp : p;
    float* stat = sm + pl.stat;            // local max | local sum | global max | 1 / global sum
    const int Hr = (H + 7) / 8 * 8;

    if (a.talk)
        for (int e = tid; e < H * Hr; e += nt) {       // talk^T, rows padded: talk_t[g][h]
            const int g = e / Hr, h = e - g * Hr;
            sm[pl.talk + e] = h < H ? __ldg(a.talk + h * H + g) : 0.f;
        }

    // ---- scores: one thread per (key, kv head), the group's query heads kAttendHeads at a time ----
    for (int e = tid; e < n * G; e += nt) {
        const int g = e / n, jl = e - g * n, j = j0 + jl;
        const T* row = nullptr;
        if (j < vis.n_blk) row = k_pool + ((size_t)j * G + g) * dp;
        else {
            const int pos = vis.w0 + j - vis.n_blk;
            if (!(fresh && pos == i)) row = k_ring + ((size_t)(pos % a.ring) * G + g) * dp;
        }
        const float* krow = sm + pl.knew + g * dp;
        for (int hb = 0; hb < rep; hb += kAttendHeads) {
            float acc[kAttendHeads] = {};
            const float* q = sm + pl.q + (g * rep + hb) * dp;
            const int nh = min(kAttendHeads, rep - hb);
            for (int d = 0; d < dp; d += 8) {
                float kv[8];
                if (row != nullptr) key_row8(row, d, kv);
                else {
#pragma unroll
                    for (int x = 0; x < 8; ++x) kv[x] = krow[d + x];
                }
#pragma unroll
                for (int r = 0; r < kAttendHeads; ++r)
                    if (r < nh) {
                        const float4 qa = *reinterpret_cast<const float4*>(q + r * dp + d);
                        const float4 qb = *reinterpret_cast<const float4*>(q + r * dp + d + 4);
                        acc[r] = fmaf(qa.x, kv[0], acc[r]); acc[r] = fmaf(qa.y, kv[1], acc[r]);
                        acc[r] = fmaf(qa.z, kv[2], acc[r]); acc[r] = fmaf(qa.w, kv[3], acc[r]);
                        acc[r] = fmaf(qb.x, kv[4], acc[r]); acc[r] = fmaf(qb.y, kv[5], acc[r]);
                        acc[r] = fmaf(qb.z, kv[6], acc[r]); acc[r] = fmaf(qb.w, kv[7], acc[r]);
                    }
            }
#pragma unroll
            for (int r = 0; r < kAttendHeads; ++r)
                if (r < nh) p[(g * rep + hb + r) * ldp + jl] = acc[r];
        }
    }
    __syncthreads();

    // ---- softmax statistics, first of this CTA's keys, then of all ----
    for (int h = warp; h < H; h += nw) {
        float m = -INFINITY;
        for (int j = lane; j < n; j += 32) m = fmaxf(m, p[h * ldp + j]);
        m = warp_max(m);
        float l = 0.f;
        for (int j = lane; j < n; j += 32) {
            const float e = expf(p[h * ldp + j] - m);
            p[h * ldp + j] = e;
            l += e;
        }
        l = warp_sum(l);
        if (lane == 0) { stat[h] = m; stat[H + h] = l; }
    }
    if (C > 1) cg::this_cluster().sync();
    else __syncthreads();
    for (int h = tid; h < H; h += nt) {
        float m = -INFINITY, l = 0.f;
        if (C > 1) {
            auto cl = cg::this_cluster();
            for (int r = 0; r < C; ++r) m = fmaxf(m, cl.map_shared_rank(stat, r)[h]);
            for (int r = 0; r < C; ++r) {
                const float* s = cl.map_shared_rank(stat, r);
                if (s[H + h] > 0.f) l += s[H + h] * expf(s[h] - m);
            }
        } else {
            m = stat[h];
            l = stat[H + h];
        }
        // a weight of this CTA = its exponential (taken against the local maximum) times this factor
        stat[2 * H + h] = n > 0 ? expf(stat[h] - m) / l : 0.f;
    }
    __syncthreads();
    if (a.talk) {
        const int nb = Hr / 8;
        for (int e = tid; e < n * nb; e += nt) {
            const int hb = e / n, jl = e - hb * n;
            float acc[8] = {};
            const float* tk = sm + pl.talk + hb * 8;
            for (int g = 0; g < H; ++g) {
                const float w = p[g * ldp + jl] * stat[2 * H + g];
                const float4 ta = *reinterpret_cast<const float4*>(tk + g * Hr);
                const float4 tb = *reinterpret_cast<const float4*>(tk + g * Hr + 4);
                acc[0] = fmaf(ta.x, w, acc[0]); acc[1] = fmaf(ta.y, w, acc[1]);
                acc[2] = fmaf(ta.z, w, acc[2]); acc[3] = fmaf(ta.w, w, acc[3]);
                acc[4] = fmaf(tb.x, w, acc[4]); acc[5] = fmaf(tb.y, w, acc[5]);
                acc[6] = fmaf(tb.z, w, acc[6]); acc[7] = fmaf(tb.w, w, acc[7]);
            }
#pragma unroll
            for (int x = 0; x < 8; ++x)
                if (hb * 8 + x < H) pm[(hb * 8 + x) * ldp + jl] = acc[x];
        }
    } else {
        for (int e = tid; e < n * H; e += nt) {
            const int h = e / n, jl = e - h * n;
            p[h * ldp + jl] *= stat[2 * H + h];
        }
    }
    __syncthreads();

    // ---- weights times values: a thread owns 8 value columns of one kv head and every split-th key ----
    const int per_g = vp / 8, slots = G * per_g;
    const int split = nt / slots > 1 ? nt / slots : 1;
    float* s_out = sm + pl.out;
    for (int hb = 0; hb < rep; hb += kAttendHeads) {
        const int nh = min(kAttendHeads, rep - hb);
        for (int e = tid; e < slots * split; e += nt) {
            const int ks = e / slots, sl = e - ks * slots, g = sl / per_g, d = (sl - g * per_g) * 8;
            float acc[kAttendHeads][8] = {};
            const float* w = pm + (g * rep + hb) * ldp;
            for (int jl = ks; jl < n; jl += split) {
                const int j = j0 + jl;
                float vv[8];
                if (j < vis.n_blk) key_row8(v_pool + ((size_t)j * G + g) * vp, d, vv);
                else {
                    const int pos = vis.w0 + j - vis.n_blk;
                    if (fresh && pos == i) {
#pragma unroll
                        for (int x = 0; x < 8; ++x) vv[x] = sm[pl.vnew + g * vp + d + x];
                    } else {
                        key_row8(v_ring + ((size_t)(pos % a.ring) * G + g) * vp, d, vv);
                    }
                }
#pragma unroll
                for (int r = 0; r < kAttendHeads; ++r)
                    if (r < nh) {
                        const float wr = w[r * ldp + jl];
#pragma unroll
                        for (int x = 0; x < 8; ++x) acc[r][x] = fmaf(wr, vv[x], acc[r][x]);
                    }
            }
            float* dst = split > 1 ? sm + pl.part + (size_t)(ks * G + g) * kAttendHeads * vp : nullptr;
#pragma unroll
            for (int r = 0; r < kAttendHeads; ++r)
                if (r < nh) {
                    float* o = split > 1 ? dst + r * vp + d : s_out + (g * rep + hb + r) * vp + d;
#pragma unroll
                    for (int x = 0; x < 8; ++x) o[x] = acc[r][x];
                }
        }
        __syncthreads();
        if (split > 1) {
            for (int e = tid; e < G * nh * vp; e += nt) {
                const int g = e / (nh * vp), x = e - g * nh * vp;
                float t = 0.f;
                for (int ks = 0; ks < split; ++ks) t += sm[pl.part + (size_t)(ks * G + g) * kAttendHeads * vp + x];
                s_out[(g * rep + hb) * vp + x] = t;
            }
            __syncthreads();
        }
    }
    if (C > 1) cg::this_cluster().sync();
    const int total = H * a.vdim, e0 = total * rank / C, e1 = total * (rank + 1) / C;
    for (int e = e0 + tid; e < e1; e += nt) {
        const int h = e / a.vdim, d = e - h * a.vdim;
        float t = 0.f;
        if (C > 1) {
            auto cl = cg::this_cluster();
            for (int r = 0; r < C; ++r) t += cl.map_shared_rank(s_out, r)[h * vp + d];
        } else {
            t = s_out[h * vp + d];
        }
        out[e] = from_f32<O>(t * out_scale);
    }
    if (C > 1) cg::this_cluster().sync();       // the other CTAs still read this one's shared memory
}

// RMS norm over a whole projection row (all heads at once): returns the factor, 1 if there is no norm.
__device__ __forceinline__ float row_factor(const float* x, const float* bias, int n, bool normed, float eps,
                                            float* s_tmp) {
    if (!normed) return 1.f;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = x[i] + (bias != nullptr ? __ldg(bias + i) : 0.f);
        ss = fmaf(v, v, ss);
    }
    return 1.f / sqrtf(cta_sum(ss, s_tmp) / (float)n + eps);
}

}  // namespace leankv
