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

// The tensor-core route of leankv_window_pool_attend (window_pool_tile.cu); LEANKV_EUNSUPPORTED for storage types,
// head counts and sizes it does not take.
int window_pool_tile_attend(const leankv_window_pool_t& a, const void* q, void* out, int out_ld, float out_scale, int rows,
                            int start, cudaStream_t st);

constexpr int kMaxCluster = 16;     // non-portable; 8 where the device does not place 16
constexpr int kAttendHeads = 4;     // query heads a thread carries at once

// Row length (elements) of bf16 operand rows in shared memory: 16-byte fragment reads of eight consecutive rows
// fall into different banks when a row is 64 bytes past a multiple of 128.
__host__ __device__ __forceinline__ int fragment_row(int n) { return n + (96 - n % 64) % 64; }

// Shared-memory plan of attend_query (floats), `threads` per CTA, at most n_local keys per CTA.
struct AttendPlan {
    int q, knew, vnew, stat, out, part, talk, p, total;    // offsets; total in floats
    int ldp;               // row length of the weight buffers, a multiple of 4
    int ldq;               // row length of the queries: fp32, or bf16 (high parts of all heads, then low parts)
    bool p_in_smem;
    __host__ __device__ AttendPlan(const leankv_window_pool_t& a, int threads, int n_local, int max_floats) {
        int o = 0;
        const auto take = [&](int n) { const int at = o; o += (n + 3) / 4 * 4; return at; };
        const bool half = a.dtype == LEANKV_DT_BF16;
        ldq = half ? fragment_row(a.dim_pad) : a.dim_pad;
        q = take(a.heads * ldq);
        knew = take(a.kv_heads * a.dim_pad / (half ? 2 : 1));
        vnew = take(a.kv_heads * a.vdim_pad / (half ? 2 : 1));
        stat = take(3 * a.heads);
        out = take(a.heads * a.vdim_pad);
        const int slots = a.kv_heads * (a.vdim_pad / 8);
        const int split = threads / slots > 1 ? threads / slots : 1;
        part = take(split > 1 ? split * a.kv_heads * kAttendHeads * a.vdim_pad : 0);
        talk = take(a.talk ? a.heads * ((a.heads + 7) / 8 * 8) : 0);
        ldp = (n_local + 3) / 4 * 4 + 4;
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

// Queries into shared memory, times the score scale.
template <typename T>
__device__ __forceinline__ void put_query(const AttendPlan& pl, float* sm, int heads, int h, int d, float v) {
    if constexpr (sizeof(T) == 4) {
        sm[pl.q + h * pl.ldq + d] = v;
    } else {
        bf16* q = reinterpret_cast<bf16*>(sm + pl.q);
        const bf16 hi = from_f32<bf16>(v);
        q[h * pl.ldq + d] = hi;
        q[(heads + h) * pl.ldq + d] = from_f32<bf16>(v - to_f32(hi));
    }
}

template <typename T>
__device__ __forceinline__ void put_query4(const AttendPlan& pl, float* sm, int heads, int h, int d, float4 v) {
    if constexpr (sizeof(T) == 4) {
        store4(sm + pl.q + h * pl.ldq + d, v);
    } else {
        bf16* q = reinterpret_cast<bf16*>(sm + pl.q);
        uint2 hi, lo;
        split_bf16(v.x, v.y, hi.x, lo.x);
        split_bf16(v.z, v.w, hi.y, lo.y);
        *reinterpret_cast<uint2*>(q + h * pl.ldq + d) = hi;
        *reinterpret_cast<uint2*>(q + (heads + h) * pl.ldq + d) = lo;
    }
}

// Scores of the keys of one kv head, row_of(jl, g) -> key row. fp32: a thread per (key, kv head), the
// group's query heads kAttendHeads at a time.
template <typename RowOf>
__device__ __forceinline__ void scores(const leankv_window_pool_t& a, const AttendPlan& pl, const float* sm, float* p,
                                       int n, RowOf row_of, float) {
    const int G = a.kv_heads, rep = a.heads / G, dp = a.dim_pad;
    for (int e = threadIdx.x; e < n * G; e += blockDim.x) {
        const int g = e / n, jl = e - g * n;
        const float* row = row_of(jl, g);
        for (int hb = 0; hb < rep; hb += kAttendHeads) {
            float acc[kAttendHeads] = {};
            const float* q = sm + pl.q + (g * rep + hb) * pl.ldq;
            const int nh = min(kAttendHeads, rep - hb);
            for (int d = 0; d < dp; d += 8) {
                float kv[8];
                key_row8(row, d, kv);
#pragma unroll
                for (int r = 0; r < kAttendHeads; ++r)
                    if (r < nh)
#pragma unroll
                        for (int x = 0; x < 8; ++x) acc[r] = fmaf(q[r * pl.ldq + d + x], kv[x], acc[r]);
            }
#pragma unroll
            for (int r = 0; r < kAttendHeads; ++r)
                if (r < nh) p[(g * rep + hb + r) * pl.ldp + jl] = acc[r];
        }
    }
}

// bf16: a warp per (16 keys, kv head) on tensor cores, keys as rows and the group's query heads as columns.
// Queries are two bf16 numbers (high + low part), so scores are exact products of the stored keys. The order
// of the dimensions inside a tile is permuted so that a lane's share of a key row is 16 consecutive bytes.
template <typename RowOf>
__device__ __forceinline__ void scores(const leankv_window_pool_t& a, const AttendPlan& pl, const float* sm, float* p,
                                       int n, RowOf row_of, bf16) {
    const int G = a.kv_heads, rep = a.heads / G, dp = a.dim_pad, ldq = pl.ldq;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int gl = lane >> 2, t = lane & 3, tiles = (n + 15) / 16, nb = dp / 32;
    const bf16* qs = reinterpret_cast<const bf16*>(sm + pl.q);
    for (int e = warp; e < tiles * G; e += nw) {
        const int g = e / tiles, k0 = (e - g * tiles) * 16;
        const int j0 = k0 + gl, j1 = j0 + 8;
        const bf16* r0 = row_of(min(j0, n - 1), g);
        const bf16* r1 = row_of(min(j1, n - 1), g);
        for (int hb = 0; hb < rep; hb += 8) {
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
            const bool on = hb + gl < rep;
            const bf16* qh = qs + (g * rep + hb + (on ? gl : 0)) * ldq;
            const bf16* ql = qh + a.heads * ldq;
            for (int b0 = 0; b0 < nb; b0 += 4) {
                uint4 x0[4], x1[4];
#pragma unroll
                for (int b = 0; b < 4; ++b)
                    if (b0 + b < nb) {
                        x0[b] = *reinterpret_cast<const uint4*>(r0 + (b0 + b) * 32 + t * 8);
                        x1[b] = *reinterpret_cast<const uint4*>(r1 + (b0 + b) * 32 + t * 8);
                    }
#pragma unroll
                for (int b = 0; b < 4; ++b)
                    if (b0 + b < nb) {
                        uint4 h = *reinterpret_cast<const uint4*>(qh + (b0 + b) * 32 + t * 8);
                        uint4 l = *reinterpret_cast<const uint4*>(ql + (b0 + b) * 32 + t * 8);
                        if (!on) h = l = make_uint4(0, 0, 0, 0);
                        mma_bf16(acc, x0[b].x, x1[b].x, x0[b].y, x1[b].y, h.x, h.y);
                        mma_bf16(acc, x0[b].z, x1[b].z, x0[b].w, x1[b].w, h.z, h.w);
                        mma_bf16(acc, x0[b].x, x1[b].x, x0[b].y, x1[b].y, l.x, l.y);
                        mma_bf16(acc, x0[b].z, x1[b].z, x0[b].w, x1[b].w, l.z, l.w);
                    }
            }
            if (dp % 32) {                              // a last half block of 16 dimensions
                const int d = nb * 32 + t * 4;
                const uint2 y0 = *reinterpret_cast<const uint2*>(r0 + d), y1 = *reinterpret_cast<const uint2*>(r1 + d);
                uint2 h = *reinterpret_cast<const uint2*>(qh + d), l = *reinterpret_cast<const uint2*>(ql + d);
                if (!on) h = l = make_uint2(0, 0);
                mma_bf16(acc, y0.x, y1.x, y0.y, y1.y, h.x, h.y);
                mma_bf16(acc, y0.x, y1.x, y0.y, y1.y, l.x, l.y);
            }
            float* dst = p + (size_t)(g * rep + hb) * pl.ldp;
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int h = 2 * t + (x & 1), j = x < 2 ? j0 : j1;
                if (hb + h < rep && j < n) dst[h * pl.ldp + j] = acc[x];
            }
        }
    }
}

// The mixing matrix into shared memory, transposed and its rows padded to 8 ([from head][to head]).
__device__ __forceinline__ void put_talk(const leankv_window_pool_t& a, const AttendPlan& pl, float* sm) {
    if (a.talk == nullptr) return;
    const int H = a.heads, Hr = (H + 7) / 8 * 8;
    for (int e = threadIdx.x; e < H * Hr; e += blockDim.x) {
        const int h = e / H, g = e - h * H;
        sm[pl.talk + g * Hr + h] = h < H ? __ldg(a.talk + e) : 0.f;
    }
}

// pm[h][j] = sum over g of talk[h][g] * (p[g][j] * factor[g]). fp32 on FMA units.
__device__ __forceinline__ void mix_heads(const leankv_window_pool_t& a, const AttendPlan& pl, float* sm,
                                          const float* factor, const float* p, float* pm, int n, float) {
    const int H = a.heads, Hr = (H + 7) / 8 * 8, nb = Hr / 8;
    for (int e = threadIdx.x; e < n * nb; e += blockDim.x) {
        const int hb = e / n, jl = e - hb * n;
        float acc[8] = {};
        const float* tk = sm + pl.talk + hb * 8;
        for (int g = 0; g < H; ++g) {
            const float w = p[g * pl.ldp + jl] * factor[g];
#pragma unroll
            for (int x = 0; x < 8; ++x) acc[x] = fmaf(tk[g * Hr + x], w, acc[x]);
        }
#pragma unroll
        for (int x = 0; x < 8; ++x)
            if (hb * 8 + x < H) pm[(hb * 8 + x) * pl.ldp + jl] = acc[x];
    }
}

// The same on tensor cores: output heads as rows, keys as columns, both operands as high + low bf16 parts
// (the product of the two low parts, 2^-16 of the result, is dropped).
__device__ __forceinline__ void mix_heads(const leankv_window_pool_t& a, const AttendPlan& pl, float* sm,
                                          const float* factor, const float* p, float* pm, int n, bf16) {
    const int H = a.heads, Hr = (H + 7) / 8 * 8, ht = (H + 15) / 16, kt = (n + 7) / 8;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, gl = lane >> 2, t = lane & 3;
    for (int e = warp; e < ht * kt; e += nw) {
        const int m0 = (e / kt) * 16, j = (e % kt) * 8 + gl;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int g0 = 0; g0 < H; g0 += 16) {
            auto tk = [&](int h, int g) { return h < H && g < H ? sm[pl.talk + g * Hr + h] : 0.f; };
            auto wt = [&](int g) { return g < H && j < n ? p[g * pl.ldp + j] * factor[g] : 0.f; };
            const int c = g0 + 2 * t;
            uint32_t ah[4], al[4], bh[2], bl[2];
            split_bf16(tk(m0 + gl, c), tk(m0 + gl, c + 1), ah[0], al[0]);
            split_bf16(tk(m0 + gl + 8, c), tk(m0 + gl + 8, c + 1), ah[1], al[1]);
            split_bf16(tk(m0 + gl, c + 8), tk(m0 + gl, c + 9), ah[2], al[2]);
            split_bf16(tk(m0 + gl + 8, c + 8), tk(m0 + gl + 8, c + 9), ah[3], al[3]);
            split_bf16(wt(c), wt(c + 1), bh[0], bl[0]);
            split_bf16(wt(c + 8), wt(c + 9), bh[1], bl[1]);
            mma_bf16(acc, ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
            mma_bf16(acc, ah[0], ah[1], ah[2], ah[3], bl[0], bl[1]);
            mma_bf16(acc, al[0], al[1], al[2], al[3], bh[0], bh[1]);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int h = m0 + gl + (x < 2 ? 0 : 8), col = (e % kt) * 8 + 2 * t + (x & 1);
            if (h < H && col < n) pm[h * pl.ldp + col] = acc[x];
        }
    }
}

// Attention of position i over this CTA's share (rank of C) of its visible keys; scores, softmax and the mix
// across heads in fp32 (bf16 operands enter as exact parts).
// sm: shared memory laid out by `pl`, with the normed queries (put_query) and the mix (put_talk) in place. If `fresh`, the key / value
// rows of position i are those at sm[pl.knew] / sm[pl.vnew] instead of the ring's (not written yet).
// p_gmem: weight buffers (2 * heads * ldp floats of this CTA) when they do not fit into shared memory.
// Writes out[h * vdim + d] times out_scale; with C > 1 the CTAs are a cluster and each writes its share.
template <typename T, typename O>
__device__ void attend_query(const leankv_window_pool_t& a, const AttendPlan& pl, float* sm, float* p_gmem, int i,
                             bool fresh, int rank, int C, O* out, float out_scale) {
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nt >> 5;
    const int H = a.heads, G = a.kv_heads, rep = H / G, dp = a.dim_pad, vp = a.vdim_pad, ldp = pl.ldp;
    const VisibleKeys vis(i, a.size, a.pool);
    const int j0 = (int)((long long)vis.n * rank / C), j1 = (int)((long long)vis.n * (rank + 1) / C), n = j1 - j0;
    float* p = pl.p_in_smem ? sm + pl.p : p_gmem;
    float* pm = a.talk ? p + H * ldp : p;
    float* stat = sm + pl.stat;            // local max | local sum | factor of this CTA's exponentials

    const int slot_w0 = vis.w0 % a.ring;
    // row of local key jl in the pooled blocks, the ring, or the fresh row
    auto row = [&](int jl, int g, const void* pool, const void* ring, int fresh_at, int width) -> const T* {
        const int j = j0 + jl;
        if (j < vis.n_blk) return static_cast<const T*>(pool) + ((size_t)j * G + g) * width;
        if (fresh && j == vis.n - 1) return reinterpret_cast<const T*>(sm + fresh_at) + g * width;
        int slot = slot_w0 + j - vis.n_blk;              // a window fits into the ring once
        if (slot >= a.ring) slot -= a.ring;
        return static_cast<const T*>(ring) + ((size_t)slot * G + g) * width;
    };
    if (n > 0) scores(a, pl, sm, p, n, [&](int jl, int g) { return row(jl, g, a.k_pool, a.k_ring, pl.knew, dp); }, T{});
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
            float mr[kMaxCluster], lr[kMaxCluster];      // all remote reads in flight together
#pragma unroll
            for (int r = 0; r < kMaxCluster; ++r) {
                const float* s = cl.map_shared_rank(stat, r < C ? r : 0);
                mr[r] = s[h];
                lr[r] = r < C ? s[H + h] : 0.f;
            }
#pragma unroll
            for (int r = 0; r < kMaxCluster; ++r) m = fmaxf(m, mr[r]);
#pragma unroll
            for (int r = 0; r < kMaxCluster; ++r)
                if (lr[r] > 0.f) l += lr[r] * expf(mr[r] - m);
        } else {
            m = stat[h];
            l = stat[H + h];
        }
        // a weight of this CTA = its exponential (taken against the local maximum) times this factor
        stat[2 * H + h] = n > 0 ? expf(stat[h] - m) / l : 0.f;
    }
    __syncthreads();
    if (a.talk) {
        mix_heads(a, pl, sm, stat + 2 * H, p, pm, n, T{});
    } else {
        for (int e = tid; e < n * H; e += nt) {
            const int h = e / n, jl = e - h * n;
            p[h * ldp + jl] *= stat[2 * H + h];
        }
    }
    __syncthreads();

    // ---- weights times values: a thread owns 8 value columns of one kv head and a range of keys ----
    const int per_g = vp / 8, slots = G * per_g;
    const int split = nt / slots > 1 ? nt / slots : 1;
    const int per_split = ((n + split - 1) / split + 3) / 4 * 4;      // 16-byte reads of the weights
    float* s_out = sm + pl.out;
    for (int hb = 0; hb < rep; hb += kAttendHeads) {
        const int nh = min(kAttendHeads, rep - hb);
        for (int e = tid; e < slots * split; e += nt) {
            const int ks = e / slots, sl = e - ks * slots, g = sl / per_g, d = (sl - g * per_g) * 8;
            float acc[kAttendHeads][8] = {};
            const float* w = pm + (g * rep + hb) * ldp;
            const int e0 = min(n, ks * per_split), e1 = min(n, e0 + per_split);
            constexpr int kBatch = sizeof(T) == 2 ? 8 : 4;      // value rows in flight per thread
            for (int jb = e0; jb < e1; jb += kBatch) {
                Raw8<T> raw[kBatch];
#pragma unroll
                for (int x = 0; x < kBatch; ++x)
                    load8(row(min(jb + x, e1 - 1), g, a.v_pool, a.v_ring, pl.vnew, vp) + d, raw[x]);
#pragma unroll
                for (int q = 0; q < kBatch; q += 4) {
                    const int jl = jb + q;
                    if (jl >= e1) break;
                    float wr[kAttendHeads][4];
#pragma unroll
                    for (int r = 0; r < kAttendHeads; ++r)
                        if (r < nh) {
                            const float4 w4 = *reinterpret_cast<const float4*>(w + r * ldp + jl);
                            wr[r][0] = w4.x; wr[r][1] = w4.y; wr[r][2] = w4.z; wr[r][3] = w4.w;
                        }
#pragma unroll
                    for (int x = 0; x < 4; ++x)
                        if (jl + x < e1) {
                            float vv[8];
                            unpack8(raw[q + x], vv);
#pragma unroll
                            for (int r = 0; r < kAttendHeads; ++r)
                                if (r < nh)
#pragma unroll
                                    for (int c = 0; c < 8; ++c) acc[r][c] = fmaf(wr[r][x], vv[c], acc[r][c]);
                        }
                }
            }
            float* dst = split > 1 ? sm + pl.part + (size_t)(ks * G + g) * kAttendHeads * vp : nullptr;
#pragma unroll
            for (int r = 0; r < kAttendHeads; ++r)
                if (r < nh) {
                    float* o = split > 1 ? dst + r * vp + d : s_out + (g * rep + hb + r) * vp + d;
                    reinterpret_cast<float4*>(o)[0] = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
                    reinterpret_cast<float4*>(o)[1] = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
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
            float part[kMaxCluster];
#pragma unroll
            for (int r = 0; r < kMaxCluster; ++r) part[r] = r < C ? cl.map_shared_rank(s_out, r)[h * vp + d] : 0.f;
#pragma unroll
            for (int r = 0; r < kMaxCluster; ++r) t += part[r];
        } else {
            t = s_out[h * vp + d];
        }
        out[e] = from_f32<O>(t * out_scale);
    }
    if (C > 1) cg::this_cluster().sync();       // the other CTAs still read this one's shared memory
}

// RMS norm over a whole projection row (all heads at once) for the q and the k part of it: the two factors.
struct RowFactors { float q, k; };
__device__ __forceinline__ RowFactors norm_factors(float sq, float sk, int nq, int nk, bool norm_q, bool norm_k,
                                                   float eps, float* s_tmp) {       // from per-thread sums of squares
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;     // nw <= 16
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { s_tmp[warp] = sq; s_tmp[16 + warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < nw; ++w) { sq += s_tmp[w]; sk += s_tmp[16 + w]; }
    return {norm_q ? 1.f / sqrtf(sq / (float)nq + eps) : 1.f, norm_k ? 1.f / sqrtf(sk / (float)nk + eps) : 1.f};
}
__device__ __forceinline__ RowFactors row_factors(const float* x, const float* bias, int nq, int nk, bool norm_q,
                                                  bool norm_k, float eps, float* s_tmp) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
        const float v = x[i] + (bias != nullptr ? __ldg(bias + i) : 0.f);
        if (i < nq) sq = fmaf(v, v, sq);
        else sk = fmaf(v, v, sk);
    }
    return norm_factors(sq, sk, nq, nk, norm_q, norm_k, eps, s_tmp);
}

}  // namespace leankv
