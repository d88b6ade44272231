// Window + pooled-block attention of a prompt portion: append (q / k norm, ring write), pooling of the blocks
// that become complete, and attention.

#include <algorithm>

#include "window_pool.cuh"

namespace leankv {
namespace {

constexpr int kAppendThreads = 256;
constexpr int kAttendThreads = 256;
constexpr int kAttendSmemFloats = 200 * 1024 / 4;

// One CTA per token: bias and norm over the whole q / k projections, q to the chunk buffer, k / v into the ring.
template <typename T>
__global__ void __launch_bounds__(kAppendThreads) window_pool_append_kernel(const leankv_window_pool_t a,
                                                                            const float* qkv, int ld, const float* bias,
                                                                            T* q_out, int start) {
    __shared__ float s_tmp[32];
    pdl_begin();
    const int t = blockIdx.x, G = a.kv_heads, nq = a.heads * a.dim, nk = G * a.dim;
    const float* row = qkv + (size_t)t * ld;
    const int slot = (start + t) % a.ring;
    const RowFactors f = row_factors(row, bias, nq, nk, a.q_norm != nullptr, a.k_norm != nullptr, a.eps, s_tmp);
    auto at = [&](int i) { return row[i] + (bias != nullptr ? __ldg(bias + i) : 0.f); };
    T* q = q_out + (size_t)t * a.heads * a.dim_pad;
    for (int e = threadIdx.x; e < a.heads * a.dim_pad; e += kAppendThreads) {
        const int h = e / a.dim_pad, d = e - h * a.dim_pad, i = h * a.dim + d;
        q[e] = from_f32<T>(d < a.dim ? at(i) * f.q * (a.q_norm ? __ldg(a.q_norm + i) : 1.f) : 0.f);
    }
    T* k = static_cast<T*>(a.k_ring) + (size_t)slot * G * a.dim_pad;
    for (int e = threadIdx.x; e < G * a.dim_pad; e += kAppendThreads) {
        const int g = e / a.dim_pad, d = e - g * a.dim_pad, i = g * a.dim + d;
        k[e] = from_f32<T>(d < a.dim ? at(nq + i) * f.k * (a.k_norm ? __ldg(a.k_norm + i) : 1.f) : 0.f);
    }
    T* v = static_cast<T*>(a.v_ring) + (size_t)slot * G * a.vdim_pad;
    for (int e = threadIdx.x; e < G * a.vdim_pad; e += kAppendThreads) {
        const int g = e / a.vdim_pad, d = e - g * a.vdim_pad;
        v[e] = from_f32<T>(d < a.vdim ? at(nq + nk + g * a.vdim + d) : 0.f);
    }
}

// The same with 4-element accesses, the row in registers (dim, vdim and ld multiples of 4, at most
// kAppendThreads * 4 * NV columns).
template <typename T, int NV>
__global__ void __launch_bounds__(kAppendThreads) window_pool_append_vec_kernel(const leankv_window_pool_t a,
                                                                                const float* qkv, int ld,
                                                                                const float* bias, T* q_out, int start) {
    __shared__ float s_tmp[32];
    pdl_begin();
    const int t = blockIdx.x, tid = threadIdx.x, G = a.kv_heads, nq = a.heads * a.dim, nk = G * a.dim, nv = G * a.vdim;
    const float* row = qkv + (size_t)t * ld;
    const int slot = (start + t) % a.ring;
    float4 x[NV];
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (tid + n * kAppendThreads) * 4;
        if (i >= nq + nk + nv) continue;
        x[n] = *reinterpret_cast<const float4*>(row + i);
        if (bias != nullptr) {
            const float4 b = *reinterpret_cast<const float4*>(bias + i);
            x[n].x += b.x; x[n].y += b.y; x[n].z += b.z; x[n].w += b.w;
        }
        const float ss = x[n].x * x[n].x + x[n].y * x[n].y + x[n].z * x[n].z + x[n].w * x[n].w;
        if (i < nq) sq += ss;
        else if (i < nq + nk) sk += ss;
    }
    const RowFactors f = norm_factors(sq, sk, nq, nk, a.q_norm != nullptr, a.k_norm != nullptr, a.eps, s_tmp);
    T* q = q_out + (size_t)t * a.heads * a.dim_pad;
    T* k = static_cast<T*>(a.k_ring) + (size_t)slot * G * a.dim_pad;
    T* v = static_cast<T*>(a.v_ring) + (size_t)slot * G * a.vdim_pad;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        int i = (tid + n * kAppendThreads) * 4;
        if (i >= nq + nk + nv) continue;
        const bool is_q = i < nq, is_k = !is_q && i < nq + nk;
        T* dst;
        if (is_q || is_k) {
            const float* w = is_q ? a.q_norm : a.k_norm;
            const float fac = is_q ? f.q : f.k;
            if (is_k) i -= nq;
            if (w != nullptr) {
                const float4 g = *reinterpret_cast<const float4*>(w + i);
                x[n].x *= g.x; x[n].y *= g.y; x[n].z *= g.z; x[n].w *= g.w;
            }
            x[n].x *= fac; x[n].y *= fac; x[n].z *= fac; x[n].w *= fac;
            const int h = i / a.dim;
            dst = (is_q ? q : k) + h * a.dim_pad + i - h * a.dim;
        } else {
            i -= nq + nk;
            const int g = i / a.vdim;
            dst = v + g * a.vdim_pad + i - g * a.vdim;
        }
        store4(dst, x[n]);
    }
    const int pd = a.dim_pad - a.dim, pv = a.vdim_pad - a.vdim;
    for (int e = tid; e < a.heads * pd; e += kAppendThreads) q[e / pd * a.dim_pad + a.dim + e % pd] = from_f32<T>(0.f);
    for (int e = tid; e < G * pd; e += kAppendThreads) k[e / pd * a.dim_pad + a.dim + e % pd] = from_f32<T>(0.f);
    for (int e = tid; e < G * pv; e += kAppendThreads) v[e / pv * a.vdim_pad + a.vdim + e % pv] = from_f32<T>(0.f);
}

// Blocks first .. : mean of the block's keys / values as the ring holds them. One CTA per block, eight columns
// per thread (both paddings are multiples of 16).
template <typename T>
__global__ void __launch_bounds__(256) window_pool_blocks_kernel(const leankv_window_pool_t a, int first) {
    pdl_begin();
    const int b = first + blockIdx.x, slot0 = (int)((long long)b * a.pool % a.ring);
    const int nk = a.kv_heads * a.dim_pad, nv = a.kv_heads * a.vdim_pad;
    const float size = (float)a.pool;
    for (int e = threadIdx.x * 8; e < nk + nv; e += 256 * 8) {
        const bool key = e < nk;
        const int n = key ? nk : nv, col = key ? e : e - nk;
        const T* src = static_cast<const T*>(key ? a.k_ring : a.v_ring) + col;
        float t[8] = {};
        int slot = slot0;
#pragma unroll 8
        for (int i = 0; i < a.pool; ++i) {
            Raw8<T> r;
            load8(src + (size_t)slot * n, r);
            float v[8];
            unpack8(r, v);
#pragma unroll
            for (int x = 0; x < 8; ++x) t[x] += v[x];
            slot = slot + 1 == a.ring ? 0 : slot + 1;
        }
        T* dst = static_cast<T*>(key ? a.k_pool : a.v_pool) + (size_t)b * n + col;
#pragma unroll
        for (int x = 0; x < 8; x += 4)
            store4(dst + x, make_float4(t[x] / size, t[x + 1] / size, t[x + 2] / size, t[x + 3] / size));
    }
}

// One CTA per query row (the fp32 route, and shapes the tile kernel does not take).
template <typename T>
__global__ void __launch_bounds__(kAttendThreads) window_pool_rows_kernel(const leankv_window_pool_t a, const T* q,
                                                                          T* out, int out_ld, float out_scale,
                                                                          int start, int n_max, float* ws) {
    extern __shared__ __align__(16) float sm[];
    pdl_begin();
    const int t = blockIdx.x;
    const AttendPlan pl(a, kAttendThreads, n_max, kAttendSmemFloats);
    const T* row = q + (size_t)t * a.heads * a.dim_pad;
    put_talk(a, pl, sm);
    for (int e = threadIdx.x; e < a.heads * a.dim_pad; e += kAttendThreads) {
        const int h = e / a.dim_pad;
        put_query<T>(pl, sm, a.heads, h, e - h * a.dim_pad, to_f32(row[e]) * a.scale);
    }
    __syncthreads();
    attend_query<T, T>(a, pl, sm, ws + (size_t)t * 2 * a.heads * pl.ldp, start + t, false, 0, 1,
                       out + (size_t)t * out_ld, out_scale);
}

int check_args(const leankv_window_pool_t* a) {
    if (!a || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 ||
        a->dim_pad < a->dim || a->vdim_pad < a->vdim || a->size <= 0 || a->pool <= 0 || a->ring <= 0 ||
        a->max_blocks < 0 || !a->k_ring || !a->v_ring || (a->max_blocks > 0 && (!a->k_pool || !a->v_pool)))
        return LEANKV_EINVAL;
    if (a->dim_pad % 16 || a->vdim_pad % 16 || !aligned16(a->k_ring) || !aligned16(a->v_ring) ||
        !aligned16(a->k_pool) || !aligned16(a->v_pool))
        return LEANKV_EALIGN;
    if (a->dtype != LEANKV_DT_BF16 && a->dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    return LEANKV_OK;
}

template <typename T>
int append(const leankv_window_pool_t& a, const float* qkv, int ld, const float* bias, void* q, int rows, int start,
           cudaStream_t st) {
    const int cols = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
    const int nv = (cols + kAppendThreads * 4 - 1) / (kAppendThreads * 4);
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && ld % 4 == 0 && nv <= 12 && aligned16(qkv) && aligned16(bias) &&
                     aligned16(a.q_norm) && aligned16(a.k_norm) && aligned16(q);
    auto go = [&](auto kernel) -> int {
        LEANKV_CUDA_TRY(launch_kernel(kernel, dim3(rows), dim3(kAppendThreads), 0, st, a, qkv, ld, bias,
                                      static_cast<T*>(q), start));
        return LEANKV_OK;
    };
    const int rc = !vec      ? go(window_pool_append_kernel<T>)
                   : nv <= 2 ? go(window_pool_append_vec_kernel<T, 2>)
                   : nv <= 6 ? go(window_pool_append_vec_kernel<T, 6>)
                             : go(window_pool_append_vec_kernel<T, 12>);
    if (rc) return rc;
    const int b0 = start / a.pool, b1 = std::min((start + rows) / a.pool, a.max_blocks);
    if (b1 > b0)
        LEANKV_CUDA_TRY(launch_kernel(window_pool_blocks_kernel<T>, dim3(b1 - b0), dim3(256), 0, st, a, b0));
    return LEANKV_OK;
}

// The most keys any position below max_pos sees (the count never falls from one position to the next).
int max_keys(const leankv_window_pool_t& a, int max_pos) {
    return VisibleKeys(std::max(max_pos - 1, 0), a.size, a.pool).n;
}

template <typename T>
int attend(const leankv_window_pool_t& a, const void* q, void* out, int out_ld, float out_scale, int rows, int start,
           float* ws, cudaStream_t st) {
    const int n_max = max_keys(a, start + rows);
    const AttendPlan pl(a, kAttendThreads, n_max, kAttendSmemFloats);
    const size_t smem = (size_t)pl.total * 4;
    if (smem > 227 * 1024) return LEANKV_ELIMIT;
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(window_pool_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem));
    LEANKV_CUDA_TRY(launch_kernel(window_pool_rows_kernel<T>, dim3(rows), dim3(kAttendThreads), smem, st, a,
                                  static_cast<const T*>(q), static_cast<T*>(out), out_ld, out_scale, start, n_max, ws));
    return LEANKV_OK;
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" int leankv_window_pool_append(const leankv_window_pool_t* a, const float* qkv, int ld, const float* bias,
                                         void* q, int rows, int start, void* stream) {
    const int rc = check_args(a);
    if (rc) return rc;
    if (!qkv || !q || rows <= 0 || start < 0 || ld < (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim)
        return LEANKV_EINVAL;
    if (rows + std::max(a->size, a->pool) - 1 > a->ring) return LEANKV_ELIMIT;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    return a->dtype == LEANKV_DT_BF16 ? append<bf16>(*a, qkv, ld, bias, q, rows, start, st)
                                      : append<float>(*a, qkv, ld, bias, q, rows, start, st);
}

extern "C" size_t leankv_window_pool_workspace_bytes(const leankv_window_pool_t* a, int rows, int max_pos) {
    if (check_args(a) || rows <= 0 || max_pos <= 0) return 0;
    const AttendPlan pl(*a, kAttendThreads, max_keys(*a, max_pos), kAttendSmemFloats);
    return pl.p_in_smem ? 0 : (size_t)rows * 2 * a->heads * pl.ldp * 4;
}

extern "C" int leankv_window_pool_attend(const leankv_window_pool_t* a, const void* q, void* out, int out_ld,
                                         float out_scale, int rows, int start, void* ws, size_t ws_bytes,
                                         void* stream) {
    const int rc = check_args(a);
    if (rc) return rc;
    if (!q || !out || rows <= 0 || start < 0 || out_ld < a->heads * a->vdim) return LEANKV_EINVAL;
    if (VisibleKeys(start + rows - 1, a->size, a->pool).n_blk > a->max_blocks) return LEANKV_ELIMIT;
    if (!aligned16(q)) return LEANKV_EALIGN;
    const int tiled = window_pool_tile_attend(*a, q, out, out_ld, out_scale, rows, start, static_cast<cudaStream_t>(stream));
    if (tiled != LEANKV_EUNSUPPORTED) return tiled;
    if (leankv_window_pool_workspace_bytes(a, rows, start + rows) > (ws ? ws_bytes : 0)) return LEANKV_EWORKSPACE;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    float* w = static_cast<float*>(ws);
    return a->dtype == LEANKV_DT_BF16 ? attend<bf16>(*a, q, out, out_ld, out_scale, rows, start, w, st)
                                      : attend<float>(*a, q, out, out_ld, out_scale, rows, start, w, st);
}
