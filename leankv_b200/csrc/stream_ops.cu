// Row-wise kernels around the projections of a prompt portion (residual sum, norm, token shift, gating) and
// the two frame kernels of a decode step whose residual stream is fp32.

#include <algorithm>

#include "decode_frame.cuh"
#include "leankv_mixers.h"

namespace leankv {
namespace {

constexpr int kRowThreads = 256;

// One CTA per row. With token shift the row above is normed a second time here (two rows of L2 reads)
// rather than handed over through memory, so rows stay independent and one launch does the whole chain.
template <typename T, typename D>
__global__ void __launch_bounds__(kRowThreads) stream_norm_kernel(const leankv_stream_norm_t a) {
    __shared__ float s_tmp[32];
    pdl_begin();
    const int t = blockIdx.x, W = a.width;
    const D* delta = static_cast<const D*>(a.delta);
    const float* scale = a.post_gain != nullptr ? a.post_gain : a.scale;
    const bool shift = a.n_mix > 0;
    auto branch_factor = [&](int row) {         // of a branch that is normed before it joins the stream
        if (a.post_gain == nullptr) return 1.f;
        float ss = 0.f;
        for (int i = threadIdx.x; i < W; i += kRowThreads) {
            const float d = to_f32(delta[(size_t)row * W + i]);
            ss = fmaf(d, d, ss);
        }
        return a.post_mult / sqrtf(cta_sum(ss, s_tmp) / (float)W + a.eps);
    };
    const float f_here = branch_factor(t), f_above = shift && t > 0 ? branch_factor(t - 1) : 1.f;
    auto value = [&](int row, int i) {
        float x = a.x_in[(size_t)row * W + i];
        if (delta != nullptr)
            x = fmaf(to_f32(delta[(size_t)row * W + i]) * (row == t ? f_here : f_above), __ldg(scale + i), x);
        return x;
    };
    float ss = 0.f, ss_above = 0.f;
    for (int i = threadIdx.x; i < W; i += kRowThreads) {
        const float x = value(t, i);
        ss = fmaf(x, x, ss);
        if (delta != nullptr) a.x_out[(size_t)t * W + i] = x;
        if (shift && t > 0) {
            const float y = value(t - 1, i);
            ss_above = fmaf(y, y, ss_above);
        }
    }
    if (a.gain == nullptr) return;
    const float gain = a.gain_per_col ? 1.f : __ldg(a.gain);
    const float rs = gain / sqrtf(cta_sum(ss, s_tmp) / (float)W + a.eps);
    float rs_above = 0.f;
    if (shift && t > 0) rs_above = gain / sqrtf(cta_sum(ss_above, s_tmp) / (float)W + a.eps);
    T* h = static_cast<T*>(a.h);
    T* mixed = static_cast<T*>(a.mixed);
    for (int i = threadIdx.x; i < W; i += kRowThreads) {
        const float ci = a.gain_per_col ? __ldg(a.gain + i) : 1.f;
        const float hv = value(t, i) * rs * ci;
        if (h != nullptr) h[(size_t)t * W + i] = from_f32<T>(hv);
        if (shift) {
            const float d = (t > 0 ? value(t - 1, i) * rs_above * ci : a.prev_in[i]) - hv;
            for (int m = 0; m < a.n_mix; ++m)
                mixed[((size_t)m * a.rows + t) * W + i] = from_f32<T>(fmaf(d, __ldg(a.mu[m] + i), hv));
        }
        if (a.prev_out != nullptr && t == a.rows - 1) a.prev_out[i] = hv;
    }
}

template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&v)[4]) { leankv::store4(p, make_float4(v[0], v[1], v[2], v[3])); }
__device__ __forceinline__ void fetch4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void fetch4(const bf16* p, float (&v)[4]) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(a.x << 16); v[1] = __uint_as_float(a.x & 0xffff0000u);
    v[2] = __uint_as_float(a.y << 16); v[3] = __uint_as_float(a.y & 0xffff0000u);
}

// The same with 4-element accesses and rows in registers (width % 4 == 0, width <= kRowThreads * 4 * NV). A CTA
// walks `per_cta` consecutive rows and keeps the row above, so only its first row is normed twice.
template <typename T, typename D, int NV>
__global__ void __launch_bounds__(kRowThreads) stream_norm_vec_kernel(const leankv_stream_norm_t a, int per_cta) {
    __shared__ float s_tmp[32];
    pdl_begin();
    const int W = a.width, r0 = blockIdx.x * per_cta, r1 = min(a.rows, r0 + per_cta), tid = threadIdx.x;
    const D* delta = static_cast<const D*>(a.delta);
    T* h = static_cast<T*>(a.h);
    T* mixed = static_cast<T*>(a.mixed);
    const bool shift = a.n_mix > 0, post = a.post_gain != nullptr, per_col = a.gain_per_col != 0;
    const float gain = a.gain == nullptr || per_col ? 1.f : __ldg(a.gain);
    const float* scale = post ? a.post_gain : a.scale;
    float cur[NV][4], above[NV][4];
    auto load = [&](int row, bool store) -> float {       // the updated stream of `row` into cur; its norm factor
        float ss = 0.f, f = 1.f;
        if (post) {                                       // the branch is normed before it joins
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int i = (tid + n * kRowThreads) * 4;
                if (i >= W) continue;
                float dv[4];
                fetch4(delta + (size_t)row * W + i, dv);
#pragma unroll
                for (int q = 0; q < 4; ++q) ss = fmaf(dv[q], dv[q], ss);
            }
            f = a.post_mult / sqrtf(cta_sum(ss, s_tmp) / (float)W + a.eps);
            ss = 0.f;
        }
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (tid + n * kRowThreads) * 4;
            if (i < W) {
                fetch4(a.x_in + (size_t)row * W + i, cur[n]);
                if (delta != nullptr) {
                    float dv[4], sv[4];
                    fetch4(delta + (size_t)row * W + i, dv);
                    fetch4(scale + i, sv);
#pragma unroll
                    for (int q = 0; q < 4; ++q) cur[n][q] = fmaf(dv[q] * f, sv[q], cur[n][q]);
                    if (store) store4(a.x_out + (size_t)row * W + i, cur[n]);
                }
#pragma unroll
                for (int q = 0; q < 4; ++q) ss = fmaf(cur[n][q], cur[n][q], ss);
            }
        }
        return a.gain == nullptr ? 1.f : gain / sqrtf(cta_sum(ss, s_tmp) / (float)W + a.eps);
    };
    auto norm = [&](int n, float rs) {
        const int i = (tid + n * kRowThreads) * 4;
        float g[4] = {1.f, 1.f, 1.f, 1.f};
        if (per_col && i < W) fetch4(a.gain + i, g);
#pragma unroll
        for (int q = 0; q < 4; ++q) cur[n][q] *= rs * g[q];
    };
    if (shift) {
        if (r0 > 0) {
            const float rs = load(r0 - 1, false);
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                norm(n, rs);
#pragma unroll
                for (int q = 0; q < 4; ++q) above[n][q] = cur[n][q];
            }
        } else {
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int i = (tid + n * kRowThreads) * 4;
                if (i < W) fetch4(a.prev_in + i, above[n]);
            }
        }
    }
    for (int row = r0; row < r1; ++row) {
        const float rs = load(row, true);
        if (a.gain == nullptr) continue;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (tid + n * kRowThreads) * 4;
            if (i >= W) continue;
            norm(n, rs);
            if (h != nullptr) store4(h + (size_t)row * W + i, cur[n]);
            if (shift) {
                for (int m = 0; m < a.n_mix; ++m) {
                    float mv[4];
                    fetch4(a.mu[m] + i, mv);
#pragma unroll
                    for (int q = 0; q < 4; ++q) mv[q] = fmaf(above[n][q] - cur[n][q], mv[q], cur[n][q]);
                    store4(mixed + ((size_t)m * a.rows + row) * W + i, mv);
                }
#pragma unroll
                for (int q = 0; q < 4; ++q) above[n][q] = cur[n][q];
                if (row == a.rows - 1) store4(a.prev_out + i, cur[n]);
            }
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) silu_mul_rows_kernel(const T* gate_up, T* out, int inter, long long total) {
    pdl_begin();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / inter, c = i - r * inter;
        const float g = to_f32(gate_up[r * 2 * inter + c]), u = to_f32(gate_up[r * 2 * inter + inter + c]);
        out[i] = from_f32<T>(g * sigmoid_f32(g) * u);
    }
}

// Eight elements per thread (inter % 8 == 0, aligned).
template <typename T>
__global__ void __launch_bounds__(256) silu_mul_vec_kernel(const T* gate_up, T* out, int inter, long long total8) {
    pdl_begin();
    const int n8 = inter >> 3;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total8;
         i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / n8;
        const int c = (int)(i - r * n8) * 8;
        Raw8<T> rg, ru;
        load8(gate_up + r * 2 * inter + c, rg);
        load8(gate_up + r * 2 * inter + inter + c, ru);
        float g[8], u[8];
        unpack8(rg, g);
        unpack8(ru, u);
        T o[8];
#pragma unroll
        for (int q = 0; q < 8; ++q) o[q] = from_f32<T>(g[q] * sigmoid_f32(g[q]) * u[q]);
        memcpy(&rg, o, sizeof(rg));
        *reinterpret_cast<Raw8<T>*>(out + r * inter + c) = rg;
    }
}

template <typename T>
__global__ void __launch_bounds__(256) tanh_split_kernel(const float* in, T* out, int n, long long total) {
    pdl_begin();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (long long)gridDim.x * blockDim.x) {
        const float v = tanhf(in[i]);
        if constexpr (sizeof(T) == 4) {
            out[i] = v;
        } else {
            const long long r = i / n, c = i - r * n;
            const T hi = from_f32<T>(v);
            out[r * 2 * n + c] = hi;
            out[r * 2 * n + n + c] = from_f32<T>(v - to_f32(hi));
        }
    }
}

__global__ void __launch_bounds__(256) softcap_kernel(float* x, long long n, float cap) {
    pdl_begin();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

template <typename T, typename D>
int launch_stream_norm(const leankv_stream_norm_t* a, cudaStream_t st) {
    bool vec = a->width % 4 == 0 && a->width <= kRowThreads * 4 * 8 && aligned16(a->x_in) && aligned16(a->x_out) &&
               aligned16(a->delta) && aligned16(a->scale) && aligned16(a->h) && aligned16(a->mixed) &&
               aligned16(a->prev_in) && aligned16(a->prev_out) && aligned16(a->post_gain) &&
               (!a->gain_per_col || aligned16(a->gain));
    for (int i = 0; i < a->n_mix; ++i) vec = vec && aligned16(a->mu[i]);
    if (!vec) {
        LEANKV_CUDA_TRY(launch_kernel(stream_norm_kernel<T, D>, dim3(a->rows), dim3(kRowThreads), 0, st, *a));
        return LEANKV_OK;
    }
    const int per = a->n_mix > 0 && a->rows >= sm_count() * 8 ? 4 : 1;
    const dim3 grid((a->rows + per - 1) / per), block(kRowThreads);
    const int nv = (a->width + kRowThreads * 4 - 1) / (kRowThreads * 4);
    if (nv <= 1) LEANKV_CUDA_TRY(launch_kernel(stream_norm_vec_kernel<T, D, 1>, grid, block, 0, st, *a, per));
    else if (nv <= 2) LEANKV_CUDA_TRY(launch_kernel(stream_norm_vec_kernel<T, D, 2>, grid, block, 0, st, *a, per));
    else if (nv <= 4) LEANKV_CUDA_TRY(launch_kernel(stream_norm_vec_kernel<T, D, 4>, grid, block, 0, st, *a, per));
    else LEANKV_CUDA_TRY(launch_kernel(stream_norm_vec_kernel<T, D, 8>, grid, block, 0, st, *a, per));
    return LEANKV_OK;
}

bool known(int dtype) { return dtype == LEANKV_DT_BF16 || dtype == LEANKV_DT_F32; }

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" int leankv_embed_begin(const void* table, int dtype, const long long* token, float* x, int width,
                                  int vocab, int32_t* state, void* stream) {
    if (!table || !token || !x || !state || width <= 0 || vocab <= 0) return LEANKV_EINVAL;
    if (!known(dtype)) return LEANKV_EUNSUPPORTED;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (dtype == LEANKV_DT_BF16)
        LEANKV_CUDA_TRY(launch_kernel(decode_begin_kernel<bf16, float>, dim3(1), dim3(256), 0, st,
                                      static_cast<const bf16*>(table), token, x, width, vocab, state));
    else
        LEANKV_CUDA_TRY(launch_kernel(decode_begin_kernel<float, float>, dim3(1), dim3(256), 0, st,
                                      static_cast<const float*>(table), token, x, width, vocab, state));
    return LEANKV_OK;
}

extern "C" int leankv_greedy_end(const float* logits, int vocab, long long* token, long long* history,
                                 int history_cap, int32_t* state, void* stream) {
    if (!logits || !token || !history || !state || vocab <= 0 || history_cap < 0) return LEANKV_EINVAL;
    if (!aligned16(logits)) return LEANKV_EALIGN;
    LEANKV_CUDA_TRY(launch_kernel(decode_end_kernel<float>, dim3(1), dim3(1024), 0, static_cast<cudaStream_t>(stream),
                                  logits, vocab, token, history, history_cap, state + kPos, state + kStep,
                                  state + kParity));
    return LEANKV_OK;
}

extern "C" int leankv_stream_norm(const leankv_stream_norm_t* a, void* stream) {
    if (!a || !a->x_in || a->rows <= 0 || a->width <= 0 || a->n_mix < 0 || a->n_mix > LEANKV_MAX_MIX) return LEANKV_EINVAL;
    if (!a->gain && (a->h || a->n_mix > 0 || !a->delta)) return LEANKV_EINVAL;
    if (a->delta && (!a->x_out || (!a->scale && !a->post_gain) || a->x_out == a->x_in)) return LEANKV_EINVAL;
    if (a->post_gain && !a->delta) return LEANKV_EINVAL;
    if (a->n_mix > 0) {
        if (!a->mixed || !a->prev_in || !a->prev_out || a->prev_in == a->prev_out) return LEANKV_EINVAL;
        for (int i = 0; i < a->n_mix; ++i)
            if (!a->mu[i]) return LEANKV_EINVAL;
    }
    if (!known(a->dtype) || (a->delta && !known(a->delta_dtype))) return LEANKV_EUNSUPPORTED;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const bool d16 = a->delta && a->delta_dtype == LEANKV_DT_BF16;
    if (a->dtype == LEANKV_DT_BF16)
        return d16 ? launch_stream_norm<bf16, bf16>(a, st) : launch_stream_norm<bf16, float>(a, st);
    return d16 ? launch_stream_norm<float, bf16>(a, st) : launch_stream_norm<float, float>(a, st);
}

extern "C" int leankv_silu_mul(const void* gate_up, void* out, int dtype, int rows, int inter, void* stream) {
    if (!gate_up || !out || rows <= 0 || inter <= 0) return LEANKV_EINVAL;
    if (!known(dtype)) return LEANKV_EUNSUPPORTED;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const bool vec = inter % 8 == 0 && aligned16(gate_up) && aligned16(out);
    const long long total = (long long)rows * inter / (vec ? 8 : 1);
    const int grid = (int)std::min<long long>((total + 255) / 256, (long long)sm_count() * 16);
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        LEANKV_CUDA_TRY(launch_kernel(vec ? silu_mul_vec_kernel<T> : silu_mul_rows_kernel<T>, dim3(grid), dim3(256), 0,
                                      st, static_cast<const T*>(gate_up), static_cast<T*>(out), inter, total));
        return LEANKV_OK;
    };
    return dtype == LEANKV_DT_BF16 ? go(bf16{}) : go(float{});
}

extern "C" int leankv_tanh_split(const float* in, void* out, int dtype, int rows, int n, void* stream) {
    if (!in || !out || rows <= 0 || n <= 0) return LEANKV_EINVAL;
    if (!known(dtype)) return LEANKV_EUNSUPPORTED;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const long long total = (long long)rows * n;
    const int grid = (int)std::min<long long>((total + 255) / 256, (long long)sm_count() * 8);
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        LEANKV_CUDA_TRY(launch_kernel(tanh_split_kernel<T>, dim3(grid), dim3(256), 0, st, in, static_cast<T*>(out), n,
                                      total));
        return LEANKV_OK;
    };
    return dtype == LEANKV_DT_BF16 ? go(bf16{}) : go(float{});
}

extern "C" int leankv_softcap(float* x, long long n, float cap, void* stream) {
    if (!x || n <= 0 || !(cap > 0.f)) return LEANKV_EINVAL;
    const int grid = (int)std::min<long long>((n + 255) / 256, (long long)sm_count() * 8);
    LEANKV_CUDA_TRY(launch_kernel(softcap_kernel, dim3(grid), dim3(256), 0, static_cast<cudaStream_t>(stream), x, n, cap));
    return LEANKV_OK;
}
