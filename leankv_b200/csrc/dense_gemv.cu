// Dense matrix-vector product over row-major [out][in] weights (bf16 or fp32), fp32 vectors and arithmetic,
// with the steps around a projection fused in: RMS norm with one gain, token shift (a mix of the normed
// vector with the previous token's, per row segment), bias, silu gating of row pairs, and the scaled
// residual sum; or a branch's post-norm and residual sum ahead of the norm, and row groups with an input slice each.
//
// A CTA owns a contiguous range of rows; its warps split the columns and every warp walks all rows of the
// range, so a lane's share of x stays in registers for the whole range and the weight stream needs no
// shared memory. Per-warp row sums go to shared memory once and are added in warp order at the end:
// bit-reproducible.

#include <algorithm>
#include <type_traits>

#include "decode_frame.cuh"
#include "leankv_mixers.h"

namespace leankv {
namespace {

constexpr int kMaxWarps = 16;
constexpr int kSmemPartials = 96 * 1024;
constexpr int kMaxStaged = 32 * 1024;        // columns of a launch that prepares its input in shared memory

struct GemvParams {
    leankv_dense_gemv_t a;
    int slabs;          // column passes of (warps * 32 * 8 * CH)
    int vec;            // cols % 8 == 0: 16-byte loads
    int x_smem;         // floats of shared memory in front of the partial sums: the prepared input
};

template <typename T>
__device__ __forceinline__ void load_w8(const T* row, int k, int cols, bool vec, Raw8<T>& r) {
    if (vec) {
        if (k < cols) stream8(row + k, r);
        else zero8(r);
    } else {
        T tmp[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) tmp[i] = k + i < cols ? row[k + i] : from_f32<T>(0.f);
        memcpy(&r, tmp, sizeof(r));
    }
}

__device__ __forceinline__ void load_x8(const float* x, int k, int cols, bool vec, float (&v)[8]) {
    if (vec) {
        if (k < cols) {
            const float4 a = ld_cg_f32x4(x + k), b = ld_cg_f32x4(x + k + 4);
            v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
            v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = 0.f;
        }
    } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = k + i < cols ? ld_cg_f32(x + k + i) : 0.f;
    }
}

// Sums of R values over the warp; lane l ends with the sum of value (l >> 2) & ... (see row_of_lane).
template <int R>
__device__ __forceinline__ float warp_reduce_rows(float (&acc)[R], int lane) {
    int n = R;
    int o = 16;
#pragma unroll
    for (int half = R / 2; half >= 1; half /= 2) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float send = up ? acc[i] : acc[i + half];
            const float keep = up ? acc[i + half] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
        o >>= 1;
        n = half;
    }
    (void)n;
    float v = acc[0];
    for (; o >= 1; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// The row whose sum warp_reduce_rows leaves in this lane: the lane's top log2(R) bits, most significant first.
template <int R>
__device__ __forceinline__ int row_of_lane(int lane) { return (lane * R) >> 5; }

// kJoined: a branch joins the stream first, or there is a gain per column; every thread prepares its columns in registers
// (one slab). kStaged: the same in shared memory, any number of slabs. kGrouped: row groups with an input slice each.
enum class Input { kPlain, kJoined, kStaged, kGrouped };
template <typename T, int CH, Input IN>
__global__ void __launch_bounds__(512, sizeof(T) == 2 ? 2 : 1) dense_gemv_kernel(const GemvParams p) {
    constexpr bool STAGED = IN == Input::kStaged, JOINED = IN == Input::kJoined, GROUPED = IN == Input::kGrouped;
    constexpr int R = 8 / CH;                        // rows in flight: R * CH 16-byte loads per lane (bf16)
    extern __shared__ __align__(16) float s_dyn[];
    float* s_part = STAGED ? s_dyn + p.x_smem : s_dyn;      // [rows of this CTA (x2 if gated)][warps]
    __shared__ float s_tmp[64];
    const leankv_dense_gemv_t& a = p.a;
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int lo = (int)((long long)a.rows * blockIdx.x / gridDim.x);
    const int hi = (int)((long long)a.rows * (blockIdx.x + 1) / gridDim.x);
    const int cols = a.cols;
    const bool vec = p.vec != 0;
    const T* W = static_cast<const T*>(a.w);
    const int mult = a.gated ? 2 : 1;
    const int slab_cols = warps * 256 * CH;

    {   // the head of this CTA's weight range into L2 while the previous kernel drains
        const size_t bytes = (size_t)(hi - lo) * cols * sizeof(T);
        const int half = blockDim.x / mult, part = a.gated ? threadIdx.x / half : 0;
        const size_t off = (size_t)(threadIdx.x - part * half) * 128;
        if (off < bytes && part < mult) {
            const char* base = reinterpret_cast<const char*>(W + ((size_t)lo + (size_t)part * a.rows) * cols);
            asm volatile("prefetch.global.L2 [%0];" ::"l"(base + off));
        }
    }
    // kJoined: the gains do not depend on the launch ahead
    float gn[CH][8], pg[CH][8];
    if constexpr (JOINED) {
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int k = (c * warps + warp) * 256 + lane * 8;
            if (a.gain_per_col) load_x8(a.gain, k, cols, vec, gn[c]);
            if (a.delta != nullptr) load_x8(a.post_gain, k, cols, vec, pg[c]);
        }
    }
    pdl_begin();

    float rs = 1.f;
    float xj[CH][8];                // kJoined: this thread's columns of x'
    if constexpr (JOINED) {
        float d[CH][8];
        const int k0 = warp * 256 + lane * 8;
        float sd = 0.f, ss = 0.f;
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            load_x8(a.x, c * warps * 256 + k0, cols, vec, xj[c]);
            if (a.delta != nullptr) load_x8(a.delta, c * warps * 256 + k0, cols, vec, d[c]);
        }
        if (a.delta != nullptr) {
#pragma unroll
            for (int c = 0; c < CH; ++c)
#pragma unroll
                for (int i = 0; i < 8; ++i) sd = fmaf(d[c][i], d[c][i], sd);
            const float f = a.post_mult / sqrtf(cta_sum_once(sd, s_tmp) / (float)cols + a.eps);
#pragma unroll
            for (int c = 0; c < CH; ++c) {
                const int k = c * warps * 256 + k0;
#pragma unroll
                for (int i = 0; i < 8; ++i) xj[c][i] = fmaf(d[c][i] * f, pg[c][i], xj[c][i]);
                if (blockIdx.x == 0)
#pragma unroll
                    for (int i = 0; i < 8; ++i)
                        if (k + i < cols) a.x_out[k + i] = xj[c][i];
            }
        }
#pragma unroll
        for (int c = 0; c < CH; ++c)
#pragma unroll
            for (int i = 0; i < 8; ++i) ss = fmaf(xj[c][i], xj[c][i], ss);
        if (a.gain != nullptr) {
            rs = (a.gain_per_col ? 1.f : __ldg(a.gain)) / sqrtf(cta_sum_once(ss, s_tmp + 32) / (float)cols + a.eps);
#pragma unroll
            for (int c = 0; c < CH; ++c)
#pragma unroll
                for (int i = 0; i < 8; ++i) xj[c][i] *= a.gain_per_col ? rs * gn[c][i] : rs;
        }
        if (a.prev != nullptr && blockIdx.x == 0) {
            float* next = a.prev + (size_t)((a.state[kParity] & 1) ^ 1) * cols;
#pragma unroll
            for (int c = 0; c < CH; ++c)
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    if (c * warps * 256 + k0 + i < cols) next[c * warps * 256 + k0 + i] = xj[c][i];
        }
    } else if constexpr (STAGED) {         // the normed input x', after a branch joined x, into shared memory
        float f = 0.f, ss = 0.f;
        if (a.delta != nullptr) {
            float sd = 0.f;
            for (int k = threadIdx.x; k < cols; k += blockDim.x) {
                const float d = ld_cg_f32(a.delta + k);
                s_dyn[k] = d;
                sd = fmaf(d, d, sd);
            }
            f = a.post_mult / sqrtf(cta_sum(sd, s_tmp) / (float)cols + a.eps);
        }
        for (int k = threadIdx.x; k < cols; k += blockDim.x) {
            float x = ld_cg_f32(a.x + k);
            if (a.delta != nullptr) {
                x = fmaf(s_dyn[k] * f, __ldg(a.post_gain + k), x);
                if (blockIdx.x == 0) a.x_out[k] = x;
            }
            s_dyn[k] = x;
            ss = fmaf(x, x, ss);
        }
        if (a.gain != nullptr) rs = (a.gain_per_col ? 1.f : __ldg(a.gain)) / sqrtf(cta_sum(ss, s_tmp) / (float)cols + a.eps);
        for (int k = threadIdx.x; k < cols; k += blockDim.x) s_dyn[k] *= rs * (a.gain_per_col ? __ldg(a.gain + k) : 1.f);
        __syncthreads();
    } else if (a.gain != nullptr) {
        float ss = 0.f;
        for (int s = 0; s < p.slabs; ++s)
#pragma unroll
            for (int c = 0; c < CH; ++c) {
                float v[8];
                load_x8(a.x, s * slab_cols + (c * warps + warp) * 256 + lane * 8, cols, vec, v);
#pragma unroll
                for (int i = 0; i < 8; ++i) ss = fmaf(v[i], v[i], ss);
            }
        rs = __ldg(a.gain) / sqrtf(cta_sum(ss, s_tmp) / (float)cols + a.eps);
    }
    const float* prev = nullptr;
    if (a.prev != nullptr) {
        const int par = a.state[kParity] & 1;
        prev = a.prev + (size_t)par * cols;
        float* next = a.prev + (size_t)(par ^ 1) * cols;
        if (!JOINED && blockIdx.x == 0)
            for (int k = threadIdx.x; k < cols; k += blockDim.x)
                next[k] = STAGED ? s_dyn[k] : ld_cg_f32(a.x + k) * rs;
    }
    const int m0 = GROUPED ? lo / a.group_rows : 0, m1 = GROUPED ? (hi - 1) / a.group_rows + 1 : max(a.n_mix, 1);

    for (int s = 0; s < p.slabs; ++s) {
        int seg_lo = GROUPED ? m0 * a.group_rows : 0;
        for (int m = m0; m < m1; ++m) {
            const int seg_hi = a.n_mix > 0 ? a.mix_end[m] : GROUPED ? seg_lo + a.group_rows : a.rows;
            const int r0 = max(lo, seg_lo), r1 = min(hi, seg_hi);
            seg_lo = seg_hi;
            if (r0 >= r1) continue;
            const float* mu = a.n_mix > 0 ? a.mu[m] : nullptr;
            float xs[CH][8];
#pragma unroll
            for (int c = 0; c < CH; ++c) {
                const int k = s * slab_cols + (c * warps + warp) * 256 + lane * 8;
                if constexpr (JOINED) {
#pragma unroll
                    for (int i = 0; i < 8; ++i) xs[c][i] = xj[c][i];
                } else if constexpr (STAGED) {
                    const bool on = vec && k < cols;
                    const float4 lo4 = on ? *reinterpret_cast<const float4*>(s_dyn + k) : make_float4(0.f, 0.f, 0.f, 0.f);
                    const float4 hi4 = on ? *reinterpret_cast<const float4*>(s_dyn + k + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
                    xs[c][0] = lo4.x; xs[c][1] = lo4.y; xs[c][2] = lo4.z; xs[c][3] = lo4.w;
                    xs[c][4] = hi4.x; xs[c][5] = hi4.y; xs[c][6] = hi4.z; xs[c][7] = hi4.w;
                    if (!vec)
#pragma unroll
                        for (int i = 0; i < 8; ++i) xs[c][i] = k + i < cols ? s_dyn[k + i] : 0.f;
                } else {
                    load_x8(GROUPED ? a.x + (size_t)m * a.group_stride : a.x, k, cols, vec, xs[c]);
#pragma unroll
                    for (int i = 0; i < 8; ++i) xs[c][i] *= rs;
                }
                if (mu != nullptr) {
                    float pv[8], mv[8];
                    load_x8(prev, k, cols, vec, pv);
                    load_x8(mu, k, cols, vec, mv);
#pragma unroll
                    for (int i = 0; i < 8; ++i) xs[c][i] = fmaf(pv[i] - xs[c][i], mv[i], xs[c][i]);
                }
            }
            const int v0 = (r0 - lo) * mult, v1 = (r1 - lo) * mult;
            for (int v = v0; v < v1; v += R) {
                Raw8<T> raw[R][CH];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const int vr = min(v + r, v1 - 1);
                    const size_t row = a.gated ? (size_t)(lo + (vr >> 1)) + (size_t)(vr & 1) * a.rows : (size_t)(lo + vr);
#pragma unroll
                    for (int c = 0; c < CH; ++c)
                        load_w8(W + row * cols, s * slab_cols + (c * warps + warp) * 256 + lane * 8, cols, vec, raw[r][c]);
                }
                float acc[R];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    acc[r] = 0.f;
#pragma unroll
                    for (int c = 0; c < CH; ++c) {
                        float w[8];
                        unpack8(raw[r][c], w);
#pragma unroll
                        for (int i = 0; i < 8; ++i) acc[r] = fmaf(w[i], xs[c][i], acc[r]);
                    }
                }
                const float sum = warp_reduce_rows<R>(acc, lane);
                const int vr = v + row_of_lane<R>(lane);
                if ((lane & (32 / R - 1)) == 0 && vr < v1) {
                    float* dst = s_part + (size_t)vr * warps + warp;
                    *dst = s == 0 ? sum : *dst + sum;
                }
            }
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < hi - lo; i += blockDim.x) {
        const int row = lo + i;
        auto total = [&](int v) {
            float t = 0.f;
            for (int w = 0; w < warps; ++w) t += s_part[(size_t)v * warps + w];
            return t;
        };
        float y;
        if (a.gated) {
            const float g = total(2 * i), u = total(2 * i + 1);
            y = g * sigmoid_f32(g) * u;
        } else {
            y = total(i);
            if (a.bias != nullptr && row < a.bias_rows) y += __ldg(a.bias + row);
        }
        if (a.softcap > 0.f) y = a.softcap * tanhf(y / a.softcap);
        if (a.residual != nullptr) y = a.residual[row] + y * __ldg(a.scale + row);
        a.y[row] = y;
    }
}

template <typename T, int CH, Input IN>
int launch_gemv(const GemvParams& p, int warps, cudaStream_t st) {
    const int per_sm = std::max(1, (sizeof(T) == 2 ? 2 : 1) * kMaxWarps / warps);
    const int mult = p.a.gated ? 2 : 1;
    int grid = std::min(sm_count() * std::min(per_sm, 8), (p.a.rows + 1) / 2);
    grid = std::max(grid, 1);
    const auto smem_for = [&](int g) { return (size_t)((p.a.rows + g - 1) / g) * mult * warps * sizeof(float); };
    while (smem_for(grid) > (size_t)kSmemPartials / 2 && grid < p.a.rows) grid = std::min(p.a.rows, grid * 2);
    const size_t smem = smem_for(grid) + (size_t)p.x_smem * sizeof(float);
    if (smem > 48 * 1024)
        LEANKV_CUDA_TRY(cudaFuncSetAttribute(dense_gemv_kernel<T, CH, IN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             kSmemPartials + kMaxStaged * (int)sizeof(float)));
    LEANKV_CUDA_TRY(launch_kernel_ex(true, dense_gemv_kernel<T, CH, IN>, dim3(grid), dim3(warps * 32), smem, st, p));
    return LEANKV_OK;
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" int leankv_dense_gemv(const leankv_dense_gemv_t* a, void* stream) {
    if (!a || !a->w || !a->x || !a->y || a->rows <= 0 || a->cols <= 0) return LEANKV_EINVAL;
    if (a->dtype != LEANKV_DT_BF16 && a->dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    if (a->x == a->y || a->n_mix < 0 || a->n_mix > LEANKV_MAX_MIX) return LEANKV_EINVAL;
    if (a->residual && !a->scale) return LEANKV_EINVAL;
    if (a->n_mix > 0) {
        if (!a->prev || !a->state || !a->gain || a->gated) return LEANKV_EINVAL;
        for (int i = 0, e = 0; i < a->n_mix; e = a->mix_end[i++])
            if (a->mix_end[i] <= e || (i == a->n_mix - 1 && a->mix_end[i] != a->rows)) return LEANKV_EINVAL;
    } else if (a->prev) {
        return LEANKV_EINVAL;
    }
    if (a->delta && (!a->post_gain || !a->x_out || a->x_out == a->x || a->x_out == a->delta || a->delta == a->y))
        return LEANKV_EINVAL;
    if ((a->delta || a->gain_per_col) && a->cols > kMaxStaged) return LEANKV_ELIMIT;
    if (a->group_rows < 0 || (a->group_rows > 0 && (a->rows % a->group_rows || a->group_stride < 0 || a->gain || a->delta ||
                                                    a->n_mix > 0 || a->gated)))
        return LEANKV_EINVAL;
    if (!aligned16(a->w) || !aligned16(a->x) || (a->gain_per_col && !aligned16(a->gain)) ||
        (a->delta && (!aligned16(a->delta) || !aligned16(a->post_gain)))) return LEANKV_EALIGN;
    GemvParams p{};
    p.a = *a;
    p.vec = a->cols % 8 == 0 && (a->group_rows == 0 || a->group_stride % 4 == 0);
    const bool staged = a->delta || (a->gain && a->gain_per_col);
    // warps x slabs x CH column chunks of 256: the widest CTA that pads least
    const int chunks = (a->cols + 255) / 256;
    int warps = 1, per = 1;
    long long best = -1;
    for (int w = 1; w <= std::min(chunks, kMaxWarps); ++w)
        for (int ch = 1; ch <= 2; ++ch) {
            const long long pad = (long long)((chunks + w * ch - 1) / (w * ch)) * w * ch;
            const long long score = pad * 64 - 2 * w - ch;      // least padding, then more warps
            if (best < 0 || score < best) { best = score; warps = w; per = ch; }
        }
    p.slabs = (chunks + warps * per - 1) / (warps * per);
    p.x_smem = staged && p.slabs > 1 ? (a->cols + 3) / 4 * 4 : 0;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        const auto with = [&](auto in) -> int {
            constexpr Input IN = decltype(in)::value;
            return per == 1 ? launch_gemv<T, 1, IN>(p, warps, st) : launch_gemv<T, 2, IN>(p, warps, st);
        };
        if (staged && p.slabs == 1) return with(std::integral_constant<Input, Input::kJoined>{});
        if (staged) return with(std::integral_constant<Input, Input::kStaged>{});
        if (a->group_rows > 0) return with(std::integral_constant<Input, Input::kGrouped>{});
        return with(std::integral_constant<Input, Input::kPlain>{});
    };
    return a->dtype == LEANKV_DT_BF16 ? go(bf16{}) : go(float{});
}
