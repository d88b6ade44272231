// Element types of the kernels that are templated over their storage precision (bf16 or fp32 weights and
// activations, fp32 arithmetic), and small helpers they share.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace leankv {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__half v) { return __half2float(v); }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// v as the storage type holds it
template <typename T> __device__ __forceinline__ float rounded(float v) { return to_f32(from_f32<T>(v)); }

// Eight consecutive elements in registers, before conversion.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> { uint4 a; };
template <> struct Raw8<float> { float4 a, b; };

__device__ __forceinline__ void unpack8(const Raw8<bf16>& r, float (&v)[8]) {
    const uint32_t w[4] = {r.a.x, r.a.y, r.a.z, r.a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void unpack8(const Raw8<float>& r, float (&v)[8]) {
    v[0] = r.a.x; v[1] = r.a.y; v[2] = r.a.z; v[3] = r.a.w;
    v[4] = r.b.x; v[5] = r.b.y; v[6] = r.b.z; v[7] = r.b.w;
}

// Plain 16-byte loads (the address must be 16-byte aligned).
__device__ __forceinline__ void load8(const bf16* p, Raw8<bf16>& r) { r.a = *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ void load8(const float* p, Raw8<float>& r) {
    r.a = reinterpret_cast<const float4*>(p)[0];
    r.b = reinterpret_cast<const float4*>(p)[1];
}

// Streaming loads that do not allocate in L1.
__device__ __forceinline__ void stream8(const bf16* p, Raw8<bf16>& r) { r.a = ld_stream_16(p); }
__device__ __forceinline__ void stream8(const float* p, Raw8<float>& r) {
    const uint4 x = ld_stream_16(p), y = ld_stream_16(p + 4);
    r.a = make_float4(__uint_as_float(x.x), __uint_as_float(x.y), __uint_as_float(x.z), __uint_as_float(x.w));
    r.b = make_float4(__uint_as_float(y.x), __uint_as_float(y.y), __uint_as_float(y.z), __uint_as_float(y.w));
}

__device__ __forceinline__ void zero8(Raw8<bf16>& r) { r.a = make_uint4(0, 0, 0, 0); }
__device__ __forceinline__ void zero8(Raw8<float>& r) { r.a = r.b = make_float4(0.f, 0.f, 0.f, 0.f); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over the CTA (whole warps), the same value in every thread; s_tmp holds 32 floats. The `once` form leaves
// s_tmp in use until the next barrier.
__device__ __forceinline__ float cta_sum_once(float v, float* s_tmp) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    if (lane == 0) s_tmp[warp] = v;
    __syncthreads();
    const int nw = (blockDim.x + 31) >> 5;
    float t = 0.f;
    for (int w = 0; w < nw; ++w) t += s_tmp[w];   // fixed order: bit-reproducible
    return t;
}
__device__ __forceinline__ float cta_sum(float v, float* s_tmp) {
    const float t = cta_sum_once(v, s_tmp);
    __syncthreads();
    return t;
}

// Two floats as packed bf16 (low half first), and what that rounding leaves over, as packed bf16.
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

// Four floats as the storage type, one 8- or 16-byte store.
__device__ __forceinline__ void store4(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }

// D += A B, one m16n8k16 tile, bf16 operands, fp32 accumulation.
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
                 "{%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }

}  // namespace leankv
