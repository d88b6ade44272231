// Causal attention of a prompt portion: rows on their way into rings and operand buffers (norm, rotation,
// padding), and attention on FMA units for the fp32 route and for sizes the tensor-core kernel does not take.

#include <algorithm>

#include "causal_attn.cuh"

namespace leankv {
namespace {

constexpr int kPlaceThreads = 256;
constexpr int kMaxPairs = 512;          // rotated pairs of a head

// One CTA per row; a thread moves pairs of elements, so that a rotation stays in one thread.
template <typename T>
__global__ void __launch_bounds__(kPlaceThreads) place_rows_kernel(const __grid_constant__ leankv_place_rows_t a) {
    __shared__ float s_tmp[32], s_sin[kMaxPairs], s_cos[kMaxPairs];
    pdl_begin();
    const int r = blockIdx.x, tid = threadIdx.x;
    int rot = 0;
    for (int s = 0; s < a.n_seg; ++s) rot = max(rot, a.seg[s].rot);
    for (int i = tid; i < rot / 2; i += kPlaceThreads) sincosf((float)(a.start + r) * __ldg(a.rate + i), &s_sin[i], &s_cos[i]);
    __syncthreads();
    for (int s = 0; s < a.n_seg; ++s) {
        const leankv_row_segment_t& g = a.seg[s];
        const float* src = g.src + (size_t)r * g.ld;
        T* dst = static_cast<T*>(g.dst) + (size_t)(g.ring > 0 ? (a.start + r) % g.ring : r) * g.dst_ld;
        float f = 1.f;
        if (g.gain != nullptr) {
            float ss = 0.f;
            for (int i = tid; i < g.n; i += kPlaceThreads) ss = fmaf(src[i], src[i], ss);
            f = 1.f / sqrtf(cta_sum(ss, s_tmp) / (float)g.n + a.eps);
        }
        const int half = (g.n_pad + 1) / 2;
        const bool pairs = (reinterpret_cast<uintptr_t>(src) & 7) == 0 && g.head_stride % 2 == 0 && g.n % 2 == 0 &&
                           (reinterpret_cast<uintptr_t>(dst) & (2 * sizeof(T) - 1)) == 0 && g.dst_head_stride % 2 == 0 &&
                           g.n_pad % 2 == 0;
        for (int e = tid; e < g.heads * half; e += kPlaceThreads) {
            const int h = e / half, i = (e - h * half) * 2;
            const float* x = src + (size_t)h * g.head_stride;
            T* y = dst + (size_t)h * g.dst_head_stride;
            float2 v;
            if (pairs) v = i < g.n ? *reinterpret_cast<const float2*>(x + i) : make_float2(0.f, 0.f);
            else v = make_float2(i < g.n ? x[i] : 0.f, i + 1 < g.n ? x[i + 1] : 0.f);
            if (g.gain != nullptr) {
                v.x *= f * (i < g.n ? __ldg(g.gain + i) : 0.f);
                v.y *= f * (i + 1 < g.n ? __ldg(g.gain + i + 1) : 0.f);
            }
            if (i < g.rot) v = turn(v.x, v.y, s_sin[i >> 1], s_cos[i >> 1]);
            if constexpr (sizeof(T) == 2) {
                if (pairs) {
                    *reinterpret_cast<uint32_t*>(y + i) = pack_bf16(v.x, v.y);
                    continue;
                }
            }
            y[i] = from_f32<T>(v.x);
            if (i + 1 < g.n_pad) y[i + 1] = from_f32<T>(v.y);
        }
    }
}

// ---- attention on FMA units -----------------------------------------------------------------------------
// A CTA holds kRows (token, query head) rows of one kv head, every warp two of them; keys come 32 at a time, a lane
// a key. Scores and softmax in fp32, outputs accumulate in shared memory.
constexpr int kWarps = 8;
constexpr int kRows = 16;
constexpr int kKeys = 32;
constexpr int kChunk = 64;              // key dimensions staged at a time

template <typename T>
__global__ void __launch_bounds__(32 * kWarps) causal_rows_kernel(const __grid_constant__ leankv_causal_attn_t a, const T* q,
                                                                  const float* gate, int gate_ld, T* out, int out_ld,
                                                                  int rows, int start) {
    extern __shared__ __align__(16) float sm[];
    pdl_begin();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rep = a.heads / a.kv_heads, g = blockIdx.y, D = a.dim_pad + a.shared_pad, V = a.vdim_pad;
    float* s_q = sm;                              // [kRows][D], times the scale
    float* s_o = s_q + kRows * D;                 // [kRows][V]
    float* s_k = s_o + kRows * V;                 // [kKeys][kChunk + 1]
    float* s_p = s_k + kKeys * (kChunk + 1);      // [kRows][kKeys]
    const long long n_rows = (long long)rows * rep, row0 = (long long)blockIdx.x * kRows;
    const int nr = (int)min((long long)kRows, n_rows - row0);
    auto token = [&](int r) { return (int)((row0 + min(r, nr - 1)) / rep); };
    auto head = [&](int r) { return g * rep + (int)((row0 + min(r, nr - 1)) % rep); };
    for (int e = tid; e < kRows * D; e += 32 * kWarps) {
        const int r = e / D, d = e - r * D;
        s_q[e] = to_f32(q[((size_t)token(r) * a.heads + head(r)) * D + d]) * a.scale;
    }
    for (int e = tid; e < kRows * V; e += 32 * kWarps) s_o[e] = 0.f;
    const int lo = first_visible(start + token(0), a.size), hi = start + token(nr - 1);
    const int r0 = 2 * warp;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const T* K = static_cast<const T*>(a.k);
    const T* S = static_cast<const T*>(a.shared);
    const T* VV = a.v != nullptr ? static_cast<const T*>(a.v) : K;
    const int v_row = a.v != nullptr ? a.vdim_pad : a.dim_pad;
    for (int j0 = lo; j0 <= hi; j0 += kKeys) {
        float s[2] = {0.f, 0.f};
        for (int c0 = 0; c0 < D; c0 += kChunk) {
            const int nc = min(kChunk, D - c0);
            __syncthreads();
            for (int e = tid; e < kKeys * nc; e += 32 * kWarps) {
                const int j = e / nc, d = c0 + e - j * nc, p = min(j0 + j, hi);
                const T* src = d < a.dim_pad ? K + ((size_t)ring_slot(p, a.k_base, a.k_ring) * a.kv_heads + g) * a.dim_pad + d
                                             : S + (size_t)ring_slot(p, 0, a.s_ring) * a.shared_pad + d - a.dim_pad;
                s_k[j * (kChunk + 1) + d - c0] = to_f32(*src);
            }
            __syncthreads();
            for (int d = 0; d < nc; ++d) {
                const float kv = s_k[lane * (kChunk + 1) + d];
#pragma unroll
                for (int x = 0; x < 2; ++x) s[x] = fmaf(s_q[(r0 + x) * D + c0 + d], kv, s[x]);
            }
        }
        float f[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = start + token(r0 + x), j = j0 + lane;
            const bool see = j <= i && j >= first_visible(i, a.size);
            const float best = fmaxf(m[x], warp_max(see ? s[x] : -INFINITY));
            const float e = see ? expf(s[x] - best) : 0.f;
            f[x] = m[x] == -INFINITY ? 0.f : expf(m[x] - best);
            l[x] = l[x] * f[x] + warp_sum(e);
            m[x] = best;
            s_p[(r0 + x) * kKeys + lane] = e;
        }
        __syncwarp();
        const int nj = min(kKeys, hi - j0 + 1);
        for (int d = lane; d < a.vdim; d += 32) {
            float acc[2] = {s_o[r0 * V + d] * f[0], s_o[(r0 + 1) * V + d] * f[1]};
            int slot = ring_slot(j0, a.k_base, a.k_ring);
            for (int j = 0; j < nj; ++j) {
                const float v = to_f32(VV[((size_t)slot * a.kv_heads + g) * v_row + d]);
#pragma unroll
                for (int x = 0; x < 2; ++x) acc[x] = fmaf(s_p[(r0 + x) * kKeys + j], v, acc[x]);
                slot = slot + 1 == a.k_ring ? 0 : slot + 1;
            }
            s_o[r0 * V + d] = acc[0];
            s_o[(r0 + 1) * V + d] = acc[1];
        }
        __syncwarp();
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        if (r0 + x >= nr) continue;
        const int t = token(r0 + x), h = head(r0 + x);
        for (int d = lane; d < a.vdim; d += 32) {
            float o = s_o[(r0 + x) * V + d] / l[x];
            if (gate != nullptr) o *= sigmoid_f32(gate[(size_t)t * gate_ld + h * a.vdim + d]);
            out[(size_t)t * out_ld + h * a.vdim + d] = from_f32<T>(o);
        }
    }
}

template <typename T>
int attend_rows(const leankv_causal_attn_t& a, const void* q, const float* gate, int gate_ld, void* out, int out_ld, int rows,
                int start, cudaStream_t st) {
    const size_t smem = 4 * (size_t)(kRows * (a.dim_pad + a.shared_pad + a.vdim_pad) + kKeys * (kChunk + 1) + kRows * kKeys);
    if (smem > 227 * 1024 || a.kv_heads > 65535) return LEANKV_ELIMIT;
    const long long n = (long long)rows * (a.heads / a.kv_heads);
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(causal_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    LEANKV_CUDA_TRY(launch_kernel(causal_rows_kernel<T>, dim3((unsigned)((n + kRows - 1) / kRows), a.kv_heads),
                                  dim3(32 * kWarps), smem, st, a, static_cast<const T*>(q), gate, gate_ld,
                                  static_cast<T*>(out), out_ld, rows, start));
    return LEANKV_OK;
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" int leankv_place_rows(const leankv_place_rows_t* a, void* stream) {
    if (!a || a->rows <= 0 || a->start < 0 || a->n_seg <= 0 || a->n_seg > LEANKV_MAX_SEGMENTS) return LEANKV_EINVAL;
    if (a->dtype != LEANKV_DT_BF16 && a->dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    for (int s = 0; s < a->n_seg; ++s) {
        const leankv_row_segment_t& g = a->seg[s];
        if (!g.src || !g.dst || g.heads <= 0 || g.n <= 0 || g.n_pad < g.n || g.ring < 0 || g.rot < 0 || g.rot > g.n || g.rot % 2 ||
            (g.rot > 0 && !a->rate) || (g.gain && g.heads != 1))
            return LEANKV_EINVAL;
        if (g.ring > 0 && a->rows > g.ring) return LEANKV_ELIMIT;
        if (g.rot > 2 * kMaxPairs) return LEANKV_EUNSUPPORTED;
    }
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a->dtype == LEANKV_DT_BF16)
        LEANKV_CUDA_TRY(launch_kernel(place_rows_kernel<bf16>, dim3(a->rows), dim3(kPlaceThreads), 0, st, *a));
    else
        LEANKV_CUDA_TRY(launch_kernel(place_rows_kernel<float>, dim3(a->rows), dim3(kPlaceThreads), 0, st, *a));
    return LEANKV_OK;
}

extern "C" int leankv_causal_attend(const leankv_causal_attn_t* a, const void* q, const float* gate, int gate_ld, void* out,
                                    int out_ld, int rows, int start, int32_t* status, void* stream) {
    const int rc = check_causal(a);
    if (rc) return rc;
    if (!q || !out || rows <= 0 || start < 0 || out_ld < a->heads * a->vdim || (gate && gate_ld < a->heads * a->vdim))
        return LEANKV_EINVAL;
    // the keys of all rows are in the ring at once
    const int keys = start + rows - first_visible(start, a->size);
    if (keys > a->k_ring || (a->shared_dim > 0 && keys > a->s_ring)) return LEANKV_ELIMIT;
    if (a->k_rows < a->k_ring && (first_visible(start, a->size) < a->k_base || start + rows - a->k_base > a->k_rows))
        return LEANKV_ELIMIT;
    if (!aligned16(q)) return LEANKV_EALIGN;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int tiled = causal_tile_attend(*a, q, gate, gate_ld, out, out_ld, rows, start, status, st);
    if (tiled != LEANKV_EUNSUPPORTED) return tiled;
    return a->dtype == LEANKV_DT_BF16 ? attend_rows<bf16>(*a, q, gate, gate_ld, out, out_ld, rows, start, st)
                                      : attend_rows<float>(*a, q, gate, gate_ld, out, out_ld, rows, start, st);
}
