// Matrix-state time mixing of a prompt portion, all in fp32: a scan over the tokens per head and value-column
// block. The columns of a head's state are independent, and a long portion is cut into pieces that run in
// parallel: (1) every piece but the last from a zero state, with the product of its decays; (2) the true
// state at the start of each piece; (3) every piece again from there, with outputs.

#include <algorithm>

#include "leankv_mixers.h"
#include "typed.cuh"

namespace leankv {
namespace {

constexpr int kCols = 32;        // value columns per CTA
constexpr int kSlices = 4;       // lanes that share a column, each with a quarter of the key channels
constexpr int kMinPiece = 64;

template <typename T>
struct ScanParams {
    const T* r;
    const T* k;
    const T* v;
    const float* z;
    const float* u;
    const float* w0;
    const float* S_in;          // [piece][head][dim][dim]; piece stride 0 when there is one piece
    float* S_out;               // pass 1: [piece][..]; pass 3: the sequence's state (last piece only)
    float* decay;               // pass 1: [piece][head][dim]
    float* o;                   // pass 3: fp32 [rows][heads * dim]
    int heads, dim, rows, piece, n_pieces;
};

// L: key channels per slice, a multiple of 4, kSlices * L >= dim.
template <typename T, int L, bool OUT>
__global__ void __launch_bounds__(kCols * kSlices) time_mix_scan_kernel(const ScanParams<T> p) {
    constexpr int kStride = kSlices * (L + 4);       // slices start in different banks
    constexpr int kTok = L > 32 ? 8 : 16;            // tokens staged in shared memory at a time
    __shared__ __align__(16) float s_r[kTok][OUT ? kStride : 4], s_k[kTok][kStride], s_w[kTok][kStride];
    __shared__ float s_v[kTok][kCols], s_bonus[kTok];
    pdl_begin();
    const int tid = threadIdx.x, slice = tid & (kSlices - 1), col = tid >> 2;
    const int head = blockIdx.x, c0 = blockIdx.y * kCols, piece = blockIdx.z, d = p.dim;
    const int t0 = piece * p.piece, t1 = min(p.rows, t0 + p.piece);
    const int N = p.heads * d;
    const bool live = c0 + col < d;
    const size_t state = (size_t)d * d;
    float S[L];
#pragma unroll
    for (int i = 0; i < L; ++i) S[i] = 0.f;
    if (OUT && live) {
        const float* src = p.S_in + ((size_t)piece * p.heads + head) * state + c0 + col;
#pragma unroll
        for (int i = 0; i < L; ++i) {
            const int k = slice * L + i;
            if (k < d) S[i] = src[(size_t)k * d];
        }
    }
    float prod[(kSlices * L + kCols * kSlices - 1) / (kCols * kSlices)];
#pragma unroll
    for (auto& x : prod) x = 1.f;

    for (int tb = t0; tb < t1; tb += kTok) {
        const int nt = min(kTok, t1 - tb);
        __syncthreads();
        for (int e = tid; e < kTok * kSlices * L; e += kCols * kSlices) {
            const int t = e / (kSlices * L), k = e - t * (kSlices * L);
            const int at = k / L * (L + 4) + k % L;
            float rv = 0.f, kv = 0.f, wv = 1.f;
            if (t < nt && k < d) {
                const size_t g = (size_t)(tb + t) * N + head * d + k;
                kv = to_f32(p.k[g]);
                wv = expf(-expf(p.z[g] + __ldg(p.w0 + head * d + k)));
                if (OUT) rv = to_f32(p.r[g]);
            }
            s_k[t][at] = kv;
            s_w[t][at] = wv;
            if (OUT) s_r[t][at] = rv;
        }
        for (int e = tid; e < kTok * kCols; e += kCols * kSlices) {
            const int t = e / kCols, c = e - t * kCols;
            s_v[t][c] = t < nt && c0 + c < d ? to_f32(p.v[(size_t)(tb + t) * N + head * d + c0 + c]) : 0.f;
        }
        __syncthreads();
        if (OUT) {      // bonus_t = sum over k of r u k: 8 threads per token
            const int t = tid >> 3, part = tid & 7;
            float b = 0.f;
            for (int k = part; k < d && t < kTok; k += 8) {
                const int at = k / L * (L + 4) + k % L;
                b = fmaf(s_r[t][at] * __ldg(p.u + head * d + k), s_k[t][at], b);
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) b += __shfl_xor_sync(0xffffffffu, b, o);
            if (part == 0 && t < kTok) s_bonus[t] = b;
            __syncthreads();
        } else if (blockIdx.y == 0) {
            int x = 0;
            for (int k = tid; k < kSlices * L; k += kCols * kSlices, ++x) {
                const int at = k / L * (L + 4) + k % L;
                float q = 1.f;
                for (int t = 0; t < nt; ++t) q *= s_w[t][at];
                prod[x] *= q;
            }
        }
        for (int tq = 0; tq < nt; tq += 4) {
            float acc[4];
#pragma unroll
            for (int tt = 0; tt < 4; ++tt) {           // tokens beyond nt: k = 0, w = 1, no effect
                const int t = tq + tt;
                const float vv = s_v[t][col];
                float a = 0.f;
#pragma unroll
                for (int i = 0; i < L; i += 4) {
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[t][slice * (L + 4) + i]);
                    const float4 w4 = *reinterpret_cast<const float4*>(&s_w[t][slice * (L + 4) + i]);
                    if (OUT) {
                        const float4 r4 = *reinterpret_cast<const float4*>(&s_r[t][slice * (L + 4) + i]);
                        a = fmaf(r4.x, S[i], a); a = fmaf(r4.y, S[i + 1], a);
                        a = fmaf(r4.z, S[i + 2], a); a = fmaf(r4.w, S[i + 3], a);
                    }
                    S[i] = fmaf(w4.x, S[i], k4.x * vv);
                    S[i + 1] = fmaf(w4.y, S[i + 1], k4.y * vv);
                    S[i + 2] = fmaf(w4.z, S[i + 2], k4.z * vv);
                    S[i + 3] = fmaf(w4.w, S[i + 3], k4.w * vv);
                }
                acc[tt] = a;
            }
            if (OUT) {      // sum over the four slices; lane `slice` keeps token tq + slice
                const bool hi2 = slice & 2, hi1 = slice & 1;
                const float a0 = (hi2 ? acc[2] : acc[0]) + __shfl_xor_sync(0xffffffffu, hi2 ? acc[0] : acc[2], 2);
                const float a1 = (hi2 ? acc[3] : acc[1]) + __shfl_xor_sync(0xffffffffu, hi2 ? acc[1] : acc[3], 2);
                const float r = (hi1 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, hi1 ? a0 : a1, 1);
                const int t = tq + slice;
                if (live && t < nt)
                    p.o[(size_t)(tb + t) * N + head * d + c0 + col] = fmaf(s_bonus[t], s_v[t][col], r);
            }
        }
    }
    if (live && (!OUT || piece == p.n_pieces - 1)) {
        float* dst = p.S_out + ((size_t)(OUT ? 0 : piece) * p.heads + head) * state + c0 + col;
#pragma unroll
        for (int i = 0; i < L; ++i) {
            const int k = slice * L + i;
            if (k < d) dst[(size_t)k * d] = S[i];
        }
    }
    if (!OUT && blockIdx.y == 0) {
        int x = 0;
        for (int k = tid; k < kSlices * L; k += kCols * kSlices, ++x)
            if (k < d) p.decay[((size_t)piece * p.heads + head) * d + k] = prod[x];
    }
}

// pieces[c] (local end state of piece c) becomes the state at the start of piece c.
__global__ void __launch_bounds__(256) time_mix_carry_kernel(const float* S, float* pieces, const float* decay,
                                                             int heads, int dim, int n_pieces) {
    pdl_begin();
    const long long total = (long long)heads * dim * dim;
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= total) return;
    const long long hk = e / dim;         // head * dim + key channel
    float s = S[e];
    for (int c = 0; c < n_pieces; ++c) {
        const float local = c + 1 < n_pieces ? pieces[c * total + e] : 0.f;
        pieces[c * total + e] = s;
        if (c + 1 < n_pieces) s = fmaf(decay[(long long)c * heads * dim + hk], s, local);
    }
}

// out = out_scale * rms(o of the head) * norm * silu(g); one warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) time_mix_out_kernel(const float* o, const T* g, const float* norm, float eps,
                                                           T* out, int out_ld, float out_scale, int rows, int heads,
                                                           int dim) {
    pdl_begin();
    const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (w >= (long long)rows * heads) return;
    const int t = (int)(w / heads), h = (int)(w - (long long)t * heads);
    const size_t base = (size_t)t * heads * dim + (size_t)h * dim;
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) ss = fmaf(o[base + i], o[base + i], ss);
    const float f = out_scale / sqrtf(warp_sum(ss) / (float)dim + eps);
    for (int i = lane; i < dim; i += 32) {
        const float gv = to_f32(g[base + i]);
        out[(size_t)t * out_ld + h * dim + i] =
            from_f32<T>(o[base + i] * f * __ldg(norm + h * dim + i) * gv * sigmoid_f32(gv));
    }
}

int pieces_for(int heads, int dim, int rows) {
    const int base = heads * ((dim + kCols - 1) / kCols);
    const int want = std::max(1, sm_count() * 8 / base);
    const int n = std::min(want, rows / kMinPiece);
    return n < 3 ? 1 : n;
}

size_t state_floats(int heads, int dim) { return (size_t)heads * dim * dim; }

template <typename T, int L>
int scan(const leankv_time_mix_t& a, const void* r, const void* k, const void* v, const float* z, float* ws, int rows,
         cudaStream_t st) {
    const int n = pieces_for(a.heads, a.dim, rows), len = (rows + n - 1) / n;
    ScanParams<T> p{};
    p.r = static_cast<const T*>(r);
    p.k = static_cast<const T*>(k);
    p.v = static_cast<const T*>(v);
    p.z = z;
    p.u = a.u;
    p.w0 = a.w0;
    p.heads = a.heads;
    p.dim = a.dim;
    p.rows = rows;
    p.piece = len;
    p.n_pieces = (rows + len - 1) / len;
    p.o = ws;
    float* pieces = ws + (size_t)rows * a.heads * a.dim;
    float* decay = pieces + (size_t)n * state_floats(a.heads, a.dim);
    const dim3 block(kCols * kSlices);
    const int cb = (a.dim + kCols - 1) / kCols;
    p.S_in = a.S;
    if (p.n_pieces > 1) {
        p.S_out = pieces;
        p.decay = decay;
        LEANKV_CUDA_TRY(launch_kernel(time_mix_scan_kernel<T, L, false>, dim3(a.heads, cb, p.n_pieces - 1), block, 0, st,
                                      p));
        const long long total = (long long)state_floats(a.heads, a.dim);
        LEANKV_CUDA_TRY(launch_kernel(time_mix_carry_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st,
                                      static_cast<const float*>(a.S), pieces, static_cast<const float*>(decay), a.heads,
                                      a.dim, p.n_pieces));
        p.S_in = pieces;
    }
    p.S_out = a.S;
    LEANKV_CUDA_TRY(launch_kernel(time_mix_scan_kernel<T, L, true>, dim3(a.heads, cb, p.n_pieces), block, 0, st, p));
    return LEANKV_OK;
}

template <typename T>
int rows_all(const leankv_time_mix_t& a, const void* r, const void* k, const void* v, const void* g, const float* z,
             void* out, int out_ld, float out_scale, int rows, float* ws, cudaStream_t st) {
    int rc = LEANKV_ELIMIT;
    if (a.dim <= 4 * 8) rc = scan<T, 8>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 4 * 16) rc = scan<T, 16>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 4 * 32) rc = scan<T, 32>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 4 * 64) rc = scan<T, 64>(a, r, k, v, z, ws, rows, st);
    if (rc) return rc;
    const long long warps = (long long)rows * a.heads;
    LEANKV_CUDA_TRY(launch_kernel(time_mix_out_kernel<T>, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, st,
                                  static_cast<const float*>(ws), static_cast<const T*>(g), a.norm, a.eps,
                                  static_cast<T*>(out), out_ld, out_scale, rows, a.heads, a.dim));
    return LEANKV_OK;
}

int check_args(const leankv_time_mix_t* a) {
    if (!a || a->heads <= 0 || a->dim <= 0 || !a->S || !a->u || !a->w0 || !a->norm) return LEANKV_EINVAL;
    if (a->dtype != LEANKV_DT_BF16 && a->dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    return LEANKV_OK;
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" size_t leankv_time_mix_workspace_bytes(const leankv_time_mix_t* a, int rows) {
    if (check_args(a) || rows <= 0) return 0;
    const size_t n = pieces_for(a->heads, a->dim, rows);
    return 4 * ((size_t)rows * a->heads * a->dim + n * (state_floats(a->heads, a->dim) + (size_t)a->heads * a->dim));
}

extern "C" int leankv_time_mix_rows(const leankv_time_mix_t* a, const void* r, const void* k, const void* v,
                                    const void* g, const float* z, void* out, int out_ld, float out_scale, int rows,
                                    void* ws, size_t ws_bytes, void* stream) {
    const int rc = check_args(a);
    if (rc) return rc;
    if (!r || !k || !v || !g || !z || !out || rows <= 0 || out_ld < a->heads * a->dim) return LEANKV_EINVAL;
    if (!ws || ws_bytes < leankv_time_mix_workspace_bytes(a, rows)) return LEANKV_EWORKSPACE;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    float* w = static_cast<float*>(ws);
    return a->dtype == LEANKV_DT_BF16 ? rows_all<bf16>(*a, r, k, v, g, z, out, out_ld, out_scale, rows, w, st)
                                      : rows_all<float>(*a, r, k, v, g, z, out, out_ld, out_scale, rows, w, st);
}
