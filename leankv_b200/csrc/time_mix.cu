// Matrix-state time mixing of a prompt portion, all in fp32: a scan over the tokens per head and value-column
// block. The columns of a head's state are independent, and a long portion is cut into pieces that run in
// parallel: (1) every piece but the last from a zero state, with the product of its decays; (2) the true
// state at the start of each piece; (3) every piece again from there, with outputs.

#include <algorithm>

#include "leankv_mixers.h"
#include "typed.cuh"

namespace leankv {
namespace {

constexpr int kSlices = 8;       // lanes that share a column group, each with an eighth of the key channels
constexpr int kColGroup = 4;     // value columns per thread: one read of r / k / w serves four columns
constexpr int kMinPiece = 64;
constexpr int kCtasPerSm = 4;

// L: key channels per slice (a power of two from 4), kSlices * L >= dim.
template <int L>
struct ScanShape {
    static constexpr int kCols = L == 4 ? 32 : 64;                   // value columns per CTA
    static constexpr int kThreads = kCols / kColGroup * kSlices;
    static constexpr int kTok = kThreads / L;                        // tokens staged at a time: 8 channels per thread
    static constexpr int kRow = kSlices * (L + 4);                   // staged row; slices start in different banks
};

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

// Eight consecutive channels of one token, zero beyond `n`.
template <typename T>
__device__ __forceinline__ void fetch8(const T* p, int n, bool vec, float (&v)[8]) {
    if (vec && n >= 8) {
        Raw8<T> r;
        load8(p, r);
        unpack8(r, v);
    } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = i < n ? to_f32(p[i]) : 0.f;
    }
}

template <typename T, int L, bool OUT>
__global__ void __launch_bounds__(ScanShape<L>::kThreads, L <= 8 ? kCtasPerSm : L == 16 ? 2 : 1) time_mix_scan_kernel(const ScanParams<T> p, bool vec) {
    using Sh = ScanShape<L>;
    constexpr int kTok = Sh::kTok, kCols = Sh::kCols, kRow = Sh::kRow;
    __shared__ __align__(16) float s_r[OUT ? kTok : 1][kRow], s_k[kTok][kRow], s_w[kTok][kRow];
    __shared__ __align__(16) float s_v[kTok][kCols], s_bonus[kTok];
    pdl_begin();
    const int tid = threadIdx.x, slice = tid & (kSlices - 1), cg = tid / kSlices;
    const int head = blockIdx.x, c0 = blockIdx.y * kCols, piece = blockIdx.z, d = p.dim;
    const int t0 = piece * p.piece, t1 = min(p.rows, t0 + p.piece);
    const int N = p.heads * d, col0 = c0 + cg * kColGroup;
    const size_t state = (size_t)d * d;

    float S[L][kColGroup];
#pragma unroll
    for (int i = 0; i < L; ++i)
#pragma unroll
        for (int c = 0; c < kColGroup; ++c) {
            const int k = slice * L + i;
            S[i][c] = OUT && k < d && col0 + c < d
                          ? p.S_in[((size_t)piece * p.heads + head) * state + (size_t)k * d + col0 + c] : 0.f;
        }

    // this thread's share of the staging: channels k8 .. k8 + 7 (and columns, for v) of token st_t
    const int st_t = tid / L, k8 = tid % L * 8, nk = d - k8;
    const int v_t = tid / (kCols / 8), v8 = tid % (kCols / 8) * 8;
    const float* w0 = p.w0 + head * d + k8;
    const float* u = p.u + head * d + k8;
    float rr[8], kk[8], zz[8], vv[8], esum[8] = {};
    auto fetch = [&](int tb) {
        const bool on = tb + st_t < t1;
        const size_t g = (size_t)(tb + st_t) * N + head * d + k8;
        fetch8(p.k + g, on ? nk : 0, vec, kk);
        fetch8(p.z + g, on ? nk : 0, vec, zz);
        if (OUT) fetch8(p.r + g, on ? nk : 0, vec, rr);
        if (v_t < kTok)
            fetch8(p.v + (size_t)(tb + v_t) * N + head * d + c0 + v8, tb + v_t < t1 ? d - c0 - v8 : 0, vec, vv);
    };
    fetch(t0);
    for (int tb = t0; tb < t1; tb += kTok) {
        const int nt = min(kTok, t1 - tb);
        __syncthreads();
        float bonus = 0.f;
#pragma unroll
        for (int h = 0; h < 8; h += 4) {
            const int k = k8 + h, at = k / L * (L + 4) + k % L;
            float w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const bool on = st_t < nt && h + i < nk;
                const float e = on ? expf(zz[h + i] + __ldg(w0 + h + i)) : 0.f;      // -log of the decay
                w[i] = expf(-e);
                if (!OUT) esum[h + i] += e;
                else if (on) bonus = fmaf(rr[h + i] * __ldg(u + h + i), kk[h + i], bonus);
            }
            if (k < kSlices * L) {
                *reinterpret_cast<float4*>(&s_k[st_t][at]) = make_float4(kk[h], kk[h + 1], kk[h + 2], kk[h + 3]);
                *reinterpret_cast<float4*>(&s_w[st_t][at]) = make_float4(w[0], w[1], w[2], w[3]);
                if (OUT) *reinterpret_cast<float4*>(&s_r[st_t][at]) = make_float4(rr[h], rr[h + 1], rr[h + 2], rr[h + 3]);
            }
        }
        if (v_t < kTok) {
            *reinterpret_cast<float4*>(&s_v[v_t][v8]) = make_float4(vv[0], vv[1], vv[2], vv[3]);
            *reinterpret_cast<float4*>(&s_v[v_t][v8 + 4]) = make_float4(vv[4], vv[5], vv[6], vv[7]);
        }
        if (OUT) {      // bonus_t = sum over k of r u k: the L threads of a token are neighbours
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, o);
            if (tid % L == 0) s_bonus[st_t] = bonus;
        }
        __syncthreads();
        if (tb + kTok < t1) fetch(tb + kTok);       // the next tokens travel while these are consumed
#pragma unroll 1
        for (int tq = 0; tq < nt; tq += 2) {        // a token beyond nt has k = 0 and w = 1: no effect
            float acc[2 * kColGroup];
#pragma unroll
            for (int tt = 0; tt < 2; ++tt) {
                const int t = tq + tt;
                const float4 v4 = *reinterpret_cast<const float4*>(&s_v[t][cg * kColGroup]);
                const float v[kColGroup] = {v4.x, v4.y, v4.z, v4.w};
                float a[kColGroup] = {};
#pragma unroll
                for (int i = 0; i < L; i += 4) {
                    const int at = slice * (L + 4) + i;
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[t][at]);
                    const float4 w4 = *reinterpret_cast<const float4*>(&s_w[t][at]);
                    const float ka[4] = {k4.x, k4.y, k4.z, k4.w}, wa[4] = {w4.x, w4.y, w4.z, w4.w};
                    float ra[4] = {};
                    if (OUT) {
                        const float4 r4 = *reinterpret_cast<const float4*>(&s_r[t][at]);
                        ra[0] = r4.x; ra[1] = r4.y; ra[2] = r4.z; ra[3] = r4.w;
                    }
#pragma unroll
                    for (int x = 0; x < 4; ++x)
#pragma unroll
                        for (int c = 0; c < kColGroup; ++c) {
                            if (OUT) a[c] = fmaf(ra[x], S[i + x][c], a[c]);
                            S[i + x][c] = fmaf(wa[x], S[i + x][c], ka[x] * v[c]);
                        }
                }
#pragma unroll
                for (int c = 0; c < kColGroup; ++c) acc[tt * kColGroup + c] = a[c];
            }
            if (OUT) {      // sum over the eight slices; lane `slice` ends with (token, column) number `slice`
#pragma unroll
                for (int o = 4; o > 0; o >>= 1)
#pragma unroll
                    for (int i = 0; i < o; ++i) {
                        const bool up = (slice & o) != 0;
                        const float send = up ? acc[i] : acc[i + o], keep = up ? acc[i + o] : acc[i];
                        acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                    }
                const int t = tq + slice / kColGroup, c = slice % kColGroup;
                if (t < nt && col0 + c < d)
                    p.o[(size_t)(tb + t) * N + head * d + col0 + c] = fmaf(s_bonus[t], s_v[t][cg * kColGroup + c], acc[0]);
            }
        }
    }
    if (!OUT || piece == p.n_pieces - 1) {
        float* dst = p.S_out + ((size_t)(OUT ? 0 : piece) * p.heads + head) * state;
#pragma unroll
        for (int i = 0; i < L; ++i)
#pragma unroll
            for (int c = 0; c < kColGroup; ++c) {
                const int k = slice * L + i;
                if (k < d && col0 + c < d) dst[(size_t)k * d + col0 + c] = S[i][c];
            }
    }
    if (!OUT && blockIdx.y == 0) {      // decay of the whole piece: exp(-sum over its tokens)
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (k8 + i < kRow) s_k[st_t][k8 + i] = esum[i];
        __syncthreads();
        for (int k = tid; k < d; k += Sh::kThreads) {
            float e = 0.f;
            for (int t = 0; t < kTok; ++t) e += s_k[t][k];
            p.decay[((size_t)piece * p.heads + head) * d + k] = expf(-e);
        }
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

// out = out_scale * rms(o of the head) * norm * silu(g); a group of `lanes` lanes per (token, head), eight
// channels per lane and pass (lanes: a power of two up to 32).
template <typename T>
__global__ void __launch_bounds__(256) time_mix_out_kernel(const float* o, const T* g, const float* norm, float eps,
                                                           T* out, int out_ld, float out_scale, long long groups, int heads,
                                                           int dim, int lanes, bool vec) {
    pdl_begin();
    const long long at = ((long long)blockIdx.x * 256 + threadIdx.x) / lanes;
    const int l = threadIdx.x % lanes;
    const bool live = at < groups;
    const long long w = live ? at : 0;
    const int t = (int)(w / heads), h = (int)(w - (long long)t * heads);
    const size_t base = (size_t)w * dim;
    float v[8], ss = 0.f;
    for (int i = l * 8; i < dim; i += lanes * 8) {
        fetch8(o + base + i, dim - i, vec, v);
#pragma unroll
        for (int x = 0; x < 8; ++x) ss = fmaf(v[x], v[x], ss);
    }
    for (int s = lanes / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    if (!live) return;
    const float f = out_scale / sqrtf(ss / (float)dim + eps);
    T* dst = out + (size_t)t * out_ld + h * dim;
    for (int i = l * 8; i < dim; i += lanes * 8) {
        float gv[8];
        if (dim > lanes * 8) fetch8(o + base + i, dim - i, vec, v);      // else still in registers
        fetch8(g + base + i, dim - i, vec, gv);
#pragma unroll
        for (int x = 0; x < 8; ++x)
            if (i + x < dim) v[x] *= f * __ldg(norm + h * dim + i + x) * gv[x] * sigmoid_f32(gv[x]);
        if (vec) {
            T r[8];
#pragma unroll
            for (int x = 0; x < 8; ++x) r[x] = from_f32<T>(v[x]);
            Raw8<T> raw;
            memcpy(&raw, r, sizeof(raw));
            *reinterpret_cast<Raw8<T>*>(dst + i) = raw;
        } else {
#pragma unroll
            for (int x = 0; x < 8; ++x)
                if (i + x < dim) dst[i + x] = from_f32<T>(v[x]);
        }
    }
}

int pieces_for(int heads, int dim, int rows) {
    const int base = heads * ((dim + 63) / 64);
    const int want = std::max(1, sm_count() * kCtasPerSm / base);
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
    using Sh = ScanShape<L>;
    const dim3 block(Sh::kThreads);
    const int cb = (a.dim + Sh::kCols - 1) / Sh::kCols;
    const bool vec = a.dim % 8 == 0 && aligned16(r) && aligned16(k) && aligned16(v) && aligned16(z);
    p.S_in = a.S;
    if (p.n_pieces > 1) {
        p.S_out = pieces;
        p.decay = decay;
        LEANKV_CUDA_TRY(launch_kernel(time_mix_scan_kernel<T, L, false>, dim3(a.heads, cb, p.n_pieces - 1), block, 0, st,
                                      p, vec));
        const long long total = (long long)state_floats(a.heads, a.dim);
        LEANKV_CUDA_TRY(launch_kernel(time_mix_carry_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st,
                                      static_cast<const float*>(a.S), pieces, static_cast<const float*>(decay), a.heads,
                                      a.dim, p.n_pieces));
        p.S_in = pieces;
    }
    p.S_out = a.S;
    LEANKV_CUDA_TRY(launch_kernel(time_mix_scan_kernel<T, L, true>, dim3(a.heads, cb, p.n_pieces), block, 0, st, p, vec));
    return LEANKV_OK;
}

template <typename T>
int rows_all(const leankv_time_mix_t& a, const void* r, const void* k, const void* v, const void* g, const float* z,
             void* out, int out_ld, float out_scale, int rows, float* ws, cudaStream_t st) {
    int rc = LEANKV_ELIMIT;
    if (a.dim <= 8 * 4) rc = scan<T, 4>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 8 * 8) rc = scan<T, 8>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 8 * 16) rc = scan<T, 16>(a, r, k, v, z, ws, rows, st);
    else if (a.dim <= 8 * 32) rc = scan<T, 32>(a, r, k, v, z, ws, rows, st);
    if (rc) return rc;
    int lanes = 1;
    while (lanes < 32 && lanes * 8 < a.dim) lanes *= 2;
    const long long groups = (long long)rows * a.heads, threads = groups * lanes;
    const bool vec = a.dim % 8 == 0 && out_ld % 8 == 0 && aligned16(ws) && aligned16(g) && aligned16(out);
    LEANKV_CUDA_TRY(launch_kernel(time_mix_out_kernel<T>, dim3((unsigned)((threads + 255) / 256)), dim3(256), 0, st,
                                  static_cast<const float*>(ws), static_cast<const T*>(g), a.norm, a.eps,
                                  static_cast<T*>(out), out_ld, out_scale, groups, a.heads, a.dim, lanes, vec));
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
