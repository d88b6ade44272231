// One decode step of a layer's token mixers, in one launch. The first thread-block cluster runs the window +
// pooled-block attention (its CTAs split the visible keys and merge through distributed shared memory), every
// further CTA one head of the matrix-state time mixing: the two mixers read the same projections and are
// independent, so they run side by side.

#include <algorithm>

#include "decode_frame.cuh"
#include "window_pool.cuh"

namespace leankv {
namespace {

constexpr int kStepThreads = 512;
constexpr int kStepSmemFloats = 200 * 1024 / 4;

struct StepParams {
    leankv_window_pool_t left;
    leankv_time_mix_t right;
    leankv_mixer_step_t s;
    int has_left, has_right, n_max, cluster, norms_aligned;
};

constexpr int kRowVecs = 6;        // float4s of the projection row a thread keeps: rows up to 12288 columns

template <typename T>
__device__ void left_step(const StepParams& p, float* sm, float* s_tmp, int rank) {
    const leankv_window_pool_t& a = p.left;
    const AttendPlan pl(a, kStepThreads, (p.n_max + p.cluster - 1) / p.cluster, kStepSmemFloats);
    const int tid = threadIdx.x, i = p.s.state[kPos], G = a.kv_heads;
    const int nq = a.heads * a.dim, nk = G * a.dim, nv = G * a.vdim;
    const float* y = p.s.y + p.s.qkv_off;       // biases are already in
    T* k_ring = static_cast<T*>(a.k_ring);
    T* v_ring = static_cast<T*>(a.v_ring);

    // before the projections are there: the mix, and this CTA's key / value rows on their way into L2
    put_talk(a, pl, sm);
    {
        const VisibleKeys vis(i, a.size, a.pool);
        const int j0 = (int)((long long)vis.n * rank / p.cluster), j1 = (int)((long long)vis.n * (rank + 1) / p.cluster);
        const int kb = G * a.dim_pad * (int)sizeof(T), per = (kb + 127) / 128;
        const int vb = G * a.vdim_pad * (int)sizeof(T), perv = (vb + 127) / 128;
        for (int e = tid; e < (j1 - j0) * (per + perv); e += kStepThreads) {
            const int jl = e / (per + perv), c = e - jl * (per + perv), j = j0 + jl;
            const int row = j < vis.n_blk ? j : (vis.w0 + j - vis.n_blk) % a.ring;
            const char* base = c < per ? static_cast<const char*>(j < vis.n_blk ? a.k_pool : a.k_ring) + (size_t)row * kb + c * 128
                                       : static_cast<const char*>(j < vis.n_blk ? a.v_pool : a.v_ring) + (size_t)row * vb + (c - per) * 128;
            asm volatile("prefetch.global.L2 [%0];" ::"l"(base));
        }
    }
    pdl_begin();

    const int slot = i % a.ring;
    T* k_new = reinterpret_cast<T*>(sm + pl.knew);
    T* v_new = reinterpret_cast<T*>(sm + pl.vnew);
    auto put_k = [&](int g, int d, float v) {
        const T r = from_f32<T>(v);
        k_new[g * a.dim_pad + d] = r;
        if (rank == 0) k_ring[((size_t)slot * G + g) * a.dim_pad + d] = r;
    };
    auto put_v = [&](int g, int d, float v) {
        const T r = from_f32<T>(v);
        v_new[g * a.vdim_pad + d] = r;
        if (rank == 0) v_ring[((size_t)slot * G + g) * a.vdim_pad + d] = r;
    };
    if (a.dim % 4 == 0 && a.vdim % 4 == 0 && p.s.qkv_off % 4 == 0 && p.norms_aligned && nq + nk + nv <= kStepThreads * 4 * kRowVecs) {
        float4 x[kRowVecs];        // the row, read once
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int n = 0; n < kRowVecs; ++n) {
            const int e = (tid + n * kStepThreads) * 4;
            x[n] = e < nq + nk + nv ? ld_cg_f32x4(y + e) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int n = 0; n < kRowVecs; ++n) {
            const int e = (tid + n * kStepThreads) * 4;
            const float ss = x[n].x * x[n].x + x[n].y * x[n].y + x[n].z * x[n].z + x[n].w * x[n].w;
            if (e < nq) sq += ss;
            else if (e < nq + nk) sk += ss;
        }
        const RowFactors f = norm_factors(sq, sk, nq, nk, a.q_norm != nullptr, a.k_norm != nullptr, a.eps, s_tmp);
#pragma unroll
        for (int n = 0; n < kRowVecs; ++n) {
            const int e = (tid + n * kStepThreads) * 4;
            if (e >= nq + nk + nv) continue;
            const bool is_q = e < nq, is_k = !is_q && e < nq + nk;
            const int at = is_q ? e : is_k ? e - nq : e - nq - nk, width = is_q || is_k ? a.dim : a.vdim;
            const int h = at / width, d = at - h * width;
            const float* w = is_q ? a.q_norm : is_k ? a.k_norm : nullptr;
            const float fac = is_q ? f.q * a.scale : is_k ? f.k : 1.f;
            float4 v = make_float4(x[n].x * fac, x[n].y * fac, x[n].z * fac, x[n].w * fac);
            if (w != nullptr) {
                const float4 g = *reinterpret_cast<const float4*>(w + at);
                v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
            }
            if (is_q) {
                put_query4<T>(pl, sm, a.heads, h, d, v);
            } else {
                const int to = h * (is_k ? a.dim_pad : a.vdim_pad) + d;
                store4((is_k ? k_new : v_new) + to, v);
                if (rank == 0)
                    store4((is_k ? k_ring : v_ring) + (size_t)slot * G * (is_k ? a.dim_pad : a.vdim_pad) + to, v);
            }
        }
    } else {
        const RowFactors f = row_factors(y, nullptr, nq, nk, a.q_norm != nullptr, a.k_norm != nullptr, a.eps, s_tmp);
        for (int e = tid; e < nq + nk + nv; e += kStepThreads) {
            if (e < nq) put_query<T>(pl, sm, a.heads, e / a.dim, e % a.dim, y[e] * f.q * (a.q_norm ? __ldg(a.q_norm + e) : 1.f) * a.scale);
            else if (e < nq + nk) put_k((e - nq) / a.dim, (e - nq) % a.dim, y[e] * f.k * (a.k_norm ? __ldg(a.k_norm + e - nq) : 1.f));
            else put_v((e - nq - nk) / a.vdim, (e - nq - nk) % a.vdim, y[e]);
        }
    }
    const int pd = a.dim_pad - a.dim, pv = a.vdim_pad - a.vdim;       // padding columns are zero
    for (int e = tid; e < a.heads * pd; e += kStepThreads) put_query<T>(pl, sm, a.heads, e / pd, a.dim + e % pd, 0.f);
    for (int e = tid; e < G * pd; e += kStepThreads) put_k(e / pd, a.dim + e % pd, 0.f);
    for (int e = tid; e < G * pv; e += kStepThreads) put_v(e / pv, a.vdim + e % pv, 0.f);
    __syncthreads();
    float* p_gmem = static_cast<float*>(p.s.ws) + (size_t)rank * 2 * a.heads * pl.ldp;
    attend_query<T, float>(a, pl, sm, p_gmem, i, true, rank, p.cluster, p.s.out, p.s.left_scale);

    // the block this token completes (not visible to it: it ends at i > i - size)
    if ((i + 1) % a.pool == 0 && (i + 1) / a.pool <= a.max_blocks) {
        const int b = i / a.pool, p0 = b * a.pool;
        auto mean = [&](const T* ring, const T* fresh, T* dst, int n) {
            for (int e = rank * kStepThreads + tid; e < n; e += p.cluster * kStepThreads) {
                float t = 0.f;
                for (int x = 0; x < a.pool - 1; ++x) t += to_f32(ring[(size_t)((p0 + x) % a.ring) * n + e]);
                dst[(size_t)b * n + e] = from_f32<T>((t + to_f32(fresh[e])) / (float)a.pool);
            }
        };
        mean(k_ring, k_new, static_cast<T*>(a.k_pool), G * a.dim_pad);
        mean(v_ring, v_new, static_cast<T*>(a.v_pool), G * a.vdim_pad);
    }
}

template <typename T>
__device__ void right_step(const StepParams& p, float* sm, float* s_tmp, int head) {
    const leankv_time_mix_t& a = p.right;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = a.dim, N = a.heads * d, c0 = head * d;
    pdl_begin();
    float* s_r = sm;
    float* s_k = s_r + d;
    float* s_w = s_k + d;
    float* s_v = s_w + d;
    float* s_o = s_v + d;                      // [slices][d]
    const float* y = p.s.y + p.s.rkvg_off + c0;
    const float* y1 = p.s.y + p.s.w1_off;
    const T* w2 = static_cast<const T*>(p.s.w2);
    float bonus = 0.f;
    for (int c = tid; c < d; c += kStepThreads) {
        const float r = y[c], k = y[N + c];
        s_r[c] = r;
        s_k[c] = k;
        s_v[c] = y[2 * N + c];
        bonus = fmaf(r * __ldg(a.u + c0 + c), k, bonus);
    }
    for (int c = warp; c < d; c += kStepThreads / 32) {
        float z = 0.f;
        for (int x = lane; x < p.s.rank; x += 32) z = fmaf(to_f32(w2[(size_t)(c0 + c) * p.s.rank + x]), tanhf(y1[x]), z);
        z = warp_sum(z);
        if (lane == 0) s_w[c] = expf(-expf(z + __ldg(a.w0 + c0 + c)));
    }
    bonus = cta_sum(bonus, s_tmp);             // synchronises
    const int slices = max(1, kStepThreads / d), sl = tid / d, col = tid - sl * d;
    float* S = a.S + (size_t)head * d * d;
    if (sl < slices) {
        const int k0 = d * sl / slices, k1 = d * (sl + 1) / slices;
        const float v = s_v[col];
        float o = 0.f;
#pragma unroll 8
        for (int k = k0; k < k1; ++k) {
            const float s = S[(size_t)k * d + col];
            o = fmaf(s_r[k], s, o);
            S[(size_t)k * d + col] = fmaf(s_w[k], s, s_k[k] * v);
        }
        s_o[sl * d + col] = o;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < d) {
        for (int x = 0; x < slices; ++x) o += s_o[x * d + tid];
        o = fmaf(bonus, s_v[tid], o);
    }
    const float f = p.s.right_scale / sqrtf(cta_sum(o * o, s_tmp) / (float)d + a.eps);
    if (tid < d) {
        const float g = y[3 * N + tid];
        p.s.out[p.s.right_off + c0 + tid] = o * f * __ldg(a.norm + c0 + tid) * g * sigmoid_f32(g);
    }
}

template <typename T>
__global__ void __launch_bounds__(kStepThreads) mixer_step_kernel(const __grid_constant__ StepParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_tmp[32];
    const int first = p.has_left ? p.cluster : 0;
    if ((int)blockIdx.x < first) left_step<T>(p, sm, s_tmp, blockIdx.x);
    else if ((int)blockIdx.x - first < p.right.heads) right_step<T>(p, sm, s_tmp, blockIdx.x - first);
}

int keys_bound(const leankv_window_pool_t& a, int max_pos) {
    return VisibleKeys(std::max(max_pos - 1, 0), a.size, a.pool).n;
}

template <typename T>
size_t step_smem(const StepParams& p) {
    size_t smem = 0;
    if (p.has_left)
        smem = 4 * (size_t)AttendPlan(p.left, kStepThreads, (p.n_max + p.cluster - 1) / p.cluster, kStepSmemFloats).total;
    if (p.has_right) smem = std::max(smem, (size_t)(4 * p.right.dim + kStepThreads + p.right.dim) * 4);
    return smem;
}

template <typename T>
int launch_step(StepParams& p, cudaStream_t st) {
    LEANKV_CUDA_TRY(cudaFuncSetAttribute(mixer_step_kernel<T>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    for (p.cluster = kMaxCluster;; p.cluster = 8) {
        const size_t smem = step_smem<T>(p);
        if (smem > 226 * 1024) return LEANKV_ELIMIT;
        LEANKV_CUDA_TRY(cudaFuncSetAttribute(mixer_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        const int heads = p.has_right ? p.right.heads : 0;
        const int grid = (p.has_left ? p.cluster : 0) + (heads + p.cluster - 1) / p.cluster * p.cluster;
        if (p.cluster > 8) {      // does a cluster of this size fit this device?
            cudaLaunchConfig_t cfg = {};
            cfg.gridDim = dim3(grid);
            cfg.blockDim = dim3(kStepThreads);
            cfg.dynamicSmemBytes = smem;
            cudaLaunchAttribute attr[1];
            attr[0].id = cudaLaunchAttributeClusterDimension;
            attr[0].val.clusterDim.x = p.cluster;
            attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
            cfg.attrs = attr;
            cfg.numAttrs = 1;
            int fits = 0;
            if (cudaOccupancyMaxActiveClusters(&fits, mixer_step_kernel<T>, &cfg) != cudaSuccess || fits < 1) {
                (void)cudaGetLastError();
                continue;
            }
        }
        LEANKV_CUDA_TRY(launch_cluster_kernel_ex(true, dim3(p.cluster), mixer_step_kernel<T>, dim3(grid),
                                                 dim3(kStepThreads), smem, st, p));
        return LEANKV_OK;
    }
}

}  // namespace
}  // namespace leankv

using namespace leankv;

extern "C" size_t leankv_mixer_step_workspace_bytes(const leankv_window_pool_t* left, int max_pos) {
    if (!left || max_pos <= 0) return 0;
    const int n = keys_bound(*left, max_pos);
    size_t need = 0;
    for (int c = 8; c <= kMaxCluster; c *= 2) {
        const AttendPlan pl(*left, kStepThreads, (n + c - 1) / c, kStepSmemFloats);
        if (!pl.p_in_smem) need = std::max(need, (size_t)c * 2 * left->heads * pl.ldp * 4);
    }
    return need;
}

extern "C" int leankv_mixer_step(const leankv_window_pool_t* left, const leankv_time_mix_t* right,
                                 const leankv_mixer_step_t* s, void* stream) {
    if (!s || (!left && !right) || !s->y || !s->out || !s->state || s->max_pos <= 0) return LEANKV_EINVAL;
    StepParams p{};
    p.s = *s;
    int dtype = 0;
    if (left) {
        if (left->heads <= 0 || left->kv_heads <= 0 || left->heads % left->kv_heads || left->dim <= 0 ||
            left->vdim <= 0 || left->size <= 0 || left->pool <= 0 || !left->k_ring || !left->v_ring)
            return LEANKV_EINVAL;
        if (left->ring < std::max(left->size, left->pool) ||
            VisibleKeys(s->max_pos - 1, left->size, left->pool).n_blk > left->max_blocks)
            return LEANKV_ELIMIT;
        if (left->dim_pad % 16 || left->vdim_pad % 16 || left->dim_pad < left->dim || left->vdim_pad < left->vdim)
            return LEANKV_EALIGN;
        if (leankv_mixer_step_workspace_bytes(left, s->max_pos) > (s->ws ? s->ws_bytes : 0)) return LEANKV_EWORKSPACE;
        p.left = *left;
        p.has_left = 1;
        p.norms_aligned = aligned16(left->q_norm) && aligned16(left->k_norm) && aligned16(s->y);
        p.n_max = keys_bound(*left, s->max_pos);
        dtype = left->dtype;
    }
    if (right) {
        if (right->heads <= 0 || right->dim <= 0 || right->dim > kStepThreads || !right->S || !right->u || !right->w0 ||
            !right->norm || !s->w2 || s->rank <= 0 || (left && left->dtype != right->dtype))
            return LEANKV_EINVAL;
        p.right = *right;
        p.has_right = 1;
        dtype = right->dtype;
    }
    if (dtype != LEANKV_DT_BF16 && dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    return dtype == LEANKV_DT_BF16 ? launch_step<bf16>(p, st) : launch_step<float>(p, st);
}
