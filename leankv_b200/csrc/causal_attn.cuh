// Causal attention over a ring of keys (whole sequence or a sliding window): what the prompt kernels
// (causal_rows.cu, causal_tile.cu) and the decode step (causal_step.cu) share. A key is a part of its kv head's own
// and a part common to all heads; values may be the leading numbers of the own part (a latent).
#pragma once

#include "leankv_mixers.h"
#include "typed.cuh"

namespace leankv {

// The visible positions of position i: first .. i.
__host__ __device__ __forceinline__ int first_visible(int i, int size) { return i - size + 1 > 0 ? i - size + 1 : 0; }

// Slot of position p in a ring whose slot 0 holds position `base` (p >= base - ring).
__host__ __device__ __forceinline__ int ring_slot(int p, int base, int ring) {
    const int s = (p - base) % ring;
    return s < 0 ? s + ring : s;
}

__device__ __forceinline__ float2 turn(float u, float v, float s, float c) {
    return make_float2(u * c - v * s, v * c + u * s);
}

inline int check_causal(const leankv_causal_attn_t* a) {
    if (!a || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 ||
        a->shared_dim < 0 || a->dim_pad < a->dim || a->vdim_pad < a->vdim || a->shared_pad < a->shared_dim ||
        a->size <= 0 || a->k_ring <= 0 || a->k_rows <= 0 || a->k_rows > a->k_ring || !a->k ||
        (a->shared_dim > 0 && (!a->shared || a->s_ring <= 0)) || (!a->v && a->vdim_pad > a->dim_pad))
        return LEANKV_EINVAL;
    if (a->dim_pad % 16 || a->vdim_pad % 16 || a->shared_pad % 16 || !aligned16(a->k) || !aligned16(a->v) ||
        !aligned16(a->shared))
        return LEANKV_EALIGN;
    if (a->dtype != LEANKV_DT_BF16 && a->dtype != LEANKV_DT_F32) return LEANKV_EUNSUPPORTED;
    return LEANKV_OK;
}

// The tensor-core route of leankv_causal_attend; LEANKV_EUNSUPPORTED for storage types and sizes it does not take.
int causal_tile_attend(const leankv_causal_attn_t& a, const void* q, const float* gate, int gate_ld, void* out, int out_ld,
                       int rows, int start, int32_t* status, cudaStream_t st);

}  // namespace leankv
