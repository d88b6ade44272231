// First and last kernel of a decode step: embedding fetch and greedy next token. Templated on the storage
// type of the table / the logits, so that every decode loop of the library frames its step the same way.
#pragma once

#include "typed.cuh"

namespace leankv {

// Decode state words (int32[8], device), as the header describes them beside leankv_decode_begin: position,
// step count, the one-sequence page table (kv_indptr[0..1], kv_last_page_len, start position), and the half
// of a double-buffered per-sequence vector that the current step reads.
enum { kPos = 0, kStep = 1, kIndptr0 = 2, kIndptr1 = 3, kLastLen = 4, kStartPos = 5, kParity = 6 };

// Fetch the embedding row of the current token and derive this step's page-table words.
template <typename In, typename Out>
__global__ void __launch_bounds__(256) decode_begin_kernel(const In* table, const long long* token, Out* h,
                                                           int hidden, int vocab, int* state) {
    pdl_begin();
    long long tok = *token;
    if (tok < 0 || tok >= vocab) tok = 0;
    if constexpr (sizeof(In) == 2 && sizeof(Out) == 2) {      // same type, hidden % 8 == 0 (checked on the host)
        const uint4* src = reinterpret_cast<const uint4*>(table + (size_t)tok * hidden);
        uint4* dst = reinterpret_cast<uint4*>(h);
        for (int i = threadIdx.x; i < hidden / 8; i += blockDim.x) dst[i] = __ldg(src + i);
    } else {
        const In* src = table + (size_t)tok * hidden;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) h[i] = to_f32(src[i]);
    }
    if (threadIdx.x == 0) {
        const int pos = state[kPos];
        state[kStartPos] = pos;
        state[kIndptr0] = 0;
        state[kIndptr1] = pos / 16 + 1;
        state[kLastLen] = pos % 16 + 1;
    }
}

// Greedy next token (lowest index wins ties), appended to the history; advances the position.
// One CTA per sequence: pos / step are that sequence's words. `parity` (optional) is flipped.
template <typename L>
__global__ void __launch_bounds__(1024) decode_end_kernel(const L* logits, int vocab, long long* token,
                                                          long long* history, int history_cap, int* pos,
                                                          int* step_ptr, int* parity) {
    __shared__ float s_v[32];
    __shared__ int s_i[32];
    pdl_begin();
    logits += (size_t)blockIdx.x * vocab;
    token += blockIdx.x;
    history += (size_t)blockIdx.x * history_cap;
    pos += blockIdx.x;
    step_ptr += blockIdx.x;
    float best = -INFINITY;
    int best_i = 0x7fffffff;
    constexpr int kPer = 16 / (int)sizeof(L);
    const int nvec = vocab / kPer;   // 16-byte loads; indices ascend within a thread, so '>' keeps the lowest
    for (int vi = threadIdx.x; vi < nvec; vi += blockDim.x) {
        const uint4 a = __ldg(reinterpret_cast<const uint4*>(logits) + vi);
        const L* hp = reinterpret_cast<const L*>(&a);
#pragma unroll
        for (int q = 0; q < kPer; ++q) {
            const float v = to_f32(hp[q]);
            if (v > best) { best = v; best_i = vi * kPer + q; }
        }
    }
    for (int i = nvec * kPer + threadIdx.x; i < vocab; i += blockDim.x) {
        const float v = to_f32(logits[i]);
        if (v > best || (v == best && i < best_i)) { best = v; best_i = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
        if (ov > best || (ov == best && oi < best_i)) { best = ov; best_i = oi; }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) { s_v[warp] = best; s_i[warp] = best_i; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < (int)(blockDim.x >> 5); ++w)
            if (s_v[w] > best || (s_v[w] == best && s_i[w] < best_i)) { best = s_v[w]; best_i = s_i[w]; }
        if (best_i == 0x7fffffff) best_i = 0;   // all-NaN row
        *token = best_i;
        const int step = *step_ptr;
        if (step < history_cap) history[step] = best_i;
        *step_ptr = step + 1;
        *pos = *pos + 1;
        if (parity != nullptr) *parity ^= 1;
    }
}

}  // namespace leankv
