// What the kernels of the matrix memory (mLSTM) share: the gates, and the hand-over of the parts of a
// head's state that its blocks have in common.
//
// Per sequence and head, with q_t (times q_scale) and k_t of D values, v_t of V values, a log input gate
// i_t and a log forget gate f_t (a soft cap around zero, the latter then through log sigmoid):
//     m_t = max(f_t + m_(t-1), i_t)
//     S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T         S is D x V
//     n_t = exp(f_t + m_(t-1) - m_t) n_(t-1) + exp(i_t - m_t) k_t
//     o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// The state of a slot is float32: S [heads][D][V], and per head a tail of D + 2 values: n, m and a counter
// (an int32, zero between launches).  All zero is a new sequence's state.
//
// Column c of S depends on no other column, so a head's columns are shared out among blocks; n and m are
// needed by all of them.  Every block works them out for itself from what the step before left, and the
// block that is the last to have READ them (the counter says which; nobody waits) writes the new ones.
#pragma once

#include "common.cuh"

#define MEM_DEN_FLOOR 1e-6f

struct MemGates {
    const float *bias_i, *bias_f;      // [heads]
    float cap;
};

__device__ __forceinline__ float mem_log_sigmoid(float x) { return fminf(x, 0.0f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float mem_soft_cap(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float mem_log_input(const MemGates& g, float z, int h) { return mem_soft_cap(z + g.bias_i[h], g.cap); }
__device__ __forceinline__ float mem_log_forget(const MemGates& g, float z, int h) {
    return mem_log_sigmoid(mem_soft_cap(z + g.bias_f[h], g.cap));
}
__device__ __forceinline__ float mem_denominator(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + MEM_DEN_FLOOR; }

// One thread of a block, after every thread of the block has read the head's n and m: whether all the
// head's other blocks have read them too (the counter is then back at zero for the next launch).
__device__ __forceinline__ bool mem_last_reader(float* tail, int D, int n_blocks) {
    if (n_blocks == 1) return true;
    int* counter = reinterpret_cast<int*>(tail + D + 1);
    __threadfence();
    if (atomicAdd(counter, 1) != n_blocks - 1) return false;
    *counter = 0;
    __threadfence();
    return true;
}
