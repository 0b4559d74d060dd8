// What the kernels of decay_scan*.cu share: a recurrence whose state decays by one number per head and token.
//
//   S_t = a_t S_(t-1) + w_t k_t v_t^T,    o_t = S_t^T q_t + skip v_t          (per head; S is [D][V])
//
// either with a constant a per head and w = 1, or with w_t = softplus(dt_t + dt_bias) and a_t = exp(-rate w_t).
#pragma once
#include "common.cuh"

// p: the step's rows, `ld` elements apart, with G heads of D queries from column q_col on, as many keys from k_col on and H
// heads of V values from v_col on (head h reads the queries and keys of group h / (H / G)).  decay, log2_decay [H]: a and
// its base-2 logarithm (at least -160), or null; dt [rows, dt_ld] 32-bit with dt_bias and rate [H] then.  skip [H] or null.
// act: queries, keys and values pass silu as they are read.  A sequence's record in `state` is [H][D][V] floats,
// state_slot floats apart.
struct SbDecay {
    const void* p;
    long long ld;
    int q_col;
    int k_col;
    int v_col;
    int act;
    const float* decay;
    const float* log2_decay;
    const float* dt;
    long long dt_ld;
    const float* dt_bias;
    const float* rate;
    const float* skip;
    float* state;
    long long state_slot;
    int H;
    int G;
    int D;
    int V;
};

__device__ __forceinline__ float silu_value(float x) { return __fdividef(x, 1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_value(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
