// What the kernels of the gated delta rule share (delta.cu, delta_chunk.cu).
#pragma once
#include "common.cuh"

#define DS_WARPS 8   // warps of a token-by-token block
#define DS_KEEP 4    // values of a head that a lane keeps in registers between the convolution and the norm

// qkv [rows, 2 G D + H V] 32-bit, [q heads | k heads | v heads], unit queries (scaled) and keys; z [rows, z_ld] 32-bit:
// the decays' inputs [H D], then the gates' [H V]; inner [rows, inner_ld] 32-bit with head h's step size, before its
// sigmoid, at column b_col + h; state [slots] records of [H][D][V] floats, state_slot floats apart.
struct SbDelta {
    const float* qkv;
    const float* z;
    long long z_ld;
    const float* inner;
    long long inner_ld;
    int b_col;
    const float* a_log;
    const float* dt_bias;
    const float* norm;
    float eps;
    float* state;
    long long state_slot;
    int H;
    int G;
    int D;
    int V;
};

// exp(rate * softplus(z)) with rate = -exp(A_log); softplus on the side that does not overflow.
__device__ __forceinline__ float delta_decay(float z, float neg_rate) {
    const float sp = z > 0.f ? z + log1pf(expf(-z)) : log1pf(expf(z));
    return expf(neg_rate * sp);
}

template <int VEC> __device__ __forceinline__ void ds_load(const float* p, float (&v)[VEC]) {
    if (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x;
        v[VEC > 1 ? 1 : 0] = f.y;
        v[VEC > 2 ? 2 : 0] = f.z;
        v[VEC > 3 ? 3 : 0] = f.w;
    } else {
        v[0] = *p;
    }
}
template <int VEC> __device__ __forceinline__ void ds_store(float* p, const float (&v)[VEC]) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[VEC > 1 ? 1 : 0], v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]);
    else *p = v[0];
}
