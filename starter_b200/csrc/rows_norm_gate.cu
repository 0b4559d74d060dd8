// The way out of a recurrence whose heads are normed together: 32-bit rows, an RMS norm in equal consecutive parts, a weight
// per column and a gate, before or behind the norm.
//
//   gate behind:  y = o / rms(part of o) * w * sigmoid(g)
//   gate first:   t = o * silu(g),  y = t / rms(part of t) * w
//
// All of it is 32-bit and rounded once, when the result is stored.
#include "common.cuh"

#define NG_THREADS 256
#define NG_KEEP 4    // groups of VEC columns that a thread keeps between the two passes

template <class T, int VEC> __device__ __forceinline__ void gate_load(const T* p, float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = to_f<T>(p[i]);
}
template <> __device__ __forceinline__ void gate_load<__nv_bfloat16, 4>(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x;
    v[1] = a.y;
    v[2] = b.x;
    v[3] = b.y;
}
template <class T, int VEC> __device__ __forceinline__ void row_store(T* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = from_f<T>(v[i]);
}
template <> __device__ __forceinline__ void row_store<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned int*>(&a);
    raw.y = *reinterpret_cast<const unsigned int*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// One block per (row, part).  VEC 4: a part's width, the gate's row stride and its start are multiples of 4.
template <class T, int VEC>
__global__ void __launch_bounds__(NG_THREADS)
norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long gate_ld, const float* __restrict__ weight,
                 T* __restrict__ y, int width, int part, float eps, int gate_first) {
    __shared__ float red[33];
    pdl_wait();
    const long long row = blockIdx.x;
    const int c0 = blockIdx.y * part, step = VEC * blockDim.x;
    const float* orow = o + row * width + c0;
    const T* grow = gate + row * gate_ld + c0;
    const float* wrow = weight + c0;
    auto value = [&](int c, float (&v)[VEC]) {
        if (VEC == 4) {
            const float4 f = *reinterpret_cast<const float4*>(orow + c);
            v[0] = f.x;
            if (VEC > 1) v[VEC > 1 ? 1 : 0] = f.y;
            if (VEC > 2) v[VEC > 2 ? 2 : 0] = f.z;
            if (VEC > 3) v[VEC > 3 ? 3 : 0] = f.w;
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] = orow[c + i];
        }
        if (gate_first) {
            float g[VEC];
            gate_load<T, VEC>(grow + c, g);
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] *= g[i] / (1.0f + expf(-g[i]));
        }
    };
    float keep[NG_KEEP][VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < NG_KEEP; ++k) {
        const int c = threadIdx.x * VEC + k * step;
        if (c < part) {
            value(c, keep[k]);
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(keep[k][i], keep[k][i], ss);
        }
    }
    for (int c = threadIdx.x * VEC + NG_KEEP * step; c < part; c += step) {
        float v[VEC];
        value(c, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)part + eps);
    auto finish = [&](int c, float (&v)[VEC]) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] *= rstd * wrow[c + i];
        if (!gate_first) {
            float g[VEC];
            gate_load<T, VEC>(grow + c, g);
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] *= 1.0f / (1.0f + expf(-g[i]));
        }
        row_store<T, VEC>(y + row * width + c0 + c, v);
    };
#pragma unroll
    for (int k = 0; k < NG_KEEP; ++k) {
        const int c = threadIdx.x * VEC + k * step;
        if (c < part) finish(c, keep[k]);
    }
    for (int c = threadIdx.x * VEC + NG_KEEP * step; c < part; c += step) {
        float v[VEC];
        value(c, v);
        finish(c, v);
    }
}

extern "C" {

// o [rows, width] floats; gate [rows, width], rows gate_ld elements apart; weight [width] floats; y [rows, width].
int sb_norm_gate(int dtype, const float* o, const void* gate, long long gate_ld, const float* weight, void* y, int rows, int width,
                 int parts, float eps, int gate_first, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (parts < 1 || width % parts || parts > 65535) return (int)cudaErrorInvalidValue;
    const int part = width / parts;
    const size_t align = dtype == SB_F32 ? 4 : 8;     // bytes that a thread's read of the gate takes: 4 floats are read one by one
    const bool vec = part % 4 == 0 && gate_ld % 4 == 0 && (reinterpret_cast<size_t>(gate) & (align - 1)) == 0
                     && (reinterpret_cast<size_t>(o) & 15) == 0 && (reinterpret_cast<size_t>(y) & 7) == 0;
    const int lanes = vec ? part / 4 : part;
    const int threads = lanes >= 1024 ? NG_THREADS : (lanes >= NG_THREADS ? NG_THREADS : (lanes + 31) / 32 * 32);
    const dim3 grid(rows, parts);
    typedef __nv_bfloat16 bf;
    if (dtype == SB_F32) {
        if (vec) sb_launch(norm_gate_kernel<float, 4>, grid, threads, 0, stream, o, (const float*)gate, gate_ld, weight, (float*)y, width, part, eps, gate_first);
        else sb_launch(norm_gate_kernel<float, 1>, grid, threads, 0, stream, o, (const float*)gate, gate_ld, weight, (float*)y, width, part, eps, gate_first);
    } else {
        if (vec) sb_launch(norm_gate_kernel<bf, 4>, grid, threads, 0, stream, o, (const bf*)gate, gate_ld, weight, (bf*)y, width, part, eps, gate_first);
        else sb_launch(norm_gate_kernel<bf, 1>, grid, threads, 0, stream, o, (const bf*)gate, gate_ld, weight, (bf*)y, width, part, eps, gate_first);
    }
    SB_LAUNCH_CHECK();
}

}  // extern "C"
