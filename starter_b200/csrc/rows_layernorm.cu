// Row kernels of a model with layer norms over a 32-bit residual, gated gelu feed-forwards and a capped head:
//
//   layernorm        (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b, with the residual sum x += delta in front
//   embed_layernorm  the same of an embedding row, 32-bit out: the first residual of a model that norms its embedding
//   gated_gelu       gelu_tanh(g) * u
//   softcap          cap * tanh(x / cap)
//
// Means, squares, the scaling and the residual sum are 32-bit; a result is rounded once, when it is stored.
#include "common.cuh"

#define LN_KEEP 4   // groups of four columns that a thread keeps in registers between the passes over its row

__device__ __forceinline__ float4 ln_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ln_load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ln_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ln_store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned int*>(&a);
    raw.y = *reinterpret_cast<const unsigned int*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// A row whose width is a multiple of 4 and at most 4 * LN_KEEP * blockDim.x: every thread keeps its columns in
// registers, so the row is read once.
template <class TX, class T, class TO>
__device__ __forceinline__ void layernorm_row_kept(const TX* src, const T* delta, float* back, const float* __restrict__ w,
                                                   const float* __restrict__ b, TO* out, int width, float eps, float* red) {
    float4 v[LN_KEEP];
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < LN_KEEP; ++i) {
        const int c = 4 * (i * blockDim.x + threadIdx.x);
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < width) {
            v[i] = ln_load4(src + c);
            if (delta != nullptr) {
                const float4 d = ln_load4(delta + c);
                v[i] = make_float4(v[i].x + d.x, v[i].y + d.y, v[i].z + d.z, v[i].w + d.w);
                ln_store4(back + c, v[i]);
            }
            sum += (v[i].x + v[i].y) + (v[i].z + v[i].w);
        }
    }
    const float mean = block_sum(sum, red) / (float)width;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < LN_KEEP; ++i) {
        const int c = 4 * (i * blockDim.x + threadIdx.x);
        if (c < width) {
            v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
        }
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < LN_KEEP; ++i) {
        const int c = 4 * (i * blockDim.x + threadIdx.x);
        if (c < width) {
            const float4 w4 = ln_load4(w + c), b4 = ln_load4(b + c);
            ln_store4(out + c, make_float4(fmaf(v[i].x * rstd, w4.x, b4.x), fmaf(v[i].y * rstd, w4.y, b4.y),
                                           fmaf(v[i].z * rstd, w4.z, b4.z), fmaf(v[i].w * rstd, w4.w, b4.w)));
        }
    }
}

// Any width: the row is read once per pass.  A thread reads back what it wrote itself.
template <class TX, class T, class TO>
__device__ __forceinline__ void layernorm_row_any(const TX* src, const T* delta, float* back, const float* __restrict__ w,
                                                  const float* __restrict__ b, TO* out, int width, float eps, float* red) {
    auto value = [&](int c) { return delta != nullptr ? back[c] : to_f<TX>(src[c]); };
    float sum = 0.f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float v = to_f<TX>(src[c]);
        if (delta != nullptr) {
            v += to_f<T>(delta[c]);
            back[c] = v;
        }
        sum += v;
    }
    const float mean = block_sum(sum, red) / (float)width;
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float d = value(c) - mean;
        ss = fmaf(d, d, ss);
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) out[c] = from_f<TO>(fmaf((value(c) - mean) * rstd, w[c], b[c]));
}

// x: the 32-bit residual, one block per row; delta may be null.
template <class T, bool KEPT>
__global__ void layernorm_kernel(float* x, const T* __restrict__ delta, const float* __restrict__ w, const float* __restrict__ b,
                                 T* __restrict__ out, int width, float eps) {
    __shared__ float red[33];
    pdl_wait();
    pdl_launch_dependents();
    const long long base = (long long)blockIdx.x * width;
    const T* d = delta != nullptr ? delta + base : nullptr;
    if (KEPT) layernorm_row_kept<float, T, T>(x + base, d, x + base, w, b, out + base, width, eps, red);
    else layernorm_row_any<float, T, T>(x + base, d, x + base, w, b, out + base, width, eps, red);
}

template <class T, bool KEPT>
__global__ void embed_layernorm_kernel(const int* __restrict__ tokens, const T* __restrict__ table, const float* __restrict__ w,
                                       const float* __restrict__ b, float* __restrict__ out, int width, int vocab, float eps, int* status) {
    __shared__ float red[33];
    pdl_wait();
    pdl_launch_dependents();
    const int row = blockIdx.x;
    int tok = tokens[row];
    if (tok < 0 || tok >= vocab) {
        if (threadIdx.x == 0) atomicOr(status, SB_STATUS_BAD_TOKEN);
        tok = 0;
    }
    const T* src = table + (long long)tok * width;
    float* dst = out + (long long)row * width;
    if (KEPT) layernorm_row_kept<T, float, float>(src, nullptr, nullptr, w, b, dst, width, eps, red);
    else layernorm_row_any<T, float, float>(src, nullptr, nullptr, w, b, dst, width, eps, red);
}

template <class T>
__global__ void gated_gelu_kernel(const T* __restrict__ gu, T* __restrict__ out, int inter, long long total) {
    pdl_wait();
    pdl_launch_dependents();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long row = i / inter;
        const int c = (int)(i - row * inter);
        const float g = to_f<T>(gu[row * 2 * inter + c]), u = to_f<T>(gu[row * 2 * inter + inter + c]);
        out[i] = from_f<T>(gelu_tanh_value(g) * u);
    }
}

// bfloat16 rows whose half-width is a multiple of 8: eight values per thread, 16-byte accesses.
__global__ void gated_gelu_vec_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, int inter, long long total8) {
    pdl_wait();
    pdl_launch_dependents();
    const int per_row = inter / 8;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total8; i += (long long)gridDim.x * blockDim.x) {
        const long long row = i / per_row;
        const int c = (int)(i % per_row) * 8;
        const uint4 graw = *reinterpret_cast<const uint4*>(gu + row * 2 * inter + c);
        const uint4 uraw = *reinterpret_cast<const uint4*>(gu + row * 2 * inter + inter + c);
        const __nv_bfloat162* gh = reinterpret_cast<const __nv_bfloat162*>(&graw);
        const __nv_bfloat162* uh = reinterpret_cast<const __nv_bfloat162*>(&uraw);
        uint4 res;
        __nv_bfloat162* rh = reinterpret_cast<__nv_bfloat162*>(&res);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 gf = __bfloat1622float2(gh[e]), uf = __bfloat1622float2(uh[e]);
            rh[e] = __floats2bfloat162_rn(gelu_tanh_value(gf.x) * uf.x, gelu_tanh_value(gf.y) * uf.y);
        }
        *reinterpret_cast<uint4*>(out + row * inter + c) = res;
    }
}

__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap) {
    pdl_wait();
    pdl_launch_dependents();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

static bool ln_aligned(const void* p) { return p == nullptr || (reinterpret_cast<size_t>(p) & 15) == 0; }

// Threads per row: enough that LN_KEEP groups of four columns each cover it (kept), or a usual block.
static int ln_threads(int width, bool kept) {
    if (!kept) return width >= 1024 ? 256 : 128;
    const int groups = width / 4;
    const int want = groups <= 512 ? groups : (groups + LN_KEEP - 1) / LN_KEEP;
    const int threads = (want + 31) / 32 * 32;
    return threads < 64 ? 64 : threads;
}

extern "C" {

// x [rows, width] 32-bit; delta (or null) and out in `dtype`; w, b 32-bit.
int sb_layernorm(int dtype, float* x, const void* delta, const float* w, const float* b, void* out, int rows, int width, float eps,
                 cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (width < 1) return (int)cudaErrorInvalidValue;
    typedef __nv_bfloat16 bf;
    const bool kept = width % 4 == 0 && width <= 4 * LN_KEEP * 1024 && ln_aligned(x) && ln_aligned(delta) && ln_aligned(w) && ln_aligned(b)
                      && ln_aligned(out);
    const int threads = ln_threads(width, kept);
    if (dtype == SB_F32) {
        if (kept) sb_launch(layernorm_kernel<float, true>, rows, threads, 0, stream, x, (const float*)delta, w, b, (float*)out, width, eps);
        else sb_launch(layernorm_kernel<float, false>, rows, threads, 0, stream, x, (const float*)delta, w, b, (float*)out, width, eps);
    } else {
        if (kept) sb_launch(layernorm_kernel<bf, true>, rows, threads, 0, stream, x, (const bf*)delta, w, b, (bf*)out, width, eps);
        else sb_launch(layernorm_kernel<bf, false>, rows, threads, 0, stream, x, (const bf*)delta, w, b, (bf*)out, width, eps);
    }
    SB_LAUNCH_CHECK();
}

int sb_embed_layernorm(int dtype, const int* tokens, const void* table, const float* w, const float* b, float* out, int rows, int width,
                       int vocab, float eps, int* status, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (width < 1 || vocab < 1) return (int)cudaErrorInvalidValue;
    typedef __nv_bfloat16 bf;
    const bool kept = width % 4 == 0 && width <= 4 * LN_KEEP * 1024 && ln_aligned(table) && ln_aligned(w) && ln_aligned(b) && ln_aligned(out);
    const int threads = ln_threads(width, kept);
    if (dtype == SB_F32) {
        if (kept)
            sb_launch(embed_layernorm_kernel<float, true>, rows, threads, 0, stream, tokens, (const float*)table, w, b, out, width, vocab, eps, status);
        else
            sb_launch(embed_layernorm_kernel<float, false>, rows, threads, 0, stream, tokens, (const float*)table, w, b, out, width, vocab, eps, status);
    } else {
        if (kept)
            sb_launch(embed_layernorm_kernel<bf, true>, rows, threads, 0, stream, tokens, (const bf*)table, w, b, out, width, vocab, eps, status);
        else
            sb_launch(embed_layernorm_kernel<bf, false>, rows, threads, 0, stream, tokens, (const bf*)table, w, b, out, width, vocab, eps, status);
    }
    SB_LAUNCH_CHECK();
}

int sb_gated_gelu(int dtype, const void* gu, void* out, int rows, int inter, cudaStream_t stream) {
    if (rows <= 0 || inter <= 0) return 0;
    if (dtype == SB_BF16 && inter % 8 == 0 && ln_aligned(gu) && ln_aligned(out)) {
        const long long total8 = (long long)rows * (inter / 8);
        const int blocks = (int)((total8 + 255) / 256 < 8192 ? (total8 + 255) / 256 : 8192);
        sb_launch(gated_gelu_vec_kernel, blocks, 256, 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, inter, total8);
        SB_LAUNCH_CHECK();
    }
    const long long total = (long long)rows * inter;
    const int blocks = (int)((total + 255) / 256 < 8192 ? (total + 255) / 256 : 8192);
    if (dtype == SB_F32) sb_launch(gated_gelu_kernel<float>, blocks, 256, 0, stream, (const float*)gu, (float*)out, inter, total);
    else sb_launch(gated_gelu_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, inter, total);
    SB_LAUNCH_CHECK();
}

int sb_softcap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) return (int)cudaErrorInvalidValue;
    const int blocks = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
    sb_launch(softcap_kernel, blocks, 256, 0, stream, x, n, cap);
    SB_LAUNCH_CHECK();
}

}  // extern "C"
