// One product per head: C[m, h, :] = A[m, h, :] * W[h]^T for W [heads, N, K], on the CUDA cores, any sizes.
//
// A and C are views with a row stride and a head stride (their last axis is contiguous), so a head's columns can
// be read out of, and written into, wider rows without a copy.  Each output is one running 32-bit sum over
// k = 0..K-1 in order: a row's result does not depend on the rows around it.  It is the product of the 32-bit
// path and of small shapes; many rows in bfloat16 go to the library's batched product.
//
// gate [rows, heads] (a view with a row stride; null: none): head h's outputs of row m are multiplied by
// sigmoid(gate[m, h]), the product as it reads back from its type.  gate_heads is that step alone, for outputs that come
// from elsewhere.
#include "common.cuh"

template <class T> __device__ __forceinline__ float head_sigmoid(const T* gate, long long gate_row, long long m, int head) {
    return 1.0f / (1.0f + expf(-to_f<T>(gate[m * gate_row + head])));
}

#define GH_BM 64
#define GH_BN 64
#define GH_BK 16

template <class T>
__global__ void __launch_bounds__(256) gemm_heads_kernel(const T* __restrict__ A, long long a_row, long long a_head,
                                                         const T* __restrict__ W, T* __restrict__ C, long long c_row,
                                                         long long c_head, const T* __restrict__ gate, long long gate_row, int M, int N, int K) {
    __shared__ float As[GH_BK][GH_BM + 4];
    __shared__ float Ws[GH_BK][GH_BN + 4];
    pdl_wait();
    const int tid = threadIdx.x, head = blockIdx.z;
    const T* Ah = A + head * a_head;
    const T* Wh = W + (long long)head * N * K;
    T* Ch = C + head * c_head;
    const int m0 = blockIdx.y * GH_BM, n0 = blockIdx.x * GH_BN;
    const int tx = tid % 16, ty = tid / 16;
    const int lr = tid / 4, lk = (tid % 4) * 4;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += GH_BK) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = k0 + lk + e;
            const int am = m0 + lr, wn = n0 + lr;
            As[lk + e][lr] = (am < M && k < K) ? to_f<T>(Ah[am * a_row + k]) : 0.f;
            Ws[lk + e][lr] = (wn < N && k < K) ? to_f<T>(Wh[(long long)wn * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < GH_BK; ++kk) {
            float a[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) w[j] = Ws[kk][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
        const float sig = gate != nullptr ? head_sigmoid<T>(gate, gate_row, m, head) : 1.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n < N) Ch[m * c_row + n] = from_f<T>(gate != nullptr ? rnd<T>(acc[i][j]) * sig : acc[i][j]);
        }
    }
}

// A handful of rows (a decode step): a warp per output column of a head, the lanes striding over K, every row's sum
// reduced across the warp.  The tiled kernel above spends a step of 8 rows on 64-row tiles and a barrier every 16
// columns of K (33 us for 16 heads of 128 x 512 on a B200); this one is bound by the few hundred KB it reads.
#define GH_SMALL_M 16

template <class T>
__global__ void __launch_bounds__(256) gemm_heads_rows_kernel(const T* __restrict__ A, long long a_row, long long a_head,
                                                              const T* __restrict__ W, T* __restrict__ C, long long c_row,
                                                              long long c_head, const T* __restrict__ gate, long long gate_row, int M, int N, int K) {
    pdl_wait();
    const int head = blockIdx.y, lane = threadIdx.x & 31;
    const int n = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (n >= N) return;
    const T* w = W + ((long long)head * N + n) * K;
    const T* a = A + head * a_head;
    float acc[GH_SMALL_M];
#pragma unroll
    for (int m = 0; m < GH_SMALL_M; ++m) acc[m] = 0.f;
    for (int k = lane; k < K; k += 32) {
        const float wv = to_f<T>(w[k]);
#pragma unroll
        for (int m = 0; m < GH_SMALL_M; ++m)
            if (m < M) acc[m] = fmaf(to_f<T>(a[m * a_row + k]), wv, acc[m]);
    }
#pragma unroll
    for (int m = 0; m < GH_SMALL_M; ++m) {
        if (m < M) {
            const float v = warp_sum(acc[m]);
            if (lane == 0)
                C[head * c_head + m * c_row + n] =
                    from_f<T>(gate != nullptr ? rnd<T>(v) * head_sigmoid<T>(gate, gate_row, m, head) : v);
        }
    }
}

// out[m, h, :] = a[m, h, :] * sigmoid(gate[m, h]); a with a row and a head stride, out contiguous.  V8: eight bfloat16
// columns at a time.
template <class T, bool V8>
__global__ void gate_heads_kernel(const T* __restrict__ a, long long a_row, long long a_head, const T* __restrict__ gate,
                                  long long gate_row, T* __restrict__ out, long long rows, int H, int V) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int W = V8 ? 8 : 1;
    const long long n = rows * H * V / W;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const long long mh = i * W / V, m = mh / H;
        const int h = (int)(mh - m * H), c = (int)(i * W - mh * V);
        const float sig = head_sigmoid<T>(gate, gate_row, m, h);
        const T* src = a + m * a_row + h * a_head + c;
        if (V8) {
            const uint4 raw = *reinterpret_cast<const uint4*>(src);
            const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw);
            uint4 res;
            __nv_bfloat162* y = reinterpret_cast<__nv_bfloat162*>(&res);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(x[e]);
                y[e] = __floats2bfloat162_rn(f.x * sig, f.y * sig);
            }
            *reinterpret_cast<uint4*>(out + i * W) = res;
        } else {
            out[i] = from_f<T>(to_f<T>(*src) * sig);
        }
    }
}

extern "C" int sb_gate_heads(int dtype, const void* a, long long a_row, long long a_head, const void* gate, long long gate_row, void* out,
                             int rows, int H, int V, cudaStream_t stream) {
    if (rows <= 0 || H <= 0 || V <= 0) return 0;
    typedef __nv_bfloat16 bf;
    const long long n = (long long)rows * H * V;
    const bool v8 = dtype == SB_BF16 && V % 8 == 0 && a_row % 8 == 0 && a_head % 8 == 0 && (reinterpret_cast<size_t>(a) & 15) == 0
                    && (reinterpret_cast<size_t>(out) & 15) == 0;
    const long long items = v8 ? n / 8 : n;
    const int blocks = (int)((items + 255) / 256 < 8192 ? (items + 255) / 256 : 8192);
    if (dtype == SB_F32)
        sb_launch(gate_heads_kernel<float, false>, blocks, 256, 0, stream, (const float*)a, a_row, a_head, (const float*)gate, gate_row,
                  (float*)out, (long long)rows, H, V);
    else if (v8)
        sb_launch(gate_heads_kernel<bf, true>, blocks, 256, 0, stream, (const bf*)a, a_row, a_head, (const bf*)gate, gate_row, (bf*)out,
                  (long long)rows, H, V);
    else
        sb_launch(gate_heads_kernel<bf, false>, blocks, 256, 0, stream, (const bf*)a, a_row, a_head, (const bf*)gate, gate_row, (bf*)out,
                  (long long)rows, H, V);
    SB_LAUNCH_CHECK();
}

// Strides in elements.
extern "C" int sb_gemm_heads(int dtype, const void* A, long long a_row, long long a_head, const void* W, void* C, long long c_row,
                             long long c_head, const void* gate, long long gate_row, int M, int N, int K, int heads, cudaStream_t stream) {
    if (M <= 0 || N <= 0 || heads <= 0) return 0;
    if (M <= GH_SMALL_M && heads <= 65535) {
        dim3 small((N + 7) / 8, heads);
        if (dtype == SB_F32)
            sb_launch(gemm_heads_rows_kernel<float>, small, 256, 0, stream, (const float*)A, a_row, a_head, (const float*)W, (float*)C,
                      c_row, c_head, (const float*)gate, gate_row, M, N, K);
        else
            sb_launch(gemm_heads_rows_kernel<__nv_bfloat16>, small, 256, 0, stream, (const __nv_bfloat16*)A, a_row, a_head,
                      (const __nv_bfloat16*)W, (__nv_bfloat16*)C, c_row, c_head, (const __nv_bfloat16*)gate, gate_row, M, N, K);
        SB_LAUNCH_CHECK();
    }
    dim3 grid((N + GH_BN - 1) / GH_BN, (M + GH_BM - 1) / GH_BM, heads);
    if (grid.y > 65535 || grid.z > 65535) return (int)cudaErrorInvalidValue;
    if (dtype == SB_F32)
        sb_launch(gemm_heads_kernel<float>, grid, 256, 0, stream, (const float*)A, a_row, a_head, (const float*)W, (float*)C, c_row,
                  c_head, (const float*)gate, gate_row, M, N, K);
    else
        sb_launch(gemm_heads_kernel<__nv_bfloat16>, grid, 256, 0, stream, (const __nv_bfloat16*)A, a_row, a_head,
                  (const __nv_bfloat16*)W, (__nv_bfloat16*)C, c_row, c_head, (const __nv_bfloat16*)gate, gate_row, M, N, K);
    SB_LAUNCH_CHECK();
}
