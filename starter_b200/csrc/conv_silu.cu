// A short causal convolution over time per channel with a bias, then silu:
//
//   y_t = silu(bias + sum_j w[:, j] u_(t - taps + 1 + j))
//
// zeros before a sequence's start (its record is zero then), inputs before the step from the sequence's record.  Sums and
// silu are 32-bit, the result is rounded once.
#include "conv_record.cuh"
#include "decay_scan.cuh"

template <class T, int VEC> __device__ __forceinline__ void channels_load(const T* p, float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = to_f<T>(p[i]);
}
template <> __device__ __forceinline__ void channels_load<__nv_bfloat16, 8>(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h[e]);
        v[2 * e] = f.x;
        v[2 * e + 1] = f.y;
    }
}
template <> __device__ __forceinline__ void channels_load<float, 8>(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x;
    v[1] = a.y;
    v[2] = a.z;
    v[3] = a.w;
    v[4] = b.x;
    v[5] = b.y;
    v[6] = b.z;
    v[7] = b.w;
}
template <class T, int VEC> __device__ __forceinline__ void channels_store(T* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = from_f<T>(v[i]);
}
template <> __device__ __forceinline__ void channels_store<__nv_bfloat16, 8>(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// A thread takes VEC channels of R consecutive rows.  u: rows `ld` elements apart; w [taps][C]; out [rows, C].  TAPS > 0: when
// all R rows have every input among the step's rows each input is read once; otherwise (and with TAPS 0: any number of
// taps) row by row.  ADVANCE (a step of one row per sequence, R 1): the thread also moves its channels' record on.
template <class T, int VEC, int R, int TAPS, bool ADVANCE>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const T* __restrict__ u, long long ld, const float* __restrict__ w, const float* __restrict__ bias, int taps, float* state,
                 long long state_slot, SbBatch batch, int C, T* __restrict__ out) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= C) return;
    float b[VEC];
    channels_load<float, VEC>(bias + c, b);
    pdl_wait();
    const int r0 = blockIdx.x * R, n_here = min(R, batch.n_rows - r0), keep = taps - 1;
    if (TAPS > 0 && R > 1) {
        const int s = batch.row_seq[r0];
        if (n_here == R && r0 - batch.cu_q[s] >= TAPS - 1 && batch.row_seq[r0 + R - 1] == s) {
            constexpr int N = TAPS > 0 ? TAPS : 1;
            float wj[N][VEC], win[N][VEC];
#pragma unroll
            for (int j = 0; j < N; ++j) {
                channels_load<float, VEC>(w + (long long)j * C + c, wj[j]);
                if (j < N - 1) channels_load<T, VEC>(u + (long long)(r0 - (N - 1) + j) * ld + c, win[j]);
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
                channels_load<T, VEC>(u + (long long)(r0 + r) * ld + c, win[(N - 1 + r) % N]);
                float y[VEC];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    y[i] = b[i];
#pragma unroll
                    for (int j = 0; j < N; ++j) y[i] = fmaf(wj[j][i], win[(r + j) % N][i], y[i]);
                    y[i] = silu_value(y[i]);
                }
                channels_store<T, VEC>(out + (long long)(r0 + r) * C + c, y);
            }
            return;
        }
    }
    for (int r = 0; r < n_here; ++r) {
        const int row = r0 + r, s = batch.row_seq[row], ahead = row - batch.cu_q[s];
        float* rec = keep > 0 ? state + (long long)batch.seq_slot[s] * state_slot : nullptr;
        float y[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = b[i];
#pragma unroll 4
        for (int j = 0; j < taps; ++j) {
            float x[VEC], wj[VEC];
            channels_load<float, VEC>(w + (long long)j * C + c, wj);
            if (ahead >= keep - j) channels_load<T, VEC>(u + (long long)(row - (keep - j)) * ld + c, x);
            else channels_load<float, VEC>(rec + (long long)(ahead + j) * C + c, x);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                y[i] = fmaf(wj[i], x[i], y[i]);
            }
            if (ADVANCE && j > 0) channels_store<float, VEC>(rec + (long long)(j - 1) * C + c, x);   // entry j - 1 was read in an earlier turn
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = silu_value(y[i]);
        channels_store<T, VEC>(out + (long long)row * C + c, y);
    }
}

extern "C" {

// one_row: every sequence of the step brings one row (the record is moved on in the same kernel).
int sb_conv_silu(int dtype, const void* u, long long ld, const float* w, const float* bias, int taps, float* state, long long state_slot,
                 SbBatch batch, int C, int one_row, void* out, cudaStream_t stream) {
    if (batch.n_rows <= 0) return 0;
    if (taps < 1 || (taps > 1 && state == nullptr) || C < 1) return (int)cudaErrorInvalidValue;
    typedef __nv_bfloat16 bf;
    const bool many = batch.n_rows >= 256 && !one_row;
    const size_t bases = reinterpret_cast<size_t>(u) | reinterpret_cast<size_t>(w) | reinterpret_cast<size_t>(bias) | reinterpret_cast<size_t>(state);
    const bool vec = dtype == SB_BF16 && batch.n_rows >= 64 && C % 8 == 0 && ld % 8 == 0 && state_slot % 4 == 0 && (bases & 15) == 0;
    const int R = many ? 4 : 1;
    const int lanes = vec ? C / 8 : C, threads = lanes >= 128 ? 128 : (lanes + 31) / 32 * 32;
    const dim3 grid((batch.n_rows + R - 1) / R, (lanes + threads - 1) / threads);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define SB_CS(T, VEC, R, TAPS, ADV)                                                                                               \
    sb_launch(conv_silu_kernel<T, VEC, R, TAPS, ADV>, grid, threads, 0, stream, (const T*)u, ld, w, bias, taps, state, state_slot, \
              batch, C, (T*)out)
#define SB_CST(T, VEC)                                      \
    do {                                                    \
        if (one_row && taps > 1) SB_CS(T, VEC, 1, 0, true); \
        else if (R == 1) SB_CS(T, VEC, 1, 0, false);        \
        else if (taps == 4) SB_CS(T, VEC, 4, 4, false);     \
        else if (taps == 3) SB_CS(T, VEC, 4, 3, false);     \
        else if (taps == 2) SB_CS(T, VEC, 4, 2, false);     \
        else SB_CS(T, VEC, 4, 0, false);                    \
    } while (0)
    if (dtype == SB_F32) SB_CST(float, 1);
    else if (vec) SB_CST(bf, 8);
    else SB_CST(bf, 1);
#undef SB_CST
#undef SB_CS
    if (taps > 1 && !one_row) launch_conv_record(dtype, u, ld, taps, state, state_slot, batch, C, stream);
    SB_LAUNCH_CHECK();
}

}  // extern "C"
