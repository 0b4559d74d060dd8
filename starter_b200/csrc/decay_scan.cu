// The decaying recurrence token by token: decoding, short steps, every 32-bit run, and sizes that decay_scan_mma.cu does not
// take.  State, decays, step sizes and sums are 32-bit.
#include "decay_scan.cuh"

#define DS_THREADS 256
#define DS_WARPS (DS_THREADS / 32)

template <int VEC> __device__ __forceinline__ void state_load(const float* p, float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = p[i];
}
template <> __device__ __forceinline__ void state_load<4>(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x;
    v[1] = f.y;
    v[2] = f.z;
    v[3] = f.w;
}
template <int VEC> __device__ __forceinline__ void state_store(float* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = v[i];
}
template <> __device__ __forceinline__ void state_store<4>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}

// One block per (sequence, head, `columns` value columns).  columns / VEC threads stand side by side along the columns, the
// others take further key channels: thread (phase, cl) holds the channels phase, phase + phases, ... of VEC neighbouring
// columns.  With EMAX > 0 (D <= EMAX * phases) they stay in registers over all rows of the step, else in the sequence's
// record (a thread meets the same entries at every row).  columns / VEC is a power of two up to 32.
template <class T, int VEC, int EMAX>
__global__ void __launch_bounds__(DS_THREADS)
decay_step_kernel(SbDecay a, SbBatch batch, float* __restrict__ out, int columns) {
    extern __shared__ float sm[];
    const int D = a.D, V = a.V, H = a.H;
    float* qs = sm;          // [D] the token's query and key, the key times its weight
    float* ks = qs + D;
    float* red = ks + D;     // [DS_WARPS][columns]
    const int s = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int tc = columns / VEC, cl = tid % tc, phase = tid / tc, phases = DS_THREADS / tc;
    const int col = blockIdx.z * columns + cl * VEC;
    const bool live = col < V;
    const int grp = head / (H / a.G);
    const float fixed = a.decay != nullptr ? a.decay[head] : 0.f;
    const float bias = a.dt != nullptr ? a.dt_bias[head] : 0.f, rate = a.dt != nullptr ? a.rate[head] : 0.f;
    const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
    pdl_wait();
    const int row0 = batch.cu_q[s], row1 = batch.cu_q[s + 1];
    float* Sg = a.state + (long long)batch.seq_slot[s] * a.state_slot + (long long)head * D * V + col;
    float S[EMAX > 0 ? EMAX : 1][VEC];
    if (EMAX > 0) {
#pragma unroll
        for (int e = 0; e < EMAX; ++e) {
            const int d = e * phases + phase;
#pragma unroll
            for (int i = 0; i < VEC; ++i) S[e][i] = 0.f;
            if (live && d < D) state_load<VEC>(Sg + (long long)d * V, S[e]);
        }
    }
    for (int row = row0; row < row1; ++row) {
        const T* in = (const T*)a.p + row * a.ld;
        float av = fixed, wv = 1.f;
        if (a.dt != nullptr) {
            wv = softplus_value(a.dt[row * a.dt_ld + head] + bias);
            av = expf(-rate * wv);
        }
        float v[VEC], o[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            v[i] = live ? to_f<T>(in[a.v_col + head * V + col + i]) : 0.f;
            if (a.act) v[i] = silu_value(v[i]);
            o[i] = phase == 0 ? skip * v[i] : 0.f;
        }
        __syncthreads();     // the row before has been read
        for (int i = tid; i < D; i += DS_THREADS) {
            float q = to_f<T>(in[a.q_col + grp * D + i]), k = to_f<T>(in[a.k_col + grp * D + i]);
            if (a.act) {
                q = silu_value(q);
                k = silu_value(k);
            }
            qs[i] = q;
            ks[i] = k * wv;
        }
        __syncthreads();
        if (EMAX > 0) {
#pragma unroll
            for (int e = 0; e < EMAX; ++e) {
                const int d = e * phases + phase;
                if (d < D) {
                    const float k = ks[d], q = qs[d];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) {
                        S[e][i] = fmaf(av, S[e][i], k * v[i]);
                        o[i] = fmaf(q, S[e][i], o[i]);
                    }
                }
            }
        } else if (live) {
#pragma unroll 4
            for (int d = phase; d < D; d += phases) {
                float cell[VEC];
                state_load<VEC>(Sg + (long long)d * V, cell);
                const float k = ks[d], q = qs[d];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    cell[i] = fmaf(av, cell[i], k * v[i]);
                    o[i] = fmaf(q, cell[i], o[i]);
                }
                state_store<VEC>(Sg + (long long)d * V, cell);
            }
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i)
            for (int off = tc; off < 32; off <<= 1) o[i] += __shfl_xor_sync(0xffffffffu, o[i], off);
        if (lane < tc) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) red[warp * columns + cl * VEC + i] = o[i];
        }
        __syncthreads();
        for (int c = tid; c < columns; c += DS_THREADS) {
            const int at = blockIdx.z * columns + c;
            if (at < V) {
                float sum = 0.f;
#pragma unroll
                for (int w = 0; w < DS_WARPS; ++w) sum += red[w * columns + c];
                out[((long long)row * H + head) * V + at] = sum;
            }
        }
    }
    if (EMAX > 0 && row0 < row1) {
#pragma unroll
        for (int e = 0; e < EMAX; ++e) {
            const int d = e * phases + phase;
            if (live && d < D) state_store<VEC>(Sg + (long long)d * V, S[e]);
        }
    }
}

// The first n columns of every row pass silu, in place.  VEC: bfloat16, n and the row stride multiples of 8.
template <class T, bool VEC>
__global__ void silu_columns_kernel(T* __restrict__ p, long long ld, int n, long long total) {
    pdl_wait();
    constexpr int W = VEC ? 8 : 1;
    const int per_row = n / W;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        T* at = p + (i / per_row) * ld + (i % per_row) * W;
        if (VEC) {
            uint4 raw = *reinterpret_cast<uint4*>(at);
            __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(h[e]);
                h[e] = __floats2bfloat162_rn(silu_value(f.x), silu_value(f.y));
            }
            *reinterpret_cast<uint4*>(at) = raw;
        } else {
            *at = from_f<T>(silu_value(to_f<T>(*at)));
        }
    }
}

template <class T>
static int launch_decay_step(SbDecay a, SbBatch batch, float* out, int columns, cudaStream_t stream) {
    const bool vec = a.V % 4 == 0 && (reinterpret_cast<size_t>(a.state) & 15) == 0 && a.state_slot % 4 == 0;
    if (!vec) columns = 32;
    const int tc = columns / (vec ? 4 : 1), phases = DS_THREADS / tc;
    const dim3 grid(batch.n_seqs, a.H, (a.V + columns - 1) / columns);
    if (grid.z > 65535) return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)(2 * a.D + DS_WARPS * columns) * sizeof(float);
#define SB_DS(VEC, EMAX)                                                                                                       \
    do {                                                                                                                       \
        if (smem > 48 * 1024) {                                                                                                \
            const cudaError_t err = cudaFuncSetAttribute(decay_step_kernel<T, VEC, EMAX>,                                      \
                                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);              \
            if (err != cudaSuccess) return (int)err;                                                                           \
        }                                                                                                                      \
        sb_launch(decay_step_kernel<T, VEC, EMAX>, grid, DS_THREADS, smem, stream, a, batch, out, columns);                    \
    } while (0)
    if (a.D <= 4 * phases) {
        if (vec) SB_DS(4, 4);
        else SB_DS(1, 4);
    } else if (a.D <= 16 * phases) {
        if (vec) SB_DS(4, 16);
        else SB_DS(1, 16);
    } else {
        if (vec) SB_DS(4, 0);
        else SB_DS(1, 0);
    }
#undef SB_DS
    SB_LAUNCH_CHECK();
}

extern "C" {

// out [rows, H V] floats; columns: value columns per block, 32, 64 or 128 (taken as 32 where 16-byte reads do not fit).
int sb_decay_step(int dtype, SbDecay a, SbBatch batch, float* out, int columns, cudaStream_t stream) {
    if (batch.n_seqs <= 0 || batch.n_rows <= 0) return 0;
    if (a.D < 1 || a.V < 1 || a.D > 4096 || a.V > 65536 || a.G < 1 || a.H % a.G || a.H > 65535 || (a.decay == nullptr) == (a.dt == nullptr)
        || (columns != 32 && columns != 64 && columns != 128))
        return (int)cudaErrorInvalidValue;
    if (dtype == SB_F32) return launch_decay_step<float>(a, batch, out, columns, stream);
    return launch_decay_step<__nv_bfloat16>(a, batch, out, columns, stream);
}

int sb_silu_columns(int dtype, void* p, long long ld, int n, int rows, cudaStream_t stream) {
    if (rows <= 0 || n <= 0) return 0;
    const bool vec = dtype == SB_BF16 && n % 8 == 0 && ld % 8 == 0 && (reinterpret_cast<size_t>(p) & 15) == 0;
    const long long total = (long long)rows * (vec ? n / 8 : n);
    const unsigned int blocks = (unsigned int)((total + 255) / 256 < 16384 ? (total + 255) / 256 : 16384);
    if (dtype == SB_F32) sb_launch(silu_columns_kernel<float, false>, blocks, 256, 0, stream, (float*)p, ld, n, total);
    else if (vec) sb_launch(silu_columns_kernel<__nv_bfloat16, true>, blocks, 256, 0, stream, (__nv_bfloat16*)p, ld, n, total);
    else sb_launch(silu_columns_kernel<__nv_bfloat16, false>, blocks, 256, 0, stream, (__nv_bfloat16*)p, ld, n, total);
    SB_LAUNCH_CHECK();
}

}  // extern "C"
