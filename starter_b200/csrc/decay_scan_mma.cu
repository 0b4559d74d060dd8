// The decaying recurrence for prompts, 64 tokens at a time on the tensor cores (bfloat16 queries, keys and values).
//
// Let c_i be the sum of the chunk's log-decays up to token i, and S0 the state at the chunk's start:
//
//   P[i][j] = (q_i . k_j) exp(c_i - c_j) w_j  for j <= i           O = P V + exp(c) (Q S0) + skip V
//   S1 = exp(c_last) S0 + sum_j (exp(c_last - c_j) w_j k_j) v_j^T
//
// The state stays in registers as 32-bit sums.  Whatever 32-bit number meets a product (P, the state that the queries read,
// the weighted keys) is written as two bfloat16 numbers hi + lo, so that it keeps 16 bits; queries, keys and values are
// bfloat16 numbers and lose nothing.  Log-decays are summed in 64-bit and kept as two 32-bit numbers, so that a chunk
// with strong decays keeps the differences between its weak ones.
//
// A step with few sequences and heads leaves most SMs without a block when every block walks a whole sequence.  The chunks
// are then dealt out in runs: decay_chunk_kernel<.., STATES> takes every run from a zero state and leaves what it adds and how
// far it decays, decay_runs_kernel walks the runs in order (one multiplication and one addition per entry of the state) and
// leaves the state at each run's start, and decay_chunk_kernel<.., OUTPUTS> takes the outputs of all runs side by side.
#include "decay_scan.cuh"
#include "mma_utils.cuh"

#define DM_L 64              // tokens of a chunk
#define DM_VB 32             // value columns per block
#define DM_VLD (DM_VB + 8)   // a row's stride in shared memory: 16-byte reads of eight rows meet no bank twice
#define DM_THREADS 128
#define DM_LEAST -160.0f     // log2 of a decay that is zero in 32-bit

__device__ __forceinline__ void cp_async_16_or_none(void* smem_dst, const void* gmem_src, bool valid) {
    const unsigned int s = (unsigned int)__cvta_generic_to_shared(smem_dst);
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem_src), "r"(n));
}

// x, y as bfloat16 pairs hi + lo.
__device__ __forceinline__ void split_pair(float x, float y, unsigned int& hi, unsigned int& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 back = __bfloat1622float2(h);
    hi = *reinterpret_cast<const unsigned int*>(&h);
    lo = pack_bf16(x - back.x, y - back.y);
}

// What a chunk's tokens need of the decays: c (as hi + lo, base 2), w, exp2(c), and exp2(c_last - c) w.
struct alignas(16) ChunkDecays {   // read two numbers at a time
    float hi[DM_L], lo[DM_L], w[DM_L], grown[DM_L], left[DM_L];
    float total;   // exp2(c_last)
};

// One warp; the chunk's tokens are rows row .. row + nt - 1, the missing ones neither decay nor weigh anything.
__device__ __forceinline__ void chunk_decays(const SbDecay& a, int head, int row, int nt, ChunkDecays& c) {
    const int lane = threadIdx.x & 31;
    double step[2];
    float w[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        float la = 0.f;
        w[e] = 0.f;
        if (t < nt) {
            if (a.dt != nullptr) {
                w[e] = softplus_value(a.dt[(row + t) * a.dt_ld + head] + a.dt_bias[head]);
                la = fmaxf(-a.rate[head] * w[e] * 1.4426950408889634f, DM_LEAST);
            } else {
                w[e] = 1.f;
                la = a.log2_decay[head];
            }
        }
        step[e] = la;
    }
    double run = step[0] + step[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
    }
    const double last = __shfl_sync(0xffffffffu, run, 31);
    const double at[2] = {run - step[1], run};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        c.hi[t] = (float)at[e];
        c.lo[t] = (float)(at[e] - (double)(float)at[e]);
        c.w[t] = w[e];
        c.grown[t] = exp2f((float)at[e]);
        c.left[t] = exp2f((float)(last - at[e])) * w[e];
    }
    if (lane == 0) c.total = exp2f((float)last);
}

enum { DM_WHOLE = 0, DM_STATES = 1, DM_OUTPUTS = 2 };

// The runs of a step: `count` per sequence of `chunks` chunks each; states [sequence][run][head][D][V] and how far each run
// decays, [sequence][run][head].
struct ChunkRuns {
    float* states;
    float* decays;
    int count;
    int chunks;
};

// A block of four warps per (sequence and run, head, DM_VB value columns) walks the run's chunks (DM_WHOLE: one run per
// sequence, from and back into its record).  Products with the queries:
// warp w owns the tokens 16 w .. 16 w + 15 of the chunk.  State: warp w owns a quarter of the key channels (DP 32: half of
// the channels and half of the columns).  DP: the key channels rounded up to 32, 64, 128 or 256.
template <int DP, int MODE>
__global__ void __launch_bounds__(DM_THREADS, DP <= 128 ? 2 : 1)
decay_chunk_kernel(SbDecay a, SbBatch batch, float* __restrict__ out, int vec, ChunkRuns runs) {
    typedef __nv_bfloat16 bf;
    constexpr int QLD = DP + 8, STAGE = 2 * DM_L * QLD + DM_L * DM_VLD;
    constexpr int MT = DP >= 64 ? DP / 64 : 1, NT = DP >= 64 ? 4 : 2;    // a warp's tiles of 16 channels and of 8 columns of the state
    extern __shared__ __align__(16) unsigned char dm_sm[];
    bf* stages = reinterpret_cast<bf*>(dm_sm);              // [2] of Q [64][QLD], K [64][QLD], V [64][DM_VLD]
    bf* Sh = stages + 2 * STAGE;                            // the state at the chunk's start, hi and lo, [DP][DM_VLD]
    bf* Sl = Sh + DP * DM_VLD;
    __shared__ ChunkDecays decays[2];
    const int D = a.D, V = a.V, H = a.H;
    const int s = MODE == DM_WHOLE ? blockIdx.x : blockIdx.x / runs.count, run = MODE == DM_WHOLE ? 0 : blockIdx.x % runs.count;
    const int head = blockIdx.y, col0 = blockIdx.z * DM_VB, nv = min(DM_VB, V - col0);
    const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g = lane >> 2, t = lane & 3;
    const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
    pdl_wait();
    int row0 = batch.cu_q[s], n = batch.cu_q[s + 1] - row0;
    if (MODE != DM_WHOLE) {                                 // the run's own rows
        row0 += run * runs.chunks * DM_L;
        n = min(n - run * runs.chunks * DM_L, runs.chunks * DM_L);
    }
    const int chunks = (n + DM_L - 1) / DM_L;
    if (n <= 0) return;
    const int grp = head / (H / a.G);
    const bf* base = (const bf*)a.p;
    auto fetch = [&](int ch) {
        bf* Q = stages + (ch & 1) * STAGE;
        bf* K = Q + DM_L * QLD;
        bf* Vs = K + DM_L * QLD;
        const int first = row0 + ch * DM_L, nt = min(DM_L, n - ch * DM_L);
        if (vec) {
            constexpr int QC = DP / 8, VC = DM_VB / 8;
            for (int e = tid; e < DM_L * QC; e += DM_THREADS) {
                const int r = e / QC, c = (e % QC) * 8;
                const bool ok = r < nt && c < D;
                const bf* src = base + (ok ? (first + r) * a.ld + grp * D + c : 0);
                if (MODE != DM_STATES) cp_async_16_or_none(Q + r * QLD + c, src + (ok ? a.q_col : 0), ok);
                cp_async_16_or_none(K + r * QLD + c, src + (ok ? a.k_col : 0), ok);
            }
            for (int e = tid; e < DM_L * VC; e += DM_THREADS) {
                const int r = e / VC, c = (e % VC) * 8;
                const bool ok = r < nt && c < nv;
                cp_async_16_or_none(Vs + r * DM_VLD + c, base + (ok ? (first + r) * a.ld + a.v_col + head * V + col0 + c : 0), ok);
            }
        } else {
            const bf zero = __float2bfloat16_rn(0.f);
            for (int e = tid; e < DM_L * DP; e += DM_THREADS) {
                const int r = e / DP, c = e % DP;
                const bool ok = r < nt && c < D;
                const bf* src = base + (first + r) * a.ld + grp * D + c;
                if (MODE != DM_STATES) Q[r * QLD + c] = ok ? src[a.q_col] : zero;
                K[r * QLD + c] = ok ? src[a.k_col] : zero;
            }
            for (int e = tid; e < DM_L * DM_VB; e += DM_THREADS) {
                const int r = e / DM_VB, c = e % DM_VB;
                Vs[r * DM_VLD + c] = r < nt && c < nv ? base[(first + r) * a.ld + a.v_col + head * V + col0 + c] : zero;
            }
        }
        cp_async_commit();
    };

    const int m_base = DP >= 64 ? w * MT * 16 : (w & 1) * 16, n_base = DP >= 64 ? 0 : (w >> 1) * 16;
    const long long cell = ((long long)blockIdx.x * H + head);     // the run's place among the runs of the step
    float* Sg = (MODE == DM_WHOLE ? a.state + (long long)batch.seq_slot[s] * a.state_slot + (long long)head * D * V
                                  : runs.states + cell * D * V) + col0;
    float S[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = m_base + mt * 16 + g + (e >> 1) * 8, c = n_base + nt * 8 + 2 * t + (e & 1);
                S[mt][nt][e] = MODE != DM_STATES && d < D && c < nv ? Sg[(long long)d * V + c] : 0.f;
            }
    float decayed = 1.f;                                    // how far the run has decayed
    auto publish = [&]() {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int at = (m_base + mt * 16 + g + half * 8) * DM_VLD + n_base + nt * 8 + 2 * t;
                    unsigned int hi, lo;
                    split_pair(S[mt][nt][2 * half], S[mt][nt][2 * half + 1], hi, lo);
                    *reinterpret_cast<unsigned int*>(Sh + at) = hi;
                    *reinterpret_cast<unsigned int*>(Sl + at) = lo;
                }
    };
    fetch(0);
    if (w == 0) chunk_decays(a, head, row0, min(DM_L, n), decays[0]);
    if (MODE != DM_STATES) publish();

    for (int ch = 0; ch < chunks; ++ch) {
        cp_async_wait<0>();
        __syncthreads();                        // the chunk's rows, its decays and the state at its start are there
        if (ch + 1 < chunks) {
            fetch(ch + 1);
            if (w == ((ch + 1) & 3)) chunk_decays(a, head, row0 + (ch + 1) * DM_L, min(DM_L, n - (ch + 1) * DM_L), decays[(ch + 1) & 1]);
        }
        const bf* Q = stages + (ch & 1) * STAGE;
        const bf* K = Q + DM_L * QLD;
        const bf* Vs = K + DM_L * QLD;
        const ChunkDecays& dc = decays[ch & 1];
        if (MODE != DM_STATES) {
        const int i0 = w * 16 + g;              // this thread's tokens: i0 and i0 + 8
        float sc[8][4], o[4][4];
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[i][e] = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
        {
            const bf* qa = Q + (w * 16 + (lane & 15)) * QLD + (lane >> 4) * 8;
            const bf* kb = K + ((lane & 7) + (lane >> 4) * 8) * QLD + ((lane >> 3) & 1) * 8;
            const bf* sh = Sh + (lane & 15) * DM_VLD + (lane >> 4) * 8;
            const bf* sl = Sl + (lane & 15) * DM_VLD + (lane >> 4) * 8;
#pragma unroll
            for (int k0 = 0; k0 < DP; k0 += 16) {
                unsigned int qf[4];
                ldmatrix_x4(qf, qa + k0);
#pragma unroll
                for (int i = 0; i < 8; i += 2) {
                    if (i <= 2 * w) {           // keys after this warp's tokens are not seen
                        unsigned int b[4];
                        ldmatrix_x4(b, kb + i * 8 * QLD + k0);
                        mma_bf16(sc[i], qf, b[0], b[1]);
                        mma_bf16(sc[i + 1], qf, b[2], b[3]);
                    }
                }
#pragma unroll
                for (int i = 0; i < 4; i += 2) {
                    unsigned int b[4];
                    ldmatrix_x4_trans(b, sh + k0 * DM_VLD + i * 8);
                    mma_bf16(o[i], qf, b[0], b[1]);
                    mma_bf16(o[i + 1], qf, b[2], b[3]);
                    ldmatrix_x4_trans(b, sl + k0 * DM_VLD + i * 8);
                    mma_bf16(o[i], qf, b[0], b[1]);
                    mma_bf16(o[i + 1], qf, b[2], b[3]);
                }
            }
        }
        {
            const float e0 = dc.grown[i0], e1 = dc.grown[i0 + 8];
            const float h0 = dc.hi[i0], h1 = dc.hi[i0 + 8], l0 = dc.lo[i0], l1 = dc.lo[i0 + 8];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                o[i][0] *= e0;
                o[i][1] *= e0;
                o[i][2] *= e1;
                o[i][3] *= e1;
            }
            const bf* vb = Vs + (lane & 15) * DM_VLD + (lane >> 4) * 8;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                if (kk <= w) {
                    unsigned int ph[4], pl[4];
#pragma unroll
                    for (int part = 0; part < 2; ++part) {
                        const int i = 2 * kk + part, j = i * 8 + 2 * t;
                        const float2 hj = *reinterpret_cast<const float2*>(dc.hi + j), lj = *reinterpret_cast<const float2*>(dc.lo + j);
                        const float2 wj = *reinterpret_cast<const float2*>(dc.w + j);
                        const float p0 = j <= i0 ? sc[i][0] * fast_exp2((h0 - hj.x) + (l0 - lj.x)) * wj.x : 0.f;
                        const float p1 = j + 1 <= i0 ? sc[i][1] * fast_exp2((h0 - hj.y) + (l0 - lj.y)) * wj.y : 0.f;
                        const float p2 = j <= i0 + 8 ? sc[i][2] * fast_exp2((h1 - hj.x) + (l1 - lj.x)) * wj.x : 0.f;
                        const float p3 = j + 1 <= i0 + 8 ? sc[i][3] * fast_exp2((h1 - hj.y) + (l1 - lj.y)) * wj.y : 0.f;
                        split_pair(p0, p1, ph[2 * part], pl[2 * part]);
                        split_pair(p2, p3, ph[2 * part + 1], pl[2 * part + 1]);
                    }
#pragma unroll
                    for (int i = 0; i < 4; i += 2) {
                        unsigned int b[4];
                        ldmatrix_x4_trans(b, vb + kk * 16 * DM_VLD + i * 8);
                        mma_bf16(o[i], ph, b[0], b[1]);
                        mma_bf16(o[i], pl, b[0], b[1]);
                        mma_bf16(o[i + 1], ph, b[2], b[3]);
                        mma_bf16(o[i + 1], pl, b[2], b[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = i0 + half * 8;
            if (ch * DM_L + i < n) {
                float* dst = out + ((long long)(row0 + ch * DM_L + i) * H + head) * V + col0;
#pragma unroll
                for (int c8 = 0; c8 < 4; ++c8) {
                    const int c = c8 * 8 + 2 * t;
                    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Vs + i * DM_VLD + c));
                    const float x = fmaf(skip, v.x, o[c8][2 * half]), y = fmaf(skip, v.y, o[c8][2 * half + 1]);
                    if (c + 1 < nv && (V & 1) == 0) {
                        *reinterpret_cast<float2*>(dst + c) = make_float2(x, y);
                    } else {
                        if (c < nv) dst[c] = x;
                        if (c + 1 < nv) dst[c + 1] = y;
                    }
                }
            }
        }
        }
        if (MODE == DM_OUTPUTS && ch + 1 == chunks) break;   // nobody asks for the state after the run
        // the state after the chunk
        const float total = dc.total;
        decayed *= total;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[mt][nt][e] *= total;
        {
            const bf* vb = Vs + (lane & 15) * DM_VLD + n_base + (lane >> 4) * 8;
            const bf* ka = K + ((lane & 7) + (lane >> 4) * 8) * QLD + m_base + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                const float2 f0 = *reinterpret_cast<const float2*>(dc.left + kk * 16 + 2 * t);
                const float2 f1 = *reinterpret_cast<const float2*>(dc.left + kk * 16 + 8 + 2 * t);
                unsigned int b[NT / 2][4];
#pragma unroll
                for (int i = 0; i < NT / 2; ++i) ldmatrix_x4_trans(b[i], vb + kk * 16 * DM_VLD + i * 16);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    unsigned int kf[4], kh[4], kl[4];
                    ldmatrix_x4_trans(kf, ka + kk * 16 * QLD + mt * 16);
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&kf[e]));
                        const float2 f = e < 2 ? f0 : f1;
                        split_pair(x.x * f.x, x.y * f.y, kh[e], kl[e]);
                    }
#pragma unroll
                    for (int i = 0; i < NT / 2; ++i) {
                        mma_bf16(S[mt][2 * i], kh, b[i][0], b[i][1]);
                        mma_bf16(S[mt][2 * i], kl, b[i][0], b[i][1]);
                        mma_bf16(S[mt][2 * i + 1], kh, b[i][2], b[i][3]);
                        mma_bf16(S[mt][2 * i + 1], kl, b[i][2], b[i][3]);
                    }
                }
            }
        }
        if (MODE != DM_STATES && ch + 1 < chunks) {
            __syncthreads();                    // nobody reads the state of this chunk's start any more
            publish();
        }
    }
    if (MODE == DM_OUTPUTS) return;
    if (MODE == DM_STATES && tid == 0 && blockIdx.z == 0) runs.decays[cell] = decayed;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = m_base + mt * 16 + g + (e >> 1) * 8, c = n_base + nt * 8 + 2 * t + (e & 1);
                if (d < D && c < nv) Sg[(long long)d * V + c] = S[mt][nt][e];
            }
}

// One thread per entry of a sequence's state: every run's place receives the state at its start, the record the state after
// the last run.  Eight runs' contributions are fetched ahead of the chain.
__global__ void __launch_bounds__(256) decay_runs_kernel(SbDecay a, SbBatch batch, ChunkRuns runs) {
    pdl_wait();
    const int s = blockIdx.x, head = blockIdx.y, size = a.D * a.V;
    const int at = blockIdx.z * blockDim.x + threadIdx.x;
    if (at >= size) return;
    const int n = batch.cu_q[s + 1] - batch.cu_q[s], per = runs.chunks * DM_L, count = min(runs.count, (n + per - 1) / per);
    float* rec = a.state + (long long)batch.seq_slot[s] * a.state_slot + (long long)head * size + at;
    float S = *rec;
    for (int r0 = 0; r0 < count; r0 += 8) {
        float add[8], keep[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const long long cell = ((long long)s * runs.count + min(r0 + i, count - 1)) * a.H + head;
            add[i] = runs.states[cell * size + at];
            keep[i] = runs.decays[cell];
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (r0 + i < count) {
                runs.states[(((long long)s * runs.count + r0 + i) * a.H + head) * size + at] = S;
                S = fmaf(keep[i], S, add[i]);
            }
    }
    if (count > 0) *rec = S;
}

template <int DP, int MODE>
static int launch_chunk_walk(SbDecay a, SbBatch batch, float* out, int vec, ChunkRuns runs, cudaStream_t stream) {
    const size_t smem = (size_t)(2 * (2 * DM_L * (DP + 8) + DM_L * DM_VLD) + 2 * DP * DM_VLD) * sizeof(__nv_bfloat16);
    const cudaError_t err = cudaFuncSetAttribute(decay_chunk_kernel<DP, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    const dim3 grid(batch.n_seqs * (MODE == DM_WHOLE ? 1 : runs.count), a.H, (a.V + DM_VB - 1) / DM_VB);
    if (grid.z > 65535) return (int)cudaErrorInvalidValue;
    sb_launch(decay_chunk_kernel<DP, MODE>, grid, DM_THREADS, smem, stream, a, batch, out, vec, runs);
    SB_LAUNCH_CHECK();
}

template <int DP>
static int launch_decay_chunk(SbDecay a, SbBatch batch, float* out, int vec, ChunkRuns runs, cudaStream_t stream) {
    if (runs.count <= 1) return launch_chunk_walk<DP, DM_WHOLE>(a, batch, out, vec, runs, stream);
    const int err = launch_chunk_walk<DP, DM_STATES>(a, batch, out, vec, runs, stream);
    if (err) return err;
    const dim3 grid(batch.n_seqs, a.H, (a.D * a.V + 255) / 256);
    if (grid.z > 65535) return (int)cudaErrorInvalidValue;
    sb_launch(decay_runs_kernel, grid, 256, 0, stream, a, batch, runs);
    return launch_chunk_walk<DP, DM_OUTPUTS>(a, batch, out, vec, runs, stream);
}

extern "C" {

// bfloat16 rows whose queries, keys and values are not to be activated any more; D up to 256; out [rows, H V] floats.
// n_runs > 1: runs of run_chunks chunks of 64 tokens (n_runs * run_chunks cover the longest sequence), with scratch for
// n_seqs * n_runs * H states of D * V floats, and as many numbers.
int sb_decay_chunk(SbDecay a, SbBatch batch, float* out, int n_runs, int run_chunks, float* run_states, float* run_decays,
                   cudaStream_t stream) {
    if (batch.n_seqs <= 0 || batch.n_rows <= 0) return 0;
    if (a.D < 1 || a.D > 256 || a.V < 1 || a.G < 1 || a.H % a.G || a.H > 65535 || a.act || (a.log2_decay == nullptr) == (a.dt == nullptr)
        || (n_runs > 1 && (run_chunks < 1 || run_states == nullptr || run_decays == nullptr)))
        return (int)cudaErrorInvalidValue;
    const ChunkRuns runs = {run_states, run_decays, n_runs, run_chunks};
    const int vec = a.ld % 8 == 0 && a.q_col % 8 == 0 && a.k_col % 8 == 0 && a.v_col % 8 == 0 && a.D % 8 == 0 && a.V % 8 == 0
                    && (reinterpret_cast<size_t>(a.p) & 15) == 0;
    if (a.D <= 32) return launch_decay_chunk<32>(a, batch, out, vec, runs, stream);
    if (a.D <= 64) return launch_decay_chunk<64>(a, batch, out, vec, runs, stream);
    if (a.D <= 128) return launch_decay_chunk<128>(a, batch, out, vec, runs, stream);
    return launch_decay_chunk<256>(a, batch, out, vec, runs, stream);
}

}  // extern "C"
