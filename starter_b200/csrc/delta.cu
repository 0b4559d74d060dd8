// The gated delta rule with a decay per key channel: what stands in front of its recurrence, and the recurrence token by
// token (decoding, short steps, and head sizes that delta_chunk.cu does not take).
//
//   conv_unit_heads  q, k, v = silu(sum_j w[:, j] u_(t - taps + 1 + j)) per channel (zeros before the sequence's start,
//                    inputs before the step from the sequence's record); q and k divided by sqrt(sum(x^2) + 1e-6) per head,
//                    q times q_scale.  32-bit results [q heads | k heads | v heads].
//   delta_step       S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      per head, over a sequence's rows
//                    g = exp(-exp(A_log) softplus(z + dt_bias)),  beta = sigmoid(b);  y = o / rms(o) * norm * sigmoid(gate)
//
// The read-out needs no second pass over the new state: with S' = g * S, r = S'^T k and p = S'^T q,
// o = p + (k . q) u, so one pass over S gives r and p, and one more writes the new state.
// Convolution, silu, unit norms, decays, state, sums, the output's norm and gate are 32-bit in every run.
#include "conv_record.cuh"
#include "delta.cuh"

// A warp per (R consecutive rows, head of q, k or v), so that the loads of R rows are in flight together.  p [rows, C] in the
// run's type, rows ld apart, C = 2 G D + H V channels; w [taps][C]; record of a sequence [taps - 1][C] floats.  inner [rows,
// inner_ld] 32-bit: its first n_inner columns are rounded into low [rows, low_ld], zeros beyond.  ADVANCE (a step of one row
// per sequence, R 1): the thread that owns a channel also moves its record on.  TAPS (0: any number): the number of taps
// when rows that have all their inputs within the step are to be taken R at a time, each input read once.
template <class T, int R, bool ADVANCE, int TAPS>
__global__ void conv_unit_heads_kernel(const T* __restrict__ p, long long ld, const float* __restrict__ w, int taps, float* state,
                                       long long state_slot, SbBatch batch, int G, int D, int H, int V, float q_scale,
                                       float* __restrict__ out, const float* __restrict__ inner, long long inner_ld, int n_inner,
                                       T* __restrict__ low, int low_ld) {
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const unsigned int wid = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const unsigned int units = 2 * G + H + 1;
    const int unit = (int)(wid % units);
    const int r0 = (int)(wid / units) * R, n_here = min(R, batch.n_rows - r0);
    if (n_here <= 0) return;
    if (unit == 2 * G + H) {   // the rows' inner vectors, side by side in the run's type
        for (int r = 0; r < n_here; ++r)
            for (int c = lane; c < low_ld; c += 32)
                low[(long long)(r0 + r) * low_ld + c] = from_f<T>(c < n_inner ? inner[(r0 + r) * inner_ld + c] : 0.f);
        return;
    }
    const int keep = taps - 1;
    const bool is_v = unit >= 2 * G;
    const int size = is_v ? V : D, c0 = is_v ? 2 * G * D + (unit - 2 * G) * V : unit * D;
    const int C = 2 * G * D + H * V;
    int ahead[R];              // rows of its sequence that the step holds before row r
    float* rec[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = r0 + min(r, n_here - 1), s = batch.row_seq[row];
        ahead[r] = row - batch.cu_q[s];
        rec[r] = keep > 0 ? state + (long long)batch.seq_slot[s] * state_slot : nullptr;
    }
    // all R rows are rows of one sequence with every input among the step's rows
    const bool inside = TAPS > 0 && n_here == R && ahead[0] >= TAPS - 1 && ahead[R - 1] == ahead[0] + R - 1;
    float kept[R][DS_KEEP], ss[R];   // a lane's values of a head of up to 32 * DS_KEEP columns; wider heads are read back from `out`
    auto values = [&](int c, float (&y)[R]) {
        const int ch = c0 + c;
#pragma unroll
        for (int r = 0; r < R; ++r) y[r] = 0.f;
        if (TAPS > 0 && inside) {
            constexpr int N = TAPS > 0 ? TAPS : 1;
            const T* src = p + (long long)(r0 - (N - 1)) * ld + ch;
            float wj[N], u[R + N - 1];
#pragma unroll
            for (int j = 0; j < N; ++j) wj[j] = w[(long long)j * C + ch];
#pragma unroll
            for (int m = 0; m < R + N - 1; ++m) {
                u[m] = to_f<T>(*src);
                src += ld;
            }
#pragma unroll
            for (int r = 0; r < R; ++r)
#pragma unroll
                for (int j = 0; j < N; ++j) y[r] = fmaf(wj[j], u[r + j], y[r]);
        } else
#pragma unroll 4
        for (int j = 0; j < taps; ++j) {
            const float wj = w[(long long)j * C + ch];
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const int row = r0 + min(r, n_here - 1), back = keep - j;
                const float u = ahead[r] >= back ? to_f<T>(p[(long long)(row - back) * ld + ch]) : rec[r][(long long)(ahead[r] + j) * C + ch];
                y[r] = fmaf(wj, u, y[r]);
                if (ADVANCE && j > 0) rec[r][(long long)(j - 1) * C + ch] = u;   // entry j - 1 was read in an earlier turn
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r) y[r] = __fdividef(y[r], 1.0f + expf(-y[r]));
    };
#pragma unroll
    for (int r = 0; r < R; ++r) ss[r] = 0.f;
#pragma unroll
    for (int i = 0; i < DS_KEEP; ++i) {
        float y[R];
        if (i * 32 + lane < size) {
            values(i * 32 + lane, y);
        } else {
#pragma unroll
            for (int r = 0; r < R; ++r) y[r] = 0.f;
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            kept[r][i] = y[r];
            ss[r] = fmaf(y[r], y[r], ss[r]);
        }
    }
    for (int c = DS_KEEP * 32 + lane; c < size; c += 32) {
        float y[R];
        values(c, y);
#pragma unroll
        for (int r = 0; r < R; ++r) {
            if (r < n_here) out[(long long)(r0 + r) * C + c0 + c] = y[r];
            ss[r] = fmaf(y[r], y[r], ss[r]);
        }
    }
    const float top = unit < G ? q_scale : 1.0f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= n_here) break;
        const float mul = is_v ? 1.0f : top / sqrtf(warp_sum(ss[r]) + 1e-6f);
        float* dst = out + (long long)(r0 + r) * C + c0;
#pragma unroll
        for (int i = 0; i < DS_KEEP; ++i) {
            const int c = i * 32 + lane;
            if (c < size) dst[c] = kept[r][i] * mul;
        }
        for (int c = DS_KEEP * 32 + lane; c < size; c += 32) dst[c] *= mul;
    }
}

// One block of eight warps per (sequence, head): warp w takes the key channels w, w + 8, ...; a lane takes VEC
// neighbouring value columns, 32 * VEC columns per turn.  The state stays in the sequence's record between the two passes
// of a token and between tokens (a thread meets the same entries every time); with EMAX > 0 (up to 8 * EMAX key channels
// and one turn of columns) a thread keeps its entries in registers over all rows.
template <class T, int VEC, int EMAX>
__global__ void __launch_bounds__(DS_WARPS * 32)
delta_step_kernel(SbDelta p, SbBatch batch, T* __restrict__ y) {
    extern __shared__ float sm[];
    const int D = p.D, V = p.V, G = p.G, H = p.H;
    float* qs = sm;              // [D] q, k and decay of the token
    float* ks = qs + D;
    float* gs = ks + D;
    float* us = gs + D;          // [V] what the token adds along k
    float* os = us + V;          // [V] its output
    float* red = os + V;         // [2][DS_WARPS][32 * VEC]
    __shared__ float red1[33];
    const int s = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    constexpr int TURN = 32 * VEC;
    const float neg_rate = -expf(p.a_log[head]);
    pdl_wait();
    const int row0 = batch.cu_q[s], row1 = batch.cu_q[s + 1];
    float* Sg = p.state + (long long)batch.seq_slot[s] * p.state_slot + (long long)head * D * V;
    const int kvh = head / (H / G), C = 2 * G * D + H * V;
    float S[EMAX > 0 ? EMAX : 1][VEC];
    if (EMAX > 0) {
#pragma unroll
        for (int e = 0; e < EMAX; ++e) {
            const int d = e * DS_WARPS + warp, j = lane * VEC;
#pragma unroll
            for (int i = 0; i < VEC; ++i) S[e][i] = 0.f;
            if (d < D && j < V) ds_load<VEC>(Sg + (long long)d * V + j, S[e]);
        }
    }
    for (int row = row0; row < row1; ++row) {
        const float* in = p.qkv + (long long)row * C;
        const float* zr = p.z + (long long)row * p.z_ld;
        __syncthreads();
        float kq = 0.f;
        for (int i = tid; i < D; i += DS_WARPS * 32) {
            const float q = in[kvh * D + i], k = in[(G + kvh) * D + i];
            qs[i] = q;
            ks[i] = k;
            gs[i] = delta_decay(zr[head * D + i] + p.dt_bias[head * D + i], neg_rate);
            kq = fmaf(k, q, kq);
        }
        kq = block_sum(kq, red1);   // also: the token's q, k and decay are in shared memory
        const float beta = 1.0f / (1.0f + expf(-p.inner[(long long)row * p.inner_ld + p.b_col + head]));
        const float* vr = in + 2 * G * D + head * V;
        for (int j0 = 0; j0 < V; j0 += TURN) {
            const int j = j0 + lane * VEC;
            float r[VEC], o[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) r[i] = o[i] = 0.f;
            if (EMAX > 0) {
#pragma unroll
                for (int e = 0; e < EMAX; ++e) {
                    const int d = e * DS_WARPS + warp;
                    if (d < D) {
                        const float g = gs[d], k = ks[d], q = qs[d];
#pragma unroll
                        for (int i = 0; i < VEC; ++i) {
                            S[e][i] *= g;
                            r[i] = fmaf(S[e][i], k, r[i]);
                            o[i] = fmaf(S[e][i], q, o[i]);
                        }
                    }
                }
            } else if (j < V) {
#pragma unroll 4
                for (int d = warp; d < D; d += DS_WARPS) {
                    float cell[VEC];
                    ds_load<VEC>(Sg + (long long)d * V + j, cell);
                    const float g = gs[d], gk = g * ks[d], gq = g * qs[d];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) {
                        r[i] = fmaf(cell[i], gk, r[i]);
                        o[i] = fmaf(cell[i], gq, o[i]);
                    }
                }
            }
            __syncthreads();
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                red[warp * TURN + lane * VEC + i] = r[i];
                red[(DS_WARPS + warp) * TURN + lane * VEC + i] = o[i];
            }
            __syncthreads();
            for (int c = tid; c < TURN; c += DS_WARPS * 32) {
                if (j0 + c < V) {
                    float rs = 0.f, ps = 0.f;
#pragma unroll
                    for (int w = 0; w < DS_WARPS; ++w) {
                        rs += red[w * TURN + c];
                        ps += red[(DS_WARPS + w) * TURN + c];
                    }
                    const float u = beta * (vr[j0 + c] - rs);
                    us[j0 + c] = u;
                    os[j0 + c] = fmaf(kq, u, ps);
                }
            }
        }
        __syncthreads();
        if (EMAX > 0) {
#pragma unroll
            for (int e = 0; e < EMAX; ++e) {
                const int d = e * DS_WARPS + warp;
                if (d < D && lane * VEC < V) {
                    const float k = ks[d];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) S[e][i] = fmaf(k, us[lane * VEC + i], S[e][i]);
                }
            }
        } else {
            for (int j = lane * VEC; j < V; j += TURN) {
#pragma unroll 4
                for (int d = warp; d < D; d += DS_WARPS) {
                    float cell[VEC];
                    ds_load<VEC>(Sg + (long long)d * V + j, cell);
                    const float g = gs[d], k = ks[d];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) cell[i] = fmaf(k, us[j + i], g * cell[i]);
                    ds_store<VEC>(Sg + (long long)d * V + j, cell);
                }
            }
        }
        float ss = 0.f;
        for (int c = tid; c < V; c += DS_WARPS * 32) ss = fmaf(os[c], os[c], ss);
        const float rstd = 1.0f / sqrtf(block_sum(ss, red1) / (float)V + p.eps);
        for (int c = tid; c < V; c += DS_WARPS * 32) {
            const float gate = 1.0f / (1.0f + expf(-zr[H * D + head * V + c]));
            y[((long long)row * H + head) * V + c] = from_f<T>(os[c] * rstd * p.norm[c] * gate);
        }
    }
    if (EMAX > 0) {
#pragma unroll
        for (int e = 0; e < EMAX; ++e) {
            const int d = e * DS_WARPS + warp, j = lane * VEC;
            if (d < D && j < V) ds_store<VEC>(Sg + (long long)d * V + j, S[e]);
        }
    }
}

template <class T>
static int launch_delta_step(SbDelta p, SbBatch batch, void* y, cudaStream_t stream) {
    const dim3 grid(batch.n_seqs, p.H);
    const bool vec = p.V % 4 == 0 && (reinterpret_cast<size_t>(p.state) & 15) == 0 && p.state_slot % 4 == 0;
    const int turn = vec ? 128 : 32;
    const size_t smem = (size_t)(3 * p.D + 2 * p.V + 2 * DS_WARPS * turn) * sizeof(float);
#define SB_DS(VEC, EMAX)                                                                                                       \
    do {                                                                                                                       \
        if (smem > 48 * 1024) {                                                                                                \
            const cudaError_t err = cudaFuncSetAttribute(delta_step_kernel<T, VEC, EMAX>,                                      \
                                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);              \
            if (err != cudaSuccess) return (int)err;                                                                           \
        }                                                                                                                      \
        sb_launch(delta_step_kernel<T, VEC, EMAX>, grid, DS_WARPS * 32, smem, stream, p, batch, (T*)y);                        \
    } while (0)
    if (p.V <= turn && p.D <= 8 * DS_WARPS) {
        if (vec) SB_DS(4, 8);
        else SB_DS(1, 8);
    } else if (p.V <= turn && p.D <= 16 * DS_WARPS) {
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

// p [rows, 2 G D + H V], rows ld apart; w [taps, channels]; state [slots][taps - 1][channels] floats; out [rows, channels]
// floats.  one_row: every sequence of the step brings one row (the record is moved on in the same kernel).
int sb_conv_unit_heads(int dtype, const void* p, long long ld, const float* w, int taps, float* state, long long state_slot, SbBatch batch,
                       int G, int D, int H, int V, float q_scale, float* out, const float* inner, long long inner_ld, int n_inner,
                       void* low, int low_ld, int one_row, cudaStream_t stream) {
    if (batch.n_rows <= 0) return 0;
    if (taps < 1 || (taps > 1 && state == nullptr) || D < 1 || V < 1 || n_inner > low_ld) return (int)cudaErrorInvalidValue;
    typedef __nv_bfloat16 bf;
    const bool advance = one_row && taps > 1 && batch.n_rows < 512;
    const int R = batch.n_rows >= 512 ? 4 : 1;   // few rows: a warp each, so that they spread over the SMs
    const long long warps = (long long)((batch.n_rows + R - 1) / R) * (2 * G + H + 1);
    if (warps > 0x7fffffffll) return (int)cudaErrorInvalidValue;
    const int per_block = batch.n_rows < 64 ? 2 : 8;
    const unsigned int blocks = (unsigned int)((warps + per_block - 1) / per_block);
#define SB_CU(T, R, A, N)                                                                                                      \
    sb_launch(conv_unit_heads_kernel<T, R, A, N>, blocks, per_block * 32, 0, stream, (const T*)p, ld, w, taps, state, state_slot, batch, G, D, \
              H, V, q_scale, out, inner, inner_ld, n_inner, (T*)low, low_ld)
#define SB_CUT(T)                                      \
    do {                                               \
        if (advance && R == 1) SB_CU(T, 1, true, 0);   \
        else if (R == 1) SB_CU(T, 1, false, 0);        \
        else if (taps == 4) SB_CU(T, 4, false, 4);     \
        else if (taps == 3) SB_CU(T, 4, false, 3);     \
        else if (taps == 2) SB_CU(T, 4, false, 2);     \
        else SB_CU(T, 4, false, 0);                    \
    } while (0)
    if (dtype == SB_F32) SB_CUT(float);
    else SB_CUT(bf);
#undef SB_CUT
#undef SB_CU
    if (taps > 1 && !advance) {
        launch_conv_record(dtype, p, ld, taps, state, state_slot, batch, 2 * G * D + H * V, stream);
    }
    SB_LAUNCH_CHECK();
}

// y [rows, H V] in `dtype`; everything else 32-bit (see SbDelta).
int sb_delta_step(int dtype, SbDelta p, SbBatch batch, void* y, cudaStream_t stream) {
    if (batch.n_seqs <= 0 || batch.n_rows <= 0) return 0;
    if (p.D < 1 || p.V < 1 || p.D > 4096 || p.V > 4096 || p.G < 1 || p.H % p.G || p.H > 65535) return (int)cudaErrorInvalidValue;
    if (dtype == SB_F32) return launch_delta_step<float>(p, batch, y, stream);
    return launch_delta_step<__nv_bfloat16>(p, batch, y, stream);
}

}  // extern "C"
