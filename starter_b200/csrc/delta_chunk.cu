// The gated delta rule for prompts: sixteen tokens at a time, everything in 32-bit on the CUDA cores.
//
// Let c_i = g_1 ... g_i (per key channel) inside a chunk that starts from the state S0, and
//
//   A[i][j] = sum_d k_i k_j (g_{j+1} ... g_i),  j < i          P[i][j] = sum_d q_i k_j (g_{j+1} ... g_i),  j <= i
//
// The rows u_i that the chunk adds along its keys solve (I + diag(beta) A) U = diag(beta) (V - (k c) S0), so with the
// unit lower triangular inverse T and M = T diag(beta):
//
//   U = M V - W S0,   W = M (k c)         O = (q c) S0 + P U         S1 = c_16 S0 + sum_j (k_j g_{j+1} ... g_16) u_j^T
//
// W, q c, P, M V, the keys carried to the chunk's end and c_16 need no state: delta_chunk_prepare works them out for all
// chunks and heads at once.  delta_chunk_scan then walks a sequence's chunks in order, a block per (sequence, head, group
// of value columns), with three small products per chunk instead of sixteen dependent tokens; delta_chunk_finish takes
// the head's norm and the gate.  The decays inside a chunk are multiplied up (never divided out and never taken as
// differences of summed logarithms), so a channel that forgets everything loses no precision afterwards.  A chunk cut
// short by the step's end stands as one with k = q = 0, beta = 0, g = 1 for the missing tokens.
#include "delta.cuh"
#include "mma_utils.cuh"

#define DC 16             // tokens of a chunk
#define DC_THREADS 128
#define DC_STAGES 4       // chunks whose operands are in shared memory or on their way

// One (chunk, head) of the workspace, in floats: [DP][2 DC] columns W | q c, then [DC][DP] keys carried to the end, then
// [DP] c_16, [DC][DC] P, [DC][VP] M V.  DP: the key channels rounded up to 32, 64 or 128; VP: the value columns rounded up
// to a multiple of 4.
__host__ __device__ __forceinline__ int dc_key_pad(int n) { return n <= 32 ? 32 : (n <= 64 ? 64 : 128); }
__host__ __device__ __forceinline__ int dc_value_pad(int n) { return (n + 3) & ~3; }
__host__ __device__ constexpr int dc_shared_part(int DP) { return (3 * DC + 1) * DP + DC * DC; }
__host__ __device__ __forceinline__ long long dc_cell(int DP, int VP) { return dc_shared_part(DP) + (long long)DC * VP; }
// First chunk of sequence s in the workspace; rows / DC + n_seqs places hold every step's chunks.
__device__ __forceinline__ int dc_base(const SbBatch& b, int s) { return b.cu_q[s] / DC + s; }

// row i of M times the sixteen values x (M is lower triangular)
__device__ __forceinline__ float dc_row_times(const float* m, int i, const float (&x)[DC]) {
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < DC; j += 4)
        if (j <= i) {
            const float4 r = *reinterpret_cast<const float4*>(m + i * DC + j);
            sum = fmaf(r.x, x[j], sum);
            sum = fmaf(r.y, x[j + 1], sum);
            sum = fmaf(r.z, x[j + 2], sum);
            sum = fmaf(r.w, x[j + 3], sum);
        }
    return sum;
}

template <int DP>
__global__ void __launch_bounds__(DC_THREADS, DP == 128 ? 4 : 6)
delta_chunk_prepare_kernel(SbDelta p, SbBatch batch, float* __restrict__ ws, int VP) {
    constexpr int LD = DP + 4, E = DP / 16;
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;               // [DC][LD]
    float* ks = qs + DC * LD;
    float* gs = ks + DC * LD;
    __shared__ float As[DC][DC + 1], bs[DC];
    __shared__ __align__(16) float Ms[DC * DC], Ps[DC * DC];
    __shared__ int s_seq;
    const int D = p.D, V = p.V, G = p.G, H = p.H;
    const int head = blockIdx.y, tid = threadIdx.x;
    const float neg_rate = -expf(p.a_log[head]);
    pdl_wait();
    if (tid == 0) {   // the last sequence whose first chunk is at or before this one
        int lo = 0, hi = batch.n_seqs - 1;
        while (lo < hi) {
            const int mid = (lo + hi + 1) / 2;
            if (dc_base(batch, mid) <= (int)blockIdx.x) lo = mid;
            else hi = mid - 1;
        }
        s_seq = lo;
    }
    __syncthreads();
    const int s = s_seq;
    const int row0 = batch.cu_q[s] + ((int)blockIdx.x - dc_base(batch, s)) * DC, nt = min(DC, batch.cu_q[s + 1] - row0);
    if (nt <= 0) return;
    const int kvh = head / (H / G), C = 2 * G * D + H * V;
    for (int e = tid; e < DC * DP; e += DC_THREADS) {
        const int t = e / DP, d = e % DP;
        float q = 0.f, k = 0.f, g = 1.f;
        if (t < nt && d < D) {
            const float* in = p.qkv + (long long)(row0 + t) * C;
            q = in[kvh * D + d];
            k = in[(G + kvh) * D + d];
            g = delta_decay(p.z[(long long)(row0 + t) * p.z_ld + head * D + d] + p.dt_bias[head * D + d], neg_rate);
        }
        qs[t * LD + d] = q;
        ks[t * LD + d] = k;
        gs[t * LD + d] = g;
    }
    if (tid < DC) bs[tid] = tid < nt ? 1.0f / (1.0f + expf(-p.inner[(long long)(row0 + tid) * p.inner_ld + p.b_col + head])) : 0.f;
    for (int e = tid; e < DC * DC; e += DC_THREADS) Ps[e] = 0.f;
    __syncthreads();
    {   // A and P: sixteen lanes per key j (and 15 - j after it), each with every 16th channel
        const int group = tid >> 4, l = tid & 15;
        const unsigned int half_mask = 0xffffu << (tid & 16);   // the two groups of a warp have loops of different lengths
#pragma unroll 1
        for (int half = 0; half < 2; ++half) {
            const int j = half == 0 ? group : DC - 1 - group;
            float kd[E];   // k_j times the decays since token j
#pragma unroll
            for (int e = 0; e < E; ++e) kd[e] = ks[j * LD + l + 16 * e];
#pragma unroll 1
            for (int i = j; i < DC; ++i) {
                float a = 0.f, o = 0.f;
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const int at = i * LD + l + 16 * e;
                    if (i > j) kd[e] *= gs[at];
                    a = fmaf(ks[at], kd[e], a);
                    o = fmaf(qs[at], kd[e], o);
                }
#pragma unroll
                for (int off = 8; off > 0; off >>= 1) {
                    a += __shfl_xor_sync(half_mask, a, off);
                    o += __shfl_xor_sync(half_mask, o, off);
                }
                if (l == 0) {
                    As[i][j] = a;
                    Ps[i * DC + j] = o;
                }
            }
        }
    }
    __syncthreads();
    if (tid < DC) {   // column tid of T by forward substitution, then M = T diag(beta)
        float t[DC];
#pragma unroll
        for (int i = 0; i < DC; ++i) {
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) sum = fmaf(As[i][j], t[j], sum);
            t[i] = (i == tid ? 1.0f : 0.f) - bs[i] * sum;
            Ms[i * DC + tid] = t[i] * bs[tid];
        }
    }
    __syncthreads();
    float* cell = ws + ((long long)blockIdx.x * H + head) * dc_cell(DP, VP);
    float* wq = cell;
    float* kh = wq + 2 * DC * DP;
    float* cg = kh + DC * DP;
    float* pg = cg + DP;
    float* mv = pg + DC * DC;
    for (int e = tid; e < DC * DC; e += DC_THREADS) pg[e] = Ps[e];
#pragma unroll 1
    for (int item = tid; item < DP + VP; item += DC_THREADS) {   // a key channel, or a value column
        float x[DC];
        if (item < DP) {
            const int d = item;
            float4* dst = reinterpret_cast<float4*>(wq + (long long)d * 2 * DC);
            float c = 1.0f;
#pragma unroll
            for (int j = DC - 1; j >= 0; --j) {
                kh[j * DP + d] = ks[j * LD + d] * c;
                c *= gs[j * LD + d];
            }
            cg[d] = c;
            c = 1.0f;
#pragma unroll
            for (int i = 0; i < DC; ++i) {
                c *= gs[i * LD + d];
                x[i] = qs[i * LD + d] * c;
            }
#pragma unroll
            for (int i = 0; i < DC; i += 4) dst[(DC + i) / 4] = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
            c = 1.0f;
#pragma unroll
            for (int i = 0; i < DC; ++i) {
                c *= gs[i * LD + d];
                x[i] = ks[i * LD + d] * c;
            }
#pragma unroll
            for (int i = 0; i < DC; i += 4)
                dst[i / 4] = make_float4(dc_row_times(Ms, i, x), dc_row_times(Ms, i + 1, x), dc_row_times(Ms, i + 2, x), dc_row_times(Ms, i + 3, x));
        } else {
            const int col = item - DP;
#pragma unroll
            for (int t = 0; t < DC; ++t)
                x[t] = t < nt && col < V ? p.qkv[(long long)(row0 + t) * C + 2 * G * D + head * V + col] : 0.f;
#pragma unroll
            for (int i = 0; i < DC; ++i) mv[(long long)i * VP + col] = dc_row_times(Ms, i, x);
        }
    }
}

// CT floats from or to 16- or 8-byte aligned shared memory.
template <int CT> __device__ __forceinline__ void dc_load(const float* p, float (&v)[CT]) {
#pragma unroll
    for (int c = 0; c < CT; c += 2) {
        const float2 f = *reinterpret_cast<const float2*>(p + c);
        v[c] = f.x;
        v[c + 1] = f.y;
    }
}
template <> __device__ __forceinline__ void dc_load<4>(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x;
    v[1] = f.y;
    v[2] = f.z;
    v[3] = f.w;
}
template <int CT> __device__ __forceinline__ void dc_store(float* p, const float (&v)[CT]) {
#pragma unroll
    for (int c = 0; c < CT; c += 2) *reinterpret_cast<float2*>(p + c) = make_float2(v[c], v[c + 1]);
}
template <> __device__ __forceinline__ void dc_store<4>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}

// A block of four warps per (sequence, head, 4 CT value columns); a warp owns CT columns of the state, of U and of O
// throughout, so that inside a chunk only the shared operands (DC_STAGES - 1 chunks ahead) need the block's barrier.
// Product with the state: lane = (row tile of 4 among the 32 rows W | q c) + 8 * (share of the key channels); the four
// shares meet by shuffles, each lane keeping one row.  What the chunk's later steps read of the operands is fetched into
// registers first: the chain from one chunk's state to the next is what the time here consists of.
template <int CT, int DP>
__global__ void __launch_bounds__(DC_THREADS)
delta_chunk_scan_kernel(SbDelta p, SbBatch batch, const float* __restrict__ ws, float* __restrict__ o_raw, int VP) {
    extern __shared__ __align__(16) float smf[];
    constexpr int VB = 4 * CT, NE = DP / 32, PART = dc_shared_part(DP), STAGE = PART + DC * VB;
    const int D = p.D, V = p.V, H = p.H;
    float* buf = smf;                           // the stages: a cell's shared part, then [DC][VB] of M V
    float* Ssm = buf + DC_STAGES * STAGE;       // [4 warps][DP][CT]
    float* Usm = Ssm + 4 * DP * CT;             // [4 warps][DC][CT]
    const int s = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int j0 = blockIdx.z * VB, col0 = j0 + warp * CT;
    pdl_wait();
    const int row0 = batch.cu_q[s], n = batch.cu_q[s + 1] - row0, chunks = (n + DC - 1) / DC;
    if (n <= 0) return;
    float* Sg = p.state + (long long)batch.seq_slot[s] * p.state_slot + (long long)head * D * V;
    float* Sw = Ssm + warp * DP * CT;
    float* Uw = Usm + warp * DC * CT;
    float S[NE][CT];
#pragma unroll
    for (int e = 0; e < NE; ++e) {
        const int d = e * 32 + lane;
#pragma unroll
        for (int c = 0; c < CT; ++c) S[e][c] = d < D && col0 + c < V ? Sg[(long long)d * V + col0 + c] : 0.f;
        dc_store<CT>(Sw + d * CT, S[e]);
    }
    const long long cell = dc_cell(DP, VP), base = dc_base(batch, s);
    auto fetch = [&](int chunk) {               // always one group of copies, so that the waits count the same
        if (chunk < chunks) {
            const float* src = ws + ((base + chunk) * H + head) * cell;
            float* dst = buf + (chunk % DC_STAGES) * STAGE;
            for (int e = tid; e < PART / 4; e += DC_THREADS) cp_async_16(dst + e * 4, src + e * 4);
            for (int e = tid; e < DC * VB / 4; e += DC_THREADS) {
                const int t = e / (VB / 4), c = (e % (VB / 4)) * 4;
                if (j0 + c < VP) cp_async_16(dst + PART + t * VB + c, src + PART + (long long)t * VP + j0 + c);
                else *reinterpret_cast<float4*>(dst + PART + t * VB + c) = make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int c = 0; c < DC_STAGES - 1; ++c) fetch(c);
    const int rt = lane & 7, share = lane >> 3;
    const int my = rt * 4 + share;              // the row among W | q c that this lane keeps
    const bool is_u = my < DC;
    for (int ch = 0; ch < chunks; ++ch) {
        cp_async_wait<DC_STAGES - 2>();
        __syncthreads();                        // the stage is there, and nobody reads the one before it any more
        fetch(ch + DC_STAGES - 1);
        const float* wq = buf + (ch % DC_STAGES) * STAGE;
        const float* kh = wq + 2 * DC * DP;
        const float* cg = kh + DC * DP;
        const float* pg = cg + DP;
        float acc[4][CT];
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int c = 0; c < CT; ++c) acc[r][c] = 0.f;
#pragma unroll
        for (int i = 0; i < DP / 4; ++i) {
            const int d = i * 4 + share;
            const float4 a = *reinterpret_cast<const float4*>(wq + d * 2 * DC + rt * 4);
            float x[CT];
            dc_load<CT>(Sw + d * CT, x);
#pragma unroll
            for (int c = 0; c < CT; ++c) {
                acc[0][c] = fmaf(a.x, x[c], acc[0][c]);
                acc[1][c] = fmaf(a.y, x[c], acc[1][c]);
                acc[2][c] = fmaf(a.z, x[c], acc[2][c]);
                acc[3][c] = fmaf(a.w, x[c], acc[3][c]);
            }
        }
        float kr[NE][DC], pr[DC], first[CT];    // this lane's keys, its row of P, its row of M V
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const float keep = cg[e * 32 + lane];
#pragma unroll
            for (int t = 0; t < DC; ++t) kr[e][t] = kh[t * DP + e * 32 + lane];
#pragma unroll
            for (int c = 0; c < CT; ++c) S[e][c] *= keep;
        }
#pragma unroll
        for (int t = 0; t < DC; t += 4) {
            const float4 r = *reinterpret_cast<const float4*>(pg + (my & (DC - 1)) * DC + t);
            pr[t] = r.x;
            pr[t + 1] = r.y;
            pr[t + 2] = r.z;
            pr[t + 3] = r.w;
        }
        dc_load<CT>(buf + (ch % DC_STAGES) * STAGE + PART + (my & (DC - 1)) * VB + warp * CT, first);
        float mine[CT];
        {
            const bool up = share & 2, odd = share & 1;
#pragma unroll
            for (int c = 0; c < CT; ++c) {
                const float send0 = up ? acc[0][c] : acc[2][c], send1 = up ? acc[1][c] : acc[3][c];
                const float keep0 = (up ? acc[2][c] : acc[0][c]) + __shfl_xor_sync(0xffffffffu, send0, 16);
                const float keep1 = (up ? acc[3][c] : acc[1][c]) + __shfl_xor_sync(0xffffffffu, send1, 16);
                mine[c] = (odd ? keep1 : keep0) + __shfl_xor_sync(0xffffffffu, odd ? keep0 : keep1, 8);
                first[c] -= mine[c];
            }
        }
        if (is_u) dc_store<CT>(Uw + my * CT, first);
        __syncwarp();
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            float u[CT];
            dc_load<CT>(Uw + t * CT, u);
#pragma unroll
            for (int c = 0; c < CT; ++c) {
#pragma unroll
                for (int e = 0; e < NE; ++e) S[e][c] = fmaf(kr[e][t], u[c], S[e][c]);
                mine[c] = fmaf(pr[t], u[c], mine[c]);     // P is zero above its diagonal
            }
        }
#pragma unroll
        for (int e = 0; e < NE; ++e) dc_store<CT>(Sw + (e * 32 + lane) * CT, S[e]);
        const int row = ch * DC + my - DC;
        if (!is_u && row < n) {
            float* o = o_raw + ((long long)(row0 + row) * H + head) * V + col0;
#pragma unroll
            for (int c = 0; c < CT; ++c)
                if (col0 + c < V) o[c] = mine[c];
        }
        __syncwarp();                           // the next chunk reads the columns that the other lanes wrote
    }
#pragma unroll
    for (int e = 0; e < NE; ++e) {
        const int d = e * 32 + lane;
#pragma unroll
        for (int c = 0; c < CT; ++c)
            if (d < D && col0 + c < V) Sg[(long long)d * V + col0 + c] = S[e][c];
    }
}

// One warp per (row, head): the head's unit norm over its V outputs, the norm weight and the gate.
template <class T>
__global__ void delta_chunk_finish_kernel(const float* __restrict__ o_raw, SbDelta p, int rows, T* __restrict__ y) {
    pdl_wait();
    const long long wid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31, H = p.H, V = p.V;
    if (wid >= (long long)rows * H) return;
    const long long row = wid / H;
    const int head = (int)(wid - row * H);
    const float* o = o_raw + wid * V;
    const float* gate = p.z + row * p.z_ld + (long long)H * p.D + (long long)head * V;
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) ss = fmaf(o[c], o[c], ss);
    const float rstd = 1.0f / sqrtf(warp_sum(ss) / (float)V + p.eps);
    for (int c = lane; c < V; c += 32) y[wid * V + c] = from_f<T>(o[c] * rstd * p.norm[c] * (1.0f / (1.0f + expf(-gate[c]))));
}

template <int CT, int DP>
static int launch_chunk_scan(SbDelta p, SbBatch batch, const float* ws, float* o_raw, int VP, cudaStream_t stream) {
    const size_t smem = (size_t)(DC_STAGES * (dc_shared_part(DP) + DC * 4 * CT) + 4 * DP * CT + 4 * DC * CT) * sizeof(float);
    const cudaError_t err = cudaFuncSetAttribute(delta_chunk_scan_kernel<CT, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    const dim3 grid(batch.n_seqs, p.H, (p.V + 4 * CT - 1) / (4 * CT));
    if (grid.z > 65535) return (int)cudaErrorInvalidValue;
    sb_launch(delta_chunk_scan_kernel<CT, DP>, grid, DC_THREADS, smem, stream, p, batch, ws, o_raw, VP);
    SB_LAUNCH_CHECK();
}

template <int DP>
static int launch_chunks(SbDelta p, SbBatch batch, float* ws, float* o_raw, int columns, cudaStream_t stream) {
    const int VP = dc_value_pad(p.V);
    const size_t smem = (size_t)(3 * DC * (DP + 4)) * sizeof(float);
    sb_launch(delta_chunk_prepare_kernel<DP>, dim3(batch.n_rows / DC + batch.n_seqs, p.H), DC_THREADS, smem, stream, p, batch, ws, VP);
    if (columns == 8) return launch_chunk_scan<2, DP>(p, batch, ws, o_raw, VP, stream);
    return launch_chunk_scan<4, DP>(p, batch, ws, o_raw, VP, stream);
}

extern "C" {

// Floats of workspace for a step of this shape, or -1 for heads the kernels do not take (more than 128 key channels).
long long sb_delta_chunk_floats(int rows, int n_seqs, int H, int D, int V) {
    if (D < 1 || D > 128 || V < 1 || V > 4096) return -1;
    return (long long)(rows / DC + n_seqs) * H * dc_cell(dc_key_pad(D), dc_value_pad(V));
}

// ws: sb_delta_chunk_floats(...) floats; o_raw [rows, H V] floats; columns: value columns per block, 8 or 16.
int sb_delta_chunk(int dtype, SbDelta p, SbBatch batch, float* ws, float* o_raw, void* y, int columns, cudaStream_t stream) {
    if (batch.n_seqs <= 0 || batch.n_rows <= 0) return 0;
    if (p.D < 1 || p.D > 128 || p.V < 1 || p.V > 4096 || p.G < 1 || p.H % p.G || p.H > 65535 || (columns != 8 && columns != 16))
        return (int)cudaErrorInvalidValue;
    const int DP = dc_key_pad(p.D);
    const int err = DP == 32 ? launch_chunks<32>(p, batch, ws, o_raw, columns, stream)
                  : DP == 64 ? launch_chunks<64>(p, batch, ws, o_raw, columns, stream)
                             : launch_chunks<128>(p, batch, ws, o_raw, columns, stream);
    if (err) return err;
    const long long warps = (long long)batch.n_rows * p.H;
    const unsigned int blocks = (unsigned int)((warps * 32 + 255) / 256);
    if (dtype == SB_F32) sb_launch(delta_chunk_finish_kernel<float>, blocks, 256, 0, stream, (const float*)o_raw, p, batch.n_rows, (float*)y);
    else
        sb_launch(delta_chunk_finish_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const float*)o_raw, p, batch.n_rows, (__nv_bfloat16*)y);
    SB_LAUNCH_CHECK();
}

}  // extern "C"
