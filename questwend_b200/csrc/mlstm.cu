// Matrix memory with exponential gates (the mLSTM of xLSTM).  Per head and token, with logarithms i and f of an input and a
// forget gate, the memory S (K x P), its normaliser n (K) and a running maximum m (0 before the first token) become
//     m' = max(m + f, i),   keep = e^(m + f - m'),   write = e^(i - m')
//     S' = keep S + write k v^T,   n' = keep n + write k
// and are read out as  S'^T q / (max(|n' . q|, e^-m') + tiny).  Both logarithms come from raw gates z through a cap,
// i = cap tanh((z_i + b_i) / cap) and f = log sigmoid(cap tanh((z_f + b_f) / cap)).  n is the memory of a value that
// is always 1, so it is kept as one more column: a head's state is [P + 1][K] floats, column by column, the last one n.
// The running maximum is kept once per column ([P + 1] floats, all equal), so that a step of one token needs no order
// between the warps that share a head.  Everything is 32-bit; running maxima and sums of logarithms inside a chunk are
// formed in 64-bit.
//
//   mlstm_gates     a step's decays (their logarithms), write strengths and running maxima, by a scan over each sequence
//   mlstm_scan      the recurrence, a warp per few columns; a step of one token per sequence makes its gates in the kernel
//   mlstm_chunked   long prompts in chunks of 64 tokens: every chunk's own sum of outer products, the carries, the outputs
// Each leaves S^T q and the denominator; the norm that follows divides.
#include "common.cuh"

#define QWB_MLSTM_CHUNK 64
#define QWB_MLSTM_WARPS 4
#define QWB_MLSTM_MAX_PER 16        // rows of a column a lane keeps: K up to 512

struct MlstmSizes { int H, K, P; };
// columns of the projection's rows: q [H * K] | k [H * K] | v [H * P] from column 0; the raw gates at i_col and f_col
struct MlstmRows { const float* x; int ld, i_col, f_col; };
struct MlstmGates { const float *i_bias, *f_bias; float cap; };

__device__ __forceinline__ float mlstm_log_sigmoid(float z) { return z > 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z)); }
__device__ __forceinline__ void mlstm_log_gates(MlstmRows rows, MlstmGates g, int t, int h, float& i, float& f) {
    const float* row = rows.x + (size_t)t * rows.ld;
    i = g.cap * tanhf((row[rows.i_col + h] + g.i_bias[h]) / g.cap);
    f = mlstm_log_sigmoid(g.cap * tanhf((row[rows.f_col + h] + g.f_bias[h]) / g.cap));
}

// ---------------------------------------------------------------------------------
// Gates of a step that brings several tokens.  grid (H, B), 256 threads.  A token is the map m -> max(m + f, i); maps compose
// into maps of the same form, so the running maxima are a scan over the tokens (in 64-bit, 256 at a time).  With the rounded
// maxima, log_decay = m + f - m' telescopes exactly.  Outputs [T, H].
// ---------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
mlstm_gates_kernel(MlstmRows rows, MlstmGates gates, const float* __restrict__ m_state, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ slots, float* __restrict__ log_decay, float* __restrict__ write, float* __restrict__ m_run, int H, int P) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ double tot_f[8], tot_x[8];
    __shared__ float last_m[8];
    const int h = blockIdx.x, b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
    double carry = (double)m_state[((size_t)slots[b] * H + h) * (P + 1)];
    for (int base = t0; base < t1; base += 256) {
        const int t = base + threadIdx.x;
        float i = 0.f, f = 0.f;
        double F = 0.0, X = -INFINITY;                              // beyond the end: the map that changes nothing
        if (t < t1) {
            mlstm_log_gates(rows, gates, t, h, i, f);
            F = (double)f; X = (double)i;
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {                          // earlier map first: (F1, X1), then (F, X)
            const double F1 = __shfl_up_sync(0xffffffffu, F, o), X1 = __shfl_up_sync(0xffffffffu, X, o);
            if (lane >= o) { X = fmax(X1 + F, X); F += F1; }
        }
        if (lane == 31) { tot_f[warp] = F; tot_x[warp] = X; }
        __syncthreads();
        double start = carry, end = carry;                          // m before this warp's tokens, and after all 256
        for (int w = 0; w < 8; ++w) {
            if (w == warp) start = end;
            end = fmax(end + tot_f[w], tot_x[w]);
        }
        const float m = (float)fmax(start + F, X);
        if (lane == 31) last_m[warp] = m;
        __syncthreads();
        float before = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) before = warp > 0 ? last_m[warp - 1] : (float)carry;
        if (t < t1) {
            const size_t at = (size_t)t * H + h;
            log_decay[at] = (float)((double)f + (double)before - (double)m);
            write[at] = expf(i - m);
            m_run[at] = m;
        }
        carry = (double)last_m[7];                                  // the rounded maximum goes on
        __syncthreads();
    }
}

// ---------------------------------------------------------------------------------
// The recurrence.  Warp = CW columns of one head of one sequence; lane l keeps rows l * PER .. l * PER + PER - 1 of each.
// STEP: one token per sequence, the gates made here from the column's running maximum.  Otherwise they come from
// mlstm_gates, and TB tokens' vectors are asked for together, a round ahead of their use.
// raw [T, H * P] = S^T q;  divisor [T, H] = max(|n . q|, e^-m) + tiny.
// ---------------------------------------------------------------------------------
template <int PER, bool VEC>
__device__ __forceinline__ void mlstm_rows(const float* __restrict__ base, int n0, int limit, float* out) {
    if (VEC) {
#pragma unroll
        for (int k = 0; k < PER; k += 4) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (n0 + k < limit) v = *reinterpret_cast<const float4*>(base + n0 + k);
            out[k] = v.x; out[k + 1] = v.y; out[k + 2] = v.z; out[k + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int k = 0; k < PER; ++k) out[k] = n0 + k < limit ? base[n0 + k] : 0.f;
    }
}

template <int PER, bool VEC, int TB, int CW, bool STEP>
__global__ void __launch_bounds__(32 * QWB_MLSTM_WARPS)
mlstm_scan_kernel(MlstmRows rows, MlstmGates gates, const float* __restrict__ log_decay, const float* __restrict__ write, const float* __restrict__ m_run,
                  float* __restrict__ state, float* __restrict__ m_state, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
                  float* __restrict__ raw, float* __restrict__ divisor, MlstmSizes z, float q_scale, float tiny, int write_state) {
    pdl_wait();
    pdl_launch_dependents();
    const int H = z.H, K = z.K, P = z.P, lane = threadIdx.x & 31;
    const int p0 = (blockIdx.x * QWB_MLSTM_WARPS + (threadIdx.x >> 5)) * CW, h = blockIdx.y, b = blockIdx.z;
    if (p0 > P) return;
    const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
    if (t0 >= t1) return;
    const int n0 = lane * PER;
    const size_t head = (size_t)slots[b] * H + h;
    float* S = state + (head * (P + 1) + p0) * K;
    float* M = m_state + head * (P + 1) + p0;
    float s[CW][PER];
#pragma unroll
    for (int c = 0; c < CW; ++c) mlstm_rows<PER, VEC>(S + (size_t)c * K, n0, p0 + c <= P ? K : 0, s[c]);
    float m_last = 0.f;
    float kn[TB][PER], qn[TB][PER], v_n[TB][CW], d_n[TB], w_n[TB], m_n[TB];
    auto load_round = [&](int tc) {
#pragma unroll
        for (int j = 0; j < TB; ++j) {
            const int t = min(tc + j, t1 - 1);                      // past the end: the last token again, not used
            const float* row = rows.x + (size_t)t * rows.ld;
            mlstm_rows<PER, VEC>(row + h * K, n0, K, qn[j]);
            mlstm_rows<PER, VEC>(row + (H + h) * K, n0, K, kn[j]);
#pragma unroll
            for (int c = 0; c < CW; ++c) v_n[j][c] = p0 + c < P ? row[2 * H * K + h * P + p0 + c] : 1.f;
            if (STEP) {
                float i, f;
                const float before = M[0];
                mlstm_log_gates(rows, gates, t, h, i, f);
                m_n[j] = (float)fmax((double)f + (double)before, (double)i);
                d_n[j] = expf((float)((double)f + (double)before - (double)m_n[j]));
                w_n[j] = expf(i - m_n[j]);
            } else {
                const size_t at = (size_t)t * H + h;
                d_n[j] = expf(log_decay[at]);
                w_n[j] = write[at];
                m_n[j] = m_run[at];
            }
        }
    };
    load_round(t0);
    for (int tc = t0; tc < t1; tc += TB) {
        float kk[TB][PER], qq[TB][PER], v[TB][CW], d[TB], w[TB], m[TB];
#pragma unroll
        for (int j = 0; j < TB; ++j) {
            d[j] = d_n[j]; w[j] = w_n[j]; m[j] = m_n[j];
#pragma unroll
            for (int k = 0; k < PER; ++k) { kk[j][k] = kn[j][k]; qq[j][k] = qn[j][k] * q_scale; }
#pragma unroll
            for (int c = 0; c < CW; ++c) v[j][c] = v_n[j][c];
        }
        if (!STEP && tc + TB < t1) load_round(tc + TB);
        float acc[TB][CW];
#pragma unroll
        for (int j = 0; j < TB; ++j) {
            if (tc + j < t1) m_last = m[j];
#pragma unroll
            for (int c = 0; c < CW; ++c) {
                acc[j][c] = 0.f;
                if (tc + j < t1) {
                    const float wv = w[j] * v[j][c];
#pragma unroll
                    for (int k = 0; k < PER; ++k) {
                        s[c][k] = d[j] * s[c][k] + wv * kk[j][k];
                        acc[j][c] += s[c][k] * qq[j][k];
                    }
                }
            }
        }
#pragma unroll
        for (int j = 0; j < TB; ++j)
#pragma unroll
            for (int c = 0; c < CW; ++c) acc[j][c] = warp_sum(acc[j][c]);
#pragma unroll
        for (int j = 0; j < TB; ++j)
#pragma unroll
            for (int c = 0; c < CW; ++c)
                if (lane == 0 && tc + j < t1) {
                    const size_t at = (size_t)(tc + j) * H + h;
                    if (p0 + c < P) raw[at * P + p0 + c] = acc[j][c];
                    else if (p0 + c == P) divisor[at] = fmaxf(fabsf(acc[j][c]), expf(-m[j])) + tiny;
                }
    }
    if (write_state) {
#pragma unroll
        for (int c = 0; c < CW; ++c) {
            if (p0 + c > P) continue;
            float* col = S + (size_t)c * K;
            if (VEC) {
#pragma unroll
                for (int k = 0; k < PER; k += 4)
                    if (n0 + k < K) *reinterpret_cast<float4*>(col + n0 + k) = make_float4(s[c][k], s[c][k + 1], s[c][k + 2], s[c][k + 3]);
            } else {
#pragma unroll
                for (int k = 0; k < PER; ++k)
                    if (n0 + k < K) col[n0 + k] = s[c][k];
            }
        }
        __syncwarp();                                               // every lane has read M[0]
        if (lane < CW && p0 + lane <= P) M[lane] = m_last;
    }
}

// ---------------------------------------------------------------------------------
// Long prompts in chunks of 64 tokens.  With G_i the sum of a chunk's log decays up to its token i (included), S0 the state
// at the chunk's start and w the write strengths,
//     S_i^T q_i = e^(G_i) S0^T q_i + sum_{j <= i} e^(G_i - G_j) w_j (q_i . k_j) v_j
//     S_end     = e^(G_end) S0 + sum_j e^(G_end - G_j) w_j k_j v_j^T
// (n likewise, its value 1), and chunks compose.  Three kernels, all sums 32-bit: chunk_state leaves every chunk's own sum
// of outer products, chunk_carry runs through a sequence's chunks and replaces each sum by the state its chunk starts from,
// chunk_out makes the chunk's scores and outputs.
// scratch: own / starts [B * chunks, H, P + 1, K], then the chunks' total decays [B * chunks, H].
// ---------------------------------------------------------------------------------
// four neighbouring floats at p + at, zeros from `limit` on
template <bool VEC>
__device__ __forceinline__ float4 mlstm_four(const float* __restrict__ p, int at, int limit) {
    if (VEC) return at < limit ? *reinterpret_cast<const float4*>(p + at) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(at < limit ? p[at] : 0.f, at + 1 < limit ? p[at + 1] : 0.f, at + 2 < limit ? p[at + 2] : 0.f, at + 3 < limit ? p[at + 3] : 0.f);
}

// G [64] of the chunk's n tokens from t0 on (constant beyond the end), by the first warp; the caller synchronises
__device__ __forceinline__ void mlstm_prefix(const float* __restrict__ log_decay, int t0, int n, int H, int h, double* G) {
    const int lane = threadIdx.x;
    if (lane >= 32) return;
    const double a = 2 * lane < n ? (double)log_decay[(size_t)(t0 + 2 * lane) * H + h] : 0.0;
    const double c = 2 * lane + 1 < n ? (double)log_decay[(size_t)(t0 + 2 * lane + 1) * H + h] : 0.0;
    double sum = a + c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
    }
    double before = __shfl_up_sync(0xffffffffu, sum, 1);
    if (lane == 0) before = 0.0;
    G[2 * lane] = before + a;
    G[2 * lane + 1] = sum;
}

// grid (chunks, H * ptiles * ktiles, B), 256 threads; a tile is PT (64 or 128) value columns x 64 key rows, a thread
// PT / 16 x 4 of it; dynamic shared memory: 64 * (64 + PT) floats
template <int PT, bool VEC>
__global__ void __launch_bounds__(256)
mlstm_chunk_state_kernel(MlstmRows rows, const float* __restrict__ log_decay, const float* __restrict__ write, const int* __restrict__ cu_seqlens,
                         float* __restrict__ own, float* __restrict__ totals, MlstmSizes z, int n_chunks, int ptiles, int ktiles) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int L = QWB_MLSTM_CHUNK;
    constexpr int CN = PT / 64;                                     // groups of four value columns a thread
    extern __shared__ __align__(16) float cs_smem[];
    float (*ks)[64] = reinterpret_cast<float (*)[64]>(cs_smem);
    float (*vs)[PT] = reinterpret_cast<float (*)[PT]>(cs_smem + L * 64);
    __shared__ double G[L];
    __shared__ float coef[L];
    const int H = z.H, K = z.K, P = z.P, c = blockIdx.x, b = blockIdx.z, tid = threadIdx.x;
    const int h = blockIdx.y / (ptiles * ktiles), tile = blockIdx.y - h * ptiles * ktiles, pt = tile / ktiles, kt = tile - pt * ktiles;
    const int t0 = cu_seqlens[b] + c * L, n = min(L, cu_seqlens[b + 1] - t0);
    if (n <= 0) return;
    mlstm_prefix(log_decay, t0, n, H, h, G);
    __syncthreads();
    if (tid < L) coef[tid] = tid < n ? expf((float)(G[L - 1] - G[tid])) * write[(size_t)(t0 + tid) * H + h] : 0.f;
    if (tid == 0 && tile == 0) totals[((size_t)b * n_chunks + c) * H + h] = expf((float)G[L - 1]);
    __syncthreads();
    const int k0 = kt * 64, p0 = pt * PT;
    for (int idx = tid; idx < L * 16; idx += 256) {
        const int j = idx >> 4, e = (idx & 15) * 4;
        float4 k4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < n) k4 = mlstm_four<VEC>(rows.x + (size_t)(t0 + j) * rows.ld + (H + h) * K, k0 + e, K);
        const float f = coef[j];
        *reinterpret_cast<float4*>(&ks[j][e]) = make_float4(k4.x * f, k4.y * f, k4.z * f, k4.w * f);
    }
    for (int idx = tid; idx < L * (PT / 4); idx += 256) {
        const int j = idx / (PT / 4), e = (idx - j * (PT / 4)) * 4;
        float4 v4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < n) v4 = mlstm_four<VEC>(rows.x + (size_t)(t0 + j) * rows.ld + 2 * H * K + h * P, p0 + e, P);
        *reinterpret_cast<float4*>(&vs[j][e]) = v4;
    }
    __syncthreads();
    const int kq = (tid & 15) * 4, pq = (tid >> 4) * 4;
    float acc[4 * CN][4];
#pragma unroll
    for (int p = 0; p < 4 * CN; ++p)
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[p][k] = 0.f;
#pragma unroll 8
    for (int j = 0; j < L; ++j) {
        const float4 kk = *reinterpret_cast<const float4*>(&ks[j][kq]);
        const float ka[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
        for (int g = 0; g < CN; ++g) {
            const float4 vv = *reinterpret_cast<const float4*>(&vs[j][64 * g + pq]);
            const float va[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
            for (int p = 0; p < 4; ++p)
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[4 * g + p][k] += va[p] * ka[k];
        }
    }
    float* U = own + (((size_t)b * n_chunks + c) * H + h) * (size_t)(P + 1) * K;
#pragma unroll
    for (int a = 0; a < 4 * CN; ++a) {
        const int p = p0 + 64 * (a >> 2) + pq + (a & 3);
        if (p >= P) continue;
        float* u = U + (size_t)p * K + k0 + kq;
        if (VEC) { if (k0 + kq < K) *reinterpret_cast<float4*>(u) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]); }
        else {
#pragma unroll
            for (int k = 0; k < 4; ++k) if (k0 + kq + k < K) u[k] = acc[a][k];
        }
    }
    if (pt == 0 && tid < 64 && k0 + tid < K) {                      // the column whose value is always 1
        float sum = 0.f;
#pragma unroll 8
        for (int j = 0; j < L; ++j) sum += ks[j][tid];
        U[(size_t)P * K + k0 + tid] = sum;
    }
}

// grid (ceil((P + 1) * K / W / 256), H, B): every element of the state runs through its sequence's chunks in order, W (4 or 1)
// neighbours a thread
template <int W>
__global__ void __launch_bounds__(256)
mlstm_chunk_carry_kernel(const int* __restrict__ cu_seqlens, const int* __restrict__ slots, float* __restrict__ state, float* __restrict__ m_state,
                         float* own, const float* __restrict__ totals, const float* __restrict__ m_run, MlstmSizes z, int n_chunks, int write_state) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int AHEAD = 8;
    const int H = z.H, K = z.K, P = z.P, h = blockIdx.y, b = blockIdx.z;
    const int e = (blockIdx.x * blockDim.x + threadIdx.x) * W, n_el = (P + 1) * K;
    const int t1 = cu_seqlens[b + 1], n_tok = t1 - cu_seqlens[b];
    if (e >= n_el || n_tok <= 0) return;
    const size_t head = (size_t)slots[b] * H + h;
    auto load = [](const float* p, float* v) {
        if (W == 4) { const float4 x = *reinterpret_cast<const float4*>(p); v[0] = x.x; v[W > 1 ? 1 : 0] = x.y; v[W > 2 ? 2 : 0] = x.z; v[W - 1] = x.w; }
        else v[0] = *p;
    };
    auto store = [](float* p, const float* v) {
        if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[W > 1 ? 1 : 0], v[W > 2 ? 2 : 0], v[W - 1]);
        else *p = v[0];
    };
    float s[W];
    load(state + head * n_el + e, s);
    const int chunks = (n_tok + QWB_MLSTM_CHUNK - 1) / QWB_MLSTM_CHUNK;
    const size_t step = (size_t)H * n_el;
    float* at = own + ((size_t)b * n_chunks * H + h) * n_el + e;
    const float* total = totals + (size_t)b * n_chunks * H + h;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float u[AHEAD][W], d[AHEAD];
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
            if (c0 + a < chunks) { load(at + (c0 + a) * step, u[a]); d[a] = total[(size_t)(c0 + a) * H]; }
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
            if (c0 + a < chunks) {
                store(at + (c0 + a) * step, s);
#pragma unroll
                for (int i = 0; i < W; ++i) s[i] = d[a] * s[i] + u[a][i];
            }
    }
    if (write_state) {
        store(state + head * n_el + e, s);
        if (e % K == 0) m_state[head * (P + 1) + e / K] = m_run[(size_t)(t1 - 1) * H + h];     // with W = 4, K is a multiple of 4
    }
}

// grid (chunks, H * ptiles, B), 256 threads; a block makes the outputs of a chunk's 64 tokens in PT (64 or 128) value
// columns.  Over the key rows in tiles of 32 it forms both the scores Q K^T (64 x 64, 4 x 4 a thread) and Q S0^T
// (64 x PT, 4 rows x PT / 16 columns a thread); then the scores, weighted by the decays between their tokens, times the values.
// Tiles are stored key row by key row, so that a thread reads four neighbours at a time.
template <int PT, bool VEC>
__global__ void __launch_bounds__(256, 2)
mlstm_chunk_out_kernel(MlstmRows rows, const float* __restrict__ log_decay, const float* __restrict__ write, const float* __restrict__ m_run,
                       const int* __restrict__ cu_seqlens, const float* __restrict__ starts, float* __restrict__ raw, float* __restrict__ divisor,
                       MlstmSizes z, int n_chunks, int ptiles, float q_scale, float tiny) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int L = QWB_MLSTM_CHUNK, KB = 32, LQ = L + 4, LP = PT + 4, CN = PT / 64;      // CN groups of four columns a thread
    extern __shared__ __align__(16) float co_smem[];
    __shared__ double G[L];
    __shared__ float eg[L], wr[L], dn[L], n0s[KB];
    float* Qt = co_smem;                    // [KB][LQ]
    float* Kt = Qt + KB * LQ;               // [KB][LQ]
    float* St = Kt + KB * LQ;               // [KB][LP]
    float* At = co_smem;                    // [L][LQ], token j's row: over the tiles above once they are read
    float* Vs = At + L * LQ;                // [L][LP]
    const int H = z.H, K = z.K, P = z.P, c = blockIdx.x, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y / ptiles, pt = blockIdx.y - h * ptiles, p0 = pt * PT;
    const int t0 = cu_seqlens[b] + c * L, n = min(L, cu_seqlens[b + 1] - t0);
    if (n <= 0) return;
    mlstm_prefix(log_decay, t0, n, H, h, G);
    __syncthreads();
    if (tid < L) {
        eg[tid] = expf((float)G[tid]) * q_scale;
        wr[tid] = tid < n ? write[(size_t)(t0 + tid) * H + h] : 0.f;
    }
    const float* S0 = starts + (((size_t)b * n_chunks + c) * H + h) * (size_t)(P + 1) * K;
    const int rg = (tid >> 4) * 4, cg = (tid & 15) * 4;
    float a[4][4], acc[4][4 * CN], nq = 0.f;
#pragma unroll
    for (int r = 0; r < 4; ++r) {
#pragma unroll
        for (int j = 0; j < 4; ++j) a[r][j] = 0.f;
#pragma unroll
        for (int j = 0; j < 4 * CN; ++j) acc[r][j] = 0.f;
    }
    // a warp fetches one group of four key rows for 32 tokens or columns at a time; a tile ahead of its use
    float4 fq[2], fk[2], fs[PT / 32];
    float fn = 0.f;
    auto fetch = [&](int k0) {
        const int k = k0 + warp * 4;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int i = lane + 32 * r;
            const float* row = rows.x + (size_t)(t0 + min(i, n - 1)) * rows.ld;
            fq[r] = mlstm_four<VEC>(row + h * K, k, i < n ? K : 0);
            fk[r] = mlstm_four<VEC>(row + (H + h) * K, k, i < n ? K : 0);
        }
#pragma unroll
        for (int r = 0; r < PT / 32; ++r) {
            const int p = p0 + lane + 32 * r;
            fs[r] = mlstm_four<VEC>(S0 + (size_t)min(p, P) * K, k, p < P ? K : 0);
        }
        if (pt == 0 && tid < KB) fn = k0 + tid < K ? S0[(size_t)P * K + k0 + tid] : 0.f;
    };
    auto put = [&](float* dst, int ld, int at, float4 v) {
        float* d = dst + (warp * 4) * ld + at;
        d[0] = v.x; d[ld] = v.y; d[2 * ld] = v.z; d[3 * ld] = v.w;
    };
    fetch(0);
    for (int k0 = 0; k0 < K; k0 += KB) {
        __syncthreads();
#pragma unroll
        for (int r = 0; r < 2; ++r) { put(Qt, LQ, lane + 32 * r, fq[r]); put(Kt, LQ, lane + 32 * r, fk[r]); }
#pragma unroll
        for (int r = 0; r < PT / 32; ++r) put(St, LP, lane + 32 * r, fs[r]);
        if (pt == 0 && tid < KB) n0s[tid] = fn;
        __syncthreads();
        if (k0 + KB < K) fetch(k0 + KB);
#pragma unroll 4
        for (int k = 0; k < KB; ++k) {
            const float4 q4 = *reinterpret_cast<const float4*>(Qt + k * LQ + rg);
            const float4 k4 = *reinterpret_cast<const float4*>(Kt + k * LQ + cg);
            const float qa[4] = {q4.x, q4.y, q4.z, q4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
                for (int j = 0; j < 4; ++j) a[r][j] += qa[r] * ka[j];
#pragma unroll
            for (int g = 0; g < CN; ++g) {
                const float4 s4 = *reinterpret_cast<const float4*>(St + k * LP + 64 * g + cg);
                const float sa[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[r][4 * g + j] += qa[r] * sa[j];
            }
        }
        if (pt == 0 && tid < L)
            for (int k = 0; k < KB; ++k) nq += Qt[k * LQ + tid] * n0s[k];
    }
    __syncthreads();                                                // the tiles are no longer read
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        float4 col;
        float* cp = reinterpret_cast<float*>(&col);
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int i = rg + r, jj = cg + j;
            cp[r] = jj <= i && i < n ? a[r][j] * q_scale * expf((float)(G[i] - G[jj])) * wr[jj] : 0.f;
        }
        *reinterpret_cast<float4*>(At + (cg + j) * LQ + rg) = col;
    }
    for (int idx = tid; idx < L * (PT / 4); idx += 256) {
        const int j = idx / (PT / 4), e = (idx - j * (PT / 4)) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < n) v = mlstm_four<VEC>(rows.x + (size_t)(t0 + j) * rows.ld + 2 * H * K + h * P, p0 + e, P);
        *reinterpret_cast<float4*>(Vs + j * LP + e) = v;
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int j = 0; j < 4 * CN; ++j) acc[r][j] *= eg[rg + r];
    if (pt == 0 && tid < L) dn[tid] = nq * eg[tid];
    __syncthreads();
    const int j_end = min(n, rg + 4);                               // no later token is seen
    for (int j = 0; j < j_end; ++j) {
        const float4 a4 = *reinterpret_cast<const float4*>(At + j * LQ + rg);
        const float aa[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
        for (int g = 0; g < CN; ++g) {
            const float4 v4 = *reinterpret_cast<const float4*>(Vs + j * LP + 64 * g + cg);
            const float va[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
                for (int q = 0; q < 4; ++q) acc[r][4 * g + q] += aa[r] * va[q];
        }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        if (rg + r >= n) continue;
        float* o = raw + ((size_t)(t0 + rg + r) * H + h) * P;
#pragma unroll
        for (int g = 0; g < CN; ++g) {
            const int p = p0 + 64 * g + cg;
            if (VEC) { if (p < P) *reinterpret_cast<float4*>(o + p) = make_float4(acc[r][4 * g], acc[r][4 * g + 1], acc[r][4 * g + 2], acc[r][4 * g + 3]); }
            else {
#pragma unroll
                for (int q = 0; q < 4; ++q) if (p + q < P) o[p + q] = acc[r][4 * g + q];
            }
        }
    }
    if (pt == 0 && tid < n) {
        float sum = dn[tid];
        for (int j = 0; j <= tid; ++j) sum += At[j * LQ + tid];
        const size_t at = (size_t)(t0 + tid) * H + h;
        divisor[at] = fmaxf(fabsf(sum), expf(-m_run[at])) + tiny;
    }
}

// ---------------------------------------------------------------------------------
static int check_mlstm(const char* what, MlstmSizes z, MlstmRows r, int B) {
    if (z.H <= 0 || z.K <= 0 || z.P <= 0 || z.K > 32 * QWB_MLSTM_MAX_PER)
        return qwb_fail(QWB_ERR_ARG, "%s: %d heads of %d x %d (up to %d key rows)", what, z.H, z.K, z.P, 32 * QWB_MLSTM_MAX_PER);
    const long long n_qkv = (long long)z.H * (2 * z.K + z.P);
    if (r.ld < n_qkv || r.i_col < n_qkv || r.f_col < n_qkv || r.i_col + z.H > r.ld || r.f_col + z.H > r.ld)
        return qwb_fail(QWB_ERR_ARG, "%s: rows of %d with gates at %d and %d", what, r.ld, r.i_col, r.f_col);
    if (B > 65535 || z.H > 65535) return qwb_fail(QWB_ERR_ARG, "%s: %d sequences or %d heads are too many", what, B, z.H);
    return 0;
}
static bool mlstm_aligned(const void* p) { return (uintptr_t)p % 16 == 0; }

// rows x [T, ld]; i_bias, f_bias [H]; state [slots, H, P + 1, K], m_state [slots, H, P + 1]; raw [T, H * P], divisor [T, H].
// single: every sequence brings one token, the gates are made in the kernel (gate_rows is then not used).
// gate_rows: 3 * T * H floats (log decays, write strengths, running maxima).
extern "C" int qwb_mlstm_scan(const float* x, int ld, int i_col, int f_col, const float* i_bias, const float* f_bias, float cap, float* state,
                              float* m_state, const int* cu_seqlens, const int* slots, float* gate_rows, float* raw, float* divisor, int T, int B, int H,
                              int K, int P, float q_scale, float tiny, int single, int write_state, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    const MlstmSizes z{H, K, P};
    const MlstmRows rows{x, ld, i_col, f_col};
    const MlstmGates gates{i_bias, f_bias, cap};
    if (int rc = check_mlstm("mlstm_scan", z, rows, B)) return rc;
    if (!(cap > 0.f) || (single && T != B) || (!single && !gate_rows)) return qwb_fail(QWB_ERR_ARG, "mlstm_scan: cap %g, %d tokens of %d sequences", (double)cap, T, B);
    float *log_decay = gate_rows, *write = gate_rows + (size_t)T * H, *m_run = gate_rows + 2 * (size_t)T * H;
    if (!single) {
        qwb_launch(mlstm_gates_kernel, dim3(H, B), 256, 0, stream, rows, gates, (const float*)m_state, cu_seqlens, slots, log_decay, write, m_run, H, P);
        if (int rc = qwb_check_launch("mlstm_gates")) return rc;
    }
    int per = 1;
    while (32 * per < K) per *= 2;
    const bool vec = per >= 4 && K % 4 == 0 && ld % 4 == 0 && mlstm_aligned(x) && mlstm_aligned(state);
    const int cw = per <= 8 ? 4 : 2;
    const dim3 grid((P / cw + 1 + QWB_MLSTM_WARPS - 1) / QWB_MLSTM_WARPS, H, B);
#define QWB_MLSTM1(PER, VEC, STEP) \
    qwb_launch(mlstm_scan_kernel<PER, VEC, (STEP ? 1 : (PER <= 4 ? 4 : (PER == 8 ? 2 : 1))), (PER <= 8 ? 4 : 2), STEP>, grid, 32 * QWB_MLSTM_WARPS, 0, stream, rows, \
               gates, (const float*)log_decay, (const float*)write, (const float*)m_run, state, m_state, cu_seqlens, slots, raw, divisor, z, q_scale, tiny, write_state)
#define QWB_MLSTM(PER, VEC) do { if (single) QWB_MLSTM1(PER, VEC, true); else QWB_MLSTM1(PER, VEC, false); } while (0)
    if (per == 1) QWB_MLSTM(1, false); else if (per == 2) QWB_MLSTM(2, false);
    else if (per == 4) { if (vec) QWB_MLSTM(4, true); else QWB_MLSTM(4, false); }
    else if (per == 8) { if (vec) QWB_MLSTM(8, true); else QWB_MLSTM(8, false); }
    else { if (vec) QWB_MLSTM(16, true); else QWB_MLSTM(16, false); }
#undef QWB_MLSTM1
#undef QWB_MLSTM
    return qwb_check_launch("mlstm_scan");
}

extern "C" int qwb_mlstm_chunk_len() { return QWB_MLSTM_CHUNK; }

extern "C" long long qwb_mlstm_scratch_floats(int B, int max_new, int H, int K, int P) {
    const long long n = (long long)B * ((max_new + QWB_MLSTM_CHUNK - 1) / QWB_MLSTM_CHUNK) * H;
    return n * (P + 1) * K + n;
}

// The same step in chunks; scratch: qwb_mlstm_scratch_floats floats.
extern "C" int qwb_mlstm_chunked(const float* x, int ld, int i_col, int f_col, const float* i_bias, const float* f_bias, float cap, float* state,
                                 float* m_state, const int* cu_seqlens, const int* slots, float* gate_rows, float* scratch, float* raw, float* divisor,
                                 int T, int B, int max_new, int H, int K, int P, float q_scale, float tiny, int write_state, cudaStream_t stream) {
    if (T <= 0 || B <= 0 || max_new <= 0) return 0;
    const MlstmSizes z{H, K, P};
    const MlstmRows rows{x, ld, i_col, f_col};
    const MlstmGates gates{i_bias, f_bias, cap};
    if (int rc = check_mlstm("mlstm_chunked", z, rows, B)) return rc;
    const int n_chunks = (max_new + QWB_MLSTM_CHUNK - 1) / QWB_MLSTM_CHUNK;
    const int pt = P > 64 ? 128 : 64, ptiles = (P + pt - 1) / pt, ktiles = (K + 63) / 64;
    if (!(cap > 0.f) || !gate_rows || !scratch || (long long)H * ptiles * ktiles > 65535 || (long long)(P + 1) * K > 0x7fffffffLL)
        return qwb_fail(QWB_ERR_ARG, "mlstm_chunked: cap %g, %d heads of %d x %d", (double)cap, H, K, P);
    float *log_decay = gate_rows, *write = gate_rows + (size_t)T * H, *m_run = gate_rows + 2 * (size_t)T * H;
    float* totals = scratch + (size_t)B * n_chunks * H * (P + 1) * K;
    const bool vec = K % 4 == 0 && P % 4 == 0 && ld % 4 == 0 && mlstm_aligned(x) && mlstm_aligned(scratch) && mlstm_aligned(raw) && mlstm_aligned(state);
    qwb_launch(mlstm_gates_kernel, dim3(H, B), 256, 0, stream, rows, gates, (const float*)m_state, cu_seqlens, slots, log_decay, write, m_run, H, P);
    if (int rc = qwb_check_launch("mlstm_gates")) return rc;
    const size_t smem1 = (size_t)QWB_MLSTM_CHUNK * (64 + pt) * sizeof(float);
    auto state_kernel = pt == 128 ? (vec ? mlstm_chunk_state_kernel<128, true> : mlstm_chunk_state_kernel<128, false>)
                                  : (vec ? mlstm_chunk_state_kernel<64, true> : mlstm_chunk_state_kernel<64, false>);
    if (smem1 + 1024 > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "mlstm_chunked: %s", cudaGetErrorString(e));
    }
    qwb_launch(state_kernel, dim3(n_chunks, H * ptiles * ktiles, B), 256, smem1, stream, rows, (const float*)log_decay, (const float*)write, cu_seqlens, scratch,
               totals, z, n_chunks, ptiles, ktiles);
    if (int rc = qwb_check_launch("mlstm_chunk_state")) return rc;
    auto carry_kernel = vec ? mlstm_chunk_carry_kernel<4> : mlstm_chunk_carry_kernel<1>;
    const int per_block = vec ? 1024 : 256;
    qwb_launch(carry_kernel, dim3(((P + 1) * K + per_block - 1) / per_block, H, B), 256, 0, stream, cu_seqlens, slots, state, m_state, scratch,
               (const float*)totals, (const float*)m_run, z, n_chunks, write_state);
    if (int rc = qwb_check_launch("mlstm_chunk_carry")) return rc;
    const size_t lq = QWB_MLSTM_CHUNK + 4, lp = pt + 4;
    const size_t smem = (QWB_MLSTM_CHUNK * lq + QWB_MLSTM_CHUNK * lp) * sizeof(float);       // the tiles of 32 key rows need less
    auto out_kernel = pt == 128 ? (vec ? mlstm_chunk_out_kernel<128, true> : mlstm_chunk_out_kernel<128, false>)
                                : (vec ? mlstm_chunk_out_kernel<64, true> : mlstm_chunk_out_kernel<64, false>);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "mlstm_chunked: %s", cudaGetErrorString(e));
    }
    qwb_launch(out_kernel, dim3(n_chunks, H * ptiles, B), 256, smem, stream, rows, (const float*)log_decay, (const float*)write, (const float*)m_run, cu_seqlens,
               (const float*)scratch, raw, divisor, z, n_chunks, ptiles, q_scale, tiny);
    return qwb_check_launch("mlstm_chunk_out");
}
