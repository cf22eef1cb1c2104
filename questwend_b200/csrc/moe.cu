// Routed experts: the router's choice, and the experts' feed-forward for the tokens that chose them.
//
//   moe_route     scores of all experts (softmax or sigmoid of the logits, 32-bit); a choice by score, or by score plus a
//                 correction per expert, over all experts or inside the best groups of neighbours; the `top` largest,
//                 ties to the lower index; weights from the scores alone
//   moe_up        act[t, k, :] = silu(Wg[e] x_t) * (Wu[e] x_t) (gated) or f(Wu[e] x_t), e = the k-th choice of token t
//   moe_down      out[t, :] = sum_k weight[t, k] * Wd[e_k] act[t, k, :]
// The weights may stand on the experts' inputs instead: act = f(Wu[e] (w x_t)), formed as f(w (Wu[e] x_t)) in 32-bit (both
// factors of the gated form), and the sum over the choices is then plain.
// A shared expert (ungated, a width of its own) that every token uses rides in the same two kernels; its output is
// multiplied by a number per token.
//
// The products read each chosen expert's rows straight from the stacked weights (Wu [E, F, D], gated: [E, 2F, D] with the
// gate rows first; Wd [E, D, F]): a warp per few rows, 32-bit sums.  This is the form for a step of few tokens, where every
// token's experts are streamed once, and for the 32-bit engine.  Many bfloat16 tokens are sorted by expert instead
// and go through a library grouped product; moe_sort, moe_spread, moe_act and moe_combine are the kernels around it.
#include "common.cuh"

#define QWB_MOE_MAX_TOP 16
#define QWB_MOE_MAX_EXPERTS 1024
#define MOE_UP_BLOCKS 5         // blocks of moe_up an SM by registers: more loads on their way beat a few spills in the shared expert's part
#define QWB_MOE_GATED 16        // activation code of the gated form, silu(gate) * up; others: qwb_activate's codes

// ---------------------------------------------------------------------------------
// route: a warp per token.  logits rows hold ld values: E experts and, with gate_out, the shared expert's gate after them.
//   score[e]  softmax(z)[e] (sigmoid = 0) or 1 / (1 + exp(-z[e])) (sigmoid = 1)
//   choice[e] score[e] + correction[e]; a group's score is the sum of its two largest choices (of one, if it has one
//             expert), and the experts of all but the `keep` best groups (ties to the lower index) are out
//   weight    score of a chosen expert, / (their sum + sum_eps) if `renorm`, * weight_scale
//   gate_out  1 / (1 + exp(-z[E]))
// ---------------------------------------------------------------------------------
// The choice works on keys, the scores' bits in an order that unsigned integers keep; 0 (below every number's key) is out.
__device__ __forceinline__ unsigned order_key(float v) {
    const unsigned b = __float_as_uint(v);
    return b ^ ((b >> 31) ? 0xffffffffu : 0x80000000u);
}
// The place of the largest of n keys in shared memory (the lowest of equal ones), which is then out; the whole warp calls.
__device__ __forceinline__ int take_best(unsigned* key, int n, int lane) {
    unsigned best = 0;
    int at = n;
    for (int e = lane; e < n; e += 32) {
        const unsigned v = key[e];
        if (v > best || at == n) { best = v; at = e; }
    }
    const unsigned top = __reduce_max_sync(0xffffffffu, best);
    const int first = (int)__reduce_min_sync(0xffffffffu, best == top && at < n ? (unsigned)at : 0x7fffffffu);
    if (lane == 0) key[first] = 0;
    __syncwarp();
    return first;
}

__global__ void moe_route_kernel(const float* logits, int ld, const float* __restrict__ correction, int* __restrict__ chosen,
                                 float* __restrict__ weight, float* __restrict__ gate_out, int T, int E, int top, int sigmoid,
                                 int groups, int keep, int renorm, float sum_eps, float weight_scale) {
    pdl_launch_dependents();            // the trigger first: see qwb_launch_link
    pdl_wait();
    extern __shared__ unsigned route_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + warp;
    if (t >= T) return;
    unsigned* key = route_smem + warp * (2 * E + groups);   // [E] keys of the choice scores
    float* score = reinterpret_cast<float*>(key + E);       // [E]
    unsigned* gkey = key + 2 * E;                           // [groups]
    const float* z = logits + (size_t)t * ld;
    float mx = 0.f, sum = 1.f;
    if (!sigmoid) {
        mx = -INFINITY;
        for (int e = lane; e < E; e += 32) mx = fmaxf(mx, __ldcg(z + e));
        mx = warp_max(mx);
        sum = 0.f;
        for (int e = lane; e < E; e += 32) sum += expf(__ldcg(z + e) - mx);
        sum = warp_sum(sum);
    }
    const bool by_logit = !sigmoid && !correction && groups == 1;       // a softmax keeps the logits' order
    for (int e = lane; e < E; e += 32) {
        const float v = __ldcg(z + e);
        const float s = sigmoid ? 1.f / (1.f + expf(-v)) : expf(v - mx) / sum;
        score[e] = s;
        key[e] = order_key(by_logit ? v : s + (correction ? correction[e] : 0.f));
    }
    __syncwarp();
    if (keep < groups) {
        const int size = E / groups;
        auto value = [&](int e) { const unsigned k = key[e]; return __uint_as_float((k >> 31) ? k ^ 0x80000000u : ~k); };
        for (int g = lane; g < groups; g += 32) {
            float a = value(g * size), b = -INFINITY;       // the two largest
            for (int e = g * size + 1; e < (g + 1) * size; ++e) {
                const float c = value(e);
                b = fmaxf(b, fminf(a, c));
                a = fmaxf(a, c);
            }
            gkey[g] = order_key(size > 1 ? a + b : a);
        }
        __syncwarp();
        for (int k = 0; k < keep; ++k) take_best(gkey, groups, lane);
        for (int e = lane; e < E; e += 32)
            if (gkey[e / size]) key[e] = 0;                 // of a group that was not taken
        __syncwarp();
    }
    int mine = 0;                                           // lane k's choice
    for (int k = 0; k < top; ++k) {
        const int at = take_best(key, E, lane);
        if (lane == k) mine = at;
    }
    const float s = lane < top ? score[mine] : 0.f;
    const float total = warp_sum(s);
    if (lane < top) {
        chosen[(size_t)t * top + lane] = mine;
        weight[(size_t)t * top + lane] = (renorm ? s / (total + sum_eps) : s) * weight_scale;
    }
    if (gate_out && lane == 31) gate_out[t] = 1.f / (1.f + expf(-__ldcg(z + E)));
}

extern "C" int qwb_moe_route(const float* logits, int ld, const float* correction, int* chosen, float* weight, float* gate_out, int T,
                             int E, int top, int sigmoid, int groups, int keep, int renorm, float sum_eps, float weight_scale,
                             cudaStream_t stream) {
    if (T <= 0) return 0;
    if (E <= 0 || E > QWB_MOE_MAX_EXPERTS || top <= 0 || top > E || top > QWB_MOE_MAX_TOP)
        return qwb_fail(QWB_ERR_ARG, "moe_route: %d of %d experts (at most %d of %d)", top, E, QWB_MOE_MAX_TOP, QWB_MOE_MAX_EXPERTS);
    if (groups <= 0 || E % groups || keep <= 0 || keep > groups || top > keep * (E / groups))
        return qwb_fail(QWB_ERR_ARG, "moe_route: %d of %d experts from %d of %d groups", top, E, keep, groups);
    if (ld < E + (gate_out ? 1 : 0)) return qwb_fail(QWB_ERR_ARG, "moe_route: rows of %d logits for %d experts", ld, E);
    const int warps = T >= 592 ? 4 : 1;                     // few tokens: a block each, side by side on the SMs
    const size_t smem = (size_t)warps * (2 * E + groups) * sizeof(float);   // at most 48 KB
    qwb_launch_link(T, QWB_LINK_ROWS_NORM, moe_route_kernel, (T + warps - 1) / warps, 32 * warps, smem, stream, logits, ld, correction, chosen, weight, gate_out, T, E, top,
               sigmoid, groups, keep, renorm, sum_eps, weight_scale);
    return qwb_check_launch("moe_route");
}

// ---------------------------------------------------------------------------------
// Rows of a matrix times vectors, a warp each: acc[r * NX + v] = this lane's part of w_r . x_v; rows `ldw` values apart, of
// which the first nr exist, vectors `ldx` apart, of which the first nx exist (a missing one repeats the last).
// ---------------------------------------------------------------------------------
template <typename T, int NR, int NX>
__device__ __forceinline__ void lane_dots(const T* __restrict__ w, size_t ldw, int nr, const T* __restrict__ x, size_t ldx, int nx, int n,
                                          int lane, float* acc) {
    constexpr int VEC = Vec16<T>::N;
#pragma unroll
    for (int i = 0; i < NR * NX; ++i) acc[i] = 0.f;
    const T* wr[NR];
    const T* xv[NX];
#pragma unroll
    for (int r = 0; r < NR; ++r) wr[r] = w + (size_t)(r < nr ? r : nr - 1) * ldw;
#pragma unroll
    for (int v = 0; v < NX; ++v) xv[v] = x + (size_t)(v < nx ? v : nx - 1) * ldx;
    if (n % VEC == 0 && ldw % VEC == 0 && (NX == 1 || ldx % VEC == 0) && (uintptr_t)w % 16 == 0 && (uintptr_t)x % 16 == 0) {
#pragma unroll 2
        for (int i = lane; i < n / VEC; i += 32) {
            float a[NR][VEC];
#pragma unroll
            for (int r = 0; r < NR; ++r) reinterpret_cast<const Vec16<T>*>(wr[r])[i].get(a[r]);
#pragma unroll
            for (int v = 0; v < NX; ++v) {
                float b[VEC];
                reinterpret_cast<const Vec16<T>*>(xv[v])[i].get(b);
#pragma unroll
                for (int r = 0; r < NR; ++r)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) acc[r * NX + v] += a[r][e] * b[e];
            }
        }
    } else {
        for (int i = lane; i < n; i += 32)
#pragma unroll
            for (int v = 0; v < NX; ++v) {
                const float b = to_f32(xv[v][i]);
#pragma unroll
                for (int r = 0; r < NR; ++r) acc[r * NX + v] += to_f32(wr[r][i]) * b;
            }
    }
}

// Blocks: per copy of a token (T * top) as many as its expert's features take, 8 warps each, then the shared expert's, with
// NT tokens a warp.
// A warp makes two features of a plain expert, one of a gated one (its gate and its up row), two of the shared expert.
template <typename T, int NT>
__global__ void __launch_bounds__(256, MOE_UP_BLOCKS)
moe_up_kernel(const T* __restrict__ x, const T* __restrict__ wu, const int* __restrict__ chosen, const float* __restrict__ weight_in, T* __restrict__ act,
              const T* __restrict__ wsu, T* __restrict__ act_s, int n_tok, int D, int F, int Fs, int top, int kind) {
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool gated = kind == QWB_MOE_GATED;
    const int per_slot = ((gated ? F : (F + 1) / 2) + 7) / 8, n_routed = n_tok * top * per_slot;
    if ((int)blockIdx.x < n_routed) {
        const int slot = blockIdx.x / per_slot, item = (blockIdx.x - slot * per_slot) * 8 + warp;
        const int f = gated ? item : 2 * item;
        if (f >= F) return;
        const size_t first = (size_t)chosen[slot] * (gated ? 2 * F : F) + f;
        float acc[2];
        lane_dots<T, 2, 1>(wu + first * D, gated ? (size_t)F * D : (size_t)D, gated ? 2 : min(2, F - f), x + (size_t)(slot / top) * D, 0, 1, D,
                           lane, acc);
        const float w = weight_in ? weight_in[slot] : 1.f;
        const float a = warp_sum(acc[0]) * w, b = warp_sum(acc[1]) * w;
        T* o = act + (size_t)slot * F + f;
        if (gated) { if (lane == 0) o[0] = from_f32<T>(a / (1.f + expf(-a)) * b); }
        else if (lane < min(2, F - f)) o[lane] = from_f32<T>(qwb_activate(lane ? b : a, kind));
    } else {
        const int per_group = ((Fs + 1) / 2 + 7) / 8, group = (blockIdx.x - n_routed) / per_group;
        const int t0 = group * NT, f = 2 * ((blockIdx.x - n_routed - group * per_group) * 8 + warp);
        if (f >= Fs) return;
        const int nt = min(NT, n_tok - t0), nf = min(2, Fs - f);
        float acc[2 * NT];
        lane_dots<T, 2, NT>(wsu + (size_t)f * D, D, nf, x + (size_t)t0 * D, D, nt, D, lane, acc);
#pragma unroll
        for (int i = 0; i < 2 * NT; ++i) {
            const float v = warp_sum(acc[i]);
            if (lane == i && i / NT < nf && i % NT < nt)
                act_s[(size_t)(t0 + i % NT) * Fs + f + i / NT] = from_f32<T>(qwb_activate(v, kind == QWB_MOE_GATED ? 3 : kind));
        }
    }
}

// grid (ceil(D / NR), T), a warp per choice and one for the shared expert: NR outputs of one token; the warps' products
// are weighted and summed in the order of the choices, the shared expert last.  out may be added onto (`onto`).
template <typename T, int NR>
__global__ void moe_down_kernel(const T* __restrict__ act, const T* __restrict__ wd, const int* __restrict__ chosen,
                                const float* __restrict__ weight, const T* __restrict__ act_s, const T* __restrict__ wsd,
                                const float* __restrict__ gate, float* out, int D, int F, int Fs, int top, int onto) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float part[QWB_MOE_MAX_TOP + 1][NR];
    const int t = blockIdx.y, d = blockIdx.x * NR;
    const int k = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nr = min(NR, D - d);
    float acc[NR], mul;
    if (k < top) {
        const size_t slot = (size_t)t * top + k;
        lane_dots<T, NR, 1>(wd + ((size_t)chosen[slot] * D + d) * F, F, nr, act + slot * F, 0, 1, F, lane, acc);
        mul = weight ? weight[slot] : 1.f;
    } else {
        lane_dots<T, NR, 1>(wsd + (size_t)d * Fs, Fs, nr, act_s + (size_t)t * Fs, 0, 1, Fs, lane, acc);
        mul = gate ? gate[t] : 1.f;
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) {
        const float v = warp_sum(acc[r]);
        if (lane == 0) part[k][r] = mul * v;
    }
    __syncthreads();
    if (threadIdx.x < nr) {
        float total = 0.f;
        for (int i = 0; i < (int)(blockDim.x >> 5); ++i) total += part[i][threadIdx.x];
        float* o = out + (size_t)t * D + d + threadIdx.x;
        *o = onto ? *o + total : total;
    }
}

template <typename T>
static void launch_moe_experts(const void* x, const void* wu, const void* wd, const int* chosen, const float* weight_in, const float* weight, const void* wsu,
                               const void* wsd, const float* gate, void* act, void* act_s, float* out, int n_tok, int D, int F, int Fs,
                               int top, int kind, int onto, cudaStream_t stream) {
    const int per_slot = ((kind == QWB_MOE_GATED ? F : (F + 1) / 2) + 7) / 8, per_group = Fs > 0 ? ((Fs + 1) / 2 + 7) / 8 : 0;
    const int nt = n_tok > 1 ? 2 : 1;
    const dim3 g1(n_tok * top * per_slot + (n_tok + nt - 1) / nt * per_group), g2((D + 3) / 4, n_tok);
    if (nt == 1)
        qwb_launch(moe_up_kernel<T, 1>, g1, 256, 0, stream, (const T*)x, (const T*)wu, chosen, weight_in, (T*)act, (const T*)wsu, (T*)act_s, n_tok, D, F, Fs, top, kind);
    else
        qwb_launch(moe_up_kernel<T, 2>, g1, 256, 0, stream, (const T*)x, (const T*)wu, chosen, weight_in, (T*)act, (const T*)wsu, (T*)act_s, n_tok, D, F, Fs, top, kind);
    qwb_launch(moe_down_kernel<T, 4>, g2, 32 * (top + (Fs > 0 ? 1 : 0)), 0, stream, (const T*)act, (const T*)wd, chosen, weight, (const T*)act_s,
               (const T*)wsd, gate, out, D, F, Fs, top, onto);
}

// weight [T, top]: on the experts' inputs (on_input) or outputs.
// wsu [Fs, D], wsd [D, Fs], gate [T] (or null: 1), act_s [T, Fs]: the shared expert, Fs = 0 for none.
extern "C" int qwb_moe_experts(const void* x, const void* wu, const void* wd, const int* chosen, const float* weight, int on_input, const void* wsu,
                               const void* wsd, const float* gate, void* act, void* act_s, float* out, int dtype, int T, int D, int F,
                               int Fs, int top, int kind, int onto, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0 || F <= 0 || Fs < 0 || top <= 0 || top > QWB_MOE_MAX_TOP)
        return qwb_fail(QWB_ERR_ARG, "moe_experts: width %d, expert width %d, shared %d, %d choices", D, F, Fs, top);
    if (Fs > 0 && (!wsu || !wsd || !act_s)) return qwb_fail(QWB_ERR_ARG, "moe_experts: a shared expert without its matrices");
    if (kind != QWB_MOE_GATED && !qwb_activation_known(kind)) return qwb_fail(QWB_ERR_ARG, "moe_experts: unknown activation %d", kind);
    if ((long long)T * top + T > 65535 || ((long long)T * top + T) * ((F > Fs ? F : Fs) / 8 + 1) > 0x7fffffffLL)
        return qwb_fail(QWB_ERR_ARG, "moe_experts: %d tokens x %d choices are too many for one launch", T, top);
    const float *weight_in = on_input ? weight : nullptr, *weight_out = on_input ? nullptr : weight;
    if (dtype == QWB_DT_F32)
        launch_moe_experts<float>(x, wu, wd, chosen, weight_in, weight_out, wsu, wsd, gate, act, act_s, out, T, D, F, Fs, top, kind, onto, stream);
    else if (dtype == QWB_DT_BF16)
        launch_moe_experts<bf16>(x, wu, wd, chosen, weight_in, weight_out, wsu, wsd, gate, act, act_s, out, T, D, F, Fs, top, kind, onto, stream);
    else return qwb_fail(QWB_ERR_ARG, "moe_experts: unknown dtype %d", dtype);
    return qwb_check_launch("moe_experts");
}

// ---------------------------------------------------------------------------------
// Around a grouped product over token copies sorted by expert (bfloat16; D and F multiples of 8):
//   moe_sort      place[c] = the row of copy c = t * top + k in the order (expert, copy); ends[e] = where expert e's run ends
//   moe_spread    xs[place[t, k], :] = x[t, :], and row_weight[place[t, k]] = weight[t, k] where the weights are on the inputs
//   moe_act       act[s, f] = f(u[s, f]), u [S, F], or silu(u[s, f]) * u[s, F + f], u [S, 2F]; u times row_weight[s] if given
//   moe_combine   out[t, :] (+)= sum_k weight[t, k] * y[place[t, k], :] + gate[t] * shared[t, :]
// ---------------------------------------------------------------------------------
// A block per expert: it counts the copies of lower experts (where its own run starts) and ranks its own ones.  Each warp
// walks over a run of neighbouring copies twice, 32 at a time (a ballot finds the ranks): once for its counts, then, knowing
// what the warps before it counted, to write the places.  Nothing depends on the order in which warps or blocks run.
#define MOE_SORT_WARPS 16
#define MOE_SORT_AHEAD 8          // groups of 32 whose loads are on their way together
__global__ void __launch_bounds__(MOE_SORT_WARPS * 32)
moe_sort_kernel(const int* __restrict__ chosen, int* __restrict__ place, int* __restrict__ ends, int S, int E) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ int own[MOE_SORT_WARPS], lower[MOE_SORT_WARPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, expert = blockIdx.x;
    const unsigned full = 0xffffffffu, before = (1u << lane) - 1u;
    const int per = ((S + MOE_SORT_WARPS - 1) / MOE_SORT_WARPS + 31) & ~31;
    const int lo = min(S, warp * per), hi = min(S, lo + per);
    auto expert_of = [&](int i) { return i < hi ? min(max(chosen[i], 0), E - 1) : E; };        // E: not a copy
    int n_own = 0, n_lower = 0;
    for (int i0 = lo; i0 < hi; i0 += 32 * MOE_SORT_AHEAD) {
        int es[MOE_SORT_AHEAD];
#pragma unroll
        for (int a = 0; a < MOE_SORT_AHEAD; ++a) es[a] = expert_of(i0 + 32 * a + lane);
#pragma unroll
        for (int a = 0; a < MOE_SORT_AHEAD; ++a) {
            n_own += __popc(__ballot_sync(full, es[a] == expert));
            n_lower += __popc(__ballot_sync(full, es[a] < expert));
        }
    }
    if (lane == 0) { own[warp] = n_own; lower[warp] = n_lower; }
    __syncthreads();
    int at = 0, total = 0;                              // the next row of this warp's copies; where the run ends
    for (int w = 0; w < MOE_SORT_WARPS; ++w) {
        at += lower[w] + (w < warp ? own[w] : 0);
        total += lower[w] + own[w];
    }
    if (threadIdx.x == 0) ends[expert] = total;
    for (int i0 = lo; i0 < hi && n_own > 0; i0 += 32 * MOE_SORT_AHEAD) {
        int es[MOE_SORT_AHEAD];
#pragma unroll
        for (int a = 0; a < MOE_SORT_AHEAD; ++a) es[a] = expert_of(i0 + 32 * a + lane);
#pragma unroll
        for (int a = 0; a < MOE_SORT_AHEAD; ++a) {
            const unsigned mine = __ballot_sync(full, es[a] == expert);
            if (es[a] == expert) place[i0 + 32 * a + lane] = at + __popc(mine & before);
            at += __popc(mine);
        }
    }
}

extern "C" int qwb_moe_sort(const int* chosen, int* place, int* ends, int S, int E, cudaStream_t stream) {
    if (S <= 0) return 0;
    if (E <= 0 || E > QWB_MOE_MAX_EXPERTS) return qwb_fail(QWB_ERR_ARG, "moe_sort: %d experts (at most %d)", E, QWB_MOE_MAX_EXPERTS);
    qwb_launch(moe_sort_kernel, E, MOE_SORT_WARPS * 32, 0, stream, chosen, place, ends, S, E);
    return qwb_check_launch("moe_sort");
}

__global__ void moe_spread_kernel(const uint4* __restrict__ x, const int* __restrict__ place, uint4* __restrict__ xs, const float* __restrict__ weight,
                                  float* __restrict__ row_weight, int pieces, int top) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    if (row_weight && (int)threadIdx.x < top) row_weight[place[(size_t)t * top + threadIdx.x]] = weight[(size_t)t * top + threadIdx.x];
    for (int i = threadIdx.x; i < pieces; i += blockDim.x) {
        const uint4 v = x[(size_t)t * pieces + i];
        for (int k = 0; k < top; ++k) xs[(size_t)place[(size_t)t * top + k] * pieces + i] = v;
    }
}

// weight [T, top] and row_weight [T * top], or both null
extern "C" int qwb_moe_spread(const void* x, const int* place, void* xs, const float* weight, float* row_weight, int T, int D, int top,
                              cudaStream_t stream) {
    if (T <= 0 || D <= 0) return 0;
    if (D % 8) return qwb_fail(QWB_ERR_ARG, "moe_spread: rows of %d values", D);
    qwb_launch(moe_spread_kernel, T, D >= 2048 ? 256 : 128, 0, stream, (const uint4*)x, place, (uint4*)xs, weight, row_weight, D / 8, top);
    return qwb_check_launch("moe_spread");
}

__device__ __forceinline__ uint4 pack_bf16x8(const float* v) {
    uint4 o;
    uint32_t* w = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 p = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        w[i] = *reinterpret_cast<const uint32_t*>(&p);
    }
    return o;
}

// 8 values a thread and step, whatever row they are in; KIND: the activation code
template <int KIND>
__global__ void moe_act_kernel(const Vec16<bf16>* __restrict__ u, const float* __restrict__ row_weight, uint4* __restrict__ act, unsigned n, unsigned pieces) {
    pdl_wait();
    pdl_launch_dependents();
    for (unsigned i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
        float a[8], b[8];
        const float w = row_weight ? row_weight[i / pieces] : 1.f;
        if (KIND == QWB_MOE_GATED) {
            const size_t gate = i + (size_t)(i / pieces) * pieces;          // row s: its gate pieces, then its up pieces
            u[gate].get(a);
            u[gate + pieces].get(b);
#pragma unroll
            for (int e = 0; e < 8; ++e) { const float g = a[e] * w; a[e] = g / (1.f + expf(-g)) * (b[e] * w); }
        } else {
            u[i].get(a);
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] = qwb_activate(a[e] * w, KIND);
        }
        act[i] = pack_bf16x8(a);
    }
}

// row_weight [S] or null
extern "C" int qwb_moe_act(const void* u, const float* row_weight, void* act, int S, int F, int kind, cudaStream_t stream) {
    if (S <= 0 || F <= 0) return 0;
    if (F % 8) return qwb_fail(QWB_ERR_ARG, "moe_act: rows of %d values", F);
    const long long n = (long long)S * (F / 8);
    if (n >= 1LL << 31) return qwb_fail(QWB_ERR_ARG, "moe_act: %d rows of %d values are too many for one launch", S, F);
    const int grid = (int)((n + 255) / 256 < 148 * 32 ? (n + 255) / 256 : 148 * 32);
#define QWB_MOE_ACT(KIND) \
    case KIND: qwb_launch(moe_act_kernel<KIND>, grid, 256, 0, stream, (const Vec16<bf16>*)u, row_weight, (uint4*)act, (unsigned)n, (unsigned)(F / 8)); break
    switch (kind) {
        QWB_MOE_ACT(0); QWB_MOE_ACT(1); QWB_MOE_ACT(2); QWB_MOE_ACT(3); QWB_MOE_ACT(5); QWB_MOE_ACT(QWB_MOE_GATED);
        default: return qwb_fail(QWB_ERR_ARG, "moe_act: unknown activation %d", kind);
    }
#undef QWB_MOE_ACT
    return qwb_check_launch("moe_act");
}

__global__ void moe_combine_kernel(const Vec16<bf16>* __restrict__ y, const int* __restrict__ place, const float* __restrict__ weight,
                                   const float* __restrict__ shared, const float* __restrict__ gate, float* out, int pieces, int top,
                                   int onto) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const float g = gate ? gate[t] : 1.f;
    for (int i = threadIdx.x; i < pieces; i += blockDim.x) {
        float total[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) total[e] = 0.f;
#pragma unroll 4
        for (int k = 0; k < top; ++k) {
            float v[8];
            y[(size_t)place[(size_t)t * top + k] * pieces + i].get(v);
            const float w = weight ? weight[(size_t)t * top + k] : 1.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) total[e] += w * v[e];
        }
        float4* o = reinterpret_cast<float4*>(out) + ((size_t)t * pieces + i) * 2;
        const float4* sh = reinterpret_cast<const float4*>(shared) + ((size_t)t * pieces + i) * 2;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            float4 r = make_float4(total[4 * j], total[4 * j + 1], total[4 * j + 2], total[4 * j + 3]);
            if (shared) { const float4 s = sh[j]; r.x += g * s.x; r.y += g * s.y; r.z += g * s.z; r.w += g * s.w; }
            if (onto) { const float4 s = o[j]; r.x += s.x; r.y += s.y; r.z += s.z; r.w += s.w; }
            o[j] = r;
        }
    }
}

// y [S, D] bfloat16; weight [T, top] (or null: 1); shared [T, D] float (or null) and gate [T] (or null: 1)
extern "C" int qwb_moe_combine(const void* y, const int* place, const float* weight, const float* shared, const float* gate, float* out,
                               int T, int D, int top, int onto, cudaStream_t stream) {
    if (T <= 0 || D <= 0) return 0;
    if (D % 8) return qwb_fail(QWB_ERR_ARG, "moe_combine: rows of %d values", D);
    qwb_launch(moe_combine_kernel, T, D >= 2048 ? 256 : 128, 0, stream, (const Vec16<bf16>*)y, place, weight, shared, gate, out, D / 8, top, onto);
    return qwb_check_launch("moe_combine");
}
