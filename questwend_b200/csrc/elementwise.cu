// Embedding gather, RMS norm (with the residual sum folded in) and the gated SiLU
// product.  The residual stream and the sums of squares are 32-bit in both engines.
#include "common.cuh"

// ---------------------------------------------------------------------------------
// h[t,:] = float(E[id_t,:]) * scale (+ float(P[p_t,:]), p_t the token's position).  A row gather (the reference, which
// neither scales nor adds: core/runtime.cpp:1001, ggml-cuda/getrows.cu:73-102).  An id outside [0, V) writes a row of
// zeros and records the first such token in *bad_token (if given); a position outside [0, NP) adds nothing.
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void embed_gather_kernel(const int* __restrict__ ids, const T* __restrict__ table, const int* __restrict__ pos,
                                    const T* __restrict__ pos_table, float* __restrict__ out, int D, int V, int NP,
                                    int* bad_token, float scale) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int id = ids[t];
    float* o = out + (size_t)t * D;
    if (id < 0 || id >= V) {
        if (bad_token && threadIdx.x == 0) atomicCAS(bad_token, -1, t);
        for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = 0.f;
        return;
    }
    const T* row = table + (size_t)id * D;
    const int p = pos_table ? pos[t] : -1;
    const T* prow = p >= 0 && p < NP ? pos_table + (size_t)p * D : nullptr;
    constexpr int VEC = Vec16<T>::N;
    if (D % VEC == 0 && (uintptr_t)table % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)pos_table % 16 == 0) {
        const Vec16<T>* src = reinterpret_cast<const Vec16<T>*>(row);                  // 16 bytes of the row a load
        const Vec16<T>* psrc = reinterpret_cast<const Vec16<T>*>(prow);
        for (int i = threadIdx.x; i < D / VEC; i += blockDim.x) {
            float v[VEC], w[VEC];
            src[i].get(v);
            if (prow) psrc[i].get(w);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = v[e] * scale + (prow ? w[e] : 0.f);
#pragma unroll
            for (int e = 0; e < VEC; e += 4)
                *reinterpret_cast<float4*>(o + (size_t)i * VEC + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
        }
        return;
    }
    for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = to_f32(row[i]) * scale + (prow ? to_f32(prow[i]) : 0.f);
}

extern "C" int qwb_embed_gather(const int* ids, const void* table, int table_dtype, const int* pos, const void* pos_table, float* out,
                                int T, int D, int V, int NP, int* bad_token, float scale, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0 || V <= 0) return qwb_fail(QWB_ERR_ARG, "embed_gather: bad sizes D=%d V=%d", D, V);
    if (pos_table && (!pos || NP <= 0)) return qwb_fail(QWB_ERR_ARG, "embed_gather: a position table of %d rows without positions", NP);
    const int block = D >= 1024 ? 256 : 128;
    if (table_dtype == QWB_DT_F32)
        qwb_launch(embed_gather_kernel<float>, T, block, 0, stream, ids, (const float*)table, pos, (const float*)pos_table, out, D, V, NP, bad_token, scale);
    else if (table_dtype == QWB_DT_BF16)
        qwb_launch(embed_gather_kernel<bf16>, T, block, 0, stream, ids, (const bf16*)table, pos, (const bf16*)pos_table, out, D, V, NP, bad_token, scale);
    else
        return qwb_fail(QWB_ERR_ARG, "embed_gather: unknown dtype %d", table_dtype);
    return qwb_check_launch("embed_gather");
}

// ---------------------------------------------------------------------------------
// h[t,:] += float(E[id_t,:]) * scale + vec[:], in place on the 32-bit stream: what a pass of a looped run of layers adds
// before its first layer (the tokens' embeddings once more and a vector of the pass).  table or vec may be null.
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void embed_add_kernel(const int* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ vec,
                                 float* h, int D, int V, float scale) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int id = table ? ids[t] : 0;
    const bool row_ok = table && id >= 0 && id < V;
    const T* row = table + (size_t)(row_ok ? id : 0) * D;
    float* o = h + (size_t)t * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = o[i];
        if (row_ok) v += to_f32(row[i]) * scale;
        if (vec) v += vec[i];
        o[i] = v;
    }
}

extern "C" int qwb_embed_add(const int* ids, const void* table, int table_dtype, const float* vec, float* h, int T, int D, int V,
                             float scale, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0 || (table && (V <= 0 || !ids))) return qwb_fail(QWB_ERR_ARG, "embed_add: bad sizes D=%d V=%d", D, V);
    if (!table && !vec) return 0;
    const int block = D >= 1024 ? 256 : 128;
    if (table_dtype == QWB_DT_F32)
        qwb_launch(embed_add_kernel<float>, T, block, 0, stream, ids, (const float*)table, vec, h, D, V, scale);
    else if (table_dtype == QWB_DT_BF16)
        qwb_launch(embed_add_kernel<bf16>, T, block, 0, stream, ids, (const bf16*)table, vec, h, D, V, scale);
    else
        return qwb_fail(QWB_ERR_ARG, "embed_add: unknown dtype %d", table_dtype);
    return qwb_check_launch("embed_add");
}

// ---------------------------------------------------------------------------------
// RMS norm over rows of D:  y = v * rsqrt(mean(v^2) + eps) * w,  v = x (+ delta).
// (the reference: core/runtime.cpp:1018-1019, ggml-cuda/norm.cu:76-155.)
//   x      [rows_in, D] float   the residual stream
//   delta  [rows_in, D] float   optional: the sum x + delta_scale * delta is formed in 32-bit first
//   planes [P, rows_in, D] float optional, instead of delta: a product that its kernel left as sums over pieces of k
//                                (gemm_ring's split form); columns 16 t .. 16 t + 15 have plane_count[t] <= 4 planes, which
//                                are added onto x in the order of the planes
//   sum_out[rows_in, D] float   optional: where x + delta is written (may be x itself)
//   rows   [n_rows] int         optional: row r of the output is made from row rows[r]
//   out    [n_rows, D]  float or bfloat16
// One block per output row; the row is kept in shared memory between the two passes.
// ---------------------------------------------------------------------------------
template <typename TOut> struct Pack4;
template <> struct Pack4<float> {
    static __device__ __forceinline__ void store(float* p, float a, float b, float c, float d) {
        *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
    }
};
template <> struct Pack4<bf16> {
    static __device__ __forceinline__ void store(bf16* p, float a, float b, float c, float d) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
        uint2 v;
        v.x = *reinterpret_cast<uint32_t*>(&lo);
        v.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = v;
    }
};

// VEC: rows are a multiple of 4 wide and 16-byte aligned, so everything moves four values at a time.
#define RMS_MAX_PLANES 4
#define RMS_W_FIRST 4             // pieces of the weight a thread asks for before the wait (rows of up to 4,096: all of it)
#define RMS_PLANE_COLS 16
template <typename TOut, bool VEC>
__global__ void rmsnorm_kernel(const float* x, const float* delta, const float* planes,
                               const unsigned char* __restrict__ plane_count, size_t plane_stride,
                               float* sum_out, const float* __restrict__ w, TOut* __restrict__ out,
                               const int* __restrict__ rows, int D, float eps, float delta_scale) {
    pdl_launch_dependents();            // the trigger first: the kernel after this one may start before the one before it ends
    // the norm's weight is nobody's output: a thread's first pieces of it are on their way before the wait
    float4 w_first[RMS_W_FIRST];
    if (VEC) {
#pragma unroll
        for (int k = 0; k < RMS_W_FIRST; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            w_first[k] = i < D / 4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    pdl_wait();
    extern __shared__ __align__(16) float row_cache[];
    __shared__ float red[32];
    const int r = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[r] : r) * D;
    float ss = 0.f;
    if (VEC) {
        const float4* x4 = reinterpret_cast<const float4*>(x + src);
        const float4* d4 = delta ? reinterpret_cast<const float4*>(delta + src) : nullptr;
        float4* s4 = sum_out ? reinterpret_cast<float4*>(sum_out + src) : nullptr;
        float4* c4 = reinterpret_cast<float4*>(row_cache);
        for (int i = threadIdx.x; i < D / 4; i += blockDim.x) {
            // plain loads (x and delta are not __restrict__: never the read-only path, see pdl_wait); with __ldcg a norm
            // of 8 rows of 4,096 took 1.4 us longer under the ring fill of the product that follows (and with a thread's four
            // loads issued together, before the first store, a step took 0.5 % longer)
            float4 v = x4[i];
            if (d4) { const float4 d = d4[i]; v.x += delta_scale * d.x; v.y += delta_scale * d.y; v.z += delta_scale * d.z; v.w += delta_scale * d.w; }
            if (planes) {
                const int n_planes = plane_count[4 * i / RMS_PLANE_COLS];
                const float4* p4 = reinterpret_cast<const float4*>(planes + src) + i;
                float4 d[RMS_MAX_PLANES];
#pragma unroll
                for (int p = 0; p < RMS_MAX_PLANES; ++p)
                    if (p < n_planes) d[p] = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p4) + p * plane_stride);
#pragma unroll
                for (int p = 0; p < RMS_MAX_PLANES; ++p)
                    if (p < n_planes) { v.x += d[p].x; v.y += d[p].y; v.z += d[p].z; v.w += d[p].w; }
            }
            if (s4) s4[i] = v;
            c4[i] = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            float v = x[src + i];
            if (delta) v += delta_scale * delta[src + i];
            if (planes)
                for (int p = 0, n_planes = plane_count[i / RMS_PLANE_COLS]; p < n_planes; ++p) v += planes[p * plane_stride + src + i];
            if (sum_out) sum_out[src + i] = v;
            row_cache[i] = v;
            ss += v * v;
        }
    }
    const float total = block_sum(ss, red);
    const float scale = rsqrtf(total / (float)D + eps);
    TOut* o = out + (size_t)r * D;
    if (VEC) {
        const float4* c4 = reinterpret_cast<const float4*>(row_cache);
        const float4* w4 = reinterpret_cast<const float4*>(w);
#pragma unroll
        for (int k = 0; k < RMS_W_FIRST; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            if (i < D / 4) {
                const float4 v = c4[i], g = w_first[k];
                Pack4<TOut>::store(o + 4 * i, v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w);
            }
        }
        for (int i = threadIdx.x + RMS_W_FIRST * blockDim.x; i < D / 4; i += blockDim.x) {
            const float4 v = c4[i], g = w4[i];
            Pack4<TOut>::store(o + 4 * i, v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w);
        }
    } else {
        for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = from_f32<TOut>(row_cache[i] * scale * w[i]);
    }
}

// Rows of up to 4 x ITERS x 256 values (ITERS 4 or 8: up to 4,096 or 8,192): the row stays in the threads' registers
// between the two passes (a thread's loads are issued together; 2,048 rows of 4,096: 8.6 us against 11.8 through shared
// memory; a decode step of 8 rows 0.5 % faster).
template <typename TOut, int ITERS>
__global__ void __launch_bounds__(256)
rmsnorm_rows_kernel(const float* x, const float* delta, const float* planes, const unsigned char* __restrict__ plane_count,
                    size_t plane_stride, float* sum_out, const float* __restrict__ w, TOut* __restrict__ out,
                    const int* __restrict__ rows, int D, float eps, float delta_scale) {
    pdl_launch_dependents();            // the trigger first, and the weight asked for before the wait: as in rmsnorm_kernel
    float4 g[ITERS];
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        g[k] = i < D / 4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    __shared__ float red[32];
    const int r = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[r] : r) * D;
    const float4* x4 = reinterpret_cast<const float4*>(x + src);
    const float4* d4 = delta ? reinterpret_cast<const float4*>(delta + src) : nullptr;
    float4 v[ITERS];
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        v[k] = i < D / 4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (d4) {
#pragma unroll
        for (int k = 0; k < ITERS; ++k) {
            const int i = threadIdx.x + k * 256;
            if (i < D / 4) { const float4 d = d4[i]; v[k].x += delta_scale * d.x; v[k].y += delta_scale * d.y; v[k].z += delta_scale * d.z; v[k].w += delta_scale * d.w; }
        }
    }
    if (planes) {                       // a product left as sums over pieces of k: a column's planes, in their order
#pragma unroll
        for (int k = 0; k < ITERS; ++k) {
            const int i = threadIdx.x + k * 256;
            if (i < D / 4) {
                const int n_planes = plane_count[4 * i / RMS_PLANE_COLS];
                const float* p4 = planes + src + 4 * (size_t)i;
                float4 pv[RMS_MAX_PLANES];
#pragma unroll
                for (int p = 0; p < RMS_MAX_PLANES; ++p)
                    if (p < n_planes) pv[p] = *reinterpret_cast<const float4*>(p4 + p * plane_stride);
#pragma unroll
                for (int p = 0; p < RMS_MAX_PLANES; ++p)
                    if (p < n_planes) { v[k].x += pv[p].x; v[k].y += pv[p].y; v[k].z += pv[p].z; v[k].w += pv[p].w; }
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        if (sum_out && i < D / 4) reinterpret_cast<float4*>(sum_out + src)[i] = v[k];
        ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    const float scale = rsqrtf(block_sum(ss, red) / (float)D + eps);
    TOut* o = out + (size_t)r * D;
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < D / 4)
            Pack4<TOut>::store(o + 4 * i, v[k].x * scale * g[k].x, v[k].y * scale * g[k].y, v[k].z * scale * g[k].z, v[k].w * scale * g[k].w);
    }
}

template <typename TOut>
static int launch_rmsnorm(const float* x, const float* delta, const float* planes, const unsigned char* plane_count,
                          size_t plane_stride, float* sum_out, const float* w, TOut* out, const int* rows,
                          int n_rows, int D, float eps, float delta_scale, size_t smem, cudaStream_t stream) {
    const bool vec = D % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                     (!delta || (uintptr_t)delta % 16 == 0) && (!sum_out || (uintptr_t)sum_out % 16 == 0) &&
                     (!planes || ((uintptr_t)planes % 16 == 0 && plane_stride % 4 == 0));
    const int work = vec ? D / 4 : D;
    const int block = work >= 1024 ? 256 : (work >= 256 ? 128 : 64);
    cudaError_t e = cudaSuccess;
    if (vec && D / 4 <= 4 * 256) {
        qwb_launch_link(n_rows, QWB_LINK_ROWS_NORM, rmsnorm_rows_kernel<TOut, 4>, n_rows, 256, 0, stream, x, delta, planes, plane_count, plane_stride, sum_out, w, out, rows, D, eps, delta_scale);
    } else if (vec && D / 4 <= 8 * 256) {
        qwb_launch_link(n_rows, QWB_LINK_ROWS_NORM, rmsnorm_rows_kernel<TOut, 8>, n_rows, 256, 0, stream, x, delta, planes, plane_count, plane_stride, sum_out, w, out, rows, D, eps, delta_scale);
    } else if (vec) {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_kernel<TOut, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm: %s", cudaGetErrorString(e));
        qwb_launch_link(n_rows, QWB_LINK_ROWS_NORM, rmsnorm_kernel<TOut, true>, n_rows, block, smem, stream, x, delta, planes, plane_count, plane_stride, sum_out, w, out, rows, D, eps, delta_scale);
    } else {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_kernel<TOut, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm: %s", cudaGetErrorString(e));
        qwb_launch(rmsnorm_kernel<TOut, false>, n_rows, block, smem, stream, x, delta, planes, plane_count, plane_stride, sum_out, w, out, rows, D, eps, delta_scale);
    }
    return qwb_check_launch("rmsnorm");
}

static int rmsnorm_any(const float* x, const float* delta, const float* planes, const unsigned char* plane_count,
                       size_t plane_stride, float* sum_out, const float* w, void* out, int out_dtype, const int* rows,
                       int n_rows, int D, float eps, float delta_scale, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (D <= 0) return qwb_fail(QWB_ERR_ARG, "rmsnorm: bad width %d", D);
    const size_t smem = (size_t)D * sizeof(float);
    if (smem > 200 * 1024) return qwb_fail(QWB_ERR_ARG, "rmsnorm: width %d does not fit in shared memory (max %d)", D, 200 * 1024 / 4);
    if (out_dtype == QWB_DT_F32)
        return launch_rmsnorm<float>(x, delta, planes, plane_count, plane_stride, sum_out, w, (float*)out, rows, n_rows, D, eps, delta_scale, smem, stream);
    if (out_dtype == QWB_DT_BF16)
        return launch_rmsnorm<bf16>(x, delta, planes, plane_count, plane_stride, sum_out, w, (bf16*)out, rows, n_rows, D, eps, delta_scale, smem, stream);
    return qwb_fail(QWB_ERR_ARG, "rmsnorm: unknown dtype %d", out_dtype);
}

extern "C" int qwb_rmsnorm(const float* x, const float* delta, float* sum_out, const float* w,
                           void* out, int out_dtype, const int* rows, int n_rows, int D, float eps, float delta_scale,
                           cudaStream_t stream) {
    return rmsnorm_any(x, delta, nullptr, nullptr, 0, sum_out, w, out, out_dtype, rows, n_rows, D, eps, delta_scale, stream);
}

// The same with a product in planes instead of delta: planes [n_planes, rows_in, D], plane_count [ceil(D / 16)] bytes.
extern "C" int qwb_rmsnorm_planes(const float* x, const float* planes, const unsigned char* plane_count, int n_planes,
                                  int rows_in, float* sum_out, const float* w, void* out, int out_dtype, const int* rows,
                                  int n_rows, int D, float eps, cudaStream_t stream) {
    if (n_planes < 1 || n_planes > RMS_MAX_PLANES)
        return qwb_fail(QWB_ERR_ARG, "rmsnorm: %d planes; this kernel adds up to %d", n_planes, RMS_MAX_PLANES);
    return rmsnorm_any(x, nullptr, planes, plane_count, (size_t)rows_in * D, sum_out, w, out, out_dtype, rows, n_rows, D, eps, 1.f, stream);
}

// x[t, :] += the planes of a product (as above), for a consumer that is not this norm.
__global__ void add_planes_kernel(float* x, const float* planes, const unsigned char* __restrict__ plane_count,
                                  size_t plane_stride, size_t n, int D) {
    pdl_wait();
    pdl_launch_dependents();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        float v = x[i];
        for (int p = 0, n_planes = plane_count[(i % D) / RMS_PLANE_COLS]; p < n_planes; ++p) v += planes[p * plane_stride + i];
        x[i] = v;
    }
}

extern "C" int qwb_add_planes(float* x, const float* planes, const unsigned char* plane_count, int T, int D, cudaStream_t stream) {
    if (T <= 0 || D <= 0) return 0;
    const size_t n = (size_t)T * D;
    const int block = 256, grid = (int)((n + block - 1) / block < 1184 ? (n + block - 1) / block : 1184);
    qwb_launch(add_planes_kernel, grid, block, 0, stream, x, planes, plane_count, n, n, D);
    return qwb_check_launch("add_planes");
}

// ---------------------------------------------------------------------------------
// a[t,f] = silu(g[t,f]) * u[t,f], silu(x) = x / (1 + exp(-x)), from one [T, 2F] float
// matrix (the reference: core/runtime.cpp:1074-1076, ggml-cuda/unary.cuh:96-98).
// interleave 0: the first F columns are the gate and the last F the up projection;
// interleave G > 0 (F a multiple of G): for every G features, their G gates and then their G ups.
// ---------------------------------------------------------------------------------
// act 0: silu(g) * u; 1: gelu(g) * u (tanh form); 2: both clamped first, g <- min(g, limit) and u <- clamp(u, -limit, limit),
// then g * sigmoid(1.702 g) * (u + 1)
__device__ __forceinline__ float gate_mul(float g, float u, int act, float limit) {
    if (act == 2) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
    }
    return (act == 1 ? 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) : g / (1.f + expf(-g))) * u;
}

template <typename TOut>
__global__ void silu_mul_kernel(const float* __restrict__ gu, TOut* __restrict__ out, int T, int F, int interleave, int act, float limit) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t n = (size_t)T * F;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / F, f = i - t * F;
        const size_t gate_at = interleave > 0 ? (f / interleave) * 2 * interleave + f % interleave : f;
        const float g = gu[t * 2 * F + gate_at];
        const float u = gu[t * 2 * F + gate_at + (interleave > 0 ? interleave : F)];
        out[i] = from_f32<TOut>(gate_mul(g, u, act, limit));
    }
}

// The same for gates and ups interleaved in eights (the layout that the products with a fused epilogue want): a thread
// takes 8 features: 64 bytes of gates and ups in four 16-byte loads, one store of 8 values.  64 rows of 12,288 features:
// 3.2 us against 5.5 with a value a thread.
template <typename TOut>
__global__ void silu_mul_eights_kernel(const float* __restrict__ gu, TOut* __restrict__ out, int T, int F, int act, float limit) {
    pdl_wait();
    pdl_launch_dependents();
    const int groups = F >> 3;
    const size_t n = (size_t)T * groups;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / groups, grp = i - t * groups;
        const float4* src = reinterpret_cast<const float4*>(gu + (t * 2 * F + grp * 16));
        const float4 g0 = src[0], g1 = src[1], u0 = src[2], u1 = src[3];
        TOut* dst = out + t * F + grp * 8;
        Pack4<TOut>::store(dst, gate_mul(g0.x, u0.x, act, limit), gate_mul(g0.y, u0.y, act, limit), gate_mul(g0.z, u0.z, act, limit), gate_mul(g0.w, u0.w, act, limit));
        Pack4<TOut>::store(dst + 4, gate_mul(g1.x, u1.x, act, limit), gate_mul(g1.y, u1.y, act, limit), gate_mul(g1.z, u1.z, act, limit), gate_mul(g1.w, u1.w, act, limit));
    }
}

extern "C" int qwb_silu_mul(const float* gate_up, void* out, int out_dtype, int T, int F, int interleave, int act, float limit, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (act < 0 || act > 2) return qwb_fail(QWB_ERR_ARG, "silu_mul: unknown gate activation %d", act);
    if (act == 2 && !(limit > 0.f)) return qwb_fail(QWB_ERR_ARG, "silu_mul: the clamped gate needs a positive limit, got %g", (double)limit);
    if (F <= 0) return qwb_fail(QWB_ERR_ARG, "silu_mul: bad width %d", F);
    if (interleave < 0 || (interleave > 0 && F % interleave))
        return qwb_fail(QWB_ERR_ARG, "silu_mul: %d features cannot be interleaved in groups of %d", F, interleave);
    const size_t n = (size_t)T * F;
    const int block = 256;
    if (interleave == 8 && F % 8 == 0 && (uintptr_t)gate_up % 16 == 0 && (uintptr_t)out % 16 == 0 &&
        (out_dtype == QWB_DT_F32 || out_dtype == QWB_DT_BF16)) {
        const size_t groups = n / 8;
        const int g8 = (int)((groups + block - 1) / block < 148 * 16 ? (groups + block - 1) / block : 148 * 16);
        if (out_dtype == QWB_DT_F32) qwb_launch(silu_mul_eights_kernel<float>, g8, block, 0, stream, gate_up, (float*)out, T, F, act, limit);
        else qwb_launch(silu_mul_eights_kernel<bf16>, g8, block, 0, stream, gate_up, (bf16*)out, T, F, act, limit);
        return qwb_check_launch("silu_mul");
    }
    const int grid = (int)((n + block - 1) / block < 148 * 16 ? (n + block - 1) / block : 148 * 16);
    if (out_dtype == QWB_DT_F32)
        qwb_launch(silu_mul_kernel<float>, grid, block, 0, stream, gate_up, (float*)out, T, F, interleave, act, limit);
    else if (out_dtype == QWB_DT_BF16)
        qwb_launch(silu_mul_kernel<bf16>, grid, block, 0, stream, gate_up, (bf16*)out, T, F, interleave, act, limit);
    else
        return qwb_fail(QWB_ERR_ARG, "silu_mul: unknown dtype %d", out_dtype);
    return qwb_check_launch("silu_mul");
}

// out[i] += scale * delta[i]: the residual sum on its own, for blocks that end without a norm.
__global__ void add_inplace_kernel(float* __restrict__ out, const float* __restrict__ delta, size_t n, float scale) {
    pdl_wait();
    pdl_launch_dependents();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        out[i] += scale * delta[i];
}

extern "C" int qwb_add_inplace(float* out, const float* delta, long long n, float scale, cudaStream_t stream) {
    if (n <= 0) return 0;
    const int block = 256;
    const long long want = (n + block - 1) / block;
    const int grid = (int)(want < 148 * 16 ? want : 148 * 16);
    qwb_launch(add_inplace_kernel, grid, block, 0, stream, out, delta, (size_t)n, scale);
    return qwb_check_launch("add_inplace");
}

// After a decode step that sampled on the device: the sampled token becomes the next
// step's input, every sequence is one token longer, the step counter goes up, and the
// token enters the sequence's penalty window (a ring of `window` ids).
__global__ void decode_advance_kernel(const int* __restrict__ sampled, int* token_ids, int* tok_pos, int* pos0,
                                      int* seq_len, unsigned int* step_counter, int* recent, int* n_seen,
                                      int window, int B) {
    pdl_wait();
    pdl_launch_dependents();
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b == 0 && step_counter) *step_counter += 1;
    if (b >= B) return;
    const int tok = sampled[b];
    token_ids[b] = tok;
    tok_pos[b] += 1;
    pos0[b] += 1;
    seq_len[b] += 1;
    if (recent && window > 0) {
        recent[(size_t)b * window + (n_seen[b] % window)] = tok;
        n_seen[b] += 1;
    }
}

extern "C" int qwb_decode_advance(const int* sampled, int* token_ids, int* tok_pos, int* pos0, int* seq_len,
                                  unsigned int* step_counter, int* recent, int* n_seen, int window, int B,
                                  cudaStream_t stream) {
    if (B <= 0) return 0;
    qwb_launch(decode_advance_kernel, (B + 127) / 128, 128, 0, stream, sampled, token_ids, tok_pos, pos0, seq_len,
                                                               step_counter, recent, n_seen, window, B);
    return qwb_check_launch("decode_advance");
}

// ---------------------------------------------------------------------------------
// The norm on a sublayer's OUTPUT:  h[t, :] += y[t, :] * rsqrt(mean(y[t, :]^2) + eps) * w, in 32-bit and in place,
// for blocks whose sublayers read the stream itself and whose results are normed before they join it.  `cast`
// (optional, float or bfloat16) receives the new h in the dtype of the next product's operands.  One block per row;
// the row of y stays in shared memory between the two passes.
// ---------------------------------------------------------------------------------
template <typename TOut>
__global__ void rmsnorm_onto_kernel(const float* __restrict__ y, const float* __restrict__ w, float* h, TOut* __restrict__ cast,
                                    int D, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float row_cache[];
    __shared__ float red[32];
    const size_t at = (size_t)blockIdx.x * D;
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = y[at + i];
        row_cache[i] = v;
        ss += v * v;
    }
    const float scale = rsqrtf(block_sum(ss, red) / (float)D + eps);
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = h[at + i] + row_cache[i] * scale * w[i];
        h[at + i] = v;
        if (cast) cast[at + i] = from_f32<TOut>(v);
    }
}

// The same for rows of up to 4 x ITERS x 256 values that are whole 16-byte pieces: the row of y stays in registers and a
// thread's loads are issued together (a step of one token is one block: its two passes are what it takes).
template <typename TOut, int ITERS>
__global__ void __launch_bounds__(256)
rmsnorm_onto_rows_kernel(const float* __restrict__ y, const float* __restrict__ w, float* h, TOut* __restrict__ cast, int D, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[32];
    const size_t at = (size_t)blockIdx.x * D;
    const float4* y4 = reinterpret_cast<const float4*>(y + at);
    float4* h4 = reinterpret_cast<float4*>(h + at);
    float4 v[ITERS], g[ITERS], r[ITERS];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        const bool in = i < D / 4;
        v[k] = in ? y4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        g[k] = in ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        r[k] = in ? h4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    const float scale = rsqrtf(block_sum(ss, red) / (float)D + eps);
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < D / 4) {
            const float4 o = make_float4(r[k].x + v[k].x * scale * g[k].x, r[k].y + v[k].y * scale * g[k].y,
                                         r[k].z + v[k].z * scale * g[k].z, r[k].w + v[k].w * scale * g[k].w);
            h4[i] = o;
            if (cast) Pack4<TOut>::store(cast + at + 4 * (size_t)i, o.x, o.y, o.z, o.w);
        }
    }
}

extern "C" int qwb_rmsnorm_onto(const float* y, const float* w, float* h, void* cast, int cast_dtype, int T, int D, float eps,
                                cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0) return qwb_fail(QWB_ERR_ARG, "rmsnorm_onto: bad width %d", D);
    if (cast && cast_dtype != QWB_DT_BF16 && cast_dtype != QWB_DT_F32) return qwb_fail(QWB_ERR_ARG, "rmsnorm_onto: unknown dtype %d", cast_dtype);
    const bool to_bf16 = cast && cast_dtype == QWB_DT_BF16;
    const bool vec = D % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)h % 16 == 0 && (!cast || (uintptr_t)cast % 16 == 0);
    if (vec && D / 4 <= 4 * 256) {
        if (D / 4 <= 2 * 256) {
            if (to_bf16) qwb_launch(rmsnorm_onto_rows_kernel<bf16, 2>, T, 256, 0, stream, y, w, h, (bf16*)cast, D, eps);
            else qwb_launch(rmsnorm_onto_rows_kernel<float, 2>, T, 256, 0, stream, y, w, h, (float*)cast, D, eps);
        } else {
            if (to_bf16) qwb_launch(rmsnorm_onto_rows_kernel<bf16, 4>, T, 256, 0, stream, y, w, h, (bf16*)cast, D, eps);
            else qwb_launch(rmsnorm_onto_rows_kernel<float, 4>, T, 256, 0, stream, y, w, h, (float*)cast, D, eps);
        }
        return qwb_check_launch("rmsnorm_onto");
    }
    const size_t smem = (size_t)D * sizeof(float);
    if (smem > 200 * 1024) return qwb_fail(QWB_ERR_ARG, "rmsnorm_onto: width %d does not fit in shared memory", D);
    const int block = D >= 1024 ? 256 : 128;
    cudaError_t e = cudaSuccess;
    if (to_bf16) {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_onto_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm_onto: %s", cudaGetErrorString(e));
        qwb_launch(rmsnorm_onto_kernel<bf16>, T, block, smem, stream, y, w, h, (bf16*)cast, D, eps);
    } else {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_onto_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm_onto: %s", cudaGetErrorString(e));
        qwb_launch(rmsnorm_onto_kernel<float>, T, block, smem, stream, y, w, h, (float*)cast, D, eps);
    }
    return qwb_check_launch("rmsnorm_onto");
}

// ---------------------------------------------------------------------------------
// The norm AFTER the sum:  h[t, :] <- norm(alpha * h[t, :] + y[t, :]) * w with norm(v) = v * rsqrt(mean(v^2) + eps), in
// 32-bit and in place, for blocks whose stream is normed after every sublayer has been added.  `cast` (optional, float or
// bfloat16) receives the new h in the dtype of the next product's operands.  One block per row; the row of sums stays in
// shared memory between the two passes.
// ---------------------------------------------------------------------------------
template <typename TOut>
__global__ void rmsnorm_mix_kernel(const float* __restrict__ y, const float* __restrict__ w, float* h, TOut* __restrict__ cast,
                                   int D, float eps, float alpha) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float row_cache[];
    __shared__ float red[32];
    const size_t at = (size_t)blockIdx.x * D;
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = alpha * h[at + i] + y[at + i];
        row_cache[i] = v;
        ss += v * v;
    }
    const float scale = rsqrtf(block_sum(ss, red) / (float)D + eps);
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = row_cache[i] * scale * w[i];
        h[at + i] = v;
        if (cast) cast[at + i] = from_f32<TOut>(v);
    }
}

// The same for rows of up to 4 x ITERS x 256 values that are whole 16-byte pieces: the row stays in registers and a
// thread's loads are issued together.
template <typename TOut, int ITERS>
__global__ void __launch_bounds__(256)
rmsnorm_mix_rows_kernel(const float* __restrict__ y, const float* __restrict__ w, float* h, TOut* __restrict__ cast, int D, float eps,
                        float alpha) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[32];
    const size_t at = (size_t)blockIdx.x * D;
    const float4* y4 = reinterpret_cast<const float4*>(y + at);
    float4* h4 = reinterpret_cast<float4*>(h + at);
    float4 v[ITERS], g[ITERS];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        const bool in = i < D / 4;
        const float4 a = in ? y4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 r = in ? h4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        g[k] = in ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        v[k] = make_float4(alpha * r.x + a.x, alpha * r.y + a.y, alpha * r.z + a.z, alpha * r.w + a.w);
        ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    const float scale = rsqrtf(block_sum(ss, red) / (float)D + eps);
#pragma unroll
    for (int k = 0; k < ITERS; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < D / 4) {
            const float4 o = make_float4(v[k].x * scale * g[k].x, v[k].y * scale * g[k].y, v[k].z * scale * g[k].z, v[k].w * scale * g[k].w);
            h4[i] = o;
            if (cast) Pack4<TOut>::store(cast + at + 4 * (size_t)i, o.x, o.y, o.z, o.w);
        }
    }
}

extern "C" int qwb_rmsnorm_mix(const float* y, const float* w, float* h, void* cast, int cast_dtype, int T, int D, float eps, float alpha,
                               cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0) return qwb_fail(QWB_ERR_ARG, "rmsnorm_mix: bad width %d", D);
    if (cast && cast_dtype != QWB_DT_BF16 && cast_dtype != QWB_DT_F32) return qwb_fail(QWB_ERR_ARG, "rmsnorm_mix: unknown dtype %d", cast_dtype);
    const bool to_bf16 = cast && cast_dtype == QWB_DT_BF16;
    const bool vec = D % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)h % 16 == 0 && (!cast || (uintptr_t)cast % 16 == 0);
    if (vec && D / 4 <= 4 * 256) {
        if (D / 4 <= 2 * 256) {
            if (to_bf16) qwb_launch(rmsnorm_mix_rows_kernel<bf16, 2>, T, 256, 0, stream, y, w, h, (bf16*)cast, D, eps, alpha);
            else qwb_launch(rmsnorm_mix_rows_kernel<float, 2>, T, 256, 0, stream, y, w, h, (float*)cast, D, eps, alpha);
        } else {
            if (to_bf16) qwb_launch(rmsnorm_mix_rows_kernel<bf16, 4>, T, 256, 0, stream, y, w, h, (bf16*)cast, D, eps, alpha);
            else qwb_launch(rmsnorm_mix_rows_kernel<float, 4>, T, 256, 0, stream, y, w, h, (float*)cast, D, eps, alpha);
        }
        return qwb_check_launch("rmsnorm_mix");
    }
    const size_t smem = (size_t)D * sizeof(float);
    if (smem > 200 * 1024) return qwb_fail(QWB_ERR_ARG, "rmsnorm_mix: width %d does not fit in shared memory", D);
    const int block = D >= 1024 ? 256 : 128;
    cudaError_t e = cudaSuccess;
    if (to_bf16) {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_mix_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm_mix: %s", cudaGetErrorString(e));
        qwb_launch(rmsnorm_mix_kernel<bf16>, T, block, smem, stream, y, w, h, (bf16*)cast, D, eps, alpha);
    } else {
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(rmsnorm_mix_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qwb_fail(QWB_ERR_CUDA, "rmsnorm_mix: %s", cudaGetErrorString(e));
        qwb_launch(rmsnorm_mix_kernel<float>, T, block, smem, stream, y, w, h, (float*)cast, D, eps, alpha);
    }
    return qwb_check_launch("rmsnorm_mix");
}

// ---------------------------------------------------------------------------------
// out[t, f] = act(x[t, f] + bias[f]) for F columns of a float matrix with rows of ld values (the caller offsets the
// pointer to the first column); out [T, F] float or bfloat16 (may be x itself when float and ld = F).
// act 0: none; 1: relu squared; 2: gelu (tanh form); 3: silu; 4: xIELU with two learned numbers p, q (`params`):
// v > 0: softplus(p) v^2 + v / 2;  v <= 0: (1/2 + softplus(q)) (e^v - 1 - v) + v / 2; 5: gelu (v times the normal
// distribution's function).  bias may be null.
// ---------------------------------------------------------------------------------
__device__ __forceinline__ float softplus32(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <typename TOut>
__global__ void bias_act_kernel(const float* x, int ld, const float* __restrict__ bias, TOut* out, size_t n, int F, int act,
                                const float* __restrict__ params) {
    pdl_wait();
    pdl_launch_dependents();
    float up = 0.f, down = 0.f;
    if (act == 4) { up = softplus32(params[0]); down = 0.5f + softplus32(params[1]); }
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / F, f = i - t * F;
        float v = x[t * ld + f] + (bias ? bias[f] : 0.f);
        if (act == 4) v = v > 0.f ? up * v * v + 0.5f * v : down * (expm1f(v) - v) + 0.5f * v;
        else v = qwb_activate(v, act);
        out[i] = from_f32<TOut>(v);
    }
}

// The same for whole rows (ld = F) with F a multiple of 4: four values a thread and step.
template <typename TOut>
__global__ void bias_act_fours_kernel(const float4* x, const float4* __restrict__ bias, TOut* out, unsigned n4, unsigned f4, int act,
                                      const float* __restrict__ params) {
    pdl_wait();
    pdl_launch_dependents();
    float up = 0.f, down = 0.f;
    if (act == 4) { up = softplus32(params[0]); down = 0.5f + softplus32(params[1]); }
    auto f = [&](float v) { return act == 4 ? (v > 0.f ? up * v * v + 0.5f * v : down * (expm1f(v) - v) + 0.5f * v) : qwb_activate(v, act); };
    for (unsigned i = blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += gridDim.x * blockDim.x) {
        float4 v = x[i];
        if (bias) { const float4 b = bias[i % f4]; v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
        Pack4<TOut>::store(out + (size_t)i * 4, f(v.x), f(v.y), f(v.z), f(v.w));
    }
}

extern "C" int qwb_bias_act(const float* x, int ld, const float* bias, void* out, int out_dtype, int T, int F, int act,
                            const float* params, cudaStream_t stream) {
    if (T <= 0 || F <= 0) return 0;
    if (ld < F) return qwb_fail(QWB_ERR_ARG, "bias_act: rows of %d values hold no %d columns", ld, F);
    if (act < 0 || act > 5) return qwb_fail(QWB_ERR_ARG, "bias_act: unknown activation %d", act);
    if (act == 4 && !params) return qwb_fail(QWB_ERR_ARG, "bias_act: this activation needs its two numbers");
    const size_t n = (size_t)T * F;
    const int block = 256;
    if (ld == F && F % 4 == 0 && n / 4 < (1u << 30) && (uintptr_t)x % 16 == 0 && (uintptr_t)bias % 16 == 0 && (uintptr_t)out % 16 == 0) {
        const unsigned n4 = (unsigned)(n / 4);
        const int g4 = (int)((n4 + block - 1) / block < 148 * 32 ? (n4 + block - 1) / block : 148 * 32);
        if (out_dtype == QWB_DT_F32)
            qwb_launch(bias_act_fours_kernel<float>, g4, block, 0, stream, (const float4*)x, (const float4*)bias, (float*)out, n4, (unsigned)(F / 4), act, params);
        else if (out_dtype == QWB_DT_BF16)
            qwb_launch(bias_act_fours_kernel<bf16>, g4, block, 0, stream, (const float4*)x, (const float4*)bias, (bf16*)out, n4, (unsigned)(F / 4), act, params);
        else return qwb_fail(QWB_ERR_ARG, "bias_act: unknown dtype %d", out_dtype);
        return qwb_check_launch("bias_act");
    }
    const int grid = (int)((n + block - 1) / block < 148 * 16 ? (n + block - 1) / block : 148 * 16);
    if (out_dtype == QWB_DT_F32) qwb_launch(bias_act_kernel<float>, grid, block, 0, stream, x, ld, bias, (float*)out, n, F, act, params);
    else if (out_dtype == QWB_DT_BF16) qwb_launch(bias_act_kernel<bf16>, grid, block, 0, stream, x, ld, bias, (bf16*)out, n, F, act, params);
    else return qwb_fail(QWB_ERR_ARG, "bias_act: unknown dtype %d", out_dtype);
    return qwb_check_launch("bias_act");
}

// ---------------------------------------------------------------------------------
// Logits in place: v <- v * scale, then cap * tanh(v / cap) if cap > 0.
// ---------------------------------------------------------------------------------
__global__ void scale_softcap_kernel(float* x, size_t n, float scale, float cap) {
    pdl_wait();
    pdl_launch_dependents();
    const float inv = cap > 0.f ? 1.f / cap : 0.f;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float v = x[i] * scale;
        x[i] = cap > 0.f ? cap * tanhf(v * inv) : v;
    }
}

extern "C" int qwb_scale_softcap(float* x, long long n, float scale, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    const int block = 256;
    const long long grid = (n + block - 1) / block;
    qwb_launch(scale_softcap_kernel, (unsigned)(grid > 148 * 16 ? 148 * 16 : grid), block, 0, stream, x, (size_t)n, scale, cap);
    return qwb_check_launch("scale_softcap");
}
