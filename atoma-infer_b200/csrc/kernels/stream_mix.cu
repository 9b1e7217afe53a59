// The kernel around the residual of blocks that carry several streams side by side (hyper-connections): every stream is
// replaced by a weighted sum of all of them plus its share of a sublayer's result, and the next sublayer's input is the
// norm of another weighted sum of the new streams.  One pass: old streams and result in, new streams and normed row out.
// The streams and all arithmetic are float32; every reduction runs in an order that depends only on the row.
#include "common.cuh"

int g_use_pdl = 1;
extern "C" void kernels_set_pdl(int mode) { g_use_pdl = mode; }

// x [T, S * H]: stream j of row t starts at (t * S + j) * H.
//   y  = (mult * (f0 a0[t] + f1 a1[t] + ...) + vec) * scale           (up to four terms; vec and scale optional)
//   x'_k = sum_j mix[j * S + k] x_j + give[k] * y                      (if there are terms; else x' = x)
//   out[r] = N(sum_k read[k] x'_k) * w                                 (if `out`; `read` null: all 1)
// With `rows`: works on rows[r] of the inputs, writes out[r], leaves x untouched.
#define MIX_MAX_TERMS 4
#define MIX_MAX_STREAMS 64
struct MixTerms {
    const void* p[MIX_MAX_TERMS];
    float f[MIX_MAX_TERMS];
    int n;
};

// V neighbouring values of the sublayer's result at row `src`, column i.
template <typename TD, int V>
__device__ __forceinline__ void load_values(const TD* p, float (&v)[V]) {
    if constexpr (V == 4) load4(p, v);
    else v[0] = to_float(p[0]);
}
template <int V>
__device__ __forceinline__ void store_values(float* p, const float (&v)[V]) {
    if constexpr (V == 4) store4(p, v);
    else p[0] = v[0];
}
template <typename TD, int V>
__device__ __forceinline__ void result_at(const MixTerms& terms, size_t at, int i, float mult, const float* vec, const float* scale,
                                          float (&y)[V]) {
    load_values<TD, V>((const TD*)terms.p[0] + at + i, y);
    if (terms.f[0] != 1.f) {
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] *= terms.f[0];
    }
#pragma unroll
    for (int j = 1; j < MIX_MAX_TERMS; ++j) {
        if (j < terms.n) {
            float t[V];
            load_values<TD, V>((const TD*)terms.p[j] + at + i, t);
#pragma unroll
            for (int k = 0; k < V; ++k) y[k] = fmaf(terms.f[j], t[k], y[k]);
        }
    }
    if (mult != 1.f) {
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] *= mult;
    }
    if (vec) {
        float t[V];
        load_values<float, V>(vec + i, t);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] += t[k];
    }
    if (scale) {
        float t[V];
        load_values<float, V>(scale + i, t);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] *= t[k];
    }
}

// S streams known at compile time: a thread holds its V columns of every stream in registers and the weighted sum that is
// normed in up to MAXC registers of V values (wider rows: in shared memory).
template <typename TD, typename TO, int S, int V, int MAXC>
__global__ void __launch_bounds__(256)
stream_mix_kernel(float* __restrict__ x, MixTerms terms, float mult, const float* __restrict__ vec, const float* __restrict__ scale,
                  const float* __restrict__ mix, const float* __restrict__ give, const float* __restrict__ read,
                  const int* __restrict__ rows, const float* __restrict__ w, float eps, TO* __restrict__ out,
                  const int* __restrict__ meta, int H) {
    __shared__ float red[33];
    // weights and the step's metadata are written by no kernel of the step: read before the wait
    float m[S][S], g[S], rd[S];
#pragma unroll
    for (int j = 0; j < S; ++j) {
        rd[j] = read ? read[j] : 1.f;
        g[j] = terms.n ? give[j] : 0.f;
#pragma unroll
        for (int k = 0; k < S; ++k) m[j][k] = terms.n ? mix[j * S + k] : (j == k ? 1.f : 0.f);
    }
    const int r = blockIdx.x, limit = rows ? meta[META_NUM_ROWS] : meta[META_NUM_TOKENS];
    const size_t src = r < limit ? (rows ? (size_t)rows[r] : (size_t)r) : 0;
    pdl_wait();
    pdl_launch_dependents();
    if (r >= limit) return;
    float* xr = x + src * S * H;
    float u[MAXC][V];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * V;
        if (i < H) {
            float v[S][V];
#pragma unroll
            for (int j = 0; j < S; ++j) load_values<float, V>(xr + (size_t)j * H + i, v[j]);
            if (terms.n) {
                float y[V], nv[S][V];
                result_at<TD, V>(terms, src * H, i, mult, vec, scale, y);
#pragma unroll
                for (int k = 0; k < S; ++k) {
#pragma unroll
                    for (int e = 0; e < V; ++e) {
                        float a = m[0][k] * v[0][e];
#pragma unroll
                        for (int j = 1; j < S; ++j) a = fmaf(m[j][k], v[j][e], a);
                        nv[k][e] = fmaf(g[k], y[e], a);
                    }
                }
#pragma unroll
                for (int k = 0; k < S; ++k) {
                    if (!rows) store_values<V>(xr + (size_t)k * H + i, nv[k]);
#pragma unroll
                    for (int e = 0; e < V; ++e) v[k][e] = nv[k][e];
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
                float a = rd[0] * v[0][e];
#pragma unroll
                for (int j = 1; j < S; ++j) a = fmaf(rd[j], v[j][e], a);
                u[c][e] = a;
                ss = fmaf(a, a, ss);
            }
        }
    }
    if (!out) return;
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)H + eps);
    TO* o = out + (size_t)r * H;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * V;
        if (i < H) {
            float wv[V];
            load_values<float, V>(w + i, wv);
#pragma unroll
            for (int e = 0; e < V; ++e) wv[e] = u[c][e] * inv * wv[e];
            if constexpr (V == 4) store4(o + i, wv);
            else o[i] = from_float<TO>(wv[0]);
        }
    }
}

// Any number of streams, any width: a thread walks its columns one by one, the weights and the weighted sum in shared
// memory (`sm`: S * S + 2 S weights, then a column's new values per thread, then H sums).
template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
stream_mix_any_kernel(float* __restrict__ x, MixTerms terms, float mult, const float* __restrict__ vec, const float* __restrict__ scale,
                      const float* __restrict__ mix, const float* __restrict__ give, const float* __restrict__ read,
                      const int* __restrict__ rows, const float* __restrict__ w, float eps, TO* __restrict__ out,
                      const int* __restrict__ meta, int H, int S) {
    __shared__ float red[33];
    extern __shared__ float sm[];
    float *m = sm, *g = m + S * S, *rd = g + S, *nv = rd + S, *u = nv + S * blockDim.x;
    for (int i = threadIdx.x; i < S * S && terms.n; i += blockDim.x) m[i] = mix[i];
    for (int i = threadIdx.x; i < S; i += blockDim.x) {
        g[i] = terms.n ? give[i] : 0.f;
        rd[i] = read ? read[i] : 1.f;
    }
    const int r = blockIdx.x, limit = rows ? meta[META_NUM_ROWS] : meta[META_NUM_TOKENS];
    const size_t src = r < limit ? (rows ? (size_t)rows[r] : (size_t)r) : 0;
    pdl_wait();
    pdl_launch_dependents();
    if (r >= limit) return;
    __syncthreads();
    float* xr = x + src * S * H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float a = 0.f;
        if (terms.n) {
            float y[1];
            result_at<TD, 1>(terms, src * H, i, mult, vec, scale, y);
            for (int k = 0; k < S; ++k) {
                float s = m[k] * xr[i];
                for (int j = 1; j < S; ++j) s = fmaf(m[j * S + k], xr[(size_t)j * H + i], s);
                nv[k * blockDim.x + threadIdx.x] = fmaf(g[k], y[0], s);
            }
            for (int k = 0; k < S; ++k) {
                const float s = nv[k * blockDim.x + threadIdx.x];
                if (!rows) xr[(size_t)k * H + i] = s;
                a = fmaf(rd[k], s, a);
            }
        } else {
            for (int k = 0; k < S; ++k) a = fmaf(rd[k], xr[(size_t)k * H + i], a);
        }
        u[i] = a;
        ss = fmaf(a, a, ss);
    }
    if (!out) return;
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) out[(size_t)r * H + i] = from_float<TO>(u[i] * inv * w[i]);
}

extern "C" int stream_mix_norm(float* x, int S, int num_terms, const void* const* term_ptrs, const float* factors, int term_dtype,
                               float mult, const float* vec, const float* scale, const float* mix, const float* give,
                               const float* read, const int* rows, const float* w, float eps, void* out, int out_dtype,
                               const int* meta, int n, int H, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (num_terms < 0 || num_terms > MIX_MAX_TERMS || S < 1 || S > MIX_MAX_STREAMS || (num_terms && (!mix || !give)) || (out && !w))
        return (int)cudaErrorInvalidValue;
    MixTerms terms = {};
    terms.n = num_terms;
    uintptr_t all = (uintptr_t)x | (uintptr_t)vec | (uintptr_t)scale | (uintptr_t)w | (uintptr_t)out;
    for (int j = 0; j < num_terms; ++j) {
        terms.p[j] = term_ptrs[j];
        terms.f[j] = factors ? factors[j] : 1.f;
        all |= (uintptr_t)term_ptrs[j];
    }
    const bool pdl = (g_use_pdl & 5) != 0;
    const bool vec4 = H % 4 == 0 && (all & 15) == 0;
    // Four columns a thread and step; enough threads that a row is one or two steps where that fits a block.
    const int V = vec4 ? 4 : 1, pieces = (H + V - 1) / V;
    const int threads = pieces <= 128 ? 128 : 256;
    const int steps = (pieces + threads - 1) / threads;
#define MIX_LAUNCH(TD, TO, SS, VV, CC)                                                                                       \
    return (int)launch_kernel_pdl(pdl, stream_mix_kernel<TD, TO, SS, VV, CC>, n, threads, 0, stream, x, terms, mult, vec, scale, mix, \
                                  give, read, rows, w, eps, (TO*)out, meta, H)
#define MIX_STEPS(TD, TO, SS)                                                                                                \
    do {                                                                                                                     \
        if (vec4 && steps == 1) MIX_LAUNCH(TD, TO, SS, 4, 1);                                                                \
        if (vec4 && steps == 2) MIX_LAUNCH(TD, TO, SS, 4, 2);                                                                \
        if (vec4 && steps <= 4) MIX_LAUNCH(TD, TO, SS, 4, 4);                                                                \
        if (vec4 && steps <= 8) MIX_LAUNCH(TD, TO, SS, 4, 8);                                                                \
    } while (0)
#define MIX_CASE(TD, TO)                                                                                                     \
    do {                                                                                                                     \
        if (S == 1) MIX_STEPS(TD, TO, 1);                                                                                    \
        if (S == 2) MIX_STEPS(TD, TO, 2);                                                                                    \
        if (S == 3) MIX_STEPS(TD, TO, 3);                                                                                    \
        if (S == 4) MIX_STEPS(TD, TO, 4);                                                                                    \
        const size_t smem = ((size_t)S * S + 2 * S + (size_t)S * 128 + H) * sizeof(float);                                   \
        if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;                                                            \
        static size_t configured = 0;                                                                                        \
        if (smem > 48 * 1024 && smem > configured) {                                                                         \
            cudaError_t e = cudaFuncSetAttribute(stream_mix_any_kernel<TD, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                             \
            configured = smem;                                                                                               \
        }                                                                                                                    \
        return (int)launch_kernel_pdl(pdl, stream_mix_any_kernel<TD, TO>, n, 128, smem, stream, x, terms, mult, vec, scale, mix, give, \
                                      read, rows, w, eps, (TO*)out, meta, H, S);                                             \
    } while (0)
    if (num_terms && term_dtype == DT_F32) {
        if (out && out_dtype != DT_F32) return (int)cudaErrorInvalidValue;
        MIX_CASE(float, float);
    }
    if (out_dtype == DT_F32) MIX_CASE(__nv_bfloat16, float);
    MIX_CASE(__nv_bfloat16, __nv_bfloat16);
#undef MIX_CASE
#undef MIX_STEPS
#undef MIX_LAUNCH
}
