// Kernels of blocks whose only norm stands on a sublayer's result: the norm of the result (layer norm or root mean square; of
// a weighted sum of terms, each of which may be normed over the width first) with the sum into the float32 stream and the
// next sublayer's input, the layer norm of chosen rows, and rows moved toward the token before by several weights at once.
// float32 and bfloat16 storage alike; all arithmetic is float32, and every reduction runs in an order that depends only on
// the row it belongs to.
#include "common.cuh"

// N sums over a block (the first `n` of them are used) with one barrier between the warps' sums and the total, which every
// warp takes for itself in the order of the warps.  `scratch` holds 8 * 33 floats; the caller separates two uses by a barrier.
#define NS_MAX_SUMS 8
template <int N>
__device__ __forceinline__ void block_totals(float (&v)[N], int n, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
#pragma unroll
    for (int k = 0; k < N; ++k)
        if (k < n) {
            v[k] = warp_sum(v[k]);
            if (lane == 0) scratch[k * 33 + warp] = v[k];
        }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < N; ++k)
        if (k < n) v[k] = warp_sum(lane < nwarps ? scratch[k * 33 + lane] : 0.f);
}

// ----------------------------------------------------------------------------- norm of the result, sum into the stream
// y[t] = mult * (f0 n0(a0[t]) + f1 n1(a1[t]) + ...) + vec, n_j(a) = a, or a * rsqrt(mean(a^2) + eps_j) * w_j where the term has
// a weight; resid[t] += norm(y[t]) with norm(y) = (y - mean) * rsqrt(mean((y - mean)^2) + eps) * w (layer_norm) or
// y * rsqrt(mean(y^2) + eps) * w; with `out` also out[t] = resid[t] in the compute type, the next sublayer's input.
#define NS_MAX_TERMS 4
struct NormedTerms {
    const void* p[NS_MAX_TERMS];
    const float* w[NS_MAX_TERMS];  // null: the term as it is
    float f[NS_MAX_TERMS], eps[NS_MAX_TERMS];
    int n;
};

#define NS_CHUNKS 4  // most fours of values a thread keeps in registers
// Four stored values as they were loaded (a bfloat16 row costs half the registers of a float32 one until it is used).
template <typename T> struct RawFour;
template <> struct RawFour<float> { float4 v; };
template <> struct RawFour<__nv_bfloat16> { uint2 v; };
template <typename T> __device__ __forceinline__ RawFour<T> raw_four(const T* p) { return *reinterpret_cast<const RawFour<T>*>(p); }
template <typename T> __device__ __forceinline__ void widen_four(const RawFour<T>& r, float (&v)[4]) { load4(reinterpret_cast<const T*>(&r), v); }

// The row form: CH fours a thread, every load of the row on its way before the first is used; NT terms (0: `terms.n`, at most
// four).  The mean of y follows from the first pass's sums (of every normed term the sum of squares and the weighted sum, of
// every other term the sum), so there are two block-wide reductions.
template <typename TD, typename TO, int NT, int CH>
__global__ void __launch_bounds__(1024)
norm_add_kernel(float* __restrict__ resid, const NormedTerms terms, float mult, const float* __restrict__ vec,
                const float* __restrict__ w, float eps, int layer_norm, TO* __restrict__ out, const int* __restrict__ meta, int H) {
    constexpr int MAXT = NT ? NT : NS_MAX_TERMS;
    __shared__ float red[3][NS_MAX_SUMS * 33];
    const int t = blockIdx.x, n = NT ? NT : terms.n;
    const bool live = t < meta[META_NUM_TOKENS];
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    const float inv_h = 1.f / (float)H;
    float* x = resid + (size_t)t * H;
    RawFour<TD> raw[MAXT][CH];
    float4 old[CH];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * 4;
        if (i < H) {
#pragma unroll
            for (int j = 0; j < MAXT; ++j)
                if (j < n) raw[j][c] = raw_four((const TD*)terms.p[j] + (size_t)t * H + i);
            old[c] = *reinterpret_cast<const float4*>(x + i);
        }
    }
    float sums[2 * MAXT] = {};
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * 4;
        if (i < H) {
#pragma unroll
            for (int j = 0; j < MAXT; ++j) {
                if (j >= n) continue;
                float a[4], wv[4] = {1.f, 1.f, 1.f, 1.f};
                widen_four(raw[j][c], a);
                if (terms.w[j]) load4(terms.w[j] + i, wv);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    sums[2 * j] = fmaf(a[k], a[k], sums[2 * j]);
                    sums[2 * j + 1] = fmaf(a[k], wv[k], sums[2 * j + 1]);
                }
            }
        }
    }
    block_totals(sums, 2 * n, red[0]);
    float fac[MAXT], mean = 0.f;
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        fac[j] = j < n ? mult * terms.f[j] * (terms.w[j] ? rsqrtf(sums[2 * j] * inv_h + terms.eps[j]) : 1.f) : 0.f;
        mean = fmaf(fac[j], sums[2 * j + 1] * inv_h, mean);
    }
    if (vec) {  // (a bias of the result: its mean joins the terms')
        float s[1] = {0.f};
        for (int i = threadIdx.x; i < H; i += blockDim.x) s[0] += vec[i];
        block_totals(s, 1, red[2]);
        mean += s[0] * inv_h;
    }
    if (!layer_norm) mean = 0.f;
    float ss[1] = {0.f}, y[CH][4];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * 4;
        if (i < H) {
            float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int j = 0; j < MAXT; ++j) {
                if (j >= n) continue;
                float a[4], wv[4] = {1.f, 1.f, 1.f, 1.f};
                widen_four(raw[j][c], a);
                if (terms.w[j]) load4(terms.w[j] + i, wv);
#pragma unroll
                for (int k = 0; k < 4; ++k) s[k] = fmaf(fac[j] * wv[k], a[k], s[k]);
            }
            if (vec) {
                float b[4];
                load4(vec + i, b);
#pragma unroll
                for (int k = 0; k < 4; ++k) s[k] += b[k];
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                y[c][k] = s[k] - mean;
                ss[0] = fmaf(y[c][k], y[c][k], ss[0]);
            }
        }
    }
    block_totals(ss, 1, red[1]);
    const float inv = rsqrtf(ss[0] * inv_h + eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * 4;
        if (i < H) {
            float wv[4], v[4] = {old[c].x, old[c].y, old[c].z, old[c].w};
            load4(w + i, wv);
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = fmaf(y[c][k] * inv, wv[k], v[k]);
            store4(x + i, v);
            if (out) store4(out + (size_t)t * H + i, v);
        }
    }
}

// The same for rows of any width and alignment, value by value; y waits in shared memory.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
norm_add_scalar_kernel(float* __restrict__ resid, const NormedTerms terms, float mult, const float* __restrict__ vec,
                       const float* __restrict__ w, float eps, int layer_norm, TO* __restrict__ out, const int* __restrict__ meta, int H) {
    __shared__ float red[3][NS_MAX_SUMS * 33];
    extern __shared__ __align__(16) float row[];
    const int t = blockIdx.x;
    const bool live = t < meta[META_NUM_TOKENS];
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    const float inv_h = 1.f / (float)H;
    float* x = resid + (size_t)t * H;
    float sums[2 * NS_MAX_TERMS] = {};
    for (int i = threadIdx.x; i < H; i += blockDim.x)
#pragma unroll
        for (int j = 0; j < NS_MAX_TERMS; ++j) {
            if (j >= terms.n) continue;
            const float a = to_float(((const TD*)terms.p[j])[(size_t)t * H + i]), wv = terms.w[j] ? terms.w[j][i] : 1.f;
            sums[2 * j] = fmaf(a, a, sums[2 * j]);
            sums[2 * j + 1] = fmaf(a, wv, sums[2 * j + 1]);
        }
    block_totals(sums, 2 * terms.n, red[0]);
    float fac[NS_MAX_TERMS], mean = 0.f;
#pragma unroll
    for (int j = 0; j < NS_MAX_TERMS; ++j) {
        fac[j] = j < terms.n ? mult * terms.f[j] * (terms.w[j] ? rsqrtf(sums[2 * j] * inv_h + terms.eps[j]) : 1.f) : 0.f;
        mean = fmaf(fac[j], sums[2 * j + 1] * inv_h, mean);
    }
    if (vec) {
        float s[1] = {0.f};
        for (int i = threadIdx.x; i < H; i += blockDim.x) s[0] += vec[i];
        block_totals(s, 1, red[2]);
        mean += s[0] * inv_h;
    }
    if (!layer_norm) mean = 0.f;
    float ss[1] = {0.f};
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NS_MAX_TERMS; ++j) {
            if (j >= terms.n) continue;
            s = fmaf(fac[j] * (terms.w[j] ? terms.w[j][i] : 1.f), to_float(((const TD*)terms.p[j])[(size_t)t * H + i]), s);
        }
        if (vec) s += vec[i];
        s -= mean;
        row[i] = s;
        ss[0] = fmaf(s, s, ss[0]);
    }
    block_totals(ss, 1, red[1]);
    const float inv = rsqrtf(ss[0] * inv_h + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = fmaf(row[i] * inv, w[i], x[i]);
        x[i] = v;
        if (out) out[(size_t)t * H + i] = from_float<TO>(v);
    }
}

extern "C" int norm_add(float* resid, int num_terms, const void* const* term_ptrs, const float* factors, const float* const* term_weights,
                        const float* term_eps, int term_dtype, float mult, const float* vec, const float* w, float eps, int layer_norm,
                        void* out, int out_dtype, const int* meta, int T, int H, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (num_terms <= 0 || num_terms > NS_MAX_TERMS) return (int)cudaErrorInvalidValue;
    NormedTerms terms = {};
    terms.n = num_terms;
    uintptr_t all = (uintptr_t)resid | (uintptr_t)vec | (uintptr_t)w | (uintptr_t)out;
    for (int j = 0; j < num_terms; ++j) {
        terms.p[j] = term_ptrs[j];
        terms.w[j] = term_weights[j];
        terms.f[j] = factors[j];
        terms.eps[j] = term_eps[j];
        all |= (uintptr_t)term_ptrs[j] | (uintptr_t)term_weights[j];
    }
    // rows of fours in registers: one, two or four of them a thread
    const int fours = (H + 3) / 4, ch = fours <= 128 ? 1 : (fours <= 1024 ? 2 : 4);
    const int threads = ((fours + ch - 1) / ch + 31) / 32 * 32;
    const bool vec4 = H % 4 == 0 && (all & 15) == 0 && threads <= 1024;
    const size_t smem = vec4 ? 0 : (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
#define NORM_ADD_ROW(TD, TO, NT, CH)                                                                                       \
    return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, norm_add_kernel<TD, TO, NT, CH>, T, threads, 0, stream, resid, terms, mult, vec, w, \
                                  eps, layer_norm, (TO*)out, meta, H)
#define NORM_ADD_TERMS(TD, TO, CH)                        \
    do {                                                  \
        if (num_terms == 1) NORM_ADD_ROW(TD, TO, 1, CH);  \
        if (num_terms == 2) NORM_ADD_ROW(TD, TO, 2, CH);  \
        NORM_ADD_ROW(TD, TO, 0, CH);                      \
    } while (0)
#define NORM_ADD_CASE(TD, TO)                                                                                              \
    do {                                                                                                                  \
        if (vec4) {                                                                                                       \
            if (ch == 1) NORM_ADD_TERMS(TD, TO, 1);                                                                       \
            if (ch == 2) NORM_ADD_TERMS(TD, TO, 2);                                                                       \
            NORM_ADD_TERMS(TD, TO, NS_CHUNKS);                                                                            \
        }                                                                                                                 \
        static size_t configured = 0;                                                                                     \
        if (smem > 40 * 1024 && smem > configured) {                                                                      \
            cudaError_t ce = cudaFuncSetAttribute(norm_add_scalar_kernel<TD, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (ce != cudaSuccess) return (int)ce;                                                                        \
            configured = smem;                                                                                            \
        }                                                                                                                 \
        return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, norm_add_scalar_kernel<TD, TO>, T, 256, smem, stream, resid, terms, mult, vec, w, \
                                      eps, layer_norm, (TO*)out, meta, H);                                                \
    } while (0)
    if (term_dtype == DT_F32 && out_dtype == DT_F32) NORM_ADD_CASE(float, float);
    if (term_dtype == DT_BF16 && out_dtype == DT_BF16) NORM_ADD_CASE(__nv_bfloat16, __nv_bfloat16);
    return (int)cudaErrorInvalidValue;
#undef NORM_ADD_CASE
#undef NORM_ADD_TERMS
#undef NORM_ADD_ROW
}

// ----------------------------------------------------------------------------- layer norm of rows
// out[r] = (x - mean) * rsqrt(mean((x - mean)^2) + eps) * w with x = resid[rows[r]] (or resid[r]).
template <typename TO>
__global__ void __launch_bounds__(256)
layer_norm_rows_kernel(const float* __restrict__ resid, const int* __restrict__ rows, const float* __restrict__ w, float eps,
                       TO* __restrict__ out, const int* __restrict__ meta, int H) {
    __shared__ float red[2][NS_MAX_SUMS * 33];
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x;
    if (r >= (rows ? meta[META_NUM_ROWS] : meta[META_NUM_TOKENS])) return;
    const float* x = resid + (size_t)(rows ? rows[r] : r) * H;
    float s[1] = {0.f}, ss[1] = {0.f};
    for (int i = threadIdx.x; i < H; i += blockDim.x) s[0] += x[i];
    block_totals(s, 1, red[0]);
    const float mean = s[0] / (float)H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) { const float d = x[i] - mean; ss[0] = fmaf(d, d, ss[0]); }
    block_totals(ss, 1, red[1]);
    const float inv = rsqrtf(ss[0] / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) out[(size_t)r * H + i] = from_float<TO>((x[i] - mean) * inv * w[i]);
}

extern "C" int layer_norm_rows(const float* resid, const int* rows, const float* w, float eps, void* out, int out_dtype, const int* meta,
                               int n, int H, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (out_dtype == DT_F32)
        return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, layer_norm_rows_kernel<float>, n, 256, 0, stream, resid, rows, w, eps, (float*)out,
                                      meta, H);
    return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, layer_norm_rows_kernel<__nv_bfloat16>, n, 256, 0, stream, resid, rows, w, eps,
                                  (__nv_bfloat16*)out, meta, H);
}

// ----------------------------------------------------------------------------- rows moved toward the token before
// out[k][t] = x[t] + (x[t - 1] - x[t]) * mu[k] for `count` weights mu[k] [H]; x[t - 1] is the row of the token before in the same
// request: of this step, or the row kept in the request's state, or zeros at position 0.  x is [T, H] float32 or the
// compute type, out [count, T, H], the state float32.  With `save` (steps in which every entry brings one token) the thread
// that has read a value of the kept row also puts the new one there.
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
token_mix_kernel(const TI* __restrict__ x, const float* __restrict__ mu, int count, float* __restrict__ state, long long slot_stride,
                 TO* __restrict__ out, const int* __restrict__ meta, const int* __restrict__ positions,
                 const int* __restrict__ token_entry, const int* __restrict__ cu_tokens, const int* __restrict__ slots, int T, int H,
                 int save, int vec4) {
    const int t = blockIdx.x;
    const bool live = t < meta[META_NUM_TOKENS];
    int first = 0, pos = 0, slot = 0;
    if (live) {
        const int e = token_entry[t];
        first = cu_tokens[e];
        pos = positions[t];
        slot = slots[e];
    }
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    const TI* xr = x + (size_t)t * H;
    const bool from_row = t > first, from_state = !from_row && pos > 0;
    float* st = state + (size_t)slot * slot_stride;
    if (vec4) {
        for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
            float v[4], b[4] = {0.f, 0.f, 0.f, 0.f};
            load4(xr + i, v);
            if (from_row) load4(xr - H + i, b);
            else if (from_state) load4(st + i, b);
            if (save) store4(st + i, v);
#pragma unroll
            for (int k = 0; k < 4; ++k) b[k] -= v[k];
            for (int j = 0; j < count; ++j) {
                float m[4], o[4];
                load4(mu + (size_t)j * H + i, m);
#pragma unroll
                for (int k = 0; k < 4; ++k) o[k] = fmaf(b[k], m[k], v[k]);
                store4(out + ((size_t)j * T + t) * H + i, o);
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_float(xr[i]), b = from_row ? to_float(xr[i - H]) : (from_state ? st[i] : 0.f);
        if (save) st[i] = v;
        for (int j = 0; j < count; ++j) out[((size_t)j * T + t) * H + i] = from_float<TO>(fmaf(b - v, mu[(size_t)j * H + i], v));
    }
}

extern "C" int token_mix(const void* x, int x_dtype, const float* mu, int count, float* state, long long slot_stride, void* out,
                         int out_dtype, const int* meta, const int* positions, const int* token_entry, const int* cu_tokens,
                         const int* slots, int T, int H, int save, cudaStream_t stream) {
    if (T <= 0 || count <= 0) return 0;
    const int threads = H >= 1024 ? 256 : 128;
    const int vec4 = H % 4 == 0 && slot_stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
#define MIX_CASE(TI, TO)                                                                                                   \
    return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, token_mix_kernel<TI, TO>, T, threads, 0, stream, (const TI*)x, mu, count, state, \
                                  slot_stride, (TO*)out, meta, positions, token_entry, cu_tokens, slots, T, H, save, vec4)
    if (x_dtype == DT_F32 && out_dtype == DT_F32) MIX_CASE(float, float);
    if (x_dtype == DT_F32) MIX_CASE(float, __nv_bfloat16);
    if (out_dtype == DT_BF16) MIX_CASE(__nv_bfloat16, __nv_bfloat16);
    return (int)cudaErrorInvalidValue;
#undef MIX_CASE
}

// The last row of every entry goes to its state (see token_mix), after everything has read the old one.  One block an entry.
template <typename TI>
__global__ void __launch_bounds__(256)
keep_last_rows_kernel(const TI* __restrict__ x, float* __restrict__ state, long long slot_stride, const int* __restrict__ meta,
                      const int* __restrict__ cu_tokens, const int* __restrict__ slots, int H) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x;
    if (e >= meta[META_NUM_ENTRIES]) return;
    const TI* row = x + (size_t)(cu_tokens[e + 1] - 1) * H;
    float* st = state + (size_t)slots[e] * slot_stride;
    for (int i = threadIdx.x; i < H; i += blockDim.x) st[i] = to_float(row[i]);
}

extern "C" int keep_last_rows(const void* x, int x_dtype, float* state, long long slot_stride, const int* meta, const int* cu_tokens,
                              const int* slots, int S, int H, cudaStream_t stream) {
    if (S <= 0) return 0;
    if (x_dtype == DT_F32)
        return (int)launch_kernel(keep_last_rows_kernel<float>, S, 256, 0, stream, (const float*)x, state, slot_stride, meta, cu_tokens, slots, H);
    return (int)launch_kernel(keep_last_rows_kernel<__nv_bfloat16>, S, 256, 0, stream, (const __nv_bfloat16*)x, state, slot_stride, meta,
                              cu_tokens, slots, H);
}

// ----------------------------------------------------------------------------- tanh on the way to the compute type
template <typename TO>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const float* __restrict__ z, TO* __restrict__ out, const int* __restrict__ meta, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < (size_t)meta[META_NUM_TOKENS] * n) out[i] = from_float<TO>(tanhf(z[i]));
}

extern "C" int tanh_rows(const float* z, void* out, int out_dtype, const int* meta, int T, int n, cudaStream_t stream) {
    if (T <= 0 || n <= 0) return 0;
    const unsigned blocks = (unsigned)(((size_t)T * n + 255) / 256);
    if (out_dtype == DT_F32) return (int)launch_kernel(tanh_rows_kernel<float>, blocks, 256, 0, stream, z, (float*)out, meta, n);
    return (int)launch_kernel(tanh_rows_kernel<__nv_bfloat16>, blocks, 256, 0, stream, z, (__nv_bfloat16*)out, meta, n);
}
