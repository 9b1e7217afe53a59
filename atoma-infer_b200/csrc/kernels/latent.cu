// Kernels of attention through low-rank latents: a root-mean-square norm over a slice of wider rows, a linear map
// applied head by head, and the rows' preparation (norm of the key/value latent, rotation of the shared key part and
// of the queries' rotated parts, the cached vector written to its page, the queries laid out for the attention
// kernels).  Storage is float32 or bfloat16, arithmetic float32.
#include <algorithm>

#include "common.cuh"

// out[t] = x[t] * rsqrt(mean(x[t]^2) + eps) * w over n elements; x is a slice of a wider row (x_stride from row to row).
template <typename T>
__global__ void __launch_bounds__(256)
rms_rows_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ w, float eps, T* __restrict__ out,
                const int* __restrict__ meta, int n) {
    __shared__ float red[33];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    if (t >= meta[META_NUM_TOKENS]) return;
    const T* xr = x + (size_t)t * x_stride;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = to_float(xr[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x) out[(size_t)t * n + i] = from_float<T>(to_float(xr[i]) * inv * w[i]);
}

extern "C" int rms_rows(const void* x, int dtype, long long x_stride, const float* w, float eps, void* out, const int* meta,
                        int T, int n, cudaStream_t stream) {
    if (T <= 0) return 0;
    const int threads = n >= 1024 ? 256 : 128;
    if (dtype == DT_F32)
        return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, rms_rows_kernel<float>, T, threads, 0, stream, (const float*)x, x_stride,
                                      w, eps, (float*)out, meta, n);
    return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, rms_rows_kernel<__nv_bfloat16>, T, threads, 0, stream,
                                  (const __nv_bfloat16*)x, x_stride, w, eps, (__nv_bfloat16*)out, meta, n);
}

// ----------------------------------------------------------------------------- a linear map per head
// y[t, h, n] = sum_k x[t, h, k] * w[h, n, k] (optionally times sigmoid(gate[t, h, n])).  x, y and gate are slices:
// element (t, h, i) lies at t * stride_t + h * stride_h + i (of a gate with one number per head: without the i).
#define HL_TM 8
#define HL_TN 128
#define HL_KC 512
// A block takes HL_TM tokens x HL_TN outputs of one head.  The tokens' x waits in shared memory (HL_KC columns at a
// time); a thread owns one output and reads its weight row itself, 16 bytes a load where the rows allow; every output
// is one accumulator running over k in order, so its value does not depend on the tile it falls in.
template <typename T>
__global__ void __launch_bounds__(HL_TN)
head_linear_kernel(const T* __restrict__ x, long long xs_t, long long xs_h, const T* __restrict__ w, T* __restrict__ y,
                   long long ys_t, long long ys_h, const T* __restrict__ gate, long long gs_t, long long gs_h,
                   int gate_per_head, const int* __restrict__ meta, int K, int N, int wvec) {
    __shared__ float xs[HL_TM][HL_KC];
    pdl_launch_dependents();
    pdl_wait();
    const int ntok = meta[META_NUM_TOKENS];
    const int t0 = blockIdx.x * HL_TM, h = blockIdx.y, n0 = blockIdx.z * blockDim.x, tid = threadIdx.x;
    if (t0 >= ntok) return;
    const int rows = min(HL_TM, ntok - t0), n = n0 + tid;
    const T* wr = w + ((size_t)h * N + min(n, N - 1)) * K;
    constexpr int V = 16 / sizeof(T);
    float acc[HL_TM];
#pragma unroll
    for (int m = 0; m < HL_TM; ++m) acc[m] = 0.f;
    for (int k0 = 0; k0 < K; k0 += HL_KC) {
        const int kc = min(HL_KC, K - k0);
        __syncthreads();
        for (int idx = tid; idx < HL_TM * kc; idx += blockDim.x) {
            const int m = idx / kc, kk = idx % kc;
            xs[m][kk] = m < rows ? to_float(x[(size_t)(t0 + m) * xs_t + (size_t)h * xs_h + k0 + kk]) : 0.f;
        }
        __syncthreads();
        int kk = 0;
        if (wvec) {
            for (; kk + V <= kc; kk += V) {
                const uint4 raw = *reinterpret_cast<const uint4*>(wr + k0 + kk);
                const T* wv = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    const float f = to_float(wv[i]);
#pragma unroll
                    for (int m = 0; m < HL_TM; ++m) acc[m] = fmaf(xs[m][kk + i], f, acc[m]);
                }
            }
        }
        for (; kk < kc; ++kk) {
            const float f = to_float(wr[k0 + kk]);
#pragma unroll
            for (int m = 0; m < HL_TM; ++m) acc[m] = fmaf(xs[m][kk], f, acc[m]);
        }
    }
    if (n >= N) return;
    for (int m = 0; m < rows; ++m) {
        float v = acc[m];
        if (gate) {
            const float g = to_float(gate[(size_t)(t0 + m) * gs_t + (size_t)h * gs_h + (gate_per_head ? 0 : n)]);
            v = v / (1.f + expf(-g));
        }
        y[(size_t)(t0 + m) * ys_t + (size_t)h * ys_h + n] = from_float<T>(v);
    }
}

// Few rows of bfloat16 (a decode step): a block takes 8 tokens x 16 outputs of one head, eight lanes share an output.  A lane's
// pieces of the weight row (16 bytes each, every eighth piece; up to P of them, K <= 64 P) are in registers before the
// dependency wait; the tokens' rows wait in shared memory as they are; the eight lanes' sums of the eight tokens are
// exchanged so that lane m ends with token m's.  The order of a sum depends on K alone.
template <int P>
__global__ void __launch_bounds__(128)
head_linear_few_kernel(const __nv_bfloat16* __restrict__ x, long long xs_t, long long xs_h, const __nv_bfloat16* __restrict__ w,
                       __nv_bfloat16* __restrict__ y, long long ys_t, long long ys_h, const __nv_bfloat16* __restrict__ gate, long long gs_t,
                       long long gs_h, int gate_per_head, const int* __restrict__ meta, int K, int N, int xvec) {
    __shared__ __align__(16) __nv_bfloat16 xs[8][64 * P];
    const int tid = threadIdx.x, lane = tid & 7, t0 = blockIdx.x * 8, h = blockIdx.y, n = blockIdx.z * 16 + tid / 8;
    const int rows = min(8, meta[META_NUM_TOKENS] - t0), pieces = K / 8;
    uint4 wr[P];
    const __nv_bfloat16* wrow = w + ((size_t)h * N + min(n, N - 1)) * K;
#pragma unroll
    for (int j = 0; j < P; ++j) wr[j] = lane + 8 * j < pieces ? *reinterpret_cast<const uint4*>(wrow + (lane + 8 * j) * 8) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    pdl_launch_dependents();
    if (rows <= 0) return;
    if (xvec) {  // the rows' slices start on 16 bytes
#pragma unroll
        for (int it = 0; it < (8 * 8 * P + 127) / 128; ++it) {
            const int idx = it * 128 + tid, m = idx / (8 * P), pc = idx % (8 * P);
            if (m < 8) {
                uint4 v = make_uint4(0, 0, 0, 0);
                if (m < rows && pc < pieces) v = *reinterpret_cast<const uint4*>(x + (size_t)(t0 + m) * xs_t + (size_t)h * xs_h + pc * 8);
                *reinterpret_cast<uint4*>(&xs[m][pc * 8]) = v;
            }
        }
    } else {
        for (int m = 0; m < 8; ++m)
            for (int k = tid; k < 64 * P; k += 128)
                xs[m][k] = m < rows && k < K ? x[(size_t)(t0 + m) * xs_t + (size_t)h * xs_h + k] : __float2bfloat16(0.f);
    }
    __syncthreads();
    float acc[8];
#pragma unroll
    for (int m = 0; m < 8; ++m) acc[m] = 0.f;
#pragma unroll
    for (int j = 0; j < P; ++j) {
        float wv[8];
        const __nv_bfloat16* we = reinterpret_cast<const __nv_bfloat16*>(&wr[j]);
#pragma unroll
        for (int k = 0; k < 8; ++k) wv[k] = to_float(we[k]);
#pragma unroll
        for (int m = 0; m < 8; ++m) {
            const uint4 raw = *reinterpret_cast<const uint4*>(&xs[m][(lane + 8 * j) * 8]);
            const __nv_bfloat16* xe = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
            for (int k = 0; k < 8; ++k) acc[m] = fmaf(to_float(xe[k]), wv[k], acc[m]);
        }
    }
    // halving: after the step with distance s a lane holds the sums of the tokens that agree with it in the bits seen so far
    float four[4], two[2];
#pragma unroll
    for (int m = 0; m < 4; ++m) {
        const float keep = lane & 4 ? acc[m + 4] : acc[m], give = lane & 4 ? acc[m] : acc[m + 4];
        four[m] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const float keep = lane & 2 ? four[m + 2] : four[m], give = lane & 2 ? four[m] : four[m + 2];
        two[m] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
    }
    float v = (lane & 1 ? two[1] : two[0]) + __shfl_xor_sync(0xffffffffu, lane & 1 ? two[0] : two[1], 1);
    if (lane >= rows || n >= N) return;
    if (gate) v = v / (1.f + expf(-to_float(gate[(size_t)(t0 + lane) * gs_t + (size_t)h * gs_h + (gate_per_head ? 0 : n)])));
    y[(size_t)(t0 + lane) * ys_t + (size_t)h * ys_h + n] = __float2bfloat16_rn(v);
}

extern "C" int head_linear(const void* x, long long xs_t, long long xs_h, const void* w, void* y, long long ys_t,
                           long long ys_h, const void* gate, long long gs_t, long long gs_h, int gate_per_head, int dtype, const int* meta,
                           int T, int heads, int K, int N, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (dtype == DT_BF16 && T < 64 && K % 8 == 0 && K <= 512 && ((uintptr_t)w & 15) == 0) {
        const dim3 few((T + 7) / 8, heads, (N + 15) / 16);
        const int xvec = xs_t % 8 == 0 && xs_h % 8 == 0 && ((uintptr_t)x & 15) == 0;
#define FEW_CASE(P)                                                                                                              \
        return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, head_linear_few_kernel<P>, few, 128, 0, stream, (const __nv_bfloat16*)x, xs_t, xs_h, \
                                      (const __nv_bfloat16*)w, (__nv_bfloat16*)y, ys_t, ys_h, (const __nv_bfloat16*)gate, gs_t, gs_h, gate_per_head, \
                                      meta, K, N, xvec)
        if (K <= 64) FEW_CASE(1);
        if (K <= 128) FEW_CASE(2);
        if (K <= 256) FEW_CASE(4);
        FEW_CASE(8);
#undef FEW_CASE
    }
    const int tn = N <= 32 ? 32 : (N <= 64 ? 64 : HL_TN);  // few outputs a head: smaller blocks, all of their threads at work
    dim3 grid((T + HL_TM - 1) / HL_TM, heads, (N + tn - 1) / tn);
    const int elem = dtype == DT_F32 ? 4 : 2;
    const int wvec = ((size_t)K * elem) % 16 == 0 && ((uintptr_t)w & 15) == 0;
    if (dtype == DT_F32)
        return (int)launch_kernel(head_linear_kernel<float>, grid, tn, 0, stream, (const float*)x, xs_t, xs_h, (const float*)w,
                                  (float*)y, ys_t, ys_h, (const float*)gate, gs_t, gs_h, gate_per_head, meta, K, N, wvec);
    return (int)launch_kernel(head_linear_kernel<__nv_bfloat16>, grid, tn, 0, stream, (const __nv_bfloat16*)x, xs_t, xs_h,
                              (const __nv_bfloat16*)w, (__nv_bfloat16*)y, ys_t, ys_h, (const __nv_bfloat16*)gate, gs_t, gs_h,
                              gate_per_head, meta, K, N, wvec);
}

// y[t, h, n] *= sigmoid(gate[t, h, n]) for a product that a library made (same slices as above).  ``vec``: every head's
// slice of y and of gate starts on 16 bytes and N is a multiple of 16 bytes' worth of elements; a thread then maps 16 bytes.
template <typename T>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(T* __restrict__ y, long long ys_t, long long ys_h, const T* __restrict__ gate, long long gs_t,
                    long long gs_h, const int* __restrict__ meta, int heads, int N, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    if (t >= meta[META_NUM_TOKENS]) return;
    if (vec) {
        constexpr int V = 16 / (int)sizeof(T);
        for (int idx = threadIdx.x * V; idx < heads * N; idx += blockDim.x * V) {
            const int h = idx / N, n = idx % N;
            uint4 gv = *reinterpret_cast<const uint4*>(gate + (size_t)t * gs_t + (size_t)h * gs_h + n);
            uint4* at = reinterpret_cast<uint4*>(y + (size_t)t * ys_t + (size_t)h * ys_h + n);
            uint4 yv = *at;
            const T* ge = reinterpret_cast<const T*>(&gv);
            T* ye = reinterpret_cast<T*>(&yv);
#pragma unroll
            for (int i = 0; i < V; ++i) ye[i] = from_float<T>(to_float(ye[i]) / (1.f + expf(-to_float(ge[i]))));
            *at = yv;
        }
        return;
    }
    for (int idx = threadIdx.x; idx < heads * N; idx += blockDim.x) {
        const int h = idx / N, n = idx % N;
        const float g = to_float(gate[(size_t)t * gs_t + (size_t)h * gs_h + n]);
        T* at = y + (size_t)t * ys_t + (size_t)h * ys_h + n;
        *at = from_float<T>(to_float(*at) / (1.f + expf(-g)));
    }
}

extern "C" int sigmoid_gate(void* y, long long ys_t, long long ys_h, const void* gate, long long gs_t, long long gs_h,
                            int dtype, const int* meta, int T, int heads, int N, cudaStream_t stream) {
    if (T <= 0) return 0;
    const long long V = dtype == DT_F32 ? 4 : 8;
    const int vec = N % V == 0 && ys_t % V == 0 && ys_h % V == 0 && gs_t % V == 0 && gs_h % V == 0 &&
                    ((uintptr_t)y | (uintptr_t)gate) % 16 == 0;
    const int threads = (int)std::min<long long>(256, std::max<long long>(32, ((long long)heads * N / (vec ? V : 1) + 31) / 32 * 32));
    if (dtype == DT_F32)
        return (int)launch_kernel(sigmoid_gate_kernel<float>, T, threads, 0, stream, (float*)y, ys_t, ys_h, (const float*)gate, gs_t,
                                  gs_h, meta, heads, N, vec);
    return (int)launch_kernel(sigmoid_gate_kernel<__nv_bfloat16>, T, threads, 0, stream, (__nv_bfloat16*)y, ys_t, ys_h,
                              (const __nv_bfloat16*)gate, gs_t, gs_h, meta, heads, N, vec);
}

// ----------------------------------------------------------------------------- the rows of latent attention
// Per token: the cached vector [c | rotated key part | zeros] with c = dkv[:rank] * rsqrt(mean(.^2) + eps) * norm_w
// goes to the key plane and to the value plane of the token's page (one key/value head of D elements); the queries, whose
// first `rank` elements are in place, get [rotated q_rot[h] | zeros] behind them, D elements a head.  Rotation: of the first `rot` dimensions of a
// rotated part, 2i pairs with 2i + 1 (`halves`: i with i + rot / 2), by the angle position * inv_freq[i] (float32 product, sincosf).
// Two neighbouring elements at once (the address a multiple of two elements): a rotation's pair.
__device__ __forceinline__ void load2(const float* p, float& a, float& b) { const float2 t = *reinterpret_cast<const float2*>(p); a = t.x; b = t.y; }
__device__ __forceinline__ void load2(const __nv_bfloat16* p, float& a, float& b) {
    const float2 t = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    a = t.x; b = t.y;
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

// Elements j and j + 1 (j even) of a rotated part whose element 0 is at `p`, turned if they belong to the first `rot`:
// interleaved, 2i pairs with 2i + 1; `halves`: i pairs with i + rot / 2 (rot / 2 even, so both partners are one access).
template <typename T>
__device__ __forceinline__ void turned2(const T* p, int j, int rot, int halves, const float* cs, const float* sn, float& a, float& b) {
    load2(p + j, a, b);
    if (j >= rot) return;
    const float a0 = a, b0 = b;
    if (!halves) {
        rotate_pair(a0, b0, cs[j >> 1], sn[j >> 1], a, b);
        return;
    }
    const int half = rot / 2;
    float c, d, unused;
    if (j < half) {
        load2(p + j + half, c, d);
        rotate_pair(a0, c, cs[j], sn[j], a, unused);
        rotate_pair(b0, d, cs[j + 1], sn[j + 1], b, unused);
    } else {
        const int f = j - half;
        load2(p + f, c, d);
        rotate_pair(c, a0, cs[f], sn[f], unused, a);
        rotate_pair(d, b0, cs[f + 1], sn[f + 1], unused, b);
    }
}
// One element likewise, any sizes.
template <typename T>
__device__ __forceinline__ float turned1(const T* p, int j, int rot, int halves, const float* cs, const float* sn) {
    const float v = to_float(p[j]);
    if (j >= rot) return v;
    const int half = rot / 2, f = halves ? (j < half ? j : j - half) : j >> 1;
    const bool low = halves ? j < half : !(j & 1);
    const float other = to_float(p[halves ? (low ? j + half : f) : j ^ 1]);
    float lo, hi;
    rotate_pair(low ? v : other, low ? other : v, cs[f], sn[f], lo, hi);
    return low ? lo : hi;
}

// A block takes one token.  `pairs`: sizes, strides and addresses are even, so a thread takes two neighbouring elements with
// one access.
template <typename T>
__global__ void __launch_bounds__(256)
latent_rows_kernel(const T* __restrict__ q_rot, long long qs_t, long long qs_h, const T* __restrict__ dkv, long long dkv_stride,
                   const float* __restrict__ norm_w, float eps, const int* __restrict__ positions,
                   const int* __restrict__ token_entry, const int* __restrict__ meta, int group,
                   const float* __restrict__ inv_freq, int rot, int halves, T* __restrict__ q_out, T* __restrict__ cache,
                   int heads, int rank, int rdim, int D, int page_size, int num_pages, int store, int pairs, int* __restrict__ status) {
    __shared__ float red[33];
    extern __shared__ float cs[];  // rot / 2 cosines, rot / 2 sines
    float* sn = cs + rot / 2;
    // The step's metadata is written by no kernel of the step: it is read before the wait.
    const int t = blockIdx.x, tid = threadIdx.x;
    const bool live = t < meta[META_NUM_TOKENS];
    const int p = live ? positions[t] : 0;
    int page = 0;
    if (live && store) page = (meta + meta[META_BT_OFFSET + group] + (size_t)token_entry[t] * meta[META_BT_STRIDE + group])[p / page_size];
    if (live)
        for (int i = tid; i < rot / 2; i += blockDim.x) sincosf((float)p * inv_freq[i], &sn[i], &cs[i]);
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    __syncthreads();  // the cosines and sines are written
    const int tail = D - rank;
    const T* qt = q_rot + (size_t)t * qs_t;
    T* qo = q_out + (size_t)t * heads * D + rank;
    if (pairs) {
        const int per = tail / 2;
        for (int it = tid; it < heads * per; it += blockDim.x) {
            const int h = it / per, j = (it % per) * 2;
            float a = 0.f, b = 0.f;
            if (j < rdim) turned2(qt + (size_t)h * qs_h, j, rot, halves, cs, sn, a, b);
            store2(qo + (size_t)h * D + j, a, b);
        }
    } else {
        for (int it = tid; it < heads * tail; it += blockDim.x) {
            const int h = it / tail, j = it % tail;
            qo[(size_t)h * D + j] = from_float<T>(j < rdim ? turned1(qt + (size_t)h * qs_h, j, rot, halves, cs, sn) : 0.f);
        }
    }
    if (!store) return;
    const T* kv = dkv + (size_t)t * dkv_stride;
    float ss = 0.f;
    if (pairs) {
        for (int i = tid * 2; i < rank; i += blockDim.x * 2) {
            float a, b;
            load2(kv + i, a, b);
            ss = fmaf(a, a, ss);
            ss = fmaf(b, b, ss);
        }
    } else {
        for (int i = tid; i < rank; i += blockDim.x) {
            const float v = to_float(kv[i]);
            ss = fmaf(v, v, ss);
        }
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)rank + eps);
    if (page <= 0 || page >= num_pages) {
        if (tid == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + t);
        return;
    }
    CacheLayout L{1, page_size, D};
    T* kdst = cache + L.offset(page, 0, 0, p % page_size);
    T* vdst = cache + L.offset(page, 1, 0, p % page_size);
    if (pairs) {
        for (int i = tid * 2; i < D; i += blockDim.x * 2) {
            float a = 0.f, b = 0.f;
            if (i < rank) {
                load2(kv + i, a, b);
                a = a * inv * norm_w[i];
                b = b * inv * norm_w[i + 1];
            } else if (i < rank + rdim) {
                turned2(kv + rank, i - rank, rot, halves, cs, sn, a, b);
            }
            store2(kdst + i, a, b);
            store2(vdst + i, a, b);
        }
        return;
    }
    for (int i = tid; i < D; i += blockDim.x) {
        float v = 0.f;
        if (i < rank) v = to_float(kv[i]) * inv * norm_w[i];
        else if (i < rank + rdim) v = turned1(kv + rank, i - rank, rot, halves, cs, sn);
        const T o = from_float<T>(v);
        kdst[i] = o;
        vdst[i] = o;
    }
}

extern "C" int latent_rows(const void* q_rot, long long qs_t, long long qs_h, const void* dkv, long long dkv_stride, const float* norm_w,
                           float eps, const int* positions, const int* token_entry, const int* meta, int group, const float* inv_freq,
                           int rot, int halves, void* q_out, void* cache, int dtype, int T, int heads, int rank, int rdim, int D,
                           int page_size, int num_pages, int store, int* status, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rot % 2 || rot > rdim || rank + rdim > D || (rot && !inv_freq)) return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)rot * sizeof(float);
    const int elem = dtype == DT_F32 ? 4 : 2;
    const int pairs = rank % 2 == 0 && rdim % 2 == 0 && D % 2 == 0 && (!halves || rot % 4 == 0) && qs_t % 2 == 0 && qs_h % 2 == 0 &&
                      dkv_stride % 2 == 0 && (((uintptr_t)q_rot | (uintptr_t)dkv | (uintptr_t)q_out | (uintptr_t)cache) % (2 * elem)) == 0;
    const int threads = T >= 512 ? 128 : 256;  // few tokens: the shortest path through a token
    if (dtype == DT_F32)
        return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, latent_rows_kernel<float>, T, threads, smem, stream, (const float*)q_rot, qs_t, qs_h,
                                      (const float*)dkv, dkv_stride, norm_w, eps, positions, token_entry, meta, group, inv_freq, rot, halves,
                                      (float*)q_out, (float*)cache, heads, rank, rdim, D, page_size, num_pages, store, pairs, status);
    return (int)launch_kernel_pdl((g_use_pdl & 5) != 0, latent_rows_kernel<__nv_bfloat16>, T, threads, smem, stream, (const __nv_bfloat16*)q_rot,
                                  qs_t, qs_h, (const __nv_bfloat16*)dkv, dkv_stride, norm_w, eps, positions, token_entry, meta, group, inv_freq,
                                  rot, halves, (__nv_bfloat16*)q_out, (__nv_bfloat16*)cache, heads, rank, rdim, D, page_size, num_pages, store,
                                  pairs, status);
}
