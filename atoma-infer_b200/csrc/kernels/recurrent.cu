// Recurrent mixers whose state is a matrix per head or per channel and whose decay differs from row to row:
//  * gated linear attention: per head S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, a_t = sigmoid(z_t)^(1/tau);
//  * the selective scan of the Mamba kind: per channel c and state n, S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n,
//    y_c = sum_n S[c, n] C_n + D_c u_c, times silu(z_c);
//  * the norm per head with a weight shared by the heads, times silu(gate), behind the first.
// Storage of projections is float32 or bfloat16; states, decays, step sizes, gates and norms are float32 always.  A
// request's tokens run in order from its state slot (pass 0), or, for long portions, cut into chunks of time that run
// side by side: pass 1 runs every chunk but the last from a zero state and leaves its end state and what its decays
// amount to, a small kernel chains the chunks' start states in order, pass 3 runs every chunk again from its start
// state and writes the outputs, the last chunk the slot.  Every sum runs in an order that depends on the sizes only.
#include "matrix_scan.cuh"

int g_use_pdl = 1;
extern "C" void kernels_set_pdl(int mode) { g_use_pdl = mode; }

// ----------------------------------------------------------------------------- gated linear attention
// q, k [T, heads * N], v [T, heads * P]: slices of wider rows (strides in elements); z float32 [T, heads * N], the decay's
// logits before their bias.  state [slots][heads][N][P]; o float32 [T, heads * P].

extern "C" size_t gla_scan_scratch_floats(int S, int heads, int N, int P, int max_chunks) {
    return scan_scratch_floats<SCAN_DECAY>(S, heads, N, P, max_chunks);
}

// mode bit 0: the decay is a constant per head, z_bias[h] (float32 [heads]; z is not read); bit 1: q, k and v pass through
// SiLU as they are loaded.
extern "C" int gla_scan_mode(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long long v_stride,
                             int dtype, const float* z, long long z_stride, const float* z_bias, float tau, float q_scale,
                             float* state, long long slot_stride, float* o, const int* meta, const int* cu_tokens, const int* slots,
                             int S, int heads, int N, int P, int chunk_len, int max_chunks, float* scratch, int mode,
                             cudaStream_t stream) {
    if (S > 0 && ((mode & 1) ? !z_bias : !z)) return (int)cudaErrorInvalidValue;
    const ScanArgs a = {q, k, v, q_stride, k_stride, v_stride, dtype, z, z_bias, z_stride, tau, q_scale, state, slot_stride, o, meta,
                        cu_tokens, slots, S, heads, N, P, chunk_len, max_chunks, scratch, mode, {}};
    return run_matrix_scan<SCAN_DECAY>(a, stream);
}

extern "C" int gla_scan(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long long v_stride,
                        int dtype, const float* z, long long z_stride, const float* z_bias, float tau, float q_scale,
                        float* state, long long slot_stride, float* o, const int* meta, const int* cu_tokens, const int* slots,
                        int S, int heads, int N, int P, int chunk_len, int max_chunks, float* scratch, cudaStream_t stream) {
    return gla_scan_mode(q, q_stride, k, k_stride, v, v_stride, dtype, z, z_stride, z_bias, tau, q_scale, state, slot_stride, o, meta,
                         cu_tokens, slots, S, heads, N, P, chunk_len, max_chunks, scratch, 0, stream);
}

// ----------------------------------------------------------------------------- norm per head, shared weight, gate
// out[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * w * silu(g[t, h, :]); o float32 [T, heads * P], g a slice of
// wider rows, w float32 [P].  A warp a (token, head).
template <typename T>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ g, long long g_stride, const float* __restrict__ w,
                      float eps, T* __restrict__ out, const int* __restrict__ meta, int heads, int P) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (t >= meta[META_NUM_TOKENS] || h >= heads) return;
    const float* row = o + ((size_t)t * heads + h) * P;
    const T* gate = g + (size_t)t * g_stride + (size_t)h * P;
    float ss = 0.f;
    for (int i = lane; i < P; i += 32) ss = fmaf(row[i], row[i], ss);
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / (float)P + eps);
    T* dst = out + ((size_t)t * heads + h) * P;
    for (int i = lane; i < P; i += 32) dst[i] = from_float<T>(row[i] * inv * w[i] * silu_f(to_float(gate[i])));
}

extern "C" int head_norm_gate(const float* o, const void* g, int dtype, long long g_stride, const float* w, float eps, void* out,
                              const int* meta, int T, int heads, int P, cudaStream_t stream) {
    if (T <= 0) return 0;
    const dim3 grid(T, (heads + 3) / 4);
    if (dtype == DT_F32)
        return (int)launch_kernel(head_norm_gate_kernel<float>, grid, 128, 0, stream, o, (const float*)g, g_stride, w, eps,
                                  (float*)out, meta, heads, P);
    return (int)launch_kernel(head_norm_gate_kernel<__nv_bfloat16>, grid, 128, 0, stream, o, (const __nv_bfloat16*)g, g_stride, w,
                              eps, (__nv_bfloat16*)out, meta, heads, P);
}

// ----------------------------------------------------------------------------- selective scan
// u [T, inner] (after convolution and activation), zg [T, inner] (the gate's input): slices of wider rows; dt_raw float32
// [T, inner] (softplus(dt_raw + dt_bias) is taken here); B at bc, C at bc + N of a row of bc_stride elements; a_log [inner, N];
// state [slots][inner][N]; out [T, inner] = (sum_n S[c, n] C_n + D_c u_c) * silu(zg_c).
// One block per (channel block, entry[, chunk]).  Thread (c, r) keeps NPT states n = r * NPT .. of channel c, as pairs of
// neighbouring states that one two-wide instruction updates.  y is the even states' sum plus the odd states', each in
// ascending order, then the R threads' sums by halving.  B and C of 16 tokens are staged in shared memory; the channel's
// own u, step size and gate input of those tokens go straight into the thread's registers.
#define LOG2E_F 1.4426950408889634f

// 2^x for x <= 0 by one approximate PTX instruction (a result below the smallest normal number is zero, which a decay of
// that size is for every state that float32 holds).
__device__ __forceinline__ float ex2_nonpositive(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <typename T, int NPT, bool WRITE_Y>
__global__ void __launch_bounds__(256)
selective_scan_kernel(const T* __restrict__ u, long long u_stride, const float* __restrict__ dt_raw,
                      const float* __restrict__ dt_bias, const T* __restrict__ bc, long long bc_stride,
                      const T* __restrict__ zg, long long z_stride, const float* __restrict__ a_log,
                      const float* __restrict__ d_skip, float* __restrict__ state, long long slot_stride, T* __restrict__ out,
                      const int* __restrict__ meta, const int* __restrict__ cu_tokens, const int* __restrict__ slots,
                      int inner, int N, int R, int CPB, int pass, int chunk_len, int max_chunks, float* __restrict__ scratch,
                      float* __restrict__ dt_sums) {
    extern __shared__ __align__(16) float sm[];
    const int SL = R > 1 ? NPT + 4 : NPT, NL = R * NPT, NP = R * SL;
    float* Bs = sm;                      // [REC_TT][NP]
    float* Cs = Bs + REC_TT * NP;        // [REC_TT][NP]
    const int e = blockIdx.y, ch = blockIdx.z;
    const int tid = threadIdx.x, cl = tid / R, r = tid % R, c = blockIdx.x * CPB + cl;
    const bool real = cl < CPB && c < inner;
    // the weights come before the wait: no kernel writes them
    float2 A2[NPT / 2];  // A log2(e), pairs of neighbouring states
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
        const int n = r * NPT + i;
        const float a = (real && n < N) ? -expf(a_log[(size_t)c * N + n]) * LOG2E_F : 0.f;
        if (i & 1) A2[i / 2].y = a; else A2[i / 2].x = a;
    }
    const float dskip = real ? d_skip[c] : 0.f, dtb = real ? dt_bias[c] : 0.f;
    pdl_launch_dependents();
    pdl_wait();
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int first = cu_tokens[e], count = cu_tokens[e + 1] - first;
    const int nchunks = pass == 0 ? 1 : (count + chunk_len - 1) / chunk_len;
    if (ch >= nchunks || (pass == 1 && ch == nchunks - 1)) return;
    const int t0 = first + (pass == 0 ? 0 : ch * chunk_len), t1 = pass == 0 ? first + count : min(first + count, t0 + chunk_len);
    const size_t HS = (size_t)inner * N;
    float* slot_state = state + (size_t)slots[e] * slot_stride;
    float* chunk_state = scratch ? scratch + ((size_t)e * max_chunks + ch) * HS : nullptr;
    const float* init = pass == 0 ? slot_state : (pass == 3 ? chunk_state : nullptr);
    float2 S[NPT / 2];
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
        const int n = r * NPT + i;
        const float s0 = (init && real && n < N) ? init[(size_t)c * N + n] : 0.f;
        if (i & 1) S[i / 2].y = s0; else S[i / 2].x = s0;
    }
    float dt_sum = 0.f;
    for (int tb = t0; tb < t1; tb += REC_TT) {
        const int nt = min(REC_TT, t1 - tb);
        // this thread's channel of the tile's tokens, straight into registers: every load is on its way before the
        // first is used (the R threads of a channel read the same addresses)
        T ur[REC_TT], zr[REC_TT];
        float dr[REC_TT];
#pragma unroll
        for (int tt = 0; tt < REC_TT; ++tt) {
            const bool in = real && tt < nt;
            const size_t t = (size_t)(tb + tt);
            ur[tt] = in ? u[t * u_stride + c] : from_float<T>(0.f);
            dr[tt] = in ? dt_raw[t * inner + c] : 0.f;
            if (WRITE_Y) zr[tt] = in ? zg[t * z_stride + c] : from_float<T>(0.f);
        }
        __syncthreads();
        for (int idx = tid; idx < nt * NL; idx += blockDim.x) {
            const int tt = idx / NL, n = idx % NL, at = tt * NP + (n / NPT) * SL + n % NPT;
            const T* row = bc + (size_t)(tb + tt) * bc_stride;
            Bs[at] = n < N ? to_float(row[n]) : 0.f;
            Cs[at] = n < N ? to_float(row[N + n]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int tt = 0; tt < REC_TT; ++tt) {
            if (tt >= nt) break;
            const float uv = to_float(ur[tt]), step = real ? softplus_f(dr[tt] + dtb) : 0.f;
            const float dx = step * uv;
            const float* Bt = Bs + tt * NP + r * SL;
            const float* Ct = Cs + tt * NP + r * SL;
            const float2 st2 = make_float2(step, step), dx2 = make_float2(dx, dx);
            float2 acc2 = make_float2(0.f, 0.f);
#pragma unroll
            for (int i = 0; i < NPT / 2; i += 2) {  // two pairs of neighbouring states a round
                const float4 b4 = *reinterpret_cast<const float4*>(Bt + 2 * i);
                float2 ea = mul2(st2, A2[i]), eb = mul2(st2, A2[i + 1]);
                ea = make_float2(ex2_nonpositive(ea.x), ex2_nonpositive(ea.y));
                eb = make_float2(ex2_nonpositive(eb.x), ex2_nonpositive(eb.y));
                S[i] = fma2(ea, S[i], mul2(dx2, make_float2(b4.x, b4.y)));
                S[i + 1] = fma2(eb, S[i + 1], mul2(dx2, make_float2(b4.z, b4.w)));
                if (WRITE_Y) {
                    const float4 c4 = *reinterpret_cast<const float4*>(Ct + 2 * i);
                    acc2 = fma2(S[i], make_float2(c4.x, c4.y), acc2);
                    acc2 = fma2(S[i + 1], make_float2(c4.z, c4.w), acc2);
                }
            }
            float acc = acc2.x + acc2.y;  // the even states' sum plus the odd states'
            if (WRITE_Y) {
                for (int s = R >> 1; s > 0; s >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, s);
                if (real && r == 0) {
                    const float y = fmaf(dskip, uv, acc);
                    out[(size_t)(tb + tt) * inner + c] = from_float<T>(y * silu_f(to_float(zr[tt])));
                }
            }
            dt_sum += step;
        }
    }
    float* fin = pass == 1 ? chunk_state + HS : ((pass == 0 || ch == nchunks - 1) ? slot_state : nullptr);
    if (fin && real) {
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
            const int n = r * NPT + i;
            if (n < N) fin[(size_t)c * N + n] = (i & 1) ? S[i / 2].y : S[i / 2].x;
        }
    }
    if (pass == 1 && real && r == 0) dt_sums[((size_t)e * max_chunks + ch) * inner + c] = dt_sum;
}

// scratch[e, 0] = the slot's state; scratch[e, c] = exp(A * (sum of the steps of chunk c - 1)) * scratch[e, c - 1] + scratch[e, c].
__global__ void __launch_bounds__(256)
selective_chunk_states_kernel(const float* __restrict__ state, long long slot_stride, float* __restrict__ scratch,
                              const float* __restrict__ dt_sums, const float* __restrict__ a_log, const int* __restrict__ meta,
                              const int* __restrict__ cu_tokens, const int* __restrict__ slots, int inner, int N, int chunk_len,
                              int max_chunks) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.y;
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int count = cu_tokens[e + 1] - cu_tokens[e], nchunks = (count + chunk_len - 1) / chunk_len;
    const long long HS = (long long)inner * N, i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= HS) return;
    const int c = (int)(i / N);
    const float a2 = -expf(a_log[i]) * LOG2E_F;
    float s = state[(size_t)slots[e] * slot_stride + i];
    scratch[((size_t)e * max_chunks) * HS + i] = s;
    for (int k = 1; k < nchunks; ++k) {
        float* at = scratch + ((size_t)e * max_chunks + k) * HS + i;
        s = fmaf(exp2f(a2 * dt_sums[((size_t)e * max_chunks + k - 1) * inner + c]), s, *at);
        *at = s;
    }
}

extern "C" size_t selective_scan_scratch_floats(int S, int inner, int N, int max_chunks) {
    return (size_t)S * max_chunks * ((size_t)inner * N + inner);
}

extern "C" int selective_scan(const void* u, long long u_stride, const float* dt_raw, const float* dt_bias, const void* bc,
                              long long bc_stride, const void* zg, long long z_stride, int dtype, const float* a_log,
                              const float* d_skip, float* state, long long slot_stride, void* out, const int* meta,
                              const int* cu_tokens, const int* slots, int S, int inner, int N, int chunk_len, int max_chunks,
                              float* scratch, cudaStream_t stream) {
    if (S <= 0) return 0;
    int NPT = 0, R = 0, CPB = 0;
    if (!rec_geometry(N, inner, &NPT, &R, &CPB)) return (int)cudaErrorInvalidValue;
    if (CPB * R > 128) CPB = 128 / R > 0 ? 128 / R : 1;  // 128 threads a block: more blocks for few requests
    const int blocks = (inner + CPB - 1) / CPB, threads = ((CPB * R + 31) / 32) * 32;
    const size_t smem = (size_t)(2 * REC_TT * R * (R > 1 ? NPT + 4 : NPT)) * sizeof(float);
    if (smem > 96 * 1024) return (int)cudaErrorInvalidValue;
    float* dt_sums = scratch ? scratch + (size_t)S * max_chunks * (size_t)inner * N : nullptr;
#define SEL_CASE(TT, K, W, pass, chunks)                                                                                    \
    case K: {                                                                                                              \
        static size_t configured = 0;                                                                                      \
        if (smem > 48 * 1024 && smem > configured) {                                                                       \
            cudaError_t ce = cudaFuncSetAttribute(selective_scan_kernel<TT, K, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (ce != cudaSuccess) return (int)ce;                                                                         \
            configured = smem;                                                                                             \
        }                                                                                                                  \
        err = (int)launch_kernel(selective_scan_kernel<TT, K, W>, dim3(blocks, S, chunks), threads, smem, stream, (const TT*)u, u_stride, \
                                 dt_raw, dt_bias, (const TT*)bc, bc_stride, (const TT*)zg, z_stride, a_log, d_skip, state,       \
                                 slot_stride, (TT*)out, meta, cu_tokens, slots, inner, N, R, CPB, pass, chunk_len, max_chunks,   \
                                 scratch, dt_sums);                                                                        \
        break;                                                                                                             \
    }
#define SEL_PASS(TT, W, pass, chunks)                                                                                       \
    switch (NPT) { SEL_CASE(TT, 8, W, pass, chunks) SEL_CASE(TT, 16, W, pass, chunks) SEL_CASE(TT, 32, W, pass, chunks) SEL_CASE(TT, 64, W, pass, chunks) }
    int err = 0;
    if (chunk_len <= 0 || max_chunks <= 1 || !scratch) {
        if (dtype == DT_F32) { SEL_PASS(float, true, 0, 1) } else { SEL_PASS(__nv_bfloat16, true, 0, 1) }
        return err;
    }
    if (dtype == DT_F32) { SEL_PASS(float, false, 1, max_chunks) } else { SEL_PASS(__nv_bfloat16, false, 1, max_chunks) }
    if (err) return err;
    const long long HS = (long long)inner * N;
    err = (int)launch_kernel(selective_chunk_states_kernel, dim3((unsigned)((HS + 255) / 256), S), 256, 0, stream,
                             (const float*)state, slot_stride, scratch, (const float*)dt_sums, a_log, meta, cu_tokens, slots,
                             inner, N, chunk_len, max_chunks);
    if (err) return err;
    if (dtype == DT_F32) { SEL_PASS(float, true, 3, max_chunks) } else { SEL_PASS(__nv_bfloat16, true, 3, max_chunks) }
    return err;
#undef SEL_PASS
#undef SEL_CASE
}
