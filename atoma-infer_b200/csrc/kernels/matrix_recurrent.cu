// Recurrent mixers on the matrix scan whose query reads more than the decayed state:
//  * the scan whose current token enters through a bonus per key channel, decay exp(-exp(z)) per key channel;
//  * the matrix memory with exponential gates: the gates of a portion's tokens (a running maximum in the log domain, taken
//    as a parallel scan over the tokens), the scan of S and n, and
//  * the norm per head behind both, with a weight per channel of every head, a gate, and (for the memory) the division by
//    max(|n . q|, exp(-m)) + 1e-6.
// Projections are stored as float32 or bfloat16; gates, states, norms and everything between are float32.
#include "matrix_scan.cuh"

int g_use_pdl = 1;
extern "C" void kernels_set_pdl(int mode) { g_use_pdl = mode; }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// ----------------------------------------------------------------------------- the two scans
extern "C" size_t bonus_scan_scratch_floats(int S, int heads, int N, int P, int max_chunks) {
    return scan_scratch_floats<SCAN_BONUS>(S, heads, N, P, max_chunks);
}

// r, k [T, heads * N], v [T, heads * P]: slices of wider rows; z float32 rows [T, heads * N], z_bias and bonus float32
// [heads * N]; state [slots][heads][N][P]; o float32 [T, heads * P].
extern "C" int bonus_scan(const void* r, long long r_stride, const void* k, long long k_stride, const void* v, long long v_stride,
                          int dtype, const float* z, long long z_stride, const float* z_bias, const float* bonus, float* state,
                          long long slot_stride, float* o, const int* meta, const int* cu_tokens, const int* slots, int S, int heads,
                          int N, int P, int chunk_len, int max_chunks, float* scratch, cudaStream_t stream) {
    ScanExtras ex = {};
    ex.bonus = bonus;
    const ScanArgs a = {r, k, v, r_stride, k_stride, v_stride, dtype, z, z_bias, z_stride, 1.f, 1.f, state, slot_stride, o, meta,
                        cu_tokens, slots, S, heads, N, P, chunk_len, max_chunks, scratch, 0, ex};
    return run_matrix_scan<SCAN_BONUS>(a, stream);
}

extern "C" size_t memory_scan_scratch_floats(int S, int heads, int N, int P, int max_chunks) {
    return scan_scratch_floats<SCAN_MEMORY>(S, heads, N, P, max_chunks);
}

// q, k [T, heads * N], v [T, heads * P]: slices of wider rows; gates float32 [T, heads, 2] (see memory_gates); state
// [slots][heads][N][P] and n_state [slots][heads][N] with one slot stride; o float32 [T, heads * P], nq float32 [T, heads].
extern "C" int memory_scan(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long long v_stride,
                           int dtype, const float* gates, float q_scale, float* state, float* n_state, long long slot_stride, float* o,
                           float* nq, const int* meta, const int* cu_tokens, const int* slots, int S, int heads, int N, int P,
                           int chunk_len, int max_chunks, float* scratch, cudaStream_t stream) {
    ScanExtras ex = {};
    ex.gates = gates;
    ex.n_state = n_state;
    ex.nq = nq;
    const ScanArgs a = {q, k, v, q_stride, k_stride, v_stride, dtype, nullptr, nullptr, 0, 1.f, q_scale, state, slot_stride, o, meta,
                        cu_tokens, slots, S, heads, N, P, chunk_len, max_chunks, scratch, 0, ex};
    return run_matrix_scan<SCAN_MEMORY>(a, stream);
}

// ----------------------------------------------------------------------------- exponential gates
// logits float32 [T, 2 * heads], the input gates' first; bias float32 [2 * heads].  Per head: i = cap * tanh((x_i + b_i) / cap),
// f = log sigmoid(cap * tanh((x_f + b_f) / cap)); m_t = max(f_t + m_(t-1), i_t) from the request's kept m (0 at its start);
// gates[t, h] = (exp(f_t + m_(t-1) - m_t), exp(i_t - m_t)); floor[t, h] = exp(-m_t); the last m goes back to the slot.
// One block per (head, entry).  A token maps m to max(m + F, I) with F = f, I = i; such maps compose to (F1 + F2,
// max(I1 + F2, I2)), so a block's tokens are taken as an inclusive scan over lanes, then over warps in order.
__global__ void __launch_bounds__(256)
memory_gates_kernel(const float* __restrict__ logits, const float* __restrict__ bias, float cap, float* __restrict__ m_state,
                    long long slot_stride, float* __restrict__ gates, float* __restrict__ floor_out, const int* __restrict__ meta,
                    const int* __restrict__ cu_tokens, const int* __restrict__ slots, int heads) {
    __shared__ float wf[8], wi[8], s_m;
    const int h = blockIdx.x, e = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    pdl_launch_dependents();
    pdl_wait();
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int first = cu_tokens[e], end = cu_tokens[e + 1];
    float* kept = m_state + (size_t)slots[e] * slot_stride + h;
    float m_in = *kept;
    const float bi = bias[h], bf = bias[heads + h];
    for (int t0 = first; t0 < end; t0 += blockDim.x) {
        const int t = t0 + threadIdx.x;
        const bool in = t < end;
        float i = -INFINITY, f = 0.f;
        if (in) {
            const float* row = logits + (size_t)t * 2 * heads;
            i = cap * tanhf((row[h] + bi) / cap);
            const float x = cap * tanhf((row[heads + h] + bf) / cap);
            f = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
        }
        float F = f, I = i;
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, F, d), pi = __shfl_up_sync(0xffffffffu, I, d);
            if (lane >= d) {
                I = fmaxf(pi + F, I);
                F = pf + F;
            }
        }
        if (lane == 31) wf[warp] = F, wi[warp] = I;
        __syncthreads();
        float m_warp = m_in;  // m before this warp's first token
        for (int w = 0; w < warp; ++w) m_warp = fmaxf(m_warp + wf[w], wi[w]);
        const float m_t = fmaxf(m_warp + F, I);
        const float below = __shfl_up_sync(0xffffffffu, m_t, 1);
        const float m_prev = lane ? below : m_warp;
        if (in) {
            float2* dst = reinterpret_cast<float2*>(gates) + (size_t)t * heads + h;
            *dst = make_float2(expf(f + m_prev - m_t), expf(i - m_t));
            floor_out[(size_t)t * heads + h] = expf(-m_t);
        }
        if (t == end - 1 || (in && threadIdx.x == blockDim.x - 1)) s_m = m_t;
        __syncthreads();  // (also: nobody reads wf and wi any more)
        m_in = s_m;
    }
    if (threadIdx.x == 0) *kept = m_in;
}

extern "C" int memory_gates(const float* logits, const float* bias, float cap, float* m_state, long long slot_stride, float* gates,
                            float* floor_out, const int* meta, const int* cu_tokens, const int* slots, int S, int heads, int longest,
                            cudaStream_t stream) {
    if (S <= 0) return 0;
    if (cap <= 0.f) return (int)cudaErrorInvalidValue;
    return (int)launch_kernel(memory_gates_kernel, dim3(heads, S), longest > 32 ? 256 : 32, 0, stream, logits, bias, cap, m_state,
                              slot_stride, gates, floor_out, meta, cu_tokens, slots, heads);
}

// ----------------------------------------------------------------------------- norm per head, a weight per channel, gate
// out[t, h, :] = v / sqrt(mean(v^2) + eps) * w[h, :] * gate_fn(g[t, h, :]) with v = o[t, h, :], or, with `nq` and `floor_in`
// (float32 [T, heads]), v = o[t, h, :] / (max(|nq|, floor) + 1e-6).  o float32 [T, heads * P], g a slice of wider rows, w float32
// [heads * P]; kind 0: sigmoid(g), 1: g * sigmoid(g).  LPH lanes (a power of two) a (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
head_weight_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ nq, const float* __restrict__ floor_in,
                             const T* __restrict__ g, long long g_stride, const float* __restrict__ w, float eps, int kind,
                             T* __restrict__ out, const int* __restrict__ meta, int heads, int P, int vec4, int LPH) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x % LPH, h = blockIdx.y * (blockDim.x / LPH) + threadIdx.x / LPH;
    if (t >= meta[META_NUM_TOKENS]) return;
    const bool live = h < heads;  // (lanes without a head still take part in their warp's sums)
    const size_t at = ((size_t)t * heads + (live ? h : 0)) * P;
    const float* row = o + at;
    const T* gate = g + (size_t)t * g_stride + (size_t)(live ? h : 0) * P;
    const float* wr = w + (size_t)(live ? h : 0) * P;
    float c = 1.f;
    if (nq && live) c = 1.f / (fmaxf(fabsf(nq[(size_t)t * heads + h]), floor_in[(size_t)t * heads + h]) + 1e-6f);
    auto group_sum = [&](float v) {
        for (int s = LPH >> 1; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
        return v;
    };
    float ss = 0.f;
    if (vec4) {
        const int step = LPH * 4;
        for (int i = lane * 4; i < P; i += step) {
            float v[4];
            load4(row + i, v);
#pragma unroll
            for (int k = 0; k < 4; ++k) { v[k] *= c; ss = fmaf(v[k], v[k], ss); }
        }
        const float inv = rsqrtf(group_sum(ss) / (float)P + eps);
        if (!live) return;
        for (int i = lane * 4; i < P; i += step) {
            float v[4], gv[4], wv[4];
            load4(row + i, v);
            load4(gate + i, gv);
            load4(wr + i, wv);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float s = sigmoid_f(gv[k]);
                v[k] = v[k] * c * inv * wv[k] * (kind == 1 ? gv[k] * s : s);
            }
            store4(out + at + i, v);
        }
        return;
    }
    for (int i = lane; i < P; i += LPH) { const float v = row[i] * c; ss = fmaf(v, v, ss); }
    const float inv = rsqrtf(group_sum(ss) / (float)P + eps);
    if (!live) return;
    for (int i = lane; i < P; i += LPH) {
        const float gv = to_float(gate[i]), s = sigmoid_f(gv);
        out[at + i] = from_float<T>(row[i] * c * inv * wr[i] * (kind == 1 ? gv * s : s));
    }
}

extern "C" int head_weight_norm_gate(const float* o, const float* nq, const float* floor_in, const void* g, int dtype, long long g_stride,
                                     const float* w, float eps, int kind, void* out, const int* meta, int T, int heads, int P,
                                     cudaStream_t stream) {
    if (T <= 0) return 0;
    const int esz = dtype == DT_F32 ? 4 : 2;
    const int vec4 = P % 4 == 0 && g_stride % 4 == 0 && (((uintptr_t)o | (uintptr_t)w) & 15) == 0 && (((uintptr_t)g | (uintptr_t)out) % (4 * esz)) == 0;
    int LPH = 1;
    while (LPH < 32 && LPH * (vec4 ? 4 : 1) < P) LPH *= 2;
    const int threads = heads * LPH > 128 ? 256 : 128;
    const dim3 grid(T, (heads + threads / LPH - 1) / (threads / LPH));
    if (dtype == DT_F32)
        return (int)launch_kernel(head_weight_norm_gate_kernel<float>, grid, threads, 0, stream, o, nq, floor_in, (const float*)g, g_stride, w, eps,
                                  kind, (float*)out, meta, heads, P, vec4, LPH);
    return (int)launch_kernel(head_weight_norm_gate_kernel<__nv_bfloat16>, grid, threads, 0, stream, o, nq, floor_in, (const __nv_bfloat16*)g,
                              g_stride, w, eps, kind, (__nv_bfloat16*)out, meta, heads, P, vec4, LPH);
}
