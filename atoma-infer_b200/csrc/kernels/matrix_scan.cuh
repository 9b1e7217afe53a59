// The scan of recurrent mixers whose state is a matrix per head: per head and token the state's rows decay, k v^T is added and
// the query reads it.  One kernel, three kinds (template parameter KIND):
//  * SCAN_DECAY: S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; the decay from logits, a_t = sigmoid(z_t)^(1/tau), or a
//    constant per head;
//  * SCAN_BONUS: a_t = exp(-exp(z_t)); the query reads the state BEFORE the update and the current token through a bonus per
//    key channel, o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t;
//  * SCAN_MEMORY: a_t and the weight of k_t are numbers per head and token that a kernel before has computed from exponential
//    gates; beside S runs n_t = a_t n_(t-1) + b_t k_t, a column whose value is always 1, and n_t . q_t is left for the norm.
// Storage of projections is float32 or bfloat16; states and everything else are float32.  A request's tokens run in order
// from its state slot (pass 0), or, for long portions, cut into chunks of time that run side by side: pass 1 runs every
// chunk but the last from a zero state and leaves its end state and what its decays amount to, a small kernel chains the
// chunks' start states in order, pass 3 runs every chunk again from its start state and writes the outputs, the last
// chunk the slot.  Every sum runs in an order that depends on the sizes only.
#pragma once
#include "common.cuh"

#define REC_TT 16  // tokens staged in shared memory at a time
#define SCAN_DECAY 0
#define SCAN_BONUS 1
#define SCAN_MEMORY 2

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

// Two float32 operations in one instruction (sm_100): the recurrences' arithmetic is bound by instruction issue, and a
// pair of neighbouring rows comes out of one 16-byte load of shared memory as two such operands.  Each half is the plain
// IEEE operation, rounded to nearest.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)),
          "l"(reinterpret_cast<const unsigned long long&>(c)));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.f32x2 %0, %1, %2;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return d;
}

// q, k [T, heads * N], v [T, heads * P]: slices of wider rows (strides in elements); z float32 [T, heads * N], the decay's
// logits before their bias.  state [slots][heads][N][P]; o float32 [T, heads * P].
// SCAN_BONUS: `bonus` float32 [heads, N].  SCAN_MEMORY: `gates` float32 [T, heads, 2], the decay a and the weight b of k;
// `n_state` [slots][heads][N] (the same slot stride), nq float32 [T, heads].
// One block per (head x column block, entry[, chunk]).  Thread (pl, r) keeps NPT rows n = r * NPT .. of CPT neighbouring
// columns in registers (a row's k, a and q are loaded once for all of them); R threads (a power of two, neighbouring
// lanes) share the columns; rows beyond N see k = q = 0 and stay zero.  P is a multiple of CPT.  An output is the sum of
// the even rows' products plus the sum of the odd rows', each in ascending order, then the R threads' sums by halving.
template <typename T>
struct alignas(4 * sizeof(T)) Raw4 { T x[4]; };  // four stored values, loaded at once

// What only some kinds read or write.
struct ScanExtras {
    const float* bonus;   // SCAN_BONUS
    const float* gates;   // SCAN_MEMORY
    float* n_state;
    float* nq;
};

template <typename T, int NPT, bool WRITE_O, int CPT, int KIND>
__global__ void __launch_bounds__(KIND == SCAN_MEMORY ? 288 : 256, NPT <= 16 ? 2 : 1)
matrix_scan_kernel(const T* __restrict__ q, long long q_stride, const T* __restrict__ k, long long k_stride,
                const T* __restrict__ v, long long v_stride, const float* __restrict__ z, long long z_stride,
                const float* __restrict__ z_bias, float inv_tau, float q_scale, float* __restrict__ state,
                long long slot_stride, float* __restrict__ o, const int* __restrict__ meta,
                const int* __restrict__ cu_tokens, const int* __restrict__ slots, int heads, int P, int N, int R, int PB,
                int col_blocks, int pass, int chunk_len, int max_chunks, float* __restrict__ scratch,
                float* __restrict__ decay, int vec, int mode, const ScanExtras ex) {
    extern __shared__ __align__(16) float sm[];
    // mode bit 0: no logits; every row of head h decays by the constant z_bias[h].  bit 1: q, k and v pass through SiLU.
    const bool fixed = mode & 1, act = mode & 2;
    const int SL = R > 1 ? NPT + 4 : NPT, NL = R * NPT, NP = R * SL;  // row n lies at (n / NPT) * SL + n % NPT
    float* qs = sm;                     // [REC_TT][NP]
    float* ks = qs + REC_TT * NP;       // [REC_TT][NP]
    float* as = ks + REC_TT * NP;       // [REC_TT][NP]
    float* vs = as + (KIND == SCAN_MEMORY ? 0 : REC_TT * NP);  // [REC_TT][PB] (one decay a token: no rows of decays)
    float* ts = vs + REC_TT * PB;       // [REC_TT]: a token's bonus, or its decay
    const int h = blockIdx.x / col_blocks, cb = blockIdx.x % col_blocks, e = blockIdx.y, c = blockIdx.z;
    pdl_launch_dependents();
    pdl_wait();
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int first = cu_tokens[e], count = cu_tokens[e + 1] - first;
    const int nchunks = pass == 0 ? 1 : (count + chunk_len - 1) / chunk_len;
    if (c >= nchunks || (pass == 1 && c == nchunks - 1)) return;
    const int t0 = first + (pass == 0 ? 0 : c * chunk_len), t1 = pass == 0 ? first + count : min(first + count, t0 + chunk_len);
    const int tid = threadIdx.x, pl = tid / R, r = tid % R, p = cb * PB + pl * CPT;
    const bool real = pl * CPT < PB && p < P;  // all CPT columns, or none
    // SCAN_MEMORY: the threads behind the first block's columns keep n, a column whose value is always 1
    const bool ones = KIND == SCAN_MEMORY && cb == 0 && pl * CPT >= PB && (pl - 1) * CPT < PB;
    const size_t HS = (size_t)N * P, CS = HS + (KIND == SCAN_MEMORY ? N : 0);  // of a chunk's end state: n behind the matrix
    float* slot_state = state + (size_t)slots[e] * slot_stride + (size_t)h * HS;
    float* slot_n = KIND == SCAN_MEMORY ? ex.n_state + (size_t)slots[e] * slot_stride + (size_t)h * N : nullptr;
    float* chunk_state = scratch ? scratch + (((size_t)e * max_chunks + c) * heads + h) * CS : nullptr;
    float2 S[CPT][NPT / 2], prod[WRITE_O || KIND == SCAN_MEMORY ? 1 : NPT / 2];
    float prod1 = 1.f;  // SCAN_MEMORY: the product of the chunk's decays, the same for every row
    const float* init = pass == 0 ? slot_state : (pass == 3 ? chunk_state : nullptr);
    const float* init_n = KIND != SCAN_MEMORY ? nullptr : (pass == 0 ? slot_n : (pass == 3 ? chunk_state + HS : nullptr));
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
        const int n = r * NPT + i;
        float row[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) row[j] = 0.f;
        if (init && real && n < N) {
            const float* src = init + (size_t)n * P + p;
            if constexpr (CPT == 4) { const float4 x = *reinterpret_cast<const float4*>(src); row[0] = x.x, row[1] = x.y, row[2] = x.z, row[3] = x.w; }
            else if constexpr (CPT == 2) { const float2 x = *reinterpret_cast<const float2*>(src); row[0] = x.x, row[1] = x.y; }
            else row[0] = src[0];
        }
        if constexpr (KIND == SCAN_MEMORY) if (init_n && ones && n < N) row[0] = init_n[n];
#pragma unroll
        for (int j = 0; j < CPT; ++j) (i & 1 ? S[j][i / 2].y : S[j][i / 2].x) = row[j];
        if constexpr (!WRITE_O && KIND != SCAN_MEMORY) prod[i / 2] = make_float2(1.f, 1.f);
    }
    for (int tb = t0; tb < t1; tb += REC_TT) {
        const int nt = min(REC_TT, t1 - tb);
        __syncthreads();  // the previous tile is no longer read
        if (CPT > 1 && vec) {  // (the one-column kernels, which run steps of few tokens, stay small: more blocks at a time)
            // four neighbouring rows (or columns) an item, two items a thread at a time, every load ahead of the first use
            const int QI = NL / 4, qitems = nt * QI, VI = PB / 4, vitems = nt * VI;
            for (int i0 = tid; i0 < qitems; i0 += 2 * blockDim.x) {
                Raw4<T> rq[2], rk[2];
                float4 rz[2];
                int at[2], hn4[2];
                bool in[2];
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int idx = i0 + u * blockDim.x, tt = idx / QI, n = (idx % QI) * 4;
                    at[u] = idx < qitems ? tt * NP + (n / NPT) * SL + n % NPT : -1;
                    in[u] = idx < qitems && n < N;
                    hn4[u] = h * N + n;
                    if (in[u]) {
                        const size_t t = (size_t)(tb + tt), hn = (size_t)h * N + n;
                        rq[u] = *reinterpret_cast<const Raw4<T>*>(q + t * q_stride + hn);
                        rk[u] = *reinterpret_cast<const Raw4<T>*>(k + t * k_stride + hn);
                        if (KIND != SCAN_MEMORY && !fixed) rz[u] = *reinterpret_cast<const float4*>(z + t * z_stride + hn);
                    }
                }
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    if (at[u] < 0) continue;
                    float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f), k4 = q4, a4 = make_float4(1.f, 1.f, 1.f, 1.f);
                    if (in[u]) {
                        // (the bias is the same for every token: it stays in the first-level cache)
                        float qv[4], kv[4];
#pragma unroll
                        for (int j = 0; j < 4; ++j) {
                            qv[j] = to_float(rq[u].x[j]), kv[j] = to_float(rk[u].x[j]);
                            if (act) qv[j] = silu_f(qv[j]), kv[j] = silu_f(kv[j]);
                        }
                        q4 = make_float4(qv[0] * q_scale, qv[1] * q_scale, qv[2] * q_scale, qv[3] * q_scale);
                        k4 = make_float4(kv[0], kv[1], kv[2], kv[3]);
                        if constexpr (KIND == SCAN_MEMORY) {
                            const float b = ex.gates[((size_t)(tb + (i0 + u * blockDim.x) / QI) * heads + h) * 2 + 1];
                            k4 = make_float4(kv[0] * b, kv[1] * b, kv[2] * b, kv[3] * b);
                        } else if constexpr (KIND == SCAN_BONUS) {
                            const float4 rb = *reinterpret_cast<const float4*>(z_bias + hn4[u]);
                            a4 = make_float4(expf(-expf(rz[u].x + rb.x)), expf(-expf(rz[u].y + rb.y)), expf(-expf(rz[u].z + rb.z)),
                                             expf(-expf(rz[u].w + rb.w)));
                        } else if (fixed) {
                            const float a = z_bias[h];
                            a4 = make_float4(a, a, a, a);
                        } else {
                        const float4 rb = z_bias ? *reinterpret_cast<const float4*>(z_bias + hn4[u]) : make_float4(0.f, 0.f, 0.f, 0.f);
                        a4 = make_float4(expf(-softplus_f(-(rz[u].x + rb.x)) * inv_tau), expf(-softplus_f(-(rz[u].y + rb.y)) * inv_tau),
                                         expf(-softplus_f(-(rz[u].z + rb.z)) * inv_tau), expf(-softplus_f(-(rz[u].w + rb.w)) * inv_tau));
                        }
                    }
                    *reinterpret_cast<float4*>(qs + at[u]) = q4;
                    *reinterpret_cast<float4*>(ks + at[u]) = k4;
                    if constexpr (KIND != SCAN_MEMORY) *reinterpret_cast<float4*>(as + at[u]) = a4;
                }
            }
            for (int i0 = tid; i0 < vitems; i0 += 2 * blockDim.x) {
                Raw4<T> rv[2];
                int at[2];
                bool in[2];
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int idx = i0 + u * blockDim.x, tt = idx / VI, pc = cb * PB + (idx % VI) * 4;
                    at[u] = idx < vitems ? idx * 4 : -1;
                    in[u] = idx < vitems && pc < P;
                    if (in[u]) rv[u] = *reinterpret_cast<const Raw4<T>*>(v + (size_t)(tb + tt) * v_stride + (size_t)h * P + pc);
                }
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    if (at[u] < 0) continue;
                    float vv4[4] = {0.f, 0.f, 0.f, 0.f};
                    if (in[u]) {
#pragma unroll
                        for (int j = 0; j < 4; ++j) vv4[j] = act ? silu_f(to_float(rv[u].x[j])) : to_float(rv[u].x[j]);
                    }
                    *reinterpret_cast<float4*>(vs + at[u]) = make_float4(vv4[0], vv4[1], vv4[2], vv4[3]);
                }
            }
        } else {
        for (int idx = tid; idx < nt * NL; idx += blockDim.x) {
            const int tt = idx / NL, n = idx % NL, at = tt * NP + (n / NPT) * SL + n % NPT;
            const size_t t = (size_t)(tb + tt);
            float qv = 0.f, kv = 0.f, av = 1.f;
            if (n < N) {
                qv = to_float(q[t * q_stride + (size_t)h * N + n]);
                kv = to_float(k[t * k_stride + (size_t)h * N + n]);
                if (act) qv = silu_f(qv), kv = silu_f(kv);
                qv *= q_scale;
                if constexpr (KIND == SCAN_MEMORY) {
                    kv *= ex.gates[(t * heads + h) * 2 + 1];
                } else if constexpr (KIND == SCAN_BONUS) {
                    av = expf(-expf(z[t * z_stride + (size_t)h * N + n] + z_bias[(size_t)h * N + n]));
                } else if (fixed) {
                    av = z_bias[h];
                } else {
                    // sigmoid(x)^(1/tau) = exp(-softplus(-x) / tau)
                    const float x = z[t * z_stride + (size_t)h * N + n] + (z_bias ? z_bias[(size_t)h * N + n] : 0.f);
                    av = expf(-softplus_f(-x) * inv_tau);
                }
            }
            qs[at] = qv;
            ks[at] = kv;
            if constexpr (KIND != SCAN_MEMORY) as[at] = av;
        }
        for (int idx = tid; idx < nt * PB; idx += blockDim.x) {
            const int tt = idx / PB, pc = cb * PB + idx % PB;
            const float x = pc < P ? to_float(v[(size_t)(tb + tt) * v_stride + (size_t)h * P + pc]) : 0.f;
            vs[idx] = act ? silu_f(x) : x;
        }
        }
        if constexpr (KIND == SCAN_MEMORY) {
            if (tid < nt) ts[tid] = ex.gates[((size_t)(tb + tid) * heads + h) * 2];
        }
        __syncthreads();
        if constexpr (KIND == SCAN_BONUS && WRITE_O) {
            // what the current token adds to its own output is v times sum_n q_n u_n k_n: a warp a token, lanes over n
            for (int tt = tid >> 5; tt < nt; tt += blockDim.x >> 5) {
                float s = 0.f;
                for (int n = tid & 31; n < N; n += 32) {
                    const int at = tt * NP + (n / NPT) * SL + n % NPT;
                    s = fmaf(qs[at] * ex.bonus[(size_t)h * N + n], ks[at], s);
                }
                s = warp_sum(s);
                if ((tid & 31) == 0) ts[tt] = s;
            }
            __syncthreads();
        }
        for (int tt = 0; tt < nt; ++tt) {
            float2 vv[CPT], acc[CPT];
            {
                const float* vt = vs + tt * PB + (pl * CPT < PB ? pl * CPT : 0);
                float x[CPT];
                if constexpr (CPT == 4) { const float4 y = *reinterpret_cast<const float4*>(vt); x[0] = y.x, x[1] = y.y, x[2] = y.z, x[3] = y.w; }
                else if constexpr (CPT == 2) { const float2 y = *reinterpret_cast<const float2*>(vt); x[0] = y.x, x[1] = y.y; }
                else x[0] = vt[0];
#pragma unroll
                for (int j = 0; j < CPT; ++j) vv[j] = make_float2(x[j], x[j]), acc[j] = make_float2(0.f, 0.f);
                if constexpr (KIND == SCAN_MEMORY) if (ones) vv[0] = make_float2(1.f, 1.f);
            }
            const float a1 = KIND == SCAN_MEMORY ? ts[tt] : 0.f;
            if constexpr (KIND == SCAN_MEMORY && !WRITE_O) prod1 *= a1;
            const float* kt = ks + tt * NP + r * SL;
            const float* at = as + tt * NP + r * SL;
            const float* qt = qs + tt * NP + r * SL;
#pragma unroll
            for (int i = 0; i < NPT; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kt + i);
                const float4 a4 = KIND == SCAN_MEMORY ? make_float4(a1, a1, a1, a1) : *reinterpret_cast<const float4*>(at + i);
                const float2 k01 = make_float2(k4.x, k4.y), k23 = make_float2(k4.z, k4.w);
                const float2 a01 = make_float2(a4.x, a4.y), a23 = make_float2(a4.z, a4.w);
                float2 q01 = make_float2(0.f, 0.f), q23 = q01;
                if constexpr (WRITE_O) {
                    const float4 q4 = *reinterpret_cast<const float4*>(qt + i);
                    q01 = make_float2(q4.x, q4.y), q23 = make_float2(q4.z, q4.w);
                } else if constexpr (KIND != SCAN_MEMORY) {
                    prod[i / 2] = mul2(prod[i / 2], a01);
                    prod[i / 2 + 1] = mul2(prod[i / 2 + 1], a23);
                }
#pragma unroll
                for (int j = 0; j < CPT; ++j) {
                    if constexpr (WRITE_O && KIND == SCAN_BONUS) {
                        acc[j] = fma2(S[j][i / 2], q01, acc[j]);
                        acc[j] = fma2(S[j][i / 2 + 1], q23, acc[j]);
                    }
                    S[j][i / 2] = fma2(a01, S[j][i / 2], mul2(k01, vv[j]));
                    S[j][i / 2 + 1] = fma2(a23, S[j][i / 2 + 1], mul2(k23, vv[j]));
                    if constexpr (WRITE_O && KIND != SCAN_BONUS) {
                        acc[j] = fma2(S[j][i / 2], q01, acc[j]);
                        acc[j] = fma2(S[j][i / 2 + 1], q23, acc[j]);
                    }
                }
            }
            if constexpr (WRITE_O) {
                float sum[CPT];
#pragma unroll
                for (int j = 0; j < CPT; ++j) {
                    sum[j] = acc[j].x + acc[j].y;
                    for (int s = R >> 1; s > 0; s >>= 1) sum[j] += __shfl_xor_sync(0xffffffffu, sum[j], s);
                    if constexpr (KIND == SCAN_BONUS) sum[j] = fmaf(ts[tt], vv[j].x, sum[j]);
                }
                if constexpr (KIND == SCAN_MEMORY) if (ones && r == 0) ex.nq[(size_t)(tb + tt) * heads + h] = sum[0];
                if (real && r == 0) {
                    float* dst = o + (size_t)(tb + tt) * heads * P + (size_t)h * P + p;
                    if constexpr (CPT == 4) *reinterpret_cast<float4*>(dst) = make_float4(sum[0], sum[1], sum[2], sum[3]);
                    else if constexpr (CPT == 2) *reinterpret_cast<float2*>(dst) = make_float2(sum[0], sum[1]);
                    else dst[0] = sum[0];
                }
            }
        }
    }
    float* fin = pass == 1 ? chunk_state + (size_t)heads * CS /* the next chunk's place */
                           : ((pass == 0 || c == nchunks - 1) ? slot_state : nullptr);
    if (fin && real) {
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
            const int n = r * NPT + i;
            if (n < N) {
                float row[CPT];
#pragma unroll
                for (int j = 0; j < CPT; ++j) row[j] = i & 1 ? S[j][i / 2].y : S[j][i / 2].x;
                float* dst = fin + (size_t)n * P + p;
                if constexpr (CPT == 4) *reinterpret_cast<float4*>(dst) = make_float4(row[0], row[1], row[2], row[3]);
                else if constexpr (CPT == 2) *reinterpret_cast<float2*>(dst) = make_float2(row[0], row[1]);
                else dst[0] = row[0];
            }
        }
    }
    if constexpr (KIND == SCAN_MEMORY) if (fin && ones) {
        float* fin_n = fin == slot_state ? slot_n : fin + HS;
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
            const int n = r * NPT + i;
            if (n < N) fin_n[n] = i & 1 ? S[0][i / 2].y : S[0][i / 2].x;
        }
    }
    if constexpr (!WRITE_O) if (pass == 1 && cb == 0 && pl == 0) {
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
            const int n = r * NPT + i;
            if (n < N) {
                float amount;
                if constexpr (KIND == SCAN_MEMORY) amount = prod1;
                else amount = i & 1 ? prod[i / 2].y : prod[i / 2].x;
                decay[(((size_t)e * max_chunks + c) * heads + h) * N + n] = amount;
            }
        }
    }
}

// scratch[e, 0] = the slot's state; scratch[e, c] = decay[e, c - 1] (a factor per row) * scratch[e, c - 1] + scratch[e, c].
// With `n_state` a chunk's state is the matrix and the N elements of n behind it, which decay as their rows do.
static __global__ void __launch_bounds__(256)
matrix_chunk_states_kernel(const float* __restrict__ state, long long slot_stride, float* __restrict__ scratch,
                           const float* __restrict__ decay, const float* __restrict__ n_state, const int* __restrict__ meta,
                           const int* __restrict__ cu_tokens, const int* __restrict__ slots, int heads, int N, int P, int chunk_len,
                           int max_chunks) {
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, e = blockIdx.y;
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int count = cu_tokens[e + 1] - cu_tokens[e], nchunks = (count + chunk_len - 1) / chunk_len;
    const long long HS = (long long)N * P, CS = HS + (n_state ? N : 0);
    const float* src = state + (size_t)slots[e] * slot_stride + (size_t)h * HS;
    const float* src_n = n_state ? n_state + (size_t)slots[e] * slot_stride + (size_t)h * N : nullptr;
    for (long long i = (long long)blockIdx.z * blockDim.x + threadIdx.x; i < CS; i += (long long)gridDim.z * blockDim.x) {
        const int n = i < HS ? (int)(i / P) : (int)(i - HS);
        float s = i < HS ? src[i] : src_n[n];
        scratch[(((size_t)e * max_chunks) * heads + h) * CS + i] = s;
        for (int c = 1; c < nchunks; ++c) {
            float* at = scratch + (((size_t)e * max_chunks + c) * heads + h) * CS + i;
            s = fmaf(decay[(((size_t)e * max_chunks + c - 1) * heads + h) * N + n], s, *at);
            *at = s;
        }
    }
}

// Rows a thread keeps and threads a column (or channel): the least padding, then 16 or 32 rows a thread.  Columns a
// block: those of up to 256 threads, ``cpt`` neighbouring columns each.
static bool rec_geometry(int N, int P, int* NPT_out, int* R_out, int* PB_out, int cpt = 1) {
    static const int sizes[] = {16, 32, 8, 64};  // in order of preference among equal paddings
    long best = -1;
    for (int k = 0; k < 4; ++k) {
        const int npt = sizes[k];
        int R = 1;
        while (R * npt < N) R *= 2;
        if (R > 32) continue;
        const long cost = (long)R * npt;
        if (best < 0 || cost < best) best = cost, *NPT_out = npt, *R_out = R;
    }
    if (best < 0) return false;
    int pb = 256 / *R_out * cpt;  // up to 256 threads a block
    if (pb > P) pb = P;
    *PB_out = pb;
    return true;
}

// What a launch of the scan needs to know; `z_bias`, `tau`, `mode` and `ex` as the kernel's kind reads them.
struct ScanArgs {
    const void *q, *k, *v;
    long long q_stride, k_stride, v_stride;
    int dtype;
    const float *z, *z_bias;
    long long z_stride;
    float tau, q_scale;
    float* state;
    long long slot_stride;
    float* o;
    const int *meta, *cu_tokens, *slots;
    int S, heads, N, P, chunk_len, max_chunks;
    float* scratch;
    int mode;
    ScanExtras ex;
};

template <int KIND>
static size_t scan_scratch_floats(int S, int heads, int N, int P, int max_chunks) {
    return (size_t)S * max_chunks * heads * ((size_t)N * P + N + (KIND == SCAN_MEMORY ? N : 0));
}

template <typename TT, int NPT, bool WRITE_O, int CPT, int KIND>
static int launch_matrix_scan(const ScanArgs& a, int R, int PB, int vec, int pass, int chunks, cudaStream_t stream) {
    const int col_blocks = (a.P + PB - 1) / PB, columns = (PB + CPT - 1) / CPT + (KIND == SCAN_MEMORY ? 1 : 0);
    const int threads = ((columns * R + 31) / 32) * 32;
    const size_t smem = (size_t)((KIND == SCAN_MEMORY ? 2 : 3) * REC_TT * R * (R > 1 ? NPT + 4 : NPT) + REC_TT * PB + REC_TT) * sizeof(float);
    if (smem > 96 * 1024 || threads > (KIND == SCAN_MEMORY ? 288 : 256)) return (int)cudaErrorInvalidValue;
    float* decay = a.scratch ? a.scratch + scan_scratch_floats<KIND>(a.S, a.heads, a.N, a.P, a.max_chunks) -
                                   (size_t)a.S * a.max_chunks * a.heads * a.N : nullptr;
    static size_t configured = 0;
    if (smem > 48 * 1024 && smem > configured) {
        cudaError_t ce = cudaFuncSetAttribute(matrix_scan_kernel<TT, NPT, WRITE_O, CPT, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (ce != cudaSuccess) return (int)ce;
        configured = smem;
    }
    return (int)launch_kernel(matrix_scan_kernel<TT, NPT, WRITE_O, CPT, KIND>, dim3(a.heads * col_blocks, a.S, chunks), threads, smem, stream,
                              (const TT*)a.q, a.q_stride, (const TT*)a.k, a.k_stride, (const TT*)a.v, a.v_stride, a.z, a.z_stride, a.z_bias,
                              1.f / a.tau, a.q_scale, a.state, a.slot_stride, a.o, a.meta, a.cu_tokens, a.slots, a.heads, a.P, a.N, R, PB,
                              col_blocks, pass, a.chunk_len, a.max_chunks, a.scratch, decay, vec, a.mode, a.ex);
}

template <typename TT, bool WRITE_O, int KIND>
static int launch_matrix_pass(const ScanArgs& a, int NPT, int R, int PB, int CPT, int vec, int pass, int chunks, cudaStream_t stream) {
    switch (NPT) {
        case 8:
            if (CPT == 4) return launch_matrix_scan<TT, 8, WRITE_O, 4, KIND>(a, R, PB, vec, pass, chunks, stream);
            if (CPT == 2) return launch_matrix_scan<TT, 8, WRITE_O, 2, KIND>(a, R, PB, vec, pass, chunks, stream);
            return launch_matrix_scan<TT, 8, WRITE_O, 1, KIND>(a, R, PB, vec, pass, chunks, stream);
        case 16:
            if (CPT == 4) return launch_matrix_scan<TT, 16, WRITE_O, 4, KIND>(a, R, PB, vec, pass, chunks, stream);
            if (CPT == 2) return launch_matrix_scan<TT, 16, WRITE_O, 2, KIND>(a, R, PB, vec, pass, chunks, stream);
            return launch_matrix_scan<TT, 16, WRITE_O, 1, KIND>(a, R, PB, vec, pass, chunks, stream);
        case 32:
            if (CPT == 2) return launch_matrix_scan<TT, 32, WRITE_O, 2, KIND>(a, R, PB, vec, pass, chunks, stream);
            return launch_matrix_scan<TT, 32, WRITE_O, 1, KIND>(a, R, PB, vec, pass, chunks, stream);
        default: return launch_matrix_scan<TT, 64, WRITE_O, 1, KIND>(a, R, PB, vec, pass, chunks, stream);
    }
}

// The scan of every entry: in order from the slots, or (chunk_len > 0, max_chunks > 1 and scratch) in chunks of time.
template <int KIND>
static int run_matrix_scan(const ScanArgs& a, cudaStream_t stream) {
    if (a.S <= 0) return 0;
    int NPT = 0, R = 0, PB = 0;
    if (a.tau <= 0.f || !rec_geometry(a.N, a.P, &NPT, &R, &PB)) return (int)cudaErrorInvalidValue;
    const bool chunked = a.chunk_len > 0 && a.max_chunks > 1 && a.scratch, bf = a.dtype != DT_F32;
    // Columns a thread: with chunks of time there are blocks enough, and a row's k, a and q serve four (or two) columns;
    // a step of few tokens per entry keeps one, for as many blocks as can be.  Vector accesses want their alignment.
    const size_t CS = (size_t)a.N * a.P + (KIND == SCAN_MEMORY ? a.N : 0);
    auto aligned = [&](int n) {
        return a.P % n == 0 && CS % n == 0 && a.slot_stride % n == 0 && ((uintptr_t)a.state | (uintptr_t)a.o | (uintptr_t)a.scratch) % (4 * n) == 0;
    };
    const int CPT = !chunked ? 1 : (NPT <= 16 && aligned(4) ? 4 : (NPT <= 32 && aligned(2) ? 2 : 1));
    rec_geometry(a.N, a.P, &NPT, &R, &PB, CPT);
    // tiles of q, k, decay logits and v in items of four: rows and columns in fours, every row's slice on its vector's boundary
    const uintptr_t esz = bf ? 2 : 4;
    const bool logits = KIND == SCAN_BONUS || (KIND == SCAN_DECAY && !(a.mode & 1));
    const int vec = a.N % 4 == 0 && a.P % 4 == 0 && PB % 4 == 0 && a.q_stride % 4 == 0 && a.k_stride % 4 == 0 && a.v_stride % 4 == 0 &&
                    ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) % (4 * esz) == 0 &&
                    (!logits || (a.z_stride % 4 == 0 && ((uintptr_t)a.z | (uintptr_t)a.z_bias) % 16 == 0));
    if (!chunked)
        return bf ? launch_matrix_pass<__nv_bfloat16, true, KIND>(a, NPT, R, PB, CPT, vec, 0, 1, stream)
                  : launch_matrix_pass<float, true, KIND>(a, NPT, R, PB, CPT, vec, 0, 1, stream);
    int err = bf ? launch_matrix_pass<__nv_bfloat16, false, KIND>(a, NPT, R, PB, CPT, vec, 1, a.max_chunks, stream)
                 : launch_matrix_pass<float, false, KIND>(a, NPT, R, PB, CPT, vec, 1, a.max_chunks, stream);
    if (err) return err;
    const float* decay = a.scratch + (size_t)a.S * a.max_chunks * a.heads * CS;
    const int zblocks = (int)((CS + 1023) / 1024);
    err = (int)launch_kernel(matrix_chunk_states_kernel, dim3(a.heads, a.S, zblocks), 256, 0, stream, (const float*)a.state, a.slot_stride,
                             a.scratch, decay, (const float*)(KIND == SCAN_MEMORY ? a.ex.n_state : nullptr), a.meta, a.cu_tokens, a.slots,
                             a.heads, a.N, a.P, a.chunk_len, a.max_chunks);
    if (err) return err;
    return bf ? launch_matrix_pass<__nv_bfloat16, true, KIND>(a, NPT, R, PB, CPT, vec, 3, a.max_chunks, stream)
              : launch_matrix_pass<float, true, KIND>(a, NPT, R, PB, CPT, vec, 3, a.max_chunks, stream);
}
