// Kernels of differential attention: the rows that enter it (biases, a short causal convolution over time, the layout in
// which the attention kernels see two maps over the same values) and the difference of the two maps behind it.
// Storage is float32 or bfloat16, arithmetic float32.
#include <type_traits>

#include "common.cuh"

// V neighbouring elements, widened; V = 8 (bfloat16 only) and 4 take one access (16-byte rows), 1 takes any address.
template <typename T, int V>
__device__ __forceinline__ void load_row(const T* p, float (&v)[V]) {
    if constexpr (V == 8) {
        float a[4], b[4];
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const T* e = reinterpret_cast<const T*>(&raw);
        load4(e, a);
        load4(e + 4, b);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] = a[k], v[4 + k] = b[k];
    } else if constexpr (V == 4) {
        load4(p, v);
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = to_float(p[k]);
    }
}
template <int V>
__device__ __forceinline__ void load_f32(const float* p, float (&v)[V]) {
    if constexpr (V % 4 == 0) {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            float t[4];
            load4(p + i, t);
#pragma unroll
            for (int k = 0; k < 4; ++k) v[i + k] = t[k];
        }
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = p[k];
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_row(T* p, const float (&v)[V]) {
    if constexpr (V == 8) {
        uint4 raw;
        T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int k = 0; k < 8; ++k) e[k] = from_float<T>(v[k]);
        *reinterpret_cast<uint4*>(p) = raw;
    } else if constexpr (V == 4) {
        store4(p, v);
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) p[k] = from_float<T>(v[k]);
    }
}

// V elements as they are stored, in one register vector where they make one (16 or 8 bytes).
template <typename T, int V>
struct RawRow {
    using type = typename std::conditional<V * sizeof(T) == 16, uint4, typename std::conditional<V * sizeof(T) == 8, uint2, T>::type>::type;
};
template <typename T, int V>
__device__ __forceinline__ void widen(const typename RawRow<T, V>::type& raw, float (&v)[V]) {
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = to_float(e[k]);
}

// ----------------------------------------------------------------------------- the rows
// A token's projected row u is [q: heads * M * d | k: kv_heads * M * d | v: kv_heads * dv] (M maps; the row may be the first
// part of a wider one).  Per channel r_t = sum_j w[j] * (u_(t - taps + 1 + j) + bias), terms before the request's start
// left out (taps 0: r_t = u_t + bias).  Query map (h, m) becomes a head of dp elements that holds its d values at m * d and
// zeros elsewhere; a key head is [its M maps side by side | zeros], a value head [its values | zeros], both dp
// elements, written to the token's page: the score of query head (h, m) and that key head is map m's alone.
// The convolution's earlier rows u come from this step or from the request's ring of taps - 1 float32 rows (the row of
// position p at place p mod (taps - 1); slot_stride floats from slot to slot).  save_own: every entry brings one token,
// so the thread that has read a channel's ring also writes the new row's place; otherwise map_rows_save writes it later.
//
// A thread owns V neighbouring channels of one output head and walks the block's tokens with its weights and biases in
// registers, four tokens at a time where their rows lie side by side.
#define MAP_ROWS_TOK 16
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128)
map_rows_kernel(const T* __restrict__ u, long long u_stride, const float* __restrict__ bias, const float* __restrict__ w,
                float* __restrict__ ring, long long slot_stride, T* __restrict__ q_out, T* __restrict__ cache,
                const int* __restrict__ meta, const int* __restrict__ positions, const int* __restrict__ token_entry,
                const int* __restrict__ cu_tokens, const int* __restrict__ slots, int group, int heads, int kv_heads, int maps, int d,
                int dv, int dp, int page_size, int num_pages, int store_kv, int save_own, int tok, int* __restrict__ status) {
    constexpr int R = TAPS > 1 ? TAPS - 1 : 0, RR = R > 0 ? R : 1;
    __shared__ int s_pos[MAP_ROWS_TOK], s_page[MAP_ROWS_TOK], s_first[MAP_ROWS_TOK], s_slot[MAP_ROWS_TOK];
    const int ntok = meta[META_NUM_TOKENS], t0 = blockIdx.x * tok, tn = min(tok, ntok - t0);
    if ((int)threadIdx.x < tn) {  // the step's metadata is written by no kernel of the step
        const int t = t0 + threadIdx.x, e = token_entry[t], p = positions[t];
        s_pos[threadIdx.x] = p;
        s_first[threadIdx.x] = cu_tokens[e];
        s_slot[threadIdx.x] = slots[e];
        int page = 0;
        if (store_kv) {
            page = (meta + meta[META_BT_OFFSET + group] + (size_t)e * meta[META_BT_STRIDE + group])[p / page_size];
            if (page <= 0 || page >= num_pages) {
                if (blockIdx.y == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + t);
                page = 0;  // its keys and values are dropped; the queries are still prepared
            }
        }
        s_page[threadIdx.x] = page;
    }
    const int nq = heads * maps, NQ = nq * d, NK = kv_heads * maps * d, N = NQ + NK + kv_heads * dv;
    const int per = dp / V, piece = blockIdx.y * blockDim.x + threadIdx.x;
    const int head = piece / per, at = (piece % per) * V;
    const bool mine = head < nq + 2 * kv_heads && tn > 0;
    // where the piece comes from (ch < 0: zeros) and where it goes
    int ch = -1, kind = 0, h = head;
    if (head < nq) {
        const int off = (head % maps) * d;
        if (at >= off && at < off + d) ch = head * d + at - off;
    } else if (head < nq + kv_heads) {
        kind = 1, h = head - nq;
        if (at < maps * d) ch = NQ + h * maps * d + at;
    } else {
        kind = 2, h = head - nq - kv_heads;
        if (at < dv) ch = NQ + NK + h * dv + at;
    }
    float b[V], wt[TAPS > 0 ? TAPS : 1][V];
#pragma unroll
    for (int k = 0; k < V; ++k) b[k] = 0.f;
    if (mine && ch >= 0) {
        if (bias) load_f32<V>(bias + ch, b);
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) load_f32<V>(w + (size_t)j * N + ch, wt[j]);
        }
    }
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    if (!mine) return;
    const size_t head_block = (size_t)page_size * dp, kv_block = (size_t)kv_heads * head_block;
    auto put = [&](int i, const float (&r)[V]) {
        if (kind == 0) {
            store_row<T, V>(q_out + ((size_t)(t0 + i) * nq + h) * dp + at, r);
        } else if (s_page[i] > 0) {
            T* page = cache + (size_t)s_page[i] * 2 * kv_block + (kind == 2 ? kv_block : 0);
            store_row<T, V>(page + (size_t)h * head_block + (size_t)(s_pos[i] % page_size) * dp + at, r);
        }
    };
    constexpr int GROUP = 4;
    for (int i = 0; i < tn;) {
        float r[V];
        if (ch < 0) {
#pragma unroll
            for (int k = 0; k < V; ++k) r[k] = 0.f;
            put(i++, r);
            continue;
        }
        const T* row = u + (size_t)(t0 + i) * u_stride + ch;
        // four tokens whose rows, and the rows before them, are all of one request and of this step: every row is loaded once
        if (i + GROUP <= tn && s_first[i + GROUP - 1] <= t0 + i - R) {
            typename RawRow<T, V>::type raw[GROUP + R];
#pragma unroll
            for (int j = 0; j < GROUP + R; ++j) raw[j] = *reinterpret_cast<const typename RawRow<T, V>::type*>(row + (long long)(j - R) * u_stride);
#pragma unroll
            for (int g = 0; g < GROUP; ++g) {
#pragma unroll
                for (int k = 0; k < V; ++k) r[k] = 0.f;
#pragma unroll
                for (int j = 0; j <= R; ++j) {
                    float v[V];
                    widen<T, V>(raw[g + j], v);
#pragma unroll
                    for (int k = 0; k < V; ++k) r[k] = TAPS > 0 ? fmaf(wt[j][k], v[k] + b[k], r[k]) : v[k] + b[k];
                }
                put(i + g, r);
            }
            i += GROUP;
            continue;
        }
        const int t = t0 + i, p = s_pos[i], first = s_first[i];
        float cur[V];
        load_row<T, V>(row, cur);
#pragma unroll
        for (int k = 0; k < V; ++k) r[k] = 0.f;
#pragma unroll
        for (int j = 0; j < R; ++j) {  // oldest tap first: a fixed order
            const int back = R - j;
            if (p - back < 0) continue;
            float v[V];
            if (t - back >= first) load_row<T, V>(u + (size_t)(t - back) * u_stride + ch, v);
            else load_f32<V>(ring + (size_t)s_slot[i] * slot_stride + (size_t)((p - back) % RR) * N + ch, v);
#pragma unroll
            for (int k = 0; k < V; ++k) r[k] = fmaf(wt[j][k], v[k] + b[k], r[k]);
        }
        if (R > 0 && save_own) {
            float* dst = ring + (size_t)s_slot[i] * slot_stride + (size_t)(p % RR) * N + ch;
#pragma unroll
            for (int k = 0; k < V; ++k) dst[k] = cur[k];
        }
#pragma unroll
        for (int k = 0; k < V; ++k) r[k] = TAPS > 0 ? fmaf(wt[TAPS > 0 ? TAPS - 1 : 0][k], cur[k] + b[k], r[k]) : cur[k] + b[k];
        put(i++, r);
    }
}

// Convolutions of more taps than the kernel above is built for, one element a thread.
template <typename T>
__global__ void __launch_bounds__(128)
map_rows_any_kernel(const T* __restrict__ u, long long u_stride, const float* __restrict__ bias, const float* __restrict__ w,
                    const float* __restrict__ ring, long long slot_stride, T* __restrict__ q_out, T* __restrict__ cache,
                    const int* __restrict__ meta, const int* __restrict__ positions, const int* __restrict__ token_entry,
                    const int* __restrict__ cu_tokens, const int* __restrict__ slots, int group, int heads, int kv_heads, int maps,
                    int d, int dv, int dp, int page_size, int num_pages, int store_kv, int taps, int* __restrict__ status) {
    const int t = blockIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    if (t >= meta[META_NUM_TOKENS]) return;
    const int e = token_entry[t], p = positions[t], first = cu_tokens[e], R = taps - 1;
    const float* st = ring + (size_t)slots[e] * slot_stride;
    int page = 0;
    if (store_kv) {
        page = (meta + meta[META_BT_OFFSET + group] + (size_t)e * meta[META_BT_STRIDE + group])[p / page_size];
        if (page <= 0 || page >= num_pages) {
            if (threadIdx.x == 0 && blockIdx.y == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + t);
            page = 0;
        }
    }
    const int nq = heads * maps, NQ = nq * d, NK = kv_heads * maps * d, N = NQ + NK + kv_heads * dv;
    const size_t head_block = (size_t)page_size * dp, kv_block = (size_t)kv_heads * head_block;
    const int it = blockIdx.y * blockDim.x + threadIdx.x, head = it / dp, at = it % dp;
    if (head >= nq + 2 * kv_heads) return;
    int ch = -1, kind = 0, h = head;
    if (head < nq) {
        const int off = (head % maps) * d;
        if (at >= off && at < off + d) ch = head * d + at - off;
    } else if (head < nq + kv_heads) {
        kind = 1, h = head - nq;
        if (at < maps * d) ch = NQ + h * maps * d + at;
    } else {
        kind = 2, h = head - nq - kv_heads;
        if (at < dv) ch = NQ + NK + h * dv + at;
    }
    float r = 0.f;
    if (ch >= 0) {
        const float b = bias ? bias[ch] : 0.f;
        for (int j = 0; j < taps; ++j) {  // oldest tap first
            const int back = R - j;
            if (p - back < 0) continue;
            const float v = t - back >= first ? to_float(u[(size_t)(t - back) * u_stride + ch]) : st[(size_t)((p - back) % R) * N + ch];
            r = fmaf(w[(size_t)j * N + ch], v + b, r);
        }
    }
    if (kind == 0) {
        q_out[((size_t)t * nq + h) * dp + at] = from_float<T>(r);
    } else if (page > 0) {
        cache[(size_t)page * 2 * kv_block + (kind == 2 ? kv_block : 0) + (size_t)h * head_block + (size_t)(p % page_size) * dp + at] =
            from_float<T>(r);
    }
}

static int map_rows_vector(int dtype, long long u_stride, long long slot_stride, int d, int dv, int dp, int N, uintptr_t all) {
    const int V = dtype == DT_F32 ? 4 : 8;
    for (int v = V; v >= 4; v /= 2)
        if (d % v == 0 && dv % v == 0 && dp % v == 0 && u_stride % v == 0 && slot_stride % 4 == 0 && N % 4 == 0 && (all & 15) == 0) return v;
    return 1;
}

extern "C" int map_rows(const void* u, int dtype, long long u_stride, const float* bias, const float* w, int taps, float* ring,
                        long long slot_stride, void* q_out, void* cache, const int* meta, const int* positions, const int* token_entry,
                        const int* cu_tokens, const int* slots, int group, int T, int heads, int kv_heads, int maps, int d, int dv, int dp,
                        int page_size, int num_pages, int store_kv, int save_own, int* status, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (taps < 0 || (taps > 0 && !w) || (taps > 1 && !ring) || maps < 1 || maps * d > dp || dv > dp) return (int)cudaErrorInvalidValue;
    const bool pdl = (g_use_pdl & 5) != 0;
    const int N = (heads + kv_heads) * maps * d + kv_heads * dv, out_heads = heads * maps + 2 * kv_heads;
    if (taps > 4) {
        if (save_own) return (int)cudaErrorInvalidValue;
        const dim3 grid(T, (out_heads * dp + 127) / 128);
        if (dtype == DT_F32)
            return (int)launch_kernel_pdl(pdl, map_rows_any_kernel<float>, grid, 128, 0, stream, (const float*)u, u_stride, bias, w, ring,
                                          slot_stride, (float*)q_out, (float*)cache, meta, positions, token_entry, cu_tokens, slots, group,
                                          heads, kv_heads, maps, d, dv, dp, page_size, num_pages, store_kv, taps, status);
        return (int)launch_kernel_pdl(pdl, map_rows_any_kernel<__nv_bfloat16>, grid, 128, 0, stream, (const __nv_bfloat16*)u, u_stride, bias,
                                      w, ring, slot_stride, (__nv_bfloat16*)q_out, (__nv_bfloat16*)cache, meta, positions, token_entry,
                                      cu_tokens, slots, group, heads, kv_heads, maps, d, dv, dp, page_size, num_pages, store_kv, taps, status);
    }
    const uintptr_t all = (uintptr_t)u | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)ring | (uintptr_t)q_out | (uintptr_t)cache;
    const int V = map_rows_vector(dtype, u_stride, slot_stride, d, dv, dp, N, all);
    // few tokens: one a block, the shortest path; many: sixteen, which read weights once and every row once
    const int tok = T >= 512 ? MAP_ROWS_TOK : T >= 128 ? 4 : 1;
    const dim3 grid((T + tok - 1) / tok, (out_heads * (dp / V) + 127) / 128);
#define ROWS_LAUNCH(TT, VV, TP)                                                                                                \
    return (int)launch_kernel_pdl(pdl, map_rows_kernel<TT, VV, TP>, grid, 128, 0, stream, (const TT*)u, u_stride, bias, w, ring, slot_stride, \
                                  (TT*)q_out, (TT*)cache, meta, positions, token_entry, cu_tokens, slots, group, heads, kv_heads, maps, d, dv, \
                                  dp, page_size, num_pages, store_kv, save_own, tok, status)
#define ROWS_CASE(TT, VV)                                                                                                      \
    do {                                                                                                                       \
        if (taps == 0) ROWS_LAUNCH(TT, VV, 0);                                                                                 \
        if (taps == 1) ROWS_LAUNCH(TT, VV, 1);                                                                                 \
        if (taps == 2) ROWS_LAUNCH(TT, VV, 2);                                                                                 \
        if (taps == 3) ROWS_LAUNCH(TT, VV, 3);                                                                                 \
        ROWS_LAUNCH(TT, VV, 4);                                                                                                \
    } while (0)
    if (dtype == DT_F32) {
        if (V == 4) ROWS_CASE(float, 4);
        ROWS_CASE(float, 1);
    }
    if (V == 8) ROWS_CASE(__nv_bfloat16, 8);
    if (V == 4) ROWS_CASE(__nv_bfloat16, 4);
    ROWS_CASE(__nv_bfloat16, 1);
#undef ROWS_CASE
#undef ROWS_LAUNCH
}

// The last taps - 1 projected rows (without biases) of every entry go to its ring.
template <typename T>
__global__ void __launch_bounds__(128)
map_rows_save_kernel(const T* __restrict__ u, long long u_stride, float* __restrict__ ring, long long slot_stride,
                     const int* __restrict__ meta, const int* __restrict__ positions, const int* __restrict__ cu_tokens,
                     const int* __restrict__ slots, int N, int R) {
    const int e = blockIdx.x / R, back = blockIdx.x % R;  // block (entry, one of its last R rows)
    const bool live = e < meta[META_NUM_ENTRIES];
    const int t = live ? cu_tokens[e + 1] - 1 - back : 0, first = live ? cu_tokens[e] : 1;
    pdl_launch_dependents();
    pdl_wait();
    if (!live || t < first) return;
    float* dst = ring + (size_t)slots[e] * slot_stride + (size_t)(positions[t] % R) * N;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < N; c += gridDim.y * blockDim.x) dst[c] = to_float(u[(size_t)t * u_stride + c]);
}

extern "C" int map_rows_save(const void* u, int dtype, long long u_stride, float* ring, long long slot_stride, const int* meta,
                             const int* positions, const int* cu_tokens, const int* slots, int S, int N, int taps, cudaStream_t stream) {
    if (S <= 0 || taps <= 1) return 0;
    const dim3 grid(S * (taps - 1), N >= 2048 ? 4 : 1);
    if (dtype == DT_F32)
        return (int)launch_kernel(map_rows_save_kernel<float>, grid, 128, 0, stream, (const float*)u, u_stride, ring, slot_stride, meta,
                                  positions, cu_tokens, slots, N, taps - 1);
    return (int)launch_kernel(map_rows_save_kernel<__nv_bfloat16>, grid, 128, 0, stream, (const __nv_bfloat16*)u, u_stride, ring, slot_stride,
                              meta, positions, cu_tokens, slots, N, taps - 1);
}

// ----------------------------------------------------------------------------- the difference of the maps
// a [T, heads, 2, dp] holds a head's two results (dv values each); o = a_1 - lambda a_2;
// out[t, h] = o * rsqrt(mean(o^2) + eps) * factor * sigmoid(gate[t, h]), out [T, heads * dv].  L lanes a (token, head), up to C
// steps of V values a lane kept in registers.
template <typename T, int V, int L, int C>
__global__ void __launch_bounds__(256)
map_difference_kernel(const T* __restrict__ a, int dp, const T* __restrict__ gate, long long gate_stride, const float* __restrict__ lambda,
                      float factor, float eps, T* __restrict__ out, const int* __restrict__ meta, int heads, int dv) {
    const int lane = threadIdx.x % L;
    const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / L;
    const int ntok = meta[META_NUM_TOKENS];
    const float lam = *lambda;
    const bool live = item < (long long)ntok * heads;
    pdl_wait();
    pdl_launch_dependents();
    const int t = live ? (int)(item / heads) : 0, h = live ? (int)(item % heads) : 0;
    const T* a1 = a + ((size_t)t * heads + h) * 2 * dp;
    float o[C][V], ss = 0.f;
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int i = (c * L + lane) * V;
        if (live && i < dv) {
            float x[V], y[V];
            load_row<T, V>(a1 + i, x);
            load_row<T, V>(a1 + dp + i, y);
#pragma unroll
            for (int k = 0; k < V; ++k) {
                o[c][k] = fmaf(-lam, y[k], x[k]);
                ss = fmaf(o[c][k], o[c][k], ss);
            }
        }
    }
#pragma unroll
    for (int s = L / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    if (!live) return;
    float f = rsqrtf(ss / (float)dv + eps) * factor;
    if (gate) f = f / (1.f + expf(-to_float(gate[(size_t)t * gate_stride + h])));
    T* dst = out + ((size_t)t * heads + h) * dv;
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int i = (c * L + lane) * V;
        if (i < dv) {
            float r[V];
#pragma unroll
            for (int k = 0; k < V; ++k) r[k] = o[c][k] * f;
            store_row<T, V>(dst + i, r);
        }
    }
}

extern "C" int map_difference(const void* a, int dtype, int dp, const void* gate, long long gate_stride, const float* lambda, float factor,
                              float eps, void* out, const int* meta, int T, int heads, int dv, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (dv > 512 || dv > dp) return (int)cudaErrorInvalidValue;
    const bool pdl = (g_use_pdl & 5) != 0;
    const int W = dtype == DT_F32 ? 4 : 8;
    const bool vec = dv % W == 0 && dp % W == 0 && (((uintptr_t)a | (uintptr_t)out) & 15) == 0;
    const int pieces = dv / (vec ? W : 1);
#define DIFF_LAUNCH(TT, VV, LL, CC)                                                                                       \
    return (int)launch_kernel_pdl(pdl, map_difference_kernel<TT, VV, LL, CC>,                                             \
                                  (unsigned)(((long long)T * heads * LL + 255) / 256), 256, 0, stream, (const TT*)a, dp, (const TT*)gate, \
                                  gate_stride, lambda, factor, eps, (TT*)out, meta, heads, dv)
#define DIFF_CASE(TT, VV)                              \
    do {                                               \
        if (pieces <= 8) DIFF_LAUNCH(TT, VV, 8, 1);    \
        if (pieces <= 16) DIFF_LAUNCH(TT, VV, 16, 1);  \
        if (pieces <= 32) DIFF_LAUNCH(TT, VV, 32, 1);  \
        DIFF_LAUNCH(TT, VV, 32, 4);                    \
    } while (0)
    if (dtype == DT_F32) {
        if (vec) DIFF_CASE(float, 4);
        DIFF_LAUNCH(float, 1, 32, 16);
    }
    if (vec) DIFF_CASE(__nv_bfloat16, 8);
    DIFF_LAUNCH(__nv_bfloat16, 1, 32, 16);
#undef DIFF_CASE
#undef DIFF_LAUNCH
}
