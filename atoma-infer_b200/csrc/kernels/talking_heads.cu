// Attention whose softmax weights are mixed across the query heads before they weigh the values, on the paged cache:
// p_h(i, j) = softmax_j(scale * q_h . k_h/(H/G)), p'_h = sum_g talk[h, g] p_g, o_h = sum_j p'_h(i, j) v_h/(H/G)(j).
// The plain kernel: float32 and bfloat16 storage, any number of heads and head size, float32 arithmetic.  The mix needs the
// finished softmax of every head, so the keys are walked twice: once for every head's maximum and sum, once for the
// weights, the mix and the values.  Keys are taken in tiles counted from the first visible key, so every sum's order depends
// on the position only.
#include "common.cuh"

#define TALK_KT 32
#define TALK_THREADS 256

template <typename T>
__global__ void __launch_bounds__(TALK_THREADS)
talk_attn_plain_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ cache, CacheLayout L, const int* __restrict__ meta,
                       int group, const int* __restrict__ token_entry, const int* __restrict__ positions, T* __restrict__ out, int H,
                       int chunk, float scale, const float* __restrict__ talk, int num_pages, int* __restrict__ status) {
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    if (t >= meta[META_NUM_TOKENS]) return;
    const int d = L.head_dim, ps = L.page_size, G = L.num_kv_heads, HG = H / G;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = TALK_THREADS / 32;
    float* qs = sm;                          // [H][d]
    float* acc = qs + (size_t)H * d;         // [H][d]
    float* m = acc + (size_t)H * d;          // [H]
    float* l = m + H;                        // [H]
    float* p = l + H;                        // [H][TALK_KT]
    float* pm = p + (size_t)H * TALK_KT;     // [H][TALK_KT], mixed
    float* tile = pm + (size_t)H * TALK_KT;  // [TALK_KT][d + 1], keys or values of one head
    const int pos = positions[t], kstart = chunk > 0 ? pos - pos % chunk : 0;
    const int* bt = meta + meta[META_BT_OFFSET + group] + (size_t)token_entry[t] * meta[META_BT_STRIDE + group];
    for (int i = tid; i < H * d; i += TALK_THREADS) {
        qs[i] = to_float(q[(size_t)t * q_stride + i]);
        acc[i] = 0.f;
    }
    for (int h = tid; h < H; h += TALK_THREADS) m[h] = -INFINITY, l[h] = 0.f;
    auto load_tile = [&](int k0, int n, int kv, int head) {
        __syncthreads();  // the previous tile is no longer read
        for (int idx = tid; idx < n * d; idx += TALK_THREADS) {
            const int j = idx / d, i = idx % d, at = k0 + j, page = bt[at / ps];
            const bool ok = page > 0 && page < num_pages;
            if (!ok) atomicExch(&status[STATUS_BAD_PAGE], 1 + t);
            tile[j * (d + 1) + i] = ok ? to_float(cache[L.offset(page, kv, head, at % ps) + i]) : 0.f;
        }
        __syncthreads();
    };
    // the scores of a tile's keys for every head, -inf behind its end
    auto score_tile = [&](int k0, int n) {
        for (int c = 0; c < G; ++c) {
            load_tile(k0, n, 0, c);
            for (int idx = tid; idx < HG * TALK_KT; idx += TALK_THREADS) {
                const int h = c * HG + idx / TALK_KT, j = idx % TALK_KT;
                float dot = 0.f;
                if (j < n)
                    for (int i = 0; i < d; ++i) dot = fmaf(qs[h * d + i], tile[j * (d + 1) + i], dot);
                p[h * TALK_KT + j] = j < n ? dot * scale : -INFINITY;
            }
        }
        __syncthreads();
    };
    for (int k0 = kstart; k0 <= pos; k0 += TALK_KT) {
        score_tile(k0, min(TALK_KT, pos - k0 + 1));
        for (int h = warp; h < H; h += nwarps) {
            const float s = p[h * TALK_KT + lane], mn = fmaxf(m[h], warp_max(s)), sum = warp_sum(expf(s - mn));
            __syncwarp();
            if (lane == 0) {
                l[h] = l[h] * expf(m[h] - mn) + sum;
                m[h] = mn;
            }
        }
    }
    for (int k0 = kstart; k0 <= pos; k0 += TALK_KT) {
        const int n = min(TALK_KT, pos - k0 + 1);
        score_tile(k0, n);
        for (int idx = tid; idx < H * TALK_KT; idx += TALK_THREADS) p[idx] = expf(p[idx] - m[idx / TALK_KT]) / l[idx / TALK_KT];
        __syncthreads();
        for (int idx = tid; idx < H * TALK_KT; idx += TALK_THREADS) {
            const int h = idx / TALK_KT, j = idx % TALK_KT;
            float s = 0.f;
            for (int g = 0; g < H; ++g) s = fmaf(talk[(size_t)h * H + g], p[g * TALK_KT + j], s);
            pm[idx] = s;
        }
        for (int c = 0; c < G; ++c) {
            load_tile(k0, n, 1, c);  // (its barriers publish pm)
            for (int idx = tid; idx < HG * d; idx += TALK_THREADS) {
                const int h = c * HG + idx / d, i = idx % d;
                float a = acc[h * d + i];
                for (int j = 0; j < n; ++j) a = fmaf(pm[h * TALK_KT + j], tile[j * (d + 1) + i], a);
                acc[h * d + i] = a;
            }
        }
    }
    __syncthreads();
    for (int i = tid; i < H * d; i += TALK_THREADS) out[(size_t)t * H * d + i] = from_float<T>(acc[i]);
}

extern "C" int talk_attn_plain(const void* q, int q_stride, const void* cache, int dtype, const int* meta, int group,
                               const int* token_entry, const int* positions, void* out, int T, int nq, int nkv, int d, int page_size,
                               int num_pages, int chunk, float scale, const float* talk, int* status, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (nkv <= 0 || nq % nkv) return (int)cudaErrorInvalidValue;
    const CacheLayout L{nkv, page_size, d};
    const size_t smem = ((size_t)2 * nq * d + 2 * nq + 2 * (size_t)nq * TALK_KT + (size_t)TALK_KT * (d + 1)) * sizeof(float);
    if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
#define TALK_PLAIN_CASE(TT)                                                                                                \
    do {                                                                                                                  \
        static size_t configured = 0;                                                                                     \
        if (smem > 48 * 1024 && smem > configured) {                                                                      \
            cudaError_t ce = cudaFuncSetAttribute(talk_attn_plain_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (ce != cudaSuccess) return (int)ce;                                                                        \
            configured = smem;                                                                                            \
        }                                                                                                                 \
        return (int)launch_kernel(talk_attn_plain_kernel<TT>, T, TALK_THREADS, smem, stream, (const TT*)q, q_stride, (const TT*)cache, L, \
                                  meta, group, token_entry, positions, (TT*)out, nq, chunk, scale, talk, num_pages, status); \
    } while (0)
    if (dtype == DT_F32) TALK_PLAIN_CASE(float);
    TALK_PLAIN_CASE(__nv_bfloat16);
#undef TALK_PLAIN_CASE
}
