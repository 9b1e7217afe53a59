// bfloat16 attention whose softmax weights are mixed across the query heads (talking_heads.cu says how), on the paged cache,
// specialised by head size (-DHEAD_DIM=...).  The mix needs every head's finished softmax, so neither kernel can run heads
// apart from one another:
//
//  * talk_decode: one thread-block cluster per request (steps in which every request brings one token), its blocks share
//    the visible keys.  Every block scores its keys for all heads (mma.sync, key fragments straight from the pages), the
//    cluster exchanges the heads' maxima and sums through distributed shared memory, every block mixes its finished
//    weights in float32 and weighs its values (mma.sync, value fragments straight from the pages), and the cluster adds
//    the blocks' results up in order.  Each key and value byte is read once; nothing goes through scratch memory.
//  * talk_prefill: one block per 16 tokens and request, all heads.  A first walk over the keys takes every head's maximum
//    and sum; a second one takes the finished weights of a key tile for all heads into shared memory, mixes them on the
//    tensor cores (a [heads x heads] times [heads x positions] product) and weighs the tile's values.
#include <cooperative_groups.h>

#include "attention_tiles.cuh"

namespace cg = cooperative_groups;

int g_use_pdl = 1;
extern "C" void kernels_set_pdl(int mode) { g_use_pdl = mode; }
extern "C" int attn_talk_head_dim() { return D; }

// ----------------------------------------------------------------------------- decode
namespace {
constexpr int TD_THREADS = D <= 64 ? 512 : 256, TD_WARPS = TD_THREADS / 32;  // (wider heads need the registers)
constexpr int TD_MAX_SPLITS = 8;
constexpr int TD_DPR = D / 8;  // dimensions of a value row that a lane of the value phase holds

// Warps that share an item (a key/value head and up to 16 of its query heads) of the value phase.
__host__ __device__ inline int td_key_parts(int H, int G) {
    const int items = G * ((H / G + 15) / 16);
    return items >= TD_WARPS ? 1 : TD_WARPS / items;
}
__host__ __device__ inline int td_row(int n) { return (n + 31) / 32 * 32 + 4; }       // floats of a head's scores
__host__ __device__ inline int td_mixed_row(int n) { return (n + 31) / 32 * 32 + 8; }  // elements of a head's mixed weights
__host__ __device__ inline int td_owned(int H, int splits) { return ((H * D + splits - 1) / splits + 3) / 4 * 4; }
// Shared memory of a block for n keys: q, the keys' places, the mixing weights transposed, weights, mixed weights, partial
// outputs, the other blocks' parts of this block's outputs, (m, l) pairs, factors.
inline size_t td_smem(int H, int G, int n, int splits) {
    return (size_t)H * D * sizeof(bf16) + (size_t)td_row(n) * sizeof(long long) + (size_t)H * ((H + 7) / 8 * 8) * sizeof(float) +
           (size_t)H * td_row(n) * sizeof(float) + (size_t)H * td_mixed_row(n) * sizeof(bf16) +
           ((size_t)td_key_parts(H, G) * H * D + (size_t)splits * td_owned(H, splits) + 3 * (size_t)H) * sizeof(float);
}
// TD_DPR consecutive elements of a row as words of two (TD_DPR is even; a row's piece starts on TD_DPR * 2 bytes).
__device__ __forceinline__ void load_words(const bf16* p, uint32_t (&w)[TD_DPR / 2]) {
    if constexpr (TD_DPR % 8 == 0) {
#pragma unroll
        for (int i = 0; i < TD_DPR / 8; ++i) {
            const uint4 v = reinterpret_cast<const uint4*>(p)[i];
            w[4 * i] = v.x, w[4 * i + 1] = v.y, w[4 * i + 2] = v.z, w[4 * i + 3] = v.w;
        }
    } else if constexpr (TD_DPR % 4 == 0) {
#pragma unroll
        for (int i = 0; i < TD_DPR / 4; ++i) {
            const uint2 v = reinterpret_cast<const uint2*>(p)[i];
            w[2 * i] = v.x, w[2 * i + 1] = v.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < TD_DPR / 2; ++i) w[i] = reinterpret_cast<const uint32_t*>(p)[i];
    }
}
}  // namespace

__global__ void __launch_bounds__(TD_THREADS)
talk_decode_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ cache, CacheLayout L, const int* __restrict__ meta,
                   int group, const int* __restrict__ positions, bf16* __restrict__ out, int H, int chunk, float scale_log2,
                   const float* __restrict__ talk, int num_pages, int splits, int max_keys, int* __restrict__ status) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int G = L.num_kv_heads, HG = H / G, HP = (H + 7) / 8 * 8, NS = td_row(max_keys), NM = td_mixed_row(max_keys), parts = td_key_parts(H, G);
    const int owned = td_owned(H, splits);
    long long* off = reinterpret_cast<long long*>(smem_raw);                   // [NS]: a key's place in the cache, -1: none
    bf16* qs = reinterpret_cast<bf16*>(off + NS);                              // [H][D]
    bf16* pm = qs + (size_t)H * D;                                             // [H][NM]: mixed weights
    float* tt = reinterpret_cast<float*>(pm + (size_t)H * NM);                 // [H][HP]: talk transposed, tt[g][h], then times g's factor
    float* sc = tt + (size_t)H * HP;                                           // [H][NS]: scores, then their exponentials
    float* po = sc + (size_t)H * NS;                                           // [parts][H][D]
    float* recv = po + (size_t)parts * H * D;                                  // [splits][owned]
    float* ml = recv + (size_t)splits * owned;                                 // [H][2]
    float* fac = ml + 2 * (size_t)H;                                           // [H]
    pdl_launch_dependents();
    const int split = blockIdx.x, e = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // (a block of a dead request leaves with its whole cluster)
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int pos = positions[e], kstart = chunk > 0 ? pos - pos % chunk : 0, len = pos + 1 - kstart;
    int per = ((len + splits - 1) / splits + 7) / 8 * 8;
    if (per > max_keys) {  // (the host's bound on the keys of a block does not hold: nothing is read beyond it)
        if (tid == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + pos);
        per = max_keys;
    }
    const int lo = kstart + split * per, n = max(0, min(per, pos + 1 - lo)), blocks32 = (n + 31) / 32;
    const int* bt = meta + meta[META_BT_OFFSET + group] + (size_t)e * meta[META_BT_STRIDE + group];
    const int ps = L.page_size;
    const size_t v_off = (size_t)G * ps * D, page_stride = 2 * v_off;
    for (int j = tid; j < blocks32 * 32; j += TD_THREADS) {
        long long at = -1;
        if (j < n) {
            const int k = lo + j, page = bt[k / ps];
            if (page > 0 && page < num_pages) at = (long long)((size_t)page * page_stride + (size_t)(k % ps) * D);
            else atomicExch(&status[STATUS_BAD_PAGE], 1 + k);
        }
        off[j] = at;
    }
    for (int i = tid; i < H * HP; i += TD_THREADS) {
        const int h = i / H, g = i % H;  // (neighbouring threads read neighbouring weights)
        tt[g * HP + h] = h < H ? talk[(size_t)h * H + g] : 0.f;
    }
    pdl_wait();
    for (int i = tid; i < H * D / 8; i += TD_THREADS)
        reinterpret_cast<uint4*>(qs)[i] = *reinterpret_cast<const uint4*>(q + (size_t)e * q_stride + (size_t)i * 8);
    __syncthreads();
    // Scores: an item is a key/value head and 32 keys; the next item's keys are on their way while one is computed.  Both
    // operands take the 16 dimensions of a k-step in the order (4t, 4t + 1 | 4t + 2, 4t + 3) for lane t of a quad, so a key
    // fragment is one 8-byte load from the page.
    const int r = lane >> 2, t4 = (lane & 3) * 4;
    {
        constexpr bool AHEAD = KSTEPS <= 8;
        const int items = G * blocks32;
        uint2 cur[4][KSTEPS], nxt[AHEAD ? 4 : 1][AHEAD ? KSTEPS : 1];
        auto load_keys = [&](int item, auto& kf) {
            const bf16* base = cache + (size_t)(item % G) * ps * D + t4;
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                const long long at = off[(item / G) * 32 + nt * 8 + r];
#pragma unroll
                for (int ks = 0; ks < KSTEPS; ++ks)
                    kf[nt][ks] = at >= 0 ? *reinterpret_cast<const uint2*>(base + at + ks * 16) : make_uint2(0u, 0u);
            }
        };
        if (AHEAD && warp < items) load_keys(warp, cur);
        for (int item = warp; item < items; item += TD_WARPS) {
            if constexpr (AHEAD) {
                if (item + TD_WARPS < items) load_keys(item + TD_WARPS, nxt);
            } else {
                load_keys(item, cur);
            }
            const int c = item % G, k0 = (item / G) * 32;
            for (int m0 = 0; m0 < HG; m0 += 16) {
                float s[4][4];
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
                const bool in0 = m0 + r < HG, in1 = m0 + r + 8 < HG;
                const bf16* q0 = qs + (size_t)(c * HG + m0 + r) * D + t4;
#pragma unroll
                for (int ks = 0; ks < KSTEPS; ++ks) {
                    const uint2 x = in0 ? *reinterpret_cast<const uint2*>(q0 + ks * 16) : make_uint2(0u, 0u);
                    const uint2 y = in1 ? *reinterpret_cast<const uint2*>(q0 + 8 * D + ks * 16) : make_uint2(0u, 0u);
                    const uint32_t a[4] = {x.x, y.x, x.y, y.y};
#pragma unroll
                    for (int nt = 0; nt < 4; ++nt) mma_bf16(s[nt], a, cur[nt][ks].x, cur[nt][ks].y);
                }
#pragma unroll
                for (int nt = 0; nt < 4; ++nt) {
                    const int key = k0 + nt * 8 + (lane & 3) * 2;
                    const bool k_in = key < n, k1_in = key + 1 < n;
                    if (in0) *reinterpret_cast<float2*>(sc + (size_t)(c * HG + m0 + r) * NS + key) =
                        make_float2(k_in ? s[nt][0] * scale_log2 : -INFINITY, k1_in ? s[nt][1] * scale_log2 : -INFINITY);
                    if (in1) *reinterpret_cast<float2*>(sc + (size_t)(c * HG + m0 + r + 8) * NS + key) =
                        make_float2(k_in ? s[nt][2] * scale_log2 : -INFINITY, k1_in ? s[nt][3] * scale_log2 : -INFINITY);
                }
            }
            if constexpr (AHEAD) {
#pragma unroll
                for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                    for (int ks = 0; ks < KSTEPS; ++ks) cur[nt][ks] = nxt[nt][ks];
            }
        }
    }
    __syncthreads();
    // every head's maximum and sum over this block's keys; the scores become exponentials against that maximum
    for (int h = warp; h < H; h += TD_WARPS) {
        float* row = sc + (size_t)h * NS;
        float mx = -INFINITY, sum = 0.f;
        for (int j = lane; j < n; j += 32) mx = fmaxf(mx, row[j]);
        mx = warp_max(mx);
        for (int j = lane; j < blocks32 * 32; j += 32) {
            const float p = j < n ? fast_exp2(row[j] - mx) : 0.f;
            row[j] = p;
            sum += p;
        }
        sum = warp_sum(sum);
        if (lane == 0) ml[2 * h] = mx, ml[2 * h + 1] = sum;
    }
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    // what turns this block's exponentials into softmax weights, over all blocks of the cluster, in order
    for (int h = tid; h < H; h += TD_THREADS) {
        float m[TD_MAX_SPLITS], l[TD_MAX_SPLITS], mx = -INFINITY, sum = 0.f;
#pragma unroll
        for (int s = 0; s < TD_MAX_SPLITS; ++s) {  // independent loads, all in flight together
            m[s] = -INFINITY, l[s] = 0.f;
            if (s < splits) {
                const float2 v = *reinterpret_cast<const float2*>(cluster.map_shared_rank(ml, s) + 2 * h);
                m[s] = v.x, l[s] = v.y;
            }
        }
#pragma unroll
        for (int s = 0; s < TD_MAX_SPLITS; ++s) mx = fmaxf(mx, m[s]);
#pragma unroll
        for (int s = 0; s < TD_MAX_SPLITS; ++s) sum += m[s] > -INFINITY ? l[s] * fast_exp2(m[s] - mx) : 0.f;
        fac[h] = n > 0 ? fast_exp2(ml[2 * h] - mx) / sum : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < H * HP; i += TD_THREADS) tt[i] *= fac[i / HP];
    __syncthreads();
    // The mix: a warp takes 32 keys and 8 heads at a time, float32.
    const int hb8 = HP / 8;
    for (int item = warp; item < hb8 * blocks32; item += TD_WARPS) {
        const int h0 = (item % hb8) * 8, j = (item / hb8) * 32 + lane;
        float acc[8] = {};
        for (int g = 0; g < H; ++g) {
            const float p = sc[(size_t)g * NS + j];
            const float4 a = *reinterpret_cast<const float4*>(tt + (size_t)g * HP + h0), b = *reinterpret_cast<const float4*>(tt + (size_t)g * HP + h0 + 4);
            acc[0] = fmaf(a.x, p, acc[0]); acc[1] = fmaf(a.y, p, acc[1]); acc[2] = fmaf(a.z, p, acc[2]); acc[3] = fmaf(a.w, p, acc[3]);
            acc[4] = fmaf(b.x, p, acc[4]); acc[5] = fmaf(b.y, p, acc[5]); acc[6] = fmaf(b.z, p, acc[6]); acc[7] = fmaf(b.w, p, acc[7]);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (h0 + i < H) pm[(size_t)(h0 + i) * NM + j] = __float2bfloat16_rn(acc[i]);
    }
    __syncthreads();
    // Values: an item is a key/value head and up to 16 of its query heads; `parts` warps share an item's keys, 16 at a step.
    // Lane (r, t) holds dimensions r * TD_DPR .. of keys 4t .. 4t + 3 of a step: the operand's column r of tile j is
    // dimension r * TD_DPR + j, its rows the keys in that order, which the weights' fragment (two 8-byte loads) takes too.
    {
        const int mt = (HG + 15) / 16, part = warp % parts, steps = blocks32 * 2;
        constexpr int UN = TD_DPR <= 8 ? 2 : 1;  // steps in flight a warp
        for (int item = warp / parts; item < G * mt; item += TD_WARPS / parts) {
            const int c = item / mt, h0 = c * HG + (item % mt) * 16, nh = min(16, (c + 1) * HG - h0);
            const bf16* base = cache + v_off + (size_t)c * ps * D + r * TD_DPR;
            float acc[TD_DPR][4];
#pragma unroll
            for (int j = 0; j < TD_DPR; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
            for (int s0 = part; s0 < steps; s0 += parts * UN) {
                uint32_t w[UN][4][TD_DPR / 2];
#pragma unroll
                for (int u = 0; u < UN; ++u)
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        const int st = s0 + u * parts;
                        const long long at = st < steps ? off[st * 16 + t4 + k] : -1;
                        if (at >= 0) {
                            load_words(base + at, w[u][k]);
                        } else {
#pragma unroll
                            for (int i = 0; i < TD_DPR / 2; ++i) w[u][k][i] = 0u;
                        }
                    }
#pragma unroll
                for (int u = 0; u < UN; ++u) {
                    const int st = s0 + u * parts;
                    if (st >= steps) continue;
                    const uint2 x = r < nh ? *reinterpret_cast<const uint2*>(pm + (size_t)(h0 + r) * NM + st * 16 + t4) : make_uint2(0u, 0u);
                    const uint2 y = r + 8 < nh ? *reinterpret_cast<const uint2*>(pm + (size_t)(h0 + r + 8) * NM + st * 16 + t4) : make_uint2(0u, 0u);
                    const uint32_t a[4] = {x.x, y.x, x.y, y.y};
#pragma unroll
                    for (int j = 0; j < TD_DPR; ++j) {
                        const uint32_t sel = j & 1 ? 0x7632u : 0x5410u;
                        mma_bf16(acc[j], a, __byte_perm(w[u][0][j / 2], w[u][1][j / 2], sel), __byte_perm(w[u][2][j / 2], w[u][3][j / 2], sel));
                    }
                }
            }
            const int d0 = (lane & 3) * 2 * TD_DPR;
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                if (r + 8 * b >= nh) continue;
                float* dst = po + ((size_t)part * H + h0 + r + 8 * b) * D + d0;
#pragma unroll
                for (int j = 0; j < TD_DPR; ++j) {
                    dst[j] = acc[j][2 * b];
                    dst[TD_DPR + j] = acc[j][2 * b + 1];
                }
            }
        }
    }
    __syncthreads();
    // Block s of the cluster owns outputs s * owned ..: every block hands it its part (an item's warps in order), and the
    // owner adds the blocks' parts up in order.
    for (int i = tid; i < H * D; i += TD_THREADS) {
        float a = 0.f;
        for (int p = 0; p < parts; ++p) a += po[(size_t)p * H * D + i];
        const int owner = i / owned;
        cluster.map_shared_rank(recv, owner)[(size_t)split * owned + (i - owner * owned)] = a;
    }
    cluster.sync();
    for (int i = tid; i < owned && split * owned + i < H * D; i += TD_THREADS) {
        float a = 0.f;
        for (int s = 0; s < splits; ++s) a += recv[(size_t)s * owned + i];
        out[(size_t)e * H * D + split * owned + i] = __float2bfloat16_rn(a);
    }
}

// The fewest blocks a request's keys (at most max_keys of them) can be shared by, at most TD_MAX_SPLITS; 0: they do not fit.
extern "C" int attn_talk_decode_min_splits(int nq, int nkv, int max_keys) {
    if (nkv <= 0 || nq % nkv) return 0;
    for (int s = 1; s <= TD_MAX_SPLITS; ++s)
        if (td_smem(nq, nkv, ((max_keys + s - 1) / s + 7) / 8 * 8, s) <= 200 * 1024) return s;
    return 0;
}

// How many decode blocks a multiprocessor holds by threads and registers; the host sizes the splits by it.
extern "C" int attn_talk_decode_blocks_per_sm() { return D <= 64 ? 1 : 2; }

extern "C" int attn_talk_decode(const void* q, int q_stride, const void* cache, const int* meta, int group, const int* positions, void* out,
                                int S, int nq, int nkv, int page_size, int num_pages, int chunk, float scale, const float* talk, int splits,
                                int max_context, int* status, cudaStream_t stream) {
    if (S <= 0) return 0;
    if (nkv <= 0 || nq % nkv || splits < 1 || splits > TD_MAX_SPLITS || q_stride % 8 || ((uintptr_t)q & 15)) return (int)cudaErrorInvalidValue;
    const int seen = chunk > 0 && chunk < max_context ? chunk : max_context;
    const int max_keys = ((seen + splits - 1) / splits + 7) / 8 * 8;
    const size_t smem = td_smem(nq, nkv, max_keys, splits);
    if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
    static size_t configured = 0;  // grows only, and is not set again inside a stream capture once large enough
    if (smem > 48 * 1024 && smem > configured) {
        cudaError_t err = cudaFuncSetAttribute(talk_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
        configured = smem;
    }
    const CacheLayout L{nkv, page_size, D};
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, S);
    cfg.blockDim = dim3(TD_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = (g_use_pdl & 1) ? 2 : 1;
    return (int)cudaLaunchKernelEx(&cfg, talk_decode_kernel, (const bf16*)q, q_stride, (const bf16*)cache, L, meta, group, positions,
                                   (bf16*)out, nq, chunk, scale * LOG2E, talk, num_pages, splits, max_keys, status);
}

// ----------------------------------------------------------------------------- prefill (and mixed steps)
namespace {
constexpr int TP_WARPS = D <= 64 ? 16 : 8, TP_THREADS = TP_WARPS * 32;  // (wider heads need the registers)
constexpr int TP_TOK = 16;  // tokens of a block

// Heads whose outputs a warp keeps in registers, for H heads (more heads than a block's warps keep: blocks share them).
inline int tp_heads_per_warp(int H) {
    const int most = D <= 128 ? 2 : 1;
    int n = 1;
    while (n < most && n * TP_WARPS < H) n *= 2;
    return n;
}
inline int pad16(int n) { return (n + 15) / 16 * 16; }
inline size_t tp_smem(int H, int G, int KT, int stages, int bt_cap) {
    return ((size_t)H * TP_TOK * LDS + (size_t)(stages + 1) * G * KT * LDS + (size_t)pad16(H) * TP_TOK * KT + (size_t)pad16(H) * (pad16(H) + 8)) * sizeof(bf16) +
           (size_t)H * TP_TOK * sizeof(float) + (size_t)(bt_cap + H) * sizeof(int);
}
}  // namespace

// Shared memory of the weights: head g's 16 x KT tile as 16-byte pieces of 8 keys, piece n * 16 + row at place (n * 16 + row) ^
// (g & 7), so that the pieces of 8 neighbouring rows, and those of one row of 8 neighbouring heads, lie in different banks.
// (The exclusive or stays inside groups of 8 pieces: n * 16 + 8 * (row / 8) + ((row % 8) ^ (g & 7)).)
constexpr int TP_STATS = D <= 64 ? 2 : 4;  // heads a warp takes at a time in the first walk
constexpr bool TP_Q_KEPT = D <= 64;        // ... with their queries' fragments in registers

// Shared memory by 32-bit address: the loops below compute an address per fragment, and generic pointers would cost three
// times the instructions.
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void sts_u32(uint32_t a, uint32_t v) { asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(a), "r"(v) : "memory"); }
__device__ __forceinline__ void cp_async_16_to(uint32_t a, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(gmem) : "memory");
}
// Bytes of (row, col) in a tile (toff in bytes), and the place of the fragment `step` steps of 16 columns behind one at `at`: in
// swizzled tiles a step of 16 columns is an exclusive or of the two piece bits above the first (a row's pieces of 128 bytes
// start on 128 bytes), in padded ones an addition.
__device__ __forceinline__ uint32_t tile_bytes(int row, int col) { return (uint32_t)toff(row, col) * 2u; }
__device__ __forceinline__ uint32_t step16(uint32_t at, int step) {
    if constexpr (SWZ) return (at ^ ((uint32_t)(step & 3) << 5)) + (uint32_t)(step >> 2) * 128u;
    return at + (uint32_t)step * 32u;
}
constexpr uint32_t ROW_BYTES = LDS * 2;

// What a lane needs to know of its two rows (g4 and g4 + 8 of the 16 tokens) and of where it reads fragments in a tile.
struct TalkLane {
    uint32_t q_at, k_at;  // bytes from the start of a head's queries, of a key tile
    int tig;
    int pa, pb, ca, cb;   // the rows' positions (-1: a padding row) and their chunks' starts
};

// The products of a head's 16 tokens with a tile's keys, unscaled; unless every token sees the tile WHOLE, -inf where a token
// does not see a key.  KEPT: the queries' fragments come from registers.
template <bool WHOLE, bool KEPT, int NK>
__device__ __forceinline__ void talk_scores(float (&s)[NK][4], const TalkLane& w, uint32_t qh, const uint32_t (*qf)[4], uint32_t kh, int k0) {
#pragma unroll
    for (int n = 0; n < NK; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
    const uint32_t q_at = qh + w.q_at, k_at = kh + w.k_at;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
        uint32_t a[4];
        if constexpr (KEPT) { a[0] = qf[ks][0]; a[1] = qf[ks][1]; a[2] = qf[ks][2]; a[3] = qf[ks][3]; }
        else ldsm_x4(a, step16(q_at, ks));
#pragma unroll
        for (int np = 0; np < NK / 2; ++np) {
            uint32_t b[4];
            ldsm_x4(b, step16(k_at, ks) + np * 16 * ROW_BYTES);
            mma_bf16(s[2 * np], a, b[0], b[1]);
            mma_bf16(s[2 * np + 1], a, b[2], b[3]);
        }
    }
    if constexpr (!WHOLE) {
#pragma unroll
        for (int n = 0; n < NK; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int key = k0 + n * 8 + w.tig * 2 + (c & 1);
                const bool sees = c < 2 ? (key <= w.pa) & (key >= w.ca) : (key <= w.pb) & (key >= w.cb);
                s[n][c] = sees ? s[n][c] : -INFINITY;
            }
    }
}

// First walk, one tile and head: the lane's running maxima and sums over its own columns of its two rows.
template <bool WHOLE, bool KEPT, int NK>
__device__ __forceinline__ void talk_stats(float (&m)[2], float (&l)[2], const TalkLane& w, uint32_t qh, const uint32_t (*qf)[4],
                                           uint32_t kh, int k0, float scale_log2) {
    float s[NK][4];
    talk_scores<WHOLE, KEPT, NK>(s, w, qh, qf, kh, k0);
#pragma unroll
    for (int b = 0; b < 2; ++b) {
        float mx = fmaxf(s[0][2 * b], s[0][2 * b + 1]);
#pragma unroll
        for (int n = 1; n < NK; ++n) mx = fmaxf(mx, fmaxf(s[n][2 * b], s[n][2 * b + 1]));
        const float m_new = fmaxf(m[b], mx), base = m_new == -INFINITY ? 0.f : m_new, off = base * scale_log2;
        float sum = l[b] * fast_exp2(m[b] * scale_log2 - off);
#pragma unroll
        for (int n = 0; n < NK; ++n)
            sum += fast_exp2(fmaf(s[n][2 * b], scale_log2, -off)) + fast_exp2(fmaf(s[n][2 * b + 1], scale_log2, -off));
        l[b] = sum;
        m[b] = m_new;
    }
}

// Second walk, one tile and head: the finished weights, to the head's pieces in shared memory.
template <bool WHOLE, int NK>
__device__ __forceinline__ void talk_weights(uint32_t dst, const TalkLane& w, uint32_t qh, uint32_t kh, int k0, float scale_log2, float s0, float s1) {
    float s[NK][4];
    talk_scores<WHOLE, false, NK>(s, w, qh, nullptr, kh, k0);
#pragma unroll
    for (int n = 0; n < NK; ++n) {
        sts_u32(dst + n * 256, pack_bf16(fast_exp2(fmaf(s[n][0], scale_log2, -s0)), fast_exp2(fmaf(s[n][1], scale_log2, -s0))));
        sts_u32(dst + n * 256 + 128, pack_bf16(fast_exp2(fmaf(s[n][2], scale_log2, -s1)), fast_exp2(fmaf(s[n][3], scale_log2, -s1))));
    }
}

template <int KT, int HPW>
__global__ void __launch_bounds__(TP_THREADS)
talk_prefill_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ cache, CacheLayout L, const int* __restrict__ meta,
                    int group, const int* __restrict__ cu_tokens, const int* __restrict__ ctx_lens, bf16* __restrict__ out, int H,
                    int chunk, float scale_log2, const float* __restrict__ talk, int num_pages, int bt_cap, int stages,
                    int* __restrict__ status) {
    constexpr int NK = KT / 8, MT = TP_WARPS * HPW > 16 ? TP_WARPS * HPW / 16 : 1, PH = TP_TOK * KT;  // PH: a head's weights
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    const int G = L.num_kv_heads, HG = H / G, HP = (H + 15) / 16 * 16, TS = HP + 8, ps = L.page_size;
    bf16* qt = reinterpret_cast<bf16*>(smem_raw);             // [H][16][LDS]
    bf16* kt = qt + (size_t)H * TP_TOK * LDS;                 // [stages][G][KT][LDS]
    bf16* vt = kt + (size_t)stages * G * KT * LDS;            // [G][KT][LDS]
    bf16* pt = vt + (size_t)G * KT * LDS;                     // [HP][PH]
    bf16* tk = pt + (size_t)HP * PH;                          // [HP][TS]: talk
    float* lse = reinterpret_cast<float*>(tk + (size_t)HP * TS);  // [H][16]: base-2 logarithm of a row's sum of exponentials
    int* kv_of = reinterpret_cast<int*>(lse + (size_t)H * TP_TOK);  // [H]: where a head's keys and values start in a tile
    int* bt_s = kv_of + H;
    pdl_launch_dependents();
    pdl_wait();
    // late query tiles see the most keys: they go first
    const int tile = gridDim.x - 1 - blockIdx.x, hpart = blockIdx.y, e = blockIdx.z;
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int row0 = cu_tokens[e], q_len = cu_tokens[e + 1] - row0, t0 = tile * TP_TOK;
    if (t0 >= q_len) return;
    const int nt = min(TP_TOK, q_len - t0), p_first = ctx_lens[e] + t0, p_last = p_first + nt - 1;
    const int* bt = meta + meta[META_BT_OFFSET + group] + (size_t)e * meta[META_BT_STRIDE + group];
    const int kbeg = chunk > 0 ? p_first - p_first % chunk : 0, kend = p_last + 1;
    const int page_lo = kbeg / ps;
    int page_cnt = (kend - 1) / ps - page_lo + 1;
    if (page_cnt > bt_cap) {
        if (tid == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + kend);
        page_cnt = bt_cap;
    }
    stage_block_table(bt_s, bt, page_lo, page_cnt, num_pages, tid, TP_THREADS, status);
    const int kend_s = min(kend, (page_lo + page_cnt) * ps), ntiles = (kend - kbeg + KT - 1) / KT;
    const int ps_shift = (ps & (ps - 1)) == 0 ? 31 - __clz(ps) : -1;
    const size_t v_off = (size_t)G * ps * D, page_stride = 2 * v_off;
    for (int idx = tid; idx < H * TP_TOK * (D / 8); idx += TP_THREADS) {
        const int c = idx % (D / 8), h = (idx / (D / 8)) % H, tok = idx / (D / 8) / H;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (tok < nt) v = *reinterpret_cast<const uint4*>(q + (size_t)(row0 + t0 + tok) * q_stride + (size_t)h * D + c * 8);
        *reinterpret_cast<uint4*>(qt + (size_t)h * TP_TOK * LDS + toff(tok, c * 8)) = v;
    }
    for (int idx = tid; idx < HP * HP; idx += TP_THREADS) {
        const int h = idx / HP, g = idx % HP;
        tk[h * TS + g] = __float2bfloat16_rn(h < H && g < H ? talk[(size_t)h * H + g] : 0.f);
    }
    for (int idx = tid; idx < (HP - H) * PH; idx += TP_THREADS) pt[(size_t)H * PH + idx] = __float2bfloat16_rn(0.f);
    for (int h = tid; h < H; h += TP_THREADS) kv_of[h] = (h / HG) * KT * LDS * 2;
    const uint32_t qt_a = smem_u32(qt), kt_a = smem_u32(kt), vt_a = smem_u32(vt), pt_a = smem_u32(pt), tk_a = smem_u32(tk);
    const uint32_t kv_bytes = (uint32_t)G * KT * ROW_BYTES;
    // Keys (kv = 0) or values (kv = 1) of a tile for every head; positions outside [kbeg, kend_s) as zeros.  A thread copies
    // 16 dimensions of the same rows of every few heads, so a row's page is looked up once.
    constexpr int PAIRS = D / 16, PP = PAIRS <= 1 ? 1 : PAIRS <= 2 ? 2 : PAIRS <= 4 ? 4 : PAIRS <= 8 ? 8 : 16;
    constexpr int RS = TP_THREADS / PP < KT ? TP_THREADS / PP : KT, CS = TP_THREADS / (PP * RS);
    const int c16 = (tid % PP) * 16, rr0 = (tid / PP) % RS, cc0 = tid / (PP * RS);
    auto load_tile = [&](uint32_t dst, int t, int kv) {
        if (c16 >= D) return;
        for (int rr = rr0; rr < KT; rr += RS) {
            const int at = kbeg + t * KT + rr;
            int page = -1, slot = 0;
            if (at < kend_s) {
                const int pi = ps_shift >= 0 ? at >> ps_shift : at / ps;
                slot = at - pi * ps;
                page = bt_s[pi - page_lo];
            }
            uint32_t d0 = dst + (uint32_t)cc0 * KT * ROW_BYTES + tile_bytes(rr, c16), d1 = dst + (uint32_t)cc0 * KT * ROW_BYTES + tile_bytes(rr, c16 + 8);
            if (page > 0) {
                const bf16* src = cache + (size_t)page * page_stride + (kv ? v_off : 0) + (size_t)(cc0 * ps + slot) * D + c16;
                for (int c = cc0; c < G; c += CS) {
                    cp_async_16_to(d0, src);
                    cp_async_16_to(d1, src + 8);
                    d0 += CS * KT * ROW_BYTES, d1 += CS * KT * ROW_BYTES, src += (size_t)CS * ps * D;
                }
            } else {
                for (int c = cc0; c < G; c += CS) {
                    asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};\n" ::"r"(d0), "r"(0) : "memory");
                    asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};\n" ::"r"(d1), "r"(0) : "memory");
                    d0 += CS * KT * ROW_BYTES, d1 += CS * KT * ROW_BYTES;
                }
            }
        }
    };
    auto k_stage = [&](int t) { return kt_a + (stages == 2 && (t & 1) ? kv_bytes : 0u); };
    const int g4 = lane >> 2, tig = lane & 3, j8 = lane >> 3, l7 = lane & 7;
    TalkLane w;
    w.tig = tig;
    const int q_row = l7 + (j8 & 1) * 8, q_col = (j8 >> 1) * 8;
    w.q_at = tile_bytes(q_row, q_col), w.k_at = tile_bytes(l7 + (j8 >> 1) * 8, (j8 & 1) * 8);
    w.pa = g4 < nt ? p_first + g4 : -1, w.pb = g4 + 8 < nt ? p_first + g4 + 8 : -1;
    w.ca = chunk > 0 && w.pa >= 0 ? w.pa - w.pa % chunk : 0, w.cb = chunk > 0 && w.pb >= 0 ? w.pb - w.pb % chunk : 0;
    const int c_last = chunk > 0 ? p_last - p_last % chunk : 0;
    // a tile that every token sees whole
    auto whole_tile = [&](int k0) { return nt == TP_TOK && k0 + KT - 1 <= p_first && k0 >= c_last; };
    __syncthreads();  // the table slice is written
    // ---- first walk: every row's maximum and sum, for every head.  A lane keeps them for its own columns; the quad's four
    // lanes are put together at the end.
    for (int h0 = warp; h0 < H + warp; h0 += TP_WARPS * TP_STATS) {  // (all warps walk alike)
        float m[TP_STATS][2], l[TP_STATS][2];
#pragma unroll
        for (int i = 0; i < TP_STATS; ++i) m[i][0] = m[i][1] = -INFINITY, l[i][0] = l[i][1] = 0.f;
        uint32_t qf[TP_STATS][TP_Q_KEPT ? KSTEPS : 1][4];
        if constexpr (TP_Q_KEPT) {
#pragma unroll
            for (int i = 0; i < TP_STATS; ++i)
#pragma unroll
                for (int ks = 0; ks < KSTEPS; ++ks)
                    ldsm_x4(qf[i][ks], step16(qt_a + (uint32_t)min(h0 + i * TP_WARPS, H - 1) * TP_TOK * ROW_BYTES + w.q_at, ks));
        }
        load_tile(k_stage(0), 0, 0);
        cp_async_commit();
        for (int t = 0; t < ntiles; ++t) {
            if (stages == 2 && t + 1 < ntiles) {
                load_tile(k_stage(t + 1), t + 1, 0);
                cp_async_commit();
                cp_async_wait<1>();
            } else {
                cp_async_wait<0>();
            }
            __syncthreads();
            const int k0 = kbeg + t * KT;
            const uint32_t keys = k_stage(t);
            if (whole_tile(k0)) {
#pragma unroll
                for (int i = 0; i < TP_STATS; ++i) {
                    const int h = h0 + i * TP_WARPS;
                    if (h < H) talk_stats<true, TP_Q_KEPT, NK>(m[i], l[i], w, qt_a + (uint32_t)h * TP_TOK * ROW_BYTES, qf[i], keys + kv_of[h], k0, scale_log2);
                }
            } else {
#pragma unroll
                for (int i = 0; i < TP_STATS; ++i) {
                    const int h = h0 + i * TP_WARPS;
                    if (h < H) talk_stats<false, TP_Q_KEPT, NK>(m[i], l[i], w, qt_a + (uint32_t)h * TP_TOK * ROW_BYTES, qf[i], keys + kv_of[h], k0, scale_log2);
                }
            }
            __syncthreads();  // the stage may be overwritten
            if (stages == 1 && t + 1 < ntiles) {
                load_tile(k_stage(t + 1), t + 1, 0);
                cp_async_commit();
            }
        }
#pragma unroll
        for (int i = 0; i < TP_STATS; ++i) {
            const int h = h0 + i * TP_WARPS;
            if (h >= H) continue;
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                float mm = m[i][b], ll = l[i][b];
#pragma unroll
                for (int o = 1; o < 4; o <<= 1) {
                    const float om = __shfl_xor_sync(0xffffffffu, mm, o), ol = __shfl_xor_sync(0xffffffffu, ll, o), mn = fmaxf(mm, om);
                    const float base = mn == -INFINITY ? 0.f : mn;
                    ll = ll * fast_exp2((mm - base) * scale_log2) + ol * fast_exp2((om - base) * scale_log2);
                    mm = mn;
                }
                // (a padding row sees nothing: every weight becomes zero)
                if (tig == 0) lse[h * TP_TOK + g4 + 8 * b] = ll > 0.f ? fmaf(mm, scale_log2, log2f(ll)) : INFINITY;
            }
        }
    }
    // ---- second walk: weights, mix, values
    const int h_lo = hpart * TP_WARPS * HPW, h_hi = min(H, h_lo + TP_WARPS * HPW);  // the heads whose outputs this block makes
    const int m0 = h_lo / 16 * 16;                                                 // first head of its tiles of 16
    float o[HPW][DTILES][4];
#pragma unroll
    for (int i = 0; i < HPW; ++i)
#pragma unroll
        for (int dt = 0; dt < DTILES; ++dt) o[i][dt][0] = o[i][dt][1] = o[i][dt][2] = o[i][dt][3] = 0.f;
    load_tile(k_stage(0), 0, 0);
    cp_async_commit();
    for (int t = 0; t < ntiles; ++t) {
        cp_async_wait<0>();
        __syncthreads();  // keys of the tile are there; values and weights of the tile before are no longer read
        load_tile(vt_a, t, 1);
        cp_async_commit();
        const bool ahead = stages == 2 && t + 1 < ntiles;
        if (ahead) {
            load_tile(k_stage(t + 1), t + 1, 0);
            cp_async_commit();
        }
        const int k0 = kbeg + t * KT;
        const uint32_t keys = k_stage(t);
        const bool whole = whole_tile(k0);
        for (int h = warp; h < H; h += TP_WARPS) {
            const float s0 = lse[h * TP_TOK + g4], s1 = lse[h * TP_TOK + g4 + 8];
            const uint32_t dst = pt_a + (uint32_t)(h * PH + (g4 ^ (h & 7)) * 8 + tig * 2) * 2u;
            if (whole) talk_weights<true, NK>(dst, w, qt_a + (uint32_t)h * TP_TOK * ROW_BYTES, keys + kv_of[h], k0, scale_log2, s0, s1);
            else talk_weights<false, NK>(dst, w, qt_a + (uint32_t)h * TP_TOK * ROW_BYTES, keys + kv_of[h], k0, scale_log2, s0, s1);
        }
        __syncthreads();
        // The mix, in place: a warp owns two pieces (16 positions) at a time of all heads, reads them and writes the heads of
        // its block's tiles of 16 (a padding head's row and column of the mixing weights are zero).
        {
            const int pc = warp * 2;  // a round moves the pieces by whole groups of 8
            const uint32_t src = pt_a + (uint32_t)((l7 + (j8 & 1) * 8) * PH + ((pc & ~7) + (((pc + (j8 >> 1)) & 7) ^ l7)) * 8) * 2u;
            const uint32_t dst = pt_a + (uint32_t)((m0 + g4) * PH + tig * 2) * 2u;
            const uint32_t ta = tk_a + (uint32_t)((m0 + q_row) * TS + q_col) * 2u;
#pragma unroll
            for (int round = 0; round < TP_TOK * NK / (TP_WARPS * 2); ++round) {
                float acc[MT][2][4];
#pragma unroll
                for (int i = 0; i < MT; ++i)
#pragma unroll
                    for (int b = 0; b < 2; ++b) acc[i][b][0] = acc[i][b][1] = acc[i][b][2] = acc[i][b][3] = 0.f;
                for (int g0 = 0; g0 < HP; g0 += 16) {
                    uint32_t b[4];
                    ldsm_x4_trans(b, src + (uint32_t)g0 * PH * 2u + round * TP_WARPS * 32);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        if (m0 + i * 16 >= h_hi) continue;
                        uint32_t a[4];
                        ldsm_x4(a, ta + (uint32_t)(i * 16 * TS + g0) * 2u);
                        mma_bf16(acc[i][0], a, b[0], b[1]);
                        mma_bf16(acc[i][1], a, b[2], b[3]);
                    }
                }
                __syncwarp();  // the warp has read its pieces
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const uint32_t place = dst + (uint32_t)((pc & ~7) + (((pc + b) & 7) ^ g4)) * 16u + round * TP_WARPS * 32;
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        if (m0 + i * 16 >= h_hi) continue;
                        sts_u32(place + i * 16 * PH * 2, pack_bf16(acc[i][b][0], acc[i][b][1]));
                        sts_u32(place + (i * 16 + 8) * PH * 2, pack_bf16(acc[i][b][2], acc[i][b][3]));
                    }
                }
            }
        }
        if (ahead) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();  // mixed weights and values are there
        if (stages == 1 && t + 1 < ntiles) {  // (one stage of keys: the next ones come while the values are weighed)
            load_tile(k_stage(t + 1), t + 1, 0);
            cp_async_commit();
        }
#pragma unroll
        for (int i = 0; i < HPW; ++i) {
            const int h = h_lo + warp + i * TP_WARPS;
            if (h < h_hi) {
                const uint32_t v = vt_a + kv_of[h] + w.q_at;
                const uint32_t p = pt_a + (uint32_t)(h * PH + ((j8 >> 1) * 16 + (l7 ^ (h & 7)) + (j8 & 1) * 8) * 8) * 2u;
#pragma unroll
                for (int ks = 0; ks < NK / 2; ++ks) {
                    uint32_t a[4];
                    ldsm_x4(a, p + ks * 512);
#pragma unroll
                    for (int dp = 0; dp < DTILES / 2; ++dp) {
                        uint32_t b[4];
                        ldsm_x4_trans(b, step16(v, dp) + ks * 16 * ROW_BYTES);
                        mma_bf16(o[i][2 * dp], a, b[0], b[1]);
                        mma_bf16(o[i][2 * dp + 1], a, b[2], b[3]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < HPW; ++i) {
        const int h = h_lo + warp + i * TP_WARPS;
        if (h >= h_hi) continue;
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int tok = g4 + 8 * b;
            if (tok >= nt) continue;
            bf16* orow = out + ((size_t)(row0 + t0 + tok) * H + h) * D;
#pragma unroll
            for (int dt = 0; dt < DTILES; ++dt)
                *reinterpret_cast<__nv_bfloat162*>(orow + dt * 8 + tig * 2) = __floats2bfloat162_rn(o[i][dt][2 * b], o[i][dt][2 * b + 1]);
        }
    }
}

namespace {
// Keys of a tile and stages of keys that fit in shared memory: the largest tile first.
bool tp_geometry(int H, int G, int bt_cap, int* KT, int* stages, size_t* smem) {
    static const int choices[][2] = {{32, 2}, {32, 1}, {16, 2}, {16, 1}};
    for (auto& c : choices) {
        *smem = tp_smem(H, G, c[0], c[1], bt_cap);
        if (*smem <= 227 * 1024) {
            *KT = c[0];
            *stages = c[1];
            return true;
        }
    }
    return false;
}
int tp_table_slice(int chunk, int max_context, int page_size) {
    const int span = chunk > 0 ? (max_context < chunk + TP_TOK ? max_context : chunk + TP_TOK) : max_context;
    return span / page_size + 2;
}
}  // namespace

extern "C" int attn_talk_prefill_supports(int nq, int nkv, int chunk, int max_context, int page_size) {
    int KT, stages;
    size_t smem;
    return nkv > 0 && nq % nkv == 0 && tp_geometry(nq, nkv, tp_table_slice(chunk, max_context, page_size), &KT, &stages, &smem);
}

extern "C" int attn_talk_prefill(const void* q, int q_stride, const void* cache, const int* meta, int group, const int* cu_tokens,
                                 const int* ctx_lens, void* out, int S, int max_q_len, int nq, int nkv, int page_size, int num_pages,
                                 int chunk, float scale, const float* talk, int max_context, int* status, cudaStream_t stream) {
    if (S <= 0 || max_q_len <= 0) return 0;
    if (nkv <= 0 || nq % nkv || q_stride % 8 || ((uintptr_t)q & 15) || scale <= 0.f) return (int)cudaErrorInvalidValue;
    const int bt_cap = tp_table_slice(chunk, max_context, page_size);
    int KT = 0, stages = 0;
    size_t smem = 0;
    if (!tp_geometry(nq, nkv, bt_cap, &KT, &stages, &smem)) return (int)cudaErrorInvalidValue;
    const int hpw = tp_heads_per_warp(nq), parts = (nq + TP_WARPS * hpw - 1) / (TP_WARPS * hpw);
    const dim3 grid((max_q_len + TP_TOK - 1) / TP_TOK, parts, S);
    const CacheLayout L{nkv, page_size, D};
#define TALK_PREFILL_CASE(KT_, HPW_)                                                                                       \
    do {                                                                                                                  \
        static size_t configured = 0;                                                                                     \
        if (smem > 48 * 1024 && smem > configured) {                                                                      \
            cudaError_t err = cudaFuncSetAttribute(talk_prefill_kernel<KT_, HPW_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (err != cudaSuccess) return (int)err;                                                                      \
            configured = smem;                                                                                            \
        }                                                                                                                 \
        return (int)launch_kernel(talk_prefill_kernel<KT_, HPW_>, grid, TP_THREADS, smem, stream, (const bf16*)q, q_stride, (const bf16*)cache, \
                                  L, meta, group, cu_tokens, ctx_lens, (bf16*)out, nq, chunk, scale * LOG2E, talk, num_pages, bt_cap, stages, \
                                  status);                                                                                \
    } while (0)
#define TALK_PREFILL_TILE(HPW_)                    \
    do {                                           \
        if (KT == 32) TALK_PREFILL_CASE(32, HPW_); \
        TALK_PREFILL_CASE(16, HPW_);               \
    } while (0)
    if (hpw == 1) TALK_PREFILL_TILE(1);
    if constexpr (D <= 128) if (hpw == 2) TALK_PREFILL_TILE(2);
    return (int)cudaErrorInvalidValue;
#undef TALK_PREFILL_TILE
#undef TALK_PREFILL_CASE
}
