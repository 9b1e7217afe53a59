// Prefill attention with softmax weights mixed across the query heads, on the 5th-generation tensor cores (-DHEAD_DIM=64 or
// 128).  The second of two kernels: the first (attn_prefill_tc_stats) has left every row's base-2 logarithm of its sum of
// exponentials, so a weight is finished the moment its score is there, and this kernel walks the keys once.
//
// One block = 8 tokens of one request, all heads; 128 keys at a time.  Everything runs TRANSPOSED: the keys are the rows
// (lanes of tensor memory), the (token, head) pairs the columns, because the mix runs over the heads at one (token, key):
//   * scores:  S^T[key, (token, head)] = K_c Q_c^T for every key/value head c, side by side in tensor memory;
//   * weights: a softmax thread owns a key; it reads its scores, takes 2^(s - lse), and writes a row of 32 head slots per token
//              to shared memory (bfloat16, two tokens to a 128-byte row);
//   * mix:     P'^T[key, head] = P^T T^T per token, a product of 128 x 32 x 32, back to tensor memory (over the scores);
//   * values:  the softmax threads write P' to shared memory as [key, (token, head)] rows, and O_c^T[dim, (token, head)] +=
//              V_c^T P'_c accumulates in tensor memory over all tiles (V is read M-major: no transpose anywhere).
// Two copy warps bring K and V tiles by TMA through one ring of stages, in the order in which two MMA warps read them: the
// next tile's keys before a tile's values, so that the softmax threads take exponentials while values are multiplied.  Head
// slots: a key/value head has HGP slots (a power of two >= its query heads), up to 32 slots in all; empty slots weigh nothing.
//
// All barrier waits are bounded; on a timeout the block raises a status word, every warp leaves its loop, and the block
// frees its tensor memory and returns.
#include "attention_tc.cuh"

int g_use_pdl = 0;
extern "C" void kernels_set_pdl(int mode) { g_use_pdl = mode; }

namespace {

constexpr int TOK = 8, BKV = 128, SLOTS = 32;
constexpr int SOFT_WARPS = 8, SOFT_THREADS = SOFT_WARPS * 32, MMA_WARP = 8, COPY_WARP = 10, THREADS = 384;
constexpr int WORKERS = 2;  // MMA warps and copy warps: number i has the ring's stages i, i + WORKERS, ...
constexpr uint32_t S_COL = 0, O_COL = 256, TMEM_COLS = 512;
constexpr int STAGE = HALVES * HALF_BYTES;     // a K or V tile of one key/value head
constexpr int NST = D == 64 ? 6 : 2;           // stages of the ring
static_assert(NST % WORKERS == 0, "a stage belongs to one copy warp and one MMA warp: their waits see its phases in order");
constexpr int Q_BYTES = TOK * SLOTS * D * 2, W_BYTES = 4 * HALF_BYTES, T_BYTES = SLOTS * 128;

// float32 accumulator, bfloat16 operands; *_mn: the operand's contiguous elements run along M or N
__host__ __device__ constexpr uint32_t idesc_of(int m, int n, bool a_mn, bool b_mn) {
    return make_idesc(m, n, b_mn) | ((a_mn ? 1u : 0u) << 15);
}

// N columns of this thread's lane without waiting for them (see tmem_wait)
template <int N> __device__ __forceinline__ void tmem_ld_issue(uint32_t taddr, uint32_t* r);
template <> __device__ __forceinline__ void tmem_ld_issue<4>(uint32_t taddr, uint32_t* r) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(taddr));
}
template <> __device__ __forceinline__ void tmem_ld_issue<8>(uint32_t taddr, uint32_t* r) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]) : "r"(taddr));
}
template <> __device__ __forceinline__ void tmem_ld_issue<16>(uint32_t taddr, uint32_t* r) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
                   "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]) : "r"(taddr));
}
// Waits for the loads issued before, and ties the registers to that wait (volatile statements keep their order).
template <int N> __device__ __forceinline__ void tmem_wait(uint32_t (&r)[N]) {
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < N; ++i) asm volatile("" : "+r"(r[i]));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

}  // namespace

template <int HGP>
__global__ void __launch_bounds__(THREADS, 1)
talk_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_kv, const bf16* __restrict__ q, int q_stride, CacheLayout L,
                       const int* __restrict__ meta, int group, const int* __restrict__ cu_tokens, const int* __restrict__ ctx_lens,
                       const float* __restrict__ lse, bf16* __restrict__ out, int H, int chunk, float scale_log2,
                       const float* __restrict__ talk, int num_pages, int bt_cap, int* __restrict__ status) {
    constexpr int GMAX = SLOTS / HGP, NS = TOK * HGP;  // key/value heads at most; columns of one
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* q_s = smem;               // [GMAX][HALVES][NS rows of 128 bytes]
    unsigned char* w_s = q_s + Q_BYTES;      // weights: [4][128 rows of 128 bytes], before the mix and after it
    unsigned char* t_s = w_s + W_BYTES;      // talk: [32 rows of 128 bytes], the first 32 elements
    unsigned char* ring = t_s + T_BYTES;     // [NST][STAGE]
    uint64_t* bars = reinterpret_cast<uint64_t*>(ring + NST * STAGE);
    uint64_t *full = bars, *empty = bars + NST, *s_done = bars + 2 * NST, *p_ready = s_done + 1, *mix_done = s_done + 2, *b_ready = s_done + 3,
             *pv_done = s_done + 4;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * NST + 6);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* lse_s = reinterpret_cast<float*>(tmem_slot + 4);  // [TOK][SLOTS]
    int* bt_s = reinterpret_cast<int*>(lse_s + TOK * SLOTS);

    const int qt = gridDim.x - 1 - blockIdx.x, e = blockIdx.z;  // late tiles see the most keys: they go first
    if (e >= meta[META_NUM_ENTRIES]) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int G = L.num_kv_heads, HG = H / G, ps = L.page_size;
    const int row0 = cu_tokens[e], q_len = cu_tokens[e + 1] - row0, t0 = qt * TOK;
    if (t0 >= q_len) return;  // before anything is allocated
    const int nt = min(TOK, q_len - t0), p_first = ctx_lens[e] + t0, p_last = p_first + nt - 1;
    const int* bt = meta + meta[META_BT_OFFSET + group] + (size_t)e * meta[META_BT_STRIDE + group];
    const int kbeg = chunk > 0 ? p_first - p_first % chunk : 0, kend = p_last + 1;
    const int k_first = (kbeg / BKV) * BKV, ntiles = (kend - k_first + BKV - 1) / BKV, page_lo = k_first / ps;
    int page_cnt = (kend - 1) / ps - page_lo + 1;
    if (page_cnt > bt_cap) {
        if (tid == 0) atomicExch(&status[STATUS_BAD_PAGE], 1 + kend);
        page_cnt = bt_cap;
    }
    for (int i = tid; i < page_cnt; i += THREADS) {
        int page = bt[page_lo + i];
        if (page >= num_pages || (page <= 0 && (page_lo + i + 1) * ps > kbeg)) {  // (pages before the chunk may have been given back)
            atomicExch(&status[STATUS_BAD_PAGE], 1 + (page_lo + i));
            page = -1;
        }
        bt_s[i] = page;
    }
    if (tid == 0) {
        for (int i = 0; i < 2 * NST; ++i) mbar_init(&bars[i], 1);
        mbar_init(s_done, WORKERS);
        mbar_init(mix_done, 1);
        mbar_init(pv_done, WORKERS);
        mbar_init(p_ready, SOFT_WARPS);
        mbar_init(b_ready, SOFT_WARPS);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == MMA_WARP) {
        tmem_alloc(tmem_slot, TMEM_COLS);
        tmem_relinquish();
    }
    // queries: row (token * HGP + head of the group) of key/value head c; empty slots and tokens are zeros
#pragma unroll 4
    for (int idx = tid; idx < GMAX * NS * (D / 8); idx += THREADS) {
        const int ch = idx % (D / 8), n = (idx / (D / 8)) % NS, c = idx / (D / 8) / NS, tok = n / HGP, hh = n % HGP;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (tok < nt && hh < HG && c < G)
            v = *reinterpret_cast<const uint4*>(q + (size_t)(row0 + t0 + tok) * q_stride + (size_t)(c * HG + hh) * D + ch * 8);
        *reinterpret_cast<uint4*>(q_s + (size_t)(c * HALVES + ch / 8) * NS * 128 + swz(n, ch % 8)) = v;
    }
    for (int idx = tid; idx < SLOTS * 8; idx += THREADS) {  // row h' of talk over slots g'; 8 elements a piece, 64 a row
        const int h = idx / 8, ch = idx % 8, hc = h / HGP, hh = h % HGP;
        uint32_t v[4] = {0u, 0u, 0u, 0u};
        if (ch < SLOTS / 8 && hc < G && hh < HG) {
            float f[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                const int g = ch * 8 + k, gc = g / HGP, gh = g % HGP;
                f[k] = gc < G && gh < HG ? talk[(size_t)(hc * HG + hh) * H + gc * HG + gh] : 0.f;
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = pack2(f[2 * k], f[2 * k + 1]);
        }
        *reinterpret_cast<uint4*>(t_s + swz(h, ch)) = make_uint4(v[0], v[1], v[2], v[3]);
    }
    for (int idx = tid; idx < TOK * SLOTS; idx += THREADS) {  // (an infinite logarithm: the weight is zero)
        const int tok = idx / SLOTS, g = idx % SLOTS, gc = g / HGP, gh = g % HGP;
        lse_s[idx] = tok < nt && gc < G && gh < HG ? lse[(size_t)(row0 + t0 + tok) * H + gc * HG + gh] : INFINITY;
    }
    fence_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp >= COPY_WARP) {
        // the ring's tiles in the order the MMA warps read them: K of tile 0 for every key/value head, K of tile 1, V of tile 0, K of
        // tile 2 ...  (A thread starts a copy in a hundred cycles or so, short ones where pages are small: two warps take turns.)
        const int cw = warp - COPY_WARP, pages = BKV / ps;
        bool ok = true;
        int n = 0, st = 0;
        uint32_t round = 0;  // how often the ring has gone round
        for (int i = 0; i < 2 * ntiles && ok; ++i) {
            const bool values = i == 2 * ntiles - 1 || (i > 0 && i % 2 == 0);
            const int t = i == 0 ? 0 : values ? (i - 1) / 2 : (i + 1) / 2;
            // one box of `ps` rows per page and 64-column half
            const int first = (k_first + t * BKV) / ps - page_lo, count = min(pages, page_cnt - first);
            const uint32_t bytes = __popc(__ballot_sync(0xffffffffu, lane < count && bt_s[first + lane] > 0)) * (uint32_t)ps * 128u * HALVES;
            for (int r = values ? G : 0, last = r + G; r < last; ++r) {  // (a page holds the K rows of every head, then the V rows)
                if (st % WORKERS == cw) {
                    if (round > 0 && !__all_sync(0xffffffffu, mbar_wait(&empty[st], (round - 1) & 1u, status, abort_flag))) { ok = false; break; }
                    if (elect_one()) {
                        mbar_expect_tx(&full[st], bytes);
                        unsigned char* dst = ring + st * STAGE;
                        for (int k = 0; k < count; ++k, dst += ps * 128) {
                            const int page = bt_s[first + k];
                            if (page <= 0) continue;
#pragma unroll
                            for (int h = 0; h < HALVES; ++h) tma_load_2d(dst + h * HALF_BYTES, &map_kv, h * 64, (page * 2 * G + r) * ps, &full[st]);
                        }
                    }
                    __syncwarp();
                }
                ++n;
                if (++st == NST) st = 0, ++round;
            }
        }
        if (*abort_flag && lane == 0)  // somebody gave up on a barrier: copies in flight land (bounded) before the block leaves
            for (int s = n > NST ? n - NST : 0; s < n; ++s)
                for (uint32_t i = 0; s % NST % WORKERS == cw && i < WAIT_LIMIT && !mbar_try_wait(&full[s % NST], (uint32_t)(s / NST) & 1u); ++i) {}
    } else if (warp >= MMA_WARP) {
        // (an MMA of these sizes runs for less time than its start takes: two warps)
        const int mw = warp - MMA_WARP;
        constexpr uint32_t idesc_s = idesc_of(BKV, NS, false, false), idesc_m = idesc_of(BKV, SLOTS, false, false),
                           idesc_o = idesc_of(D, NS, true, true);
        bool ok = true;
        int st = 0;
        uint32_t round = 0;
        // descriptors of the buffers' starts: another place in a buffer is a sum in the address field (units of 16 bytes)
        const uint64_t ring_k = make_desc(smem_u32(ring), 0), ring_v = make_desc(smem_u32(ring), HALF_BYTES), q_desc = make_desc(smem_u32(q_s), 0),
                       w_desc = make_desc(smem_u32(w_s), 0), w_desc_mn = make_desc(smem_u32(w_s), HALF_BYTES), t_desc = make_desc(smem_u32(t_s), 0);
        auto next = [&]() { if (++st == NST) st = 0, ++round; };
        auto wait_all = [&](uint64_t* bar, uint32_t parity) {
            ok = __all_sync(0xffffffffu, mbar_wait(bar, parity, status, abort_flag));
            tc_fence_after();
            return ok;
        };
        auto scores = [&]() {  // of the next tile
            for (int c = 0; c < G; ++c, next()) {
                if (st % WORKERS != mw) continue;
                if (!wait_all(&full[st], round & 1u)) return;
                if (elect_one()) {
                    const uint64_t a = ring_k + (uint32_t)(st * (STAGE / 16)), b = q_desc + (uint32_t)(c * (HALVES * NS * 128 / 16));
#pragma unroll
                    for (int kd = 0; kd < D / 16; ++kd)
                        umma_bf16(tmem_base + S_COL + c * NS, a + ((kd / 4) * HALF_BYTES + (kd % 4) * 32) / 16,
                                  b + ((kd / 4) * NS * 128 + (kd % 4) * 32) / 16, idesc_s, kd > 0);
                    umma_commit(&empty[st]);
                }
            }
            if (elect_one()) umma_commit(s_done);
        };
        scores();
        for (int t = 0; t < ntiles && ok; ++t) {
            const uint32_t par = (uint32_t)t & 1u;
            const int k0 = k_first + t * BKV;
            if (mw == 0) {
                if (!wait_all(p_ready, par)) break;
                if (elect_one()) {
#pragma unroll
                    for (int tok = 0; tok < TOK; ++tok)
#pragma unroll
                        for (int ks = 0; ks < SLOTS / 16; ++ks)
                            umma_bf16(tmem_base + S_COL + tok * SLOTS, w_desc + ((tok >> 1) * HALF_BYTES + (tok & 1) * 64 + ks * 32) / 16,
                                      t_desc + ks * 2, idesc_m, ks > 0);
                    umma_commit(mix_done);
                }
            }
            if (!wait_all(b_ready, par)) break;
            // the next tile's scores come first: the softmax warps work on them while the values are multiplied
            if (t + 1 < ntiles) scores();
            if (!ok) break;
            const bool edge = k0 < kbeg || k0 + BKV > kend;  // keys that nobody sees: their value rows must be zeros (0 * NaN)
            for (int c = 0; c < G; ++c, next()) {
                if (st % WORKERS != mw) continue;
                if (!wait_all(&full[st], round & 1u)) break;
                if (edge) {
                    for (int r = lane; r < BKV; r += 32) {
                        const int key = k0 + r;
                        if (key < kbeg || key >= kend) {
#pragma unroll
                            for (int ch = 0; ch < D / 8; ++ch)
                                *reinterpret_cast<uint4*>(ring + st * STAGE + (ch / 8) * HALF_BYTES + swz(r, ch % 8)) = make_uint4(0u, 0u, 0u, 0u);
                        }
                    }
                    fence_async_smem();
                    __syncwarp();
                }
                if (elect_one()) {
                    const uint32_t at = (uint32_t)c * NS * 2;
                    const uint64_t a = ring_v + (uint32_t)(st * (STAGE / 16)), b = w_desc_mn + (at / 128 * HALF_BYTES + at % 128) / 16;
#pragma unroll
                    for (int ks = 0; ks < BKV / 16; ++ks)
                        umma_bf16(tmem_base + O_COL + c * NS, a + ks * 128, b + ks * 128, idesc_o, ks > 0 ? 1u : (t > 0));
                    umma_commit(&empty[st]);
                }
            }
            if (!ok) break;
            if (elect_one()) umma_commit(pv_done);
        }
    } else {
        const int quarter = warp & 3, th = warp >> 2, j = quarter * 32 + lane;  // a warp reaches the lanes of its quarter
        const uint32_t tmem_row = tmem_base + ((uint32_t)(quarter * 32) << 16);
        bool ok = true;
        for (int t = 0; t < ntiles && ok; ++t) {
            const uint32_t par = (uint32_t)t & 1u;
            const int key = k_first + t * BKV + j;
            ok = __all_sync(0xffffffffu, mbar_wait(s_done, par, status, abort_flag));
            if (!ok) break;
            tc_fence_after();
            uint32_t pk[4][SLOTS / 2];  // the weights of my key and four tokens, two a register
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                uint32_t r[64];
#pragma unroll
                for (int c = 0; c < GMAX; ++c) tmem_ld_issue<2 * HGP>(tmem_row + S_COL + c * NS + (4 * th + 2 * u) * HGP, r + c * 2 * HGP);
                tmem_wait(r);
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const int tok = 4 * th + 2 * u + k, p = p_first + tok;
                    const bool vis = tok < nt && key <= p && key >= (chunk > 0 ? p - p % chunk : 0);
                    const float* ls = lse_s + tok * SLOTS;
#pragma unroll
                    for (int ch = 0; ch < SLOTS / 8; ++ch) {
                        const float4 l0 = *reinterpret_cast<const float4*>(ls + ch * 8), l1 = *reinterpret_cast<const float4*>(ls + ch * 8 + 4);
                        const float l8[8] = {l0.x, l0.y, l0.z, l0.w, l1.x, l1.y, l1.z, l1.w};
                        float w8[8];
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const int g = ch * 8 + i, c = g / HGP;
                            const float x = fast_exp2(fmaf(__uint_as_float(r[c * 2 * HGP + k * HGP + g % HGP]), scale_log2, -l8[i]));
                            w8[i] = vis && c < G ? x : 0.f;  // (columns of absent heads hold anything)
                        }
#pragma unroll
                        for (int i = 0; i < 4; ++i) pk[2 * u + k][ch * 4 + i] = pack2(w8[2 * i], w8[2 * i + 1]);
                    }
                }
            }
            // (the values' product of the tile before reads the weights' space)
            if (t > 0) ok = __all_sync(0xffffffffu, mbar_wait(pv_done, par ^ 1u, status, abort_flag));
            if (!ok) break;
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
                for (int ch = 0; ch < SLOTS / 8; ++ch)
                    *reinterpret_cast<uint4*>(w_s + (2 * th + k / 2) * HALF_BYTES + swz(j, (k & 1) * 4 + ch)) =
                        make_uint4(pk[k][ch * 4], pk[k][ch * 4 + 1], pk[k][ch * 4 + 2], pk[k][ch * 4 + 3]);
            fence_async_smem();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_ready);
            ok = __all_sync(0xffffffffu, mbar_wait(mix_done, par, status, abort_flag));
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                uint32_t r[64];
#pragma unroll
                for (int i = 0; i < 4; ++i) tmem_ld_issue<16>(tmem_row + S_COL + (4 * th + 2 * u) * SLOTS + i * 16, r + i * 16);
                tmem_wait(r);
#pragma unroll
                for (int k = 0; k < 2; ++k)
#pragma unroll
                    for (int i = 0; i < SLOTS / 2; ++i)
                        pk[2 * u + k][i] = pack2(__uint_as_float(r[k * SLOTS + 2 * i]), __uint_as_float(r[k * SLOTS + 2 * i + 1]));
            }
#pragma unroll
            for (int c = 0; c < GMAX; ++c) {
                if (c >= G) continue;
                const uint32_t b = (uint32_t)c * NS * 2 + (uint32_t)(4 * th * HGP) * 2;
#pragma unroll
                for (int ch = 0; ch < HGP / 2; ++ch) {
                    uint32_t v[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int el = 2 * (4 * ch + i);
                        v[i] = pk[el / HGP][c * (HGP / 2) + el % HGP / 2];
                    }
                    *reinterpret_cast<uint4*>(w_s + b / 128 * HALF_BYTES + swz(j, (int)(b % 128) / 16 + ch)) = make_uint4(v[0], v[1], v[2], v[3]);
                }
            }
            fence_async_smem();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_ready);
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(pv_done, (uint32_t)(ntiles - 1) & 1u, status, abort_flag));
        if (ok) {
            tc_fence_after();
            bf16* out_s = reinterpret_cast<bf16*>(w_s);  // the tokens' rows as they lie in `out`, where the weights were
            // rows of O are dimensions: 64 of them lie in the first 16 lanes of every quarter, 128 in all lanes
            const int dim = D == 64 ? quarter * 16 + lane : quarter * 32 + lane;
            const bool mine = D == 128 || lane < 16;
            for (int c = th * (GMAX / 2); c < (th + 1) * (GMAX / 2) && c < G; ++c) {
#pragma unroll
                for (int n0 = 0; n0 < NS; n0 += 16) {
                    uint32_t r[16];
                    tmem_ld_issue<16>(tmem_row + O_COL + c * NS + n0, r);
                    tmem_wait(r);
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const int tok = (n0 + i) / HGP, hh = (n0 + i) % HGP;
                        if (mine && tok < nt && hh < HG) out_s[(tok * H + c * HG + hh) * D + dim] = __float2bfloat16_rn(__uint_as_float(r[i]));
                    }
                }
            }
        }
        asm volatile("bar.sync 1, %0;" ::"n"(SOFT_THREADS) : "memory");  // (every softmax warp comes here, whether it gave up or not)
        if (ok) {
            uint4* dst = reinterpret_cast<uint4*>(out + (size_t)(row0 + t0) * H * D);
            for (int i = tid; i < nt * H * D / 8; i += SOFT_THREADS) dst[i] = reinterpret_cast<const uint4*>(w_s)[i];
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == MMA_WARP) tmem_dealloc(tmem_base, TMEM_COLS);
}

// ----------------------------------------------------------------------------- host side
namespace {
size_t talk_tc_smem(int bt_cap) {
    return 1024 + Q_BYTES + W_BYTES + T_BYTES + (size_t)NST * STAGE + (2 * NST + 6) * 8 + 16 + TOK * SLOTS * 4 + (size_t)bt_cap * 4;
}
int talk_tc_table(int chunk, int max_context, int page_size) {
    const int span = chunk > 0 && chunk + TOK + 2 * BKV < max_context ? chunk + TOK + 2 * BKV : max_context;
    return span / page_size + 2 + BKV / page_size;
}
int head_slots(int nq, int nkv) {  // a power of two, 2 at least
    int n = 2;
    while (n < nq / nkv) n *= 2;
    return n;
}
}  // namespace

extern "C" int attn_talk_tc_head_dim() { return D; }

// Up to 32 head slots (groups of up to 8 query heads); page sizes as the statistics kernel takes them.
extern "C" int attn_talk_prefill_tc_supports(int nq, int nkv, int chunk, int max_context, int page_size) {
    if (nkv <= 0 || nq % nkv || page_size < 8 || page_size > 128 || (page_size & (page_size - 1))) return 0;
    const int hgp = head_slots(nq, nkv);
    return hgp <= 8 && hgp * nkv <= SLOTS && talk_tc_smem(talk_tc_table(chunk, max_context, page_size)) <= 227 * 1024;
}

// lse: what attn_prefill_tc_stats has left, float32 [rows, nq].
extern "C" int attn_talk_prefill_tc(const void* q, int q_stride, const void* cache, const int* meta, int group, const int* cu_tokens,
                                    const int* ctx_lens, const float* lse, void* out, int S, int max_q_len, int nq, int nkv, int page_size,
                                    int num_pages, int chunk, float scale, const float* talk, int max_context, int* status,
                                    cudaStream_t stream) {
    if (S <= 0 || max_q_len <= 0) return 0;
    if (!attn_talk_prefill_tc_supports(nq, nkv, chunk, max_context, page_size) || q_stride % 8 || (((uintptr_t)q | (uintptr_t)out) & 15) || scale <= 0.f)
        return (int)cudaErrorInvalidValue;
    CUtensorMap map;
    if (!cache_map(&map, cache, num_pages, nkv, page_size)) return (int)cudaErrorNotSupported;
    const CacheLayout L{nkv, page_size, D};
    const int bt_cap = talk_tc_table(chunk, max_context, page_size), hgp = head_slots(nq, nkv);
    const size_t smem = talk_tc_smem(bt_cap);
    const dim3 grid((max_q_len + TOK - 1) / TOK, 1, S);
#define TALK_TC_CASE(HGP_)                                                                                                 \
    if (hgp == HGP_) {                                                                                                    \
        static size_t configured = 0;                                                                                     \
        if (smem > configured) {                                                                                          \
            cudaError_t err = cudaFuncSetAttribute(talk_prefill_tc_kernel<HGP_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (err != cudaSuccess) return (int)err;                                                                      \
            configured = smem;                                                                                            \
        }                                                                                                                 \
        talk_prefill_tc_kernel<HGP_><<<grid, THREADS, smem, stream>>>(map, (const bf16*)q, q_stride, L, meta, group, cu_tokens, ctx_lens, lse, \
                                                                      (bf16*)out, nq, chunk, scale * LOG2E, talk, num_pages, bt_cap, status); \
        LAUNCH_RETURN();                                                                                                  \
    }
    TALK_TC_CASE(2)
    TALK_TC_CASE(4)
    TALK_TC_CASE(8)
    return (int)cudaErrorInvalidValue;
#undef TALK_TC_CASE
}
