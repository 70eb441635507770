// Paged causal attention for prompt portions on the 5th-generation tensor cores where the values are the keys and many
// query heads share one cached row (attention over low-rank latents), for one row length: compile with
// -DTW_HEAD_DIM=<values of a cached row, a multiple of 16 up to 256>, -DTW_V_COLS=<leading values of a row that count as the
// value, a multiple of 16> and -DTW_KEY_TILE=96 or 64.
//
// A block serves 128 rows of one (request, key/value head), a row being a (token, query head of the group) pair, and walks
// the request's keys in tiles.  A tile is copied to shared memory once and read twice: K-major for S = Q K^T, and
// "MN-major" in the same layout for O += P V.  Tensor memory holds two S buffers (P is stored over S) and O, which fills
// it, so the block has one row tile; the second S buffer lets the tensor cores make S of the next tile while the softmax
// warps work on this one, and O += P V follows while they work on the next:
//
//     tensor cores    S(1)        O += P(0) V(0)   S(2)        O += P(1) V(1)   S(3) ...
//     softmax warps   ... P(0)           P(1)                         P(2)
//
// The rules are those of attention_tcgen05.cu: one warp issues the copies (one TMA box per page and 64 columns, no
// multicast), one thread issues every MMA, four warps own a row (a TMEM lane) per thread; O is rescaled only when a row's
// maximum grows by more than 2^8; rows of the last tile beyond the last key are zeroed in shared memory before P meets
// them; pages wholly before the first visible key are not read.
//
//   score = (q . k) * scale,  visible iff  tw_first_key(position, window) <= p <= position
//   `sink` (fp32 [Hq], or null): exp(sink[h]) joins the denominator; `gate` (fp32 [rows][Hq], or null) multiplies a head's output
//
// Every wait on an mbarrier is bounded; a wait that runs out sets TW_ERR_WAIT in the status word, every role stops, the
// block waits (bounded) for its copies in flight, frees its tensor memory and returns.
#include "tcgen05_softmax.cuh"

#ifndef TW_HEAD_DIM
#define TW_HEAD_DIM 256
#endif
#ifndef TW_V_COLS
#define TW_V_COLS TW_HEAD_DIM
#endif
#ifndef TW_KEY_TILE
#define TW_KEY_TILE 96
#endif

namespace {

using namespace tc5;

constexpr int D = TW_HEAD_DIM, DV = TW_V_COLS;
static_assert(D % 16 == 0 && D >= 16 && D <= 256 && DV % 16 == 0 && DV >= 16 && DV <= D, "row sizes");
constexpr int BM = 128;                       // rows of a block = TMEM lanes
constexpr int BN = TW_KEY_TILE;               // keys per tile
static_assert(BN == 96 || BN == 64, "key tiles");
constexpr int KB = (D + 63) / 64;             // 64-column blocks of a row (the copy fills what lies beyond the row with zeros)
constexpr int Q_BLK = BM * 128, BLK = BN * 128;
constexpr int Q_BYTES = KB * Q_BLK, STAGE_BYTES = KB * BLK;
constexpr int EXTRA = 1024 /* alignment slack */ + 256 /* barriers */;
constexpr int ROOM = (227 * 1024 - EXTRA - Q_BYTES) / STAGE_BYTES;
constexpr int STAGES = ROOM < 6 ? ROOM : 6;
static_assert(STAGES >= 3, "three tiles in flight");
constexpr int TILES = Q_BYTES + STAGES * STAGE_BYTES;
constexpr int SMEM = (TILES + EXTRA) > 120 * 1024 ? (TILES + EXTRA) : 120 * 1024;      // one block per SM: it takes all of the tensor memory
constexpr int THREADS = 192;                  // warp 0: TMA, warp 1: MMA, warps 2-5: softmax
constexpr int TMEM_COLS = 512, S_COLS = 128, O_COL = 256;
constexpr float RESCALE_THRESHOLD = 8.f;      // log2 units
#define NEG_INF (-INFINITY)

__global__ void __launch_bounds__(THREADS, 1)
attn_latent_tc5_kernel(const __grid_constant__ CUtensorMap map, bf16* __restrict__ out, int out_stride, const bf16* __restrict__ q,
                       int q_stride, const int* __restrict__ seq_q_start, const int* __restrict__ seq_q_len,
                       const int* __restrict__ seq_kv_len, const int* __restrict__ seq_slot, const int* __restrict__ block_table,
                       int table_stride, int Hq, int Hkv, int page_size, int num_pages, int window, float scale_log2e,
                       int skip_single, const float* __restrict__ sink, const float* __restrict__ gate, int* status) {
    extern __shared__ unsigned char smem_raw[];
    TW_TIMELINE_SCOPE(TW_K_ATTN_PREFILL);
    tw_grid_wait();
    TW_TIMELINE_MARK();
    // the longest blocks start first (see attention_tcgen05.cu)
    const int s = blockIdx.y, kvh = (int)blockIdx.x % Hkv, xt = (int)blockIdx.x / Hkv;
    const int q_len = seq_q_len[s];
    if (q_len <= 0 || (skip_single && q_len == 1)) return;
    const int G = Hq / Hkv;
    const int rows_total = q_len * G;
    const int mtiles = (rows_total + BM - 1) / BM;
    if (xt >= mtiles) return;
    const int row0 = (mtiles - 1 - xt) * BM;
    const int kv_len = seq_kv_len[s];
    const int pos0 = kv_len - q_len;                                 // position of the first token of this portion
    const int n0 = seq_q_start[s];
    const int* table = block_table + (size_t)seq_slot[s] * table_stride;
    const int row_end = min(rows_total, row0 + BM);
    const int pos_first = pos0 + row0 / G, pos_last = pos0 + (row_end - 1) / G;
    const int lo_block = tw_first_key(pos_first, window);            // no row of the block sees a key before this one
    const int j_begin = lo_block / BN;
    const int ntiles = pos_last / BN + 1 - j_begin;
    const int tail_rows = max(0, (j_begin + ntiles) * BN - kv_len);  // rows of the last tile that hold no key

    unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    unsigned char* q_s = tiles;                                      // [KB][128 rows][128 B]
    unsigned char* k_s = q_s + Q_BYTES;                              // [STAGES][KB][BN keys][128 B]
    uint64_t* full = reinterpret_cast<uint64_t*>(tiles + TILES);
    uint64_t* empty = full + STAGES;
    uint64_t* s_full = empty + STAGES;                               // S of a buffer is complete
    // (two barriers each, for even and odd tiles: a role may be a tile behind, never two, when it looks at one)
    uint64_t* p_full = s_full + 2;                                   // P of the tile is written, S read, O rescaled
    uint64_t* o_done = p_full + 2;                                   // P V of the tile, and of those before, have retired
    uint64_t* v_fixed = o_done + 2;                                  // rows past the last key are zeroed
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(v_fixed + 1);
    volatile int* aborted = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int i = 0; i < STAGES; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&s_full[b], 1); mbar_init(&p_full[b], BM / 32); mbar_init(&o_done[b], 1); }
        mbar_init(v_fixed, 1);
        *aborted = 0;
        mbar_fence_init();
    }
    // key tile i: one TMA box per page and 64 columns; lane b owns box b
    const int box_rows = min(page_size, BN), boxes = BN / box_rows;
    auto issue_tile = [&](int i) -> bool {
        const int st = i % STAGES;
        int row_coord = -1;
        if (lane < boxes) {
            const int key0 = (j_begin + i) * BN + lane * box_rows;
            if (key0 < kv_len && key0 + box_rows <= lo_block) {
                row_coord = num_pages * Hkv * page_size;             // beyond the cache: zeros
            } else if (key0 < kv_len) {
                const int blk = key0 / page_size;
                const int page = blk < table_stride ? table[blk] : -1;
                if (page < 0 || page >= num_pages) atomicOr(status, TW_ERR_PAGE);
                else row_coord = (page * Hkv + kvh) * page_size + (key0 - blk * page_size);
            }
        }
        const uint32_t box_bytes = (uint32_t)__popc(__ballot_sync(0xffffffffu, row_coord >= 0)) * box_rows * 128;
        int ok = 1;
        if (lane == 0) {
            ok = (!*aborted && mbar_wait(&empty[st], ((i / STAGES) & 1) ^ 1, status)) ? 1 : 0;
            if (ok) mbar_expect_tx(&full[st], box_bytes * KB); else *aborted = 1;
        }
        ok = __shfl_sync(0xffffffffu, ok, 0);
        if (!ok) return false;
        if (row_coord >= 0) {
#pragma unroll
            for (int kb = 0; kb < KB; ++kb)
                tma_load_2d(k_s + st * STAGE_BYTES + kb * BLK + lane * box_rows * 128, &map, &full[st], kb * 64, row_coord);
        }
        return true;
    };
    if (warp == 1) tmem_alloc(tmem_slot, TMEM_COLS);
    int issued = 0;
    if (warp == 0) {
        __syncwarp();
        while (issued < ntiles && issued < STAGES && issue_tile(issued)) ++issued;
    }
    // the block's query rows into the swizzled K-major layout (rows beyond the portion, and columns beyond D, are zero)
    {
        constexpr int CH = KB * 8, ITEMS = BM * CH, QT = THREADS - 32;
        constexpr int PER = (ITEMS + QT - 1) / QT, GROUP = PER < 14 ? PER : 14;
        for (int j0 = 0; warp != 0 && j0 < PER; j0 += GROUP) {
            uint4 vals[GROUP];
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                const int i = (int)threadIdx.x - 32 + (j0 + j) * QT;
                const int rr = i / CH, c = i - rr * CH, r = row0 + rr;
                vals[j] = make_uint4(0u, 0u, 0u, 0u);
                if (i < ITEMS && r < rows_total && c * 8 < D) {
                    const int t = r / G;
                    vals[j] = *reinterpret_cast<const uint4*>(q + (size_t)(n0 + t) * q_stride + (size_t)(kvh * G + (r - t * G)) * D + c * 8);
                }
            }
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                const int i = (int)threadIdx.x - 32 + (j0 + j) * QT;
                const int rr = i / CH, c = i - rr * CH;
                if (i < ITEMS) *reinterpret_cast<uint4*>(q_s + (c >> 3) * Q_BLK + rr * 128 + (((c & 7) ^ (rr & 7)) << 4)) = vals[j];
            }
        }
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        while (issued < ntiles && !*aborted && issue_tile(issued)) ++issued;
        if (tail_rows && issued == ntiles) {
            const int last = ntiles - 1, st = last % STAGES;
            if (mbar_wait(&full[st], (last / STAGES) & 1, status)) {
                // (S of this tile may be reading these rows at the same time: its columns for them are masked)
                unsigned char* vt = k_s + st * STAGE_BYTES;
                for (int idx = lane; idx < tail_rows * KB * 8; idx += 32) {
                    const int r = BN - tail_rows + idx / (KB * 8), rest = idx % (KB * 8);
                    *reinterpret_cast<uint4*>(vt + (rest >> 3) * BLK + r * 128 + ((rest & 7) << 4)) = make_uint4(0u, 0u, 0u, 0u);
                }
                fence_proxy_async();
                __syncwarp();
                if (lane == 0) mbar_arrive(v_fixed);
            } else {
                *aborted = 1;
            }
        }
        if (*aborted && lane == 0) {
            for (int i = max(0, issued - STAGES); i < issued; ++i) mbar_wait(&full[i % STAGES], (i / STAGES) & 1, status);
        }
    } else if (warp == 1) {
        if (lane == 0 && ntiles > 0) {
            const uint32_t idesc_s = instr_desc(BN), idesc_o = instr_desc(DV, true);
            const uint64_t q_desc = smem_desc(q_s, 0), k_desc = smem_desc(k_s, 0), v_desc = smem_desc_mn_major(k_s, BLK);
            auto issue_s = [&](int i) {
                const uint64_t kd = k_desc + (uint64_t)((i % STAGES) * (STAGE_BYTES >> 4));
                const uint32_t dst = tmem_base + (i & 1) * S_COLS;
#pragma unroll
                for (int k = 0; k < D / 16; ++k)
                    umma_bf16(dst, q_desc + (uint64_t)((k >> 2) * (Q_BLK >> 4) + (k & 3) * 2), kd + (uint64_t)((k >> 2) * (BLK >> 4) + (k & 3) * 2),
                              idesc_s, k > 0 ? 1u : 0u);
                umma_commit(&s_full[i & 1]);
            };
            auto issue_o = [&](int i) {
                const uint64_t vd = v_desc + (uint64_t)((i % STAGES) * (STAGE_BYTES >> 4));
                const uint32_t p = tmem_base + (i & 1) * S_COLS;
#pragma unroll
                for (int k = 0; k < BN / 16; ++k)
                    umma_bf16_ts(tmem_base + O_COL, p + k * 8, vd + (uint64_t)(k * (2048 >> 4)), idesc_o, (i > 0 || k > 0) ? 1u : 0u);
                umma_commit(&empty[i % STAGES]);                     // this tile has been read for the last time
                umma_commit(&o_done[i & 1]);
            };
            bool ok = mbar_wait(&full[0], 0, status);
            if (ok) {
                tc_fence_after();
                issue_s(0);
            }
            for (int i = 0; ok && i < ntiles; ++i) {
                if (i + 1 < ntiles) {
                    // the buffer of S(i + 1) held P(i - 1), whose product was issued before: MMAs of a block retire in order
                    ok = mbar_wait(&full[(i + 1) % STAGES], ((i + 1) / STAGES) & 1, status);
                    if (!ok) break;
                    tc_fence_after();
                    issue_s(i + 1);
                } else if (tail_rows) {
                    ok = mbar_wait(v_fixed, 0, status);
                    if (!ok) break;
                }
                ok = mbar_wait(&p_full[i & 1], (i >> 1) & 1, status);
                if (!ok) break;
                tc_fence_after();
                issue_o(i);
            }
            if (!ok) *aborted = 1;
        }
        __syncwarp();
    } else {
        // ---- softmax: thread = row rt = TMEM lane rt
        const int quarter = warp & 3;                        // the TMEM lanes this warp may touch
        const int rt = quarter * 32 + lane, r = row0 + rt;
        const bool valid = r < rows_total;
        const int t = valid ? r / G : (rows_total - 1) / G;
        const int head = kvh * G + (valid ? r - t * G : 0);
        const int pos = pos0 + t;
        const int lo = tw_first_key(pos, window);
        const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16), o_addr = lane_addr + O_COL;
        float m_used = NEG_INF, l = 0.f;
        bool ok = true;
        for (int i = 0; i < ntiles; ++i) {
            const int kbase = (j_begin + i) * BN;
            const uint32_t s_addr = lane_addr + (i & 1) * S_COLS;
            ok = !*aborted && mbar_wait(&s_full[i & 1], (i >> 1) & 1, status);
            if (!ok) break;
            tc_fence_after();
            uint32_t v[BN];
#pragma unroll
            for (int c = 0; c < BN; c += 32) tmem_ld32_nowait(s_addr + c, v + c);
            tmem_wait_ld();
            const bool all_visible = kbase + BN - 1 <= pos && kbase >= lo;
            if (!__all_sync(0xffffffffu, all_visible)) {
#pragma unroll
                for (int c = 0; c < BN; ++c) {
                    const int key = kbase + c;
                    if (key > pos || key < lo) v[c] = __float_as_uint(NEG_INF);
                }
            }
            float mx[4] = {NEG_INF, NEG_INF, NEG_INF, NEG_INF};
#pragma unroll
            for (int c = 0; c < BN; c += 8) {
#pragma unroll
                for (int k = 0; k < 4; ++k) mx[k] = max3(mx[k], __uint_as_float(v[c + 2 * k]), __uint_as_float(v[c + 2 * k + 1]));
            }
            const float mt = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * scale_log2e;   // scale > 0: the maximum commutes with it
            const bool rescale = mt > m_used + RESCALE_THRESHOLD;     // also the first finite maximum (m_used = -inf)
            float factor = 1.f;
            if (rescale) {
                factor = m_used == NEG_INF ? 0.f : ex2(m_used - mt);
                m_used = mt;
            }
            const float neg_mu = m_used == NEG_INF ? 0.f : -m_used;
            float2 acc[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
            for (int c = 0; c < BN; c += 8) {
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    float2 e = fma2(__uint_as_float(v[c + 2 * k]), __uint_as_float(v[c + 2 * k + 1]), scale_log2e, neg_mu);
                    e.x = ex2(e.x);
                    e.y = ex2(e.y);
                    acc[k] = add2(acc[k], e);
                    v[(c >> 1) + k] = pack_bf16(e.x, e.y);
                }
            }
            const float sum = ((acc[0].x + acc[0].y) + (acc[1].x + acc[1].y)) + ((acc[2].x + acc[2].y) + (acc[3].x + acc[3].y));
            l = l * factor + sum;
            if (i > 0 && __any_sync(0xffffffffu, rescale)) {
                ok = mbar_wait(&o_done[(i - 1) & 1], ((i - 1) >> 1) & 1, status);     // O is complete up to the tile before
                if (!ok) break;
                tc_fence_after();
#pragma unroll
                for (int c = 0; c < DV; c += 16) {
                    uint32_t o[16];
                    tmem_ld16(o_addr + c, o);
#pragma unroll
                    for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * factor);
                    tmem_st16_nowait(o_addr + c, o);
                }
                tmem_wait_st();
            }
            // P over the first half of S: the whole row of S is in registers by now
            tmem_st32_nowait(s_addr, v);
            if constexpr (BN == 96) tmem_st16_nowait(s_addr + 32, v + 32);
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[i & 1]);
        }
        if (ok && ntiles > 0) ok = mbar_wait(&o_done[(ntiles - 1) & 1], ((ntiles - 1) >> 1) & 1, status);
        if (!ok) {
            *aborted = 1;
        } else if (ntiles > 0) {
            tc_fence_after();
            // the sink counts with the same stale maximum as the sums (one far above it leaves an output of zero)
            if (sink) l += ex2(__ldg(sink + head) * 1.4426950408889634f - m_used);
            float inv = l > 0.f ? 1.f / l : 0.f;
            if (gate && valid) inv *= __ldg(gate + (size_t)(n0 + t) * Hq + head);
            bf16* orow = out + (size_t)(n0 + t) * out_stride + (size_t)head * D;
#pragma unroll
            for (int c = 0; c < DV; c += 16) {
                uint32_t o[16];
                tmem_ld16(o_addr + c, o);
                if (valid) {
#pragma unroll
                    for (int k = 0; k < 16; k += 8) {
                        uint4 w;
                        w.x = pack_bf16(__uint_as_float(o[k]) * inv, __uint_as_float(o[k + 1]) * inv);
                        w.y = pack_bf16(__uint_as_float(o[k + 2]) * inv, __uint_as_float(o[k + 3]) * inv);
                        w.z = pack_bf16(__uint_as_float(o[k + 4]) * inv, __uint_as_float(o[k + 5]) * inv);
                        w.w = pack_bf16(__uint_as_float(o[k + 6]) * inv, __uint_as_float(o[k + 7]) * inv);
                        *reinterpret_cast<uint4*>(orow + c + k) = w;
                    }
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, TMEM_COLS);
}

}  // namespace

// Attention for the requests of the batch that bring several tokens (with skip_single, requests with one token are left
// to the decode kernel).  q [tokens, Hq * D] and out [tokens, Hq * D] are bf16 with 16-byte aligned rows, of a head's D
// outputs the first DV are written; the cache is [pages, Hkv, page_size, D] bf16.
TW_EXPORT int tw_attn_latent_tc5(void* out, int out_stride, const void* q, int q_stride, const int* seq_q_start, const int* seq_q_len,
                                 const int* seq_kv_len, const int* seq_slot, const int* block_table, int table_stride,
                                 const void* k_cache, int n_seqs, int max_q_len, int Hq, int Hkv, int page_size, int num_pages,
                                 int window, float scale, int skip_single, const float* sink, const float* gate, int* status,
                                 cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return 0;
    if (Hkv <= 0 || Hq % Hkv || page_size < 4 || (BN % page_size && page_size % BN) || !(scale > 0.f)) return (int)cudaErrorInvalidValue;
    if ((reinterpret_cast<uintptr_t>(out) & 15) || (reinterpret_cast<uintptr_t>(q) & 15) || (out_stride & 7) || (q_stride & 7) ||
        (reinterpret_cast<uintptr_t>(k_cache) & 15))
        return (int)cudaErrorMisalignedAddress;
    static bool attr_set = false;
    if (!attr_set) {
        const cudaError_t e = cudaFuncSetAttribute(attn_latent_tc5_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) return (int)e;
        attr_set = true;
    }
    const int box_rows = page_size < BN ? page_size : BN;
    const long long rows = (long long)num_pages * Hkv * page_size;
    if (rows >= (1ll << 31) - 1) return (int)cudaErrorInvalidValue;
    CUtensorMap map;
    if (int e = get_map(k_cache, rows, D, box_rows, &map)) return e;
    const dim3 grid(((max_q_len * (Hq / Hkv) + BM - 1) / BM) * Hkv, n_seqs);
    return tw_launch(attn_latent_tc5_kernel, grid, dim3(THREADS), (size_t)SMEM, stream, 1, map, (bf16*)out, out_stride, (const bf16*)q,
                     q_stride, seq_q_start, seq_q_len, seq_kv_len, seq_slot, block_table, table_stride, Hq, Hkv, page_size, num_pages,
                     window, scale * 1.4426950408889634f, skip_single, sink, gate, status);
}
