// Differential prefill attention on the 5th-generation tensor cores: every head has two attention maps over the same
// values, the second is taken off the first, the difference is normalised and gated.  Causal, optionally within blocks
// of positions, grouped query heads, sequences of unequal length packed back to back, keys and values read from the
// paged bfloat16 cache whose key rows hold the keys of both maps side by side.
//
// An item is 128 consecutive new tokens of one sequence and one query head; for each the block walks the keys the item
// may see in blocks of 128 (two pages of 64), for both maps m = 0, 1:
//
//   S_m  = Q_m K_m^T    tcgen05.mma, M = 128 queries, N = 128 keys, K = one map's key channels (padded with zeros)
//   P_m  = exp2(capped scaled S_m - reference)   in 32-bit, by the threads that own the row (TMEM lane = row);
//          rounded to bfloat16 and written back over S_m, where the next product reads it as its A operand
//   O_m += P_m V        tcgen05.mma, N = value channels; both maps use the block's values from one stage
//
// and ends with  o = O_0 / l_0 - lambda O_1 / l_1  (l: a row's sum of weights),  o / sqrt(mean(o^2) + eps) * out_scale *
// sigmoid(gate), all in 32-bit, on its way out.  Two groups of row threads take a map each, so the two maps are what
// keeps the tensor core busy while the other's scores are turned into weights.
//
// Soft cap: a scaled score s becomes cap tanh(s / cap).  For |s / cap| <= 5/8 it is an odd polynomial (interpolated at
// Chebyshev points; relative error 1.2e-7), evaluated for two scores at a time on the multiply-add units, with the scale
// and the cap in its coefficients; a warp that holds a larger one in a run of 32 keys takes tanh(x) = 1 - 2 / (1 + e^(2x))
// for that run.
//
// FIXED: with a cap of at most 60 no score leaves +-60 log2(e) < 87 in powers of two, so the weights are taken as they
// are (reference 0): float and bfloat16 have the range, and there is no maximum to find and nothing to rescale.  Else
// the reference is the row's running maximum, allowed to lag by 2^8 as in attn_prefill_tc05.cu.
//
// Warp 0 loads queries and keys, the last warp the values (TMA; a ring per kind), warp 1 issues the products, the others
// are the row threads, ROWT of them to a row and map.  A thread's weights lie in the first half of its own columns of
// S, so it may write those of one run of keys before it has read the next.  Every wait is bounded.
//
// Sizes: a map's keys up to 128 channels, values up to 256, both multiples of 8; pages of 64 positions.  Values of more
// than 128 channels take two items a head, half the channels each; the maps' outputs then go to a float buffer
// [tokens, heads, 2, value channels] for diff_combine_kernel (elementwise.cu).
#include "tc05.cuh"
#include <cstring>

namespace {
using namespace tc05;
constexpr int BM = 128, BN = 128, PAGE = 64, MAPS = 2, ROWT = 2;
constexpr int ATOM_BYTES = 128 * 128;           // 128 rows of 128 bytes: one 64-wide slice of a 128-row operand
constexpr int POLY = 5;
// tanh(x) / x as a polynomial in x^2 on |x| <= 5/8
constexpr double TANH_POLY[POLY] = {0.99999988079, -0.33331942558, 0.13304379582, -0.051815912127, 0.015043356456};
constexpr float TANH_POLY_MAX = 0.625f;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float FIXED_CAP_MAX = 60.f;

struct DiffAttnParams {
    bf16* out;                // [tokens, nh, vd]
    float* maps_out;          // [tokens, nh, 2, vd]: used in place of ``out`` when the values take several items
    const int* tile_seq;
    const int* tile_first;
    const int* seq_start;
    const int* seq_past;
    const int* block_table;
    const float* gate;        // [tokens, ldg] or null
    long long ldg;
    int table_stride, n_pages, nh, nkv, vd, v_parts, chunk, kv_rows, n_tiles, smem_bytes;
    int* status;
    float to_unit;            // scores to the argument of tanh (scale / cap); without a cap to powers of two (scale log2 e)
    float cap2;               // cap log2(e), or 0: no cap
    float lambda, eps, out_scale;
    float raw_max;            // raw scores up to here take the polynomial
    unsigned long long poly[POLY];   // TANH_POLY[k] cap2 to_unit^(2k + 1), each twice: a polynomial in the raw score's square
};

__device__ __forceinline__ unsigned idesc_attn(int n, bool b_mn_major) {
    return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn_major ? (1u << 16) : 0u) | ((unsigned)(n >> 3) << 17) |
           ((unsigned)(128 >> 4) << 24);
}
// descriptor of an MN-major operand: rows are 16 consecutive k (keys), 128 bytes of n (head columns) each;
// the next 64 columns lie ``lbo`` bytes further, the next 8 keys 1024 bytes further
__device__ __forceinline__ unsigned long long smem_desc_mn(const void* p, unsigned lbo) {
    unsigned long long d = 0;
    d |= (unsigned long long)((smem_u32(p) & 0x3FFFFu) >> 4);
    d |= (unsigned long long)((lbo >> 4) & 0x3FFFu) << 16;
    d |= (unsigned long long)(1024 >> 4) << 32;
    d |= (unsigned long long)1 << 46;
    d |= (unsigned long long)2 << 61;
    return d;
}
// 2^x by the special function unit (ex2.approx: relative error about 2^-22; -inf gives 0)
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// two floats in one 64-bit register: one instruction does the arithmetic of both
__device__ __forceinline__ unsigned long long pack2(float a, float b) {
    unsigned long long d;
    asm("mov.b64 %0, {%1, %2};\n" : "=l"(d) : "f"(a), "f"(b));
    return d;
}
__device__ __forceinline__ void unpack2(unsigned long long d, float& a, float& b) {
    asm("mov.b64 {%0, %1}, %2;\n" : "=f"(a), "=f"(b) : "l"(d));
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
    unsigned long long d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ unsigned long long add2(unsigned long long a, unsigned long long b) {
    unsigned long long d;
    asm("add.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
// the largest magnitude of three
__device__ __forceinline__ float max_abs3(float a, float b, float c) {
    float d;
    asm("max.abs.f32 %0, %1, %2, %3;\n" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}
// the ``count`` threads that meet at named barrier ``id`` learn whether all of them are well
__device__ __forceinline__ bool pair_agree(bool ok, int id, int count) {
    unsigned all;
    asm volatile(
        "{\n.reg .pred p, q;\n"
        "setp.ne.u32 p, %1, 0;\n"
        "bar.red.and.pred q, %2, %3, p;\n"
        "selp.u32 %0, 1, 0, q;\n}\n"
        : "=r"(all) : "r"(ok ? 1u : 0u), "r"(id), "r"(count) : "memory");
    return all != 0;
}
__device__ __forceinline__ void named_sync(int id, int count) {
    asm volatile("bar.sync %0, %1;\n" ::"r"(id), "r"(count) : "memory");
}

// the tile of 128 query rows, the head and the part of the value channels that a block works on
struct Item {
    int seq, h, kvh, part, row0, rows, pos0, pos_last, blk_lo, nb, page_lo;
};
__device__ __forceinline__ Item load_item(const DiffAttnParams& p, int item) {
    Item it;
    const int per_tile = p.nh * p.v_parts;
    const int tile = item / per_tile, rest = item - tile * per_tile;
    it.h = rest / p.v_parts;
    it.part = rest - it.h * p.v_parts;
    it.kvh = it.h / (p.nh / p.nkv);
    it.seq = p.tile_seq[tile];
    const int first = p.tile_first[tile];
    it.row0 = p.seq_start[it.seq] + first;                               // the tile's first row among the packed tokens
    it.rows = min(BM, p.seq_start[it.seq + 1] - p.seq_start[it.seq] - first);
    it.pos0 = p.seq_past[it.seq] + first;
    it.pos_last = it.pos0 + it.rows - 1;
    const int key_lo = first_visible_key(it.pos0, 0, p.chunk);
    it.blk_lo = key_lo / BN;
    it.page_lo = key_lo / PAGE;                                          // the first page that holds a key any row sees
    it.nb = it.pos_last / BN - it.blk_lo + 1;
    return it;
}

template <int KD, int VD> struct Layout {
    static constexpr int K_TILE = KD / 64 * ATOM_BYTES;                  // 128 keys of one map
    static constexpr int V_TILE = VD / 64 * ATOM_BYTES;
    static constexpr int Q_BYTES = MAPS * K_TILE;
    static constexpr int K_STAGES = KD == 64 ? 6 : 3;                    // tiles of one map's keys: 96 KB
    static constexpr int V_STAGES = VD == 64 ? 4 : KD == 64 ? 3 : 2;
    static constexpr int TILES = Q_BYTES + K_STAGES * K_TILE + V_STAGES * V_TILE;
    static constexpr int TAIL = 256 + MAPS * ROWT * 128 * 4;             // barriers and two words; the row threads' exchange
    static constexpr int N_BARS = 8 + 2 * K_STAGES + 2 * V_STAGES;
};

// Persistent: the (tile, head) items are listed with the most keys first; block b takes the items
// b, 2G-1-b, 2G+b, 4G-1-b, ... (G blocks).  Every role derives the same run of items, and the counters of key blocks
// that choose the stage and the phase of each mbarrier run on from one item to the next.
template <int KD, int VD, bool FIXED>
__global__ void __launch_bounds__(96 + MAPS * ROWT * 128, 1)
attn_diff_tc05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_v, const __grid_constant__ DiffAttnParams p) {
    using L = Layout<KD, VD>;
    constexpr int HK = KD / 64, HV = VD / 64;             // 64-column slices of a map's key and of a value
    constexpr int KST = L::K_STAGES, VST = L::V_STAGES;
    const int n_items = p.n_tiles * p.nh * p.v_parts, G = gridDim.x;
    auto item_of = [&](int round) { return round * G + ((round & 1) ? G - 1 - (int)blockIdx.x : (int)blockIdx.x); };

    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* q_s = smem;                            // [map]
    unsigned char* k_s = q_s + L::Q_BYTES;                // [KST]: tile (block, map) goes to stage (2 block + map) % KST
    unsigned char* v_s = k_s + KST * L::K_TILE;           // [VST]
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(v_s + VST * L::V_TILE);
    unsigned long long* q_full = bars;                    // [1]
    unsigned long long* q_empty = bars + 1;               // [1]
    unsigned long long* o_full = bars + 2;                // [1] every product of the item is done
    unsigned long long* o_free = bars + 3;                // [1] the row threads have read the item's O
    unsigned long long* s_full = bars + 4;                // [MAPS]
    unsigned long long* p_ready = bars + 6;               // [MAPS]
    unsigned long long* k_full = bars + 8;                // [KST]
    unsigned long long* k_empty = k_full + KST;           // [KST]
    unsigned long long* v_full = k_empty + KST;           // [VST]
    unsigned long long* v_empty = v_full + VST;           // [VST]
    unsigned* tmem_slot = reinterpret_cast<unsigned*>(bars + L::N_BARS);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    static_assert(L::N_BARS * 8 + 8 <= 256, "the barriers and the two words after them take 256 bytes");
    float* xchg = reinterpret_cast<float*>(bars) + 64;    // [MAPS][ROWT][128]
    // where shared memory is too short for the slack that rounding up to 1024 bytes needs, its start has to
    // be aligned already; the block refuses to run otherwise
    if (smem + L::TILES + L::TAIL > smem_raw + p.smem_bytes) {
        if (threadIdx.x == 0) atomicOr(p.status, ESP_STATUS_SMEM_LAYOUT);
        return;
    }

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    constexpr int V_WARP = 2 + MAPS * ROWT * 4;           // warps: 0 queries and keys, 1 products, row threads, values
    if (threadIdx.x == 0) {
        // o_free: one arrival per warp of row threads; p_ready: one per warp of the map's; the others one
        for (int i = 0; i < L::N_BARS; i++) mbar_init(&bars[i], i == 3 ? MAPS * ROWT * 4 : (i == 6 || i == 7) ? ROWT * 4 : 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(tmem_slot)), "r"(512));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const unsigned tmem_base = *tmem_slot;
    const unsigned tm_s = tmem_base, tm_o = tmem_base + 256;           // S of the maps at columns 0 and 128, O at 256 and 384

    if (warp == 0 || warp == V_WARP) {
        // ---- loads.  Warp 0: the queries of both maps and the keys (a tile per block and map); the last warp: the values
        // (a tile per block).  A lane's box: (page of the block, 64-column slice); the pages of 16 blocks are read from
        // the block table at once, one per lane, and handed out by shuffle.
        const bool is_k = warp == 0;
        const int per_block = is_k ? MAPS : 1, slices = is_k ? HK : HV, stages = is_k ? KST : VST;
        const int tile_bytes = is_k ? L::K_TILE : L::V_TILE;
        unsigned char* ring = is_k ? k_s : v_s;
        unsigned long long* full = is_k ? k_full : v_full;
        unsigned long long* empty = is_k ? k_empty : v_empty;
        bool ok = true;
        const int pg_in_blk = lane / slices, slice = lane % slices;     // lanes 0 .. 2 * slices - 1 issue boxes
        int issued_q = 0, issued = 0;                                   // tiles of this warp's ring so far
        for (int round = 0; ok; round++) {
            const int item = item_of(round);
            if (item >= n_items) break;
            const Item t = load_item(p, item);
            if (is_k) {
                if (lane == 0) {                                         // the last item's S products have read its queries
                    ok = !*abort_flag && mbar_wait(q_empty, (round & 1) ^ 1);
                    if (ok) mbar_expect_tx(q_full, L::Q_BYTES);
                }
                ok = __shfl_sync(0xffffffffu, ok, 0);
                if (!ok) break;
                if (lane < MAPS * HK)
                    tma_load_3d(q_s + lane * ATOM_BYTES, &map_q, (lane % HK) * 64, t.h * MAPS + lane / HK, t.row0, q_full);
                issued_q = round + 1;
            }
            int rows16 = p.kv_rows;                                      // this lane's page of the 16 blocks at hand
            for (int j = 0; j < t.nb && ok; j++) {
                if ((j & 15) == 0) {
                    // a page past the tile's last key, or ahead of the first key that any of its rows sees (the sequence
                    // may have given it back), is read as zeros (a row past the cache)
                    rows16 = p.kv_rows;
                    const int page_idx = (t.blk_lo + j) * 2 + lane;
                    if (page_idx <= t.pos_last / PAGE && page_idx >= t.page_lo) {
                        const int pg = p.block_table[(size_t)t.seq * p.table_stride + page_idx];
                        if (pg >= 0 && pg < p.n_pages) rows16 = (pg * p.nkv + t.kvh) * PAGE;
                        else atomicOr(p.status, ESP_STATUS_BAD_INDEX);
                    }
                }
                const int box_row = __shfl_sync(0xffffffffu, rows16, ((j & 15) * 2 + pg_in_blk) & 31);
                for (int m = 0; m < per_block && ok; m++) {
                    const int s = issued % stages, ph = (issued / stages) & 1;
                    if (lane == 0) {
                        ok = !*abort_flag && mbar_wait(&empty[s], ph ^ 1);
                        if (ok) mbar_expect_tx(&full[s], tile_bytes);
                    }
                    ok = __shfl_sync(0xffffffffu, ok, 0);
                    if (!ok) break;
                    if (lane < 2 * slices) {
                        unsigned char* dst = ring + s * tile_bytes + slice * ATOM_BYTES + pg_in_blk * (PAGE * 128);
                        if (is_k) tma_load_3d(dst, &map_k, slice * 64, m, box_row, &full[s]);
                        else tma_load_2d(dst, &map_v, t.part * 128 + slice * 64, box_row, &full[s]);
                    }
                    issued++;
                }
            }
        }
        if (lane == 0 && (!ok || *abort_flag)) {
            atomicOr(p.status, ESP_STATUS_WAIT_EXPIRED);
            *abort_flag = 1;
            // let this warp's own copies land before the block's shared memory is given up
            if (issued_q > 0) mbar_wait(q_full, (issued_q - 1) & 1);
            for (int j = max(0, issued - stages); j < issued; j++) mbar_wait(&full[j % stages], (j / stages) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const unsigned idesc_s = idesc_attn(BN, false), idesc_pv = idesc_attn(VD, true);
            const unsigned long long dq = smem_desc(q_s), dk = smem_desc(k_s);
            const unsigned long long dv = smem_desc_mn(v_s, ATOM_BYTES);
            bool ok = true;
            int g0 = 0;                                                   // key blocks before this item
            for (int round = 0; ok && !*abort_flag; round++) {
                const int item = item_of(round);
                if (item >= n_items) break;
                const Item t = load_item(p, item);
                // S_m of the item's key block j, over where the map's last P stood: the tensor core runs one thread's
                // products in the order in which they were issued
                auto issue_s = [&](int j, int m) {
                    const int c = (g0 + j) * MAPS + m, st = c % KST;
                    if (!mbar_wait(&k_full[st], (c / KST) & 1)) return false;
                    tc_fence_after();
#pragma unroll
                    for (int kk = 0; kk < KD / 16; kk++) {
                        const unsigned off = ((kk >> 2) * ATOM_BYTES + (kk & 3) * 32) >> 4;
                        tc_mma(tm_s + m * BN, dq + ((m * L::K_TILE) >> 4) + off, dk + ((st * L::K_TILE) >> 4) + off, idesc_s, kk > 0 ? 1u : 0u);
                    }
                    tc_commit(&k_empty[st]);                              // the keys are free once S is done
                    if (j + 1 == t.nb && m + 1 == MAPS) tc_commit(q_empty);   // and so are the queries after the item's last S
                    tc_commit(&s_full[m]);
                    return true;
                };
                ok = mbar_wait(q_full, round & 1);
                for (int m = 0; m < MAPS && ok; m++) ok = issue_s(0, m);
                // the row threads have read the O of the item before
                if (ok) ok = mbar_wait(o_free, (round & 1) ^ 1);
                for (int j = 0; j < t.nb && ok && !*abort_flag; j++) {
                    const int gg = g0 + j, st = gg % VST;
                    if (!mbar_wait(&v_full[st], (gg / VST) & 1)) {
                        ok = false;
                        break;
                    }
#pragma unroll
                    for (int m = 0; m < MAPS; m++) {
                        // the map's P stands where its S stood (and its O has been rescaled if it had to be)
                        if (!ok || !mbar_wait(&p_ready[m], gg & 1)) {
                            ok = false;
                            break;
                        }
                        tc_fence_after();
#pragma unroll
                        for (int kk = 0; kk < BN / 16; kk++) {            // O_m += P_m V; the item's first block starts it
                            const unsigned b_off = (st * L::V_TILE + kk * 16 * 128) >> 4;
                            // a row thread's 64 keys are 32 columns of weights at the start of its 64 columns of scores
                            const unsigned a_at = tm_s + m * BN + (kk >> 2) * (BN / ROWT) + (kk & 3) * 8;
                            tc_mma_ta(tm_o + m * BN, a_at, dv + b_off, idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
                        }
                        if (m + 1 == MAPS) {
                            tc_commit(&v_empty[st]);
                            if (j + 1 == t.nb) tc_commit(o_full);         // all of the item's products
                        }
                        if (j + 1 < t.nb) ok = issue_s(j + 1, m);         // the map's next block
                    }
                }
                g0 += t.nb;
            }
            if (!ok) {
                atomicOr(p.status, ESP_STATUS_WAIT_EXPIRED);
                *abort_flag = 1;
            }
        }
    } else {
        // ---- row threads: TMEM lane = query row of the tile; a group of them per map.  ROWT threads of a group share a
        // row: thread ``side`` takes the keys side * CW .. of a block.
        const int quad = warp & 3, r = quad * 32 + lane, grp = (warp - 2) / (4 * ROWT), side = ((warp - 2) >> 2) % ROWT;
        const unsigned lane_sel = (unsigned)(quad * 32) << 16;
        constexpr int CW = BN / ROWT;                                    // keys of a block that this thread takes
        constexpr int OW = VD / ROWT;                                    // columns of the map's O that this thread rescales
        constexpr int FW = VD / (MAPS * ROWT);                           // columns of the result that this thread writes
        constexpr int MATES = ROWT * 32, ROW_ALL = MAPS * ROWT * 32;     // threads at the map's and at the row's barrier
        constexpr float LAZY = 8.f;                                      // O is rescaled when the maximum grew by more (log2)
        static_assert(CW == 64, "a thread's weights take the first half of its columns of scores");
        static_assert(FW == 16 || FW == 32, "columns are read 32 or 16 at a time");
        const int bar_grp = 1 + grp * 4 + quad, bar_row = 1 + MAPS * 4 + quad;
        float* xg = xchg + grp * (ROWT * 128);                            // the group's [side][row]
        const unsigned s_addr = tm_s + grp * BN + lane_sel + side * CW;
        const bool capped = FIXED || p.cap2 > 0.f;
        const float unit = p.to_unit, cap2 = p.cap2;
        bool ok = true;
        int n_b = 0;                                                      // key blocks so far
        for (int round = 0; ok; round++) {
            const int item = item_of(round);
            if (item >= n_items) break;
            const Item t = load_item(p, item);
            const int pos = t.pos0 + r;
            const int key_first = first_visible_key(pos, 0, p.chunk);     // the keys this row sees: key_first .. pos
            const int key_first_last = first_visible_key(t.pos0 + BM - 1, 0, p.chunk);   // of the tile's last row
            float m_ref = FIXED ? 0.f : -INFINITY, l_run = 0.f;           // what O and l_run are scaled by
            for (int j = 0; j < t.nb && ok; j++, n_b++) {
                const int key0 = (t.blk_lo + j) * BN;
                ok = !*abort_flag && mbar_wait(&s_full[grp], n_b & 1);
                ok = FIXED ? __all_sync(0xffffffffu, ok) : pair_agree(ok, bar_grp, MATES);   // a warp goes on or leaves together
                if (!ok) break;
                // S is done, and so are the products issued before it: O holds the map's blocks so far
                tc_fence_after();
                // does any (row of the tile, key of the block) pair need the mask?
                const bool edge = key0 + BN - 1 > t.pos0 || key0 < key_first_last;
                // live columns of this row: c_lo .. c_lo + c_span; one unsigned comparison per element, no branch
                const int c_lo = key_first - key0 - side * CW;
                const unsigned c_span = (unsigned)(pos - key_first);
                if constexpr (!FIXED) {
                    float mx = -INFINITY;                                 // of the raw scores: what is done to them is monotonic
#pragma unroll
                    for (int c = 0; c < CW / 32; c++) {
                        float sv[32];
                        tc_ld32(s_addr + c * 32, sv);
#pragma unroll
                        for (int i = 0; i < 32; i++) {
                            const bool live = !edge || (unsigned)(c * 32 + i - c_lo) <= c_span;
                            mx = fmaxf(mx, live ? sv[i] : -INFINITY);
                        }
                    }
                    xg[side * 128 + r] = mx;
                    named_sync(bar_grp, MATES);
#pragma unroll
                    for (int o2 = 0; o2 < ROWT; o2++) mx = fmaxf(mx, xg[o2 * 128 + r]);
                    named_sync(bar_grp, MATES);                           // all have read: the next block may write
                    float m_blk = mx * unit;                              // the maximum in powers of two
                    if (capped && mx != -INFINITY) m_blk = cap2 * tanhf(m_blk);
                    const float m_new = fmaxf(m_ref, m_blk);
                    // A row whose maximum outgrew the reference by more than LAZY is brought up to date: the sum here, O
                    // in tensor memory, which the warp reads and writes as a whole (the other rows take the factor 1).
                    const bool grew = m_new > m_ref + LAZY;               // the same for all threads of the row
                    if (j == 0) {
                        m_ref = m_new;
                    } else if (__any_sync(0xffffffffu, grew)) {
                        const float alpha = grew ? fast_exp2(m_ref - m_new) : 1.f;   // m_ref = -inf gives 0
                        if (grew) m_ref = m_new;
                        l_run *= alpha;
#pragma unroll
                        for (int c = 0; c < OW / 16; c++) {
                            const unsigned o_addr = tm_o + grp * BN + lane_sel + side * OW + c * 16;
                            float v[16];
                            unsigned w[16];
                            tc_ld16(o_addr, v);
#pragma unroll
                            for (int i = 0; i < 16; i++) w[i] = __float_as_uint(v[i] * alpha);
                            tc_st16(o_addr, w);
                        }
                    }
                }
                const float m_use = FIXED || m_ref == -INFINITY ? 0.f : m_ref;
                const unsigned long long neg_m = pack2(-m_use, -m_use), unit2 = pack2(unit, unit);
                unsigned long long l_add = 0;                              // two sums: of the even and of the odd keys
                // the weights of keys 2c and 2c + 1 of this thread's run go to column c of its columns of S
#pragma unroll
                for (int c = 0; c < CW / 32; c++) {
                    float sv[32];
                    unsigned packed[16];
                    tc_ld32(s_addr + c * 32, sv);
                    bool small = false;
                    if (capped) {
                        float am = max_abs3(sv[0], sv[1], sv[2]), bm = max_abs3(sv[3], sv[4], sv[5]);
#pragma unroll
                        for (int i = 6; i < 30; i += 4) {
                            am = max_abs3(am, sv[i], sv[i + 1]);
                            bm = max_abs3(bm, sv[i + 2], sv[i + 3]);
                        }
                        small = __all_sync(0xffffffffu, fmaxf(max_abs3(am, sv[30], sv[31]), bm) <= p.raw_max);
                    }
                    if (small) {
#pragma unroll
                        for (int i = 0; i < 32; i += 2) {
                            const unsigned long long x = pack2(sv[i], sv[i + 1]), y = mul2(x, x);
                            unsigned long long f = fma2(p.poly[4], y, p.poly[3]);
                            f = fma2(f, y, p.poly[2]);
                            f = fma2(f, y, p.poly[1]);
                            f = fma2(f, y, p.poly[0]);
                            unpack2(FIXED ? mul2(f, x) : fma2(f, x, neg_m), sv[i], sv[i + 1]);
                        }
                    } else if (capped) {
#pragma unroll
                        for (int i = 0; i < 32; i++)
                            sv[i] = cap2 - m_use - __fdividef(2.f * cap2, 1.f + fast_exp2(sv[i] * (2.f * LOG2E * unit)));
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; i += 2)
                            unpack2(fma2(pack2(sv[i], sv[i + 1]), unit2, neg_m), sv[i], sv[i + 1]);
                    }
                    if (edge) {
#pragma unroll
                        for (int i = 0; i < 32; i++) sv[i] = (unsigned)(c * 32 + i - c_lo) <= c_span ? sv[i] : -INFINITY;
                    }
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {                     // a masked score is -inf: its weight is 0
                        __nv_bfloat162 b2 = __floats2bfloat162_rn(fast_exp2(sv[i]), fast_exp2(sv[i + 1]));
                        // the sum is of the weights as the product will see them: a row with one key then returns its value
                        // exactly in either map, whatever the weight (the maps' difference may be all that is left of it)
                        const unsigned w2 = *reinterpret_cast<unsigned*>(&b2);
                        l_add = add2(l_add, pack2(__uint_as_float(w2 << 16), __uint_as_float(w2 & 0xffff0000u)));
                        packed[i >> 1] = w2;
                    }
                    tc_st16(s_addr + c * 16, packed);
                }
                tc_wait_st();
                float l_even, l_odd;
                unpack2(l_add, l_even, l_odd);
                l_run += l_even + l_odd;
                tc_fence_before();                                        // S has been read, P and O written
                __syncwarp();
                if (lane == 0) mbar_arrive(&p_ready[grp]);
            }
            // ---- the item's end: the sums of both maps to all the row's threads, who wait for the last products and
            // each make FW columns
            ok = pair_agree(ok, bar_row, ROW_ALL);                        // (all have read what the last item left in xchg)
            if (!ok) break;
            xg[side * 128 + r] = l_run;
            ok = !*abort_flag && mbar_wait(o_full, round & 1);
            ok = pair_agree(ok, bar_row, ROW_ALL);                        // all threads of the row: written, and well
            if (!ok) break;
            tc_fence_after();
            float inv[MAPS];
#pragma unroll
            for (int m = 0; m < MAPS; m++) {
                float l = 0.f;
#pragma unroll
                for (int o2 = 0; o2 < ROWT; o2++) l += xchg[(m * ROWT + o2) * 128 + r];   // keys in ascending order
                inv[m] = l > 0.f ? 1.0f / l : 0.f;
            }
            const int col0 = (grp * ROWT + side) * FW;
            float o1[FW], o2v[FW];
            if constexpr (FW == 32) {
                tc_ld32(tm_o + lane_sel + col0, o1);
                tc_ld32(tm_o + BN + lane_sel + col0, o2v);
            } else {
                tc_ld16(tm_o + lane_sel + col0, o1);
                tc_ld16(tm_o + BN + lane_sel + col0, o2v);
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(o_free);
            const int vcol = t.part * 128 + col0;                         // of the head's value channels
            if (p.v_parts > 1) {
                if (r < t.rows) {
                    float* mrow = p.maps_out + ((size_t)(t.row0 + r) * p.nh + t.h) * MAPS * p.vd + vcol;
#pragma unroll
                    for (int i = 0; i < FW; i += 4)
                        if (vcol + i < p.vd) {
                            *reinterpret_cast<float4*>(mrow + i) =
                                make_float4(o1[i] * inv[0], o1[i + 1] * inv[0], o1[i + 2] * inv[0], o1[i + 3] * inv[0]);
                            *reinterpret_cast<float4*>(mrow + p.vd + i) =
                                make_float4(o2v[i] * inv[1], o2v[i + 1] * inv[1], o2v[i + 2] * inv[1], o2v[i + 3] * inv[1]);
                        }
                }
                if constexpr (!FIXED) named_sync(bar_row, ROW_ALL);       // all have read the sums: the next item may write
                continue;
            }
            float ss = 0.f;
            const float f2 = p.lambda * inv[1];
#pragma unroll
            for (int i = 0; i < FW; i++) {                                // columns beyond vd are zero
                o1[i] = o1[i] * inv[0] - f2 * o2v[i];
                ss = fmaf(o1[i], o1[i], ss);
            }
            named_sync(bar_row, ROW_ALL);                                 // all have read the sums
            xchg[(grp * ROWT + side) * 128 + r] = ss;
            named_sync(bar_row, ROW_ALL);
            ss = 0.f;
#pragma unroll
            for (int q = 0; q < MAPS * ROWT; q++) ss += xchg[q * 128 + r];
            // the next item's maxima go to the same place (FIXED has none: its next write lies behind a row's barrier)
            if constexpr (!FIXED) named_sync(bar_row, ROW_ALL);
            if (r < t.rows) {
                float f = p.out_scale / sqrtf(ss / (float)p.vd + p.eps);
                if (p.gate) f *= 1.0f / (1.0f + expf(-p.gate[(size_t)(t.row0 + r) * p.ldg + t.h]));
                bf16* orow = p.out + ((size_t)(t.row0 + r) * p.nh + t.h) * p.vd + vcol;
#pragma unroll
                for (int i = 0; i < FW; i += 8) {
                    if (vcol + i >= p.vd) break;
                    __nv_bfloat162 b0 = __floats2bfloat162_rn(o1[i] * f, o1[i + 1] * f);
                    __nv_bfloat162 b1 = __floats2bfloat162_rn(o1[i + 2] * f, o1[i + 3] * f);
                    __nv_bfloat162 b2 = __floats2bfloat162_rn(o1[i + 4] * f, o1[i + 5] * f);
                    __nv_bfloat162 b3 = __floats2bfloat162_rn(o1[i + 6] * f, o1[i + 7] * f);
                    *reinterpret_cast<uint4*>(orow + i) = make_uint4(*reinterpret_cast<unsigned*>(&b0), *reinterpret_cast<unsigned*>(&b1),
                                                                     *reinterpret_cast<unsigned*>(&b2), *reinterpret_cast<unsigned*>(&b3));
                }
            }
        }
        if (!ok && lane == 0) {
            atomicOr(p.status, ESP_STATUS_WAIT_EXPIRED);
            *abort_flag = 1;
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base), "r"(512));
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// a contiguous bfloat16 array [rows, mid, cols] in boxes of box_rows x 1 x 64, 128-byte swizzle, zeros outside (mid 0:
// two dimensions)
int make_map(CUtensorMap* map, const void* base, unsigned long long cols, unsigned long long mid, unsigned long long rows,
             unsigned box_rows) {
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) != cudaSuccess ||
            qres != cudaDriverEntryPointSuccess)
            return (int)cudaErrorNotSupported;
        fn = reinterpret_cast<EncodeTiledFn>(ptr);
    }
    const bool three = mid > 0;
    const cuuint64_t dims[3] = {cols, three ? mid : rows, rows};
    const cuuint64_t strides[2] = {cols * 2, cols * (three ? mid : 1) * 2};
    const cuuint32_t box[3] = {64, three ? 1 : box_rows, box_rows};
    const cuuint32_t elem[3] = {1, 1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, three ? 3 : 2, const_cast<void*>(base), dims, strides, box, elem,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : (int)cudaErrorInvalidValue;
}

template <int KD, int VD, bool FIXED>
int launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, DiffAttnParams p, cudaStream_t stream) {
    using L = Layout<KD, VD>;
    // 1024 bytes to round the start up with, where the 227 KB of a block have room for them
    size_t smem = (size_t)L::TILES + L::TAIL;
    if (smem + 1024 <= 232448) smem += 1024;
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(attn_diff_tc05_kernel<KD, VD, FIXED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        raised = true;
    }
    static int sm_count = 0;
    if (!sm_count) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&sm_count, cudaDevAttrMultiProcessorCount, dev);
        if (sm_count <= 0) sm_count = 148;
    }
    const long long items = (long long)p.n_tiles * p.nh * p.v_parts;
    const long long grid = items < sm_count ? items : sm_count;
    p.smem_bytes = (int)smem;
    attn_diff_tc05_kernel<KD, VD, FIXED><<<(int)grid, 96 + MAPS * ROWT * 128, smem, stream>>>(mq, mk, mv, p);
    return esp_launch_status();
}
}  // namespace

// q [n_tokens, nh, 2, kd] and out [n_tokens, nh, vd], bfloat16; keys [pages, nkv, 64, 2 * kd], values [pages, nkv, 64,
// vd]; tile_seq / tile_first: the tiles of 128 new tokens, best listed with the tiles that see the most keys first.
// kd: a multiple of 8 up to 128; vd: a multiple of 8 up to 256.  vd > 128: the maps' outputs go to maps_out float
// [n_tokens, nh, 2, vd] and ``out``, lambda, eps, out_scale and the gate are not used.  softcap 0: none.  chunk 0: every
// earlier key.
ESP_API int esp_attn_diff_tc05(const void* q, long long n_tokens, const void* k_cache, const void* v_cache, void* out,
                               float* maps_out, const int* tile_seq, const int* tile_first, const int* seq_start,
                               const int* seq_past, const int* block_table, int table_stride, int n_pages, int page, int n_tiles,
                               int nh, int nkv, int kd, int vd, float scale, float softcap, int chunk, float lambda, float eps,
                               float out_scale, const float* gate, long long ldg, int* status, cudaStream_t stream) {
    if (n_tiles <= 0) return 0;
    if (page != PAGE || kd <= 0 || kd % 8 != 0 || kd > 128 || vd <= 0 || vd % 8 != 0 || vd > 256 || nkv <= 0 || nh % nkv != 0 ||
        nh > 32767 || n_tokens <= 0 || !(scale > 0.f) || softcap < 0.f || (vd > 128 ? !maps_out : !out))
        return (int)cudaErrorInvalidValue;
    const unsigned long long kv_rows = (unsigned long long)n_pages * nkv * PAGE;
    if (kv_rows >= (1ull << 31)) return (int)cudaErrorInvalidValue;
    CUtensorMap mq, mk, mv;
    int rc = make_map(&mq, q, (unsigned long long)kd, (unsigned long long)nh * MAPS, (unsigned long long)n_tokens, BM);
    if (rc) return rc;
    rc = make_map(&mk, k_cache, (unsigned long long)kd, MAPS, kv_rows, PAGE);
    if (rc) return rc;
    rc = make_map(&mv, v_cache, (unsigned long long)vd, 0, kv_rows, PAGE);
    if (rc) return rc;
    DiffAttnParams p{};
    p.out = (bf16*)out; p.maps_out = maps_out; p.tile_seq = tile_seq; p.tile_first = tile_first; p.seq_start = seq_start;
    p.seq_past = seq_past; p.block_table = block_table; p.gate = gate; p.ldg = ldg; p.table_stride = table_stride;
    p.n_pages = n_pages; p.nh = nh; p.nkv = nkv; p.vd = vd; p.v_parts = vd > 128 ? 2 : 1; p.chunk = chunk;
    p.kv_rows = (int)kv_rows; p.n_tiles = n_tiles; p.status = status; p.lambda = lambda; p.eps = eps; p.out_scale = out_scale;
    p.cap2 = softcap * LOG2E;
    p.to_unit = softcap > 0.f ? scale / softcap : scale * LOG2E;
    p.raw_max = TANH_POLY_MAX / p.to_unit;
    double power = (double)p.cap2 * p.to_unit;
    for (int i = 0; i < POLY; i++, power *= (double)p.to_unit * p.to_unit) {
        const float c = (float)(TANH_POLY[i] * power);
        if (softcap > 0.f && !(c < -1e-36f || c > 1e-36f)) p.raw_max = -1.f;      // too small for float: the other form throughout
        unsigned bits;
        memcpy(&bits, &c, 4);
        p.poly[i] = ((unsigned long long)bits << 32) | bits;
    }
    const bool fixed = softcap > 0.f && softcap <= FIXED_CAP_MAX;
#define ESP_DIFF_TC(KD, VD) return fixed ? launch<KD, VD, true>(mq, mk, mv, p, stream) : launch<KD, VD, false>(mq, mk, mv, p, stream)
    if (kd <= 64 && vd <= 64) ESP_DIFF_TC(64, 64);
    if (kd <= 64) ESP_DIFF_TC(64, 128);
    if (vd <= 64) ESP_DIFF_TC(128, 64);
    ESP_DIFF_TC(128, 128);
#undef ESP_DIFF_TC
}
