// Attention over a cached latent on the fifth-generation tensor cores (bfloat16): all query heads share one cached
// row per position, [latent (rank) | rotated key part], and the values are the first `rank` columns of the same rows.
//
// The query rows of a request are its (token, head) pairs in that order, which is how they lie in memory.  A block takes
// 128 consecutive rows of them and up to 256 value columns: the accumulators of a tile, two of 128 scores a row and one
// of the value columns, fill the 512 columns of tensor memory.  A rank above 256 is cut into column blocks, each with the
// scores of its own (computed twice for a rank of 512; the products of the values, and the reads of the cached rows
// for them, are not).  Six warps:
//   warp 0   one lane issues the TMA loads: the query rows once, [128 rows x 64 columns] a box, which stay; then, through
//            one ring of 16 KB stages in the order in which the products want them, for every tile of 128 keys the row's
//            pieces [128 keys x 64 columns] (two boxes of 64 keys: a box never crosses a page) and the value columns as
//            pieces [32 keys x up to 256 columns].  Columns past a row's end arrive as zeros;
//   warp 1   allocates tensor memory; one lane issues S_(j+1) = Q K^T piece by piece as the ring delivers (128 x 128 x 16
//            products, both operands k-major), waits for P_j, then issues O += P_j V_j (128 x columns x 16 products, V as it
//            lies in the cache, which is the MN-major form of the B operand, P_j from tensor memory), so that the
//            tensor cores work on the next scores while the softmax of the current ones runs;
//   warps 2-5  one thread a query row, which holds the row's 128 scores in registers: maximum, then P = exp2(s * scale -
//            max) as bfloat16 pairs over the S columns it came from, running maximum and sum in float32.  The maximum that P is taken against moves only when the true one is 2^8 ahead (O is rescaled in
//            tensor memory then).  At the end O is divided by the sum and stored.
//
// Decode is the same kernel with one new token a request at position seq_len - 1: a tile is one token's heads, and the keys
// may be cut into ranges of whole tiles whose (max, sum, output) go to scratch in the layout the combine kernel merges
// (lily_attention_combine: [requests, heads, ranges, rank] outputs, then [.., 2]).  Fewer than 128 heads leave rows of
// the products unused (their time is the tensor cores' for 128 rows whatever the heads).
//
// With `sinks` a row's running maximum starts at the head's sink (in the units of the unscaled scores) and its sum at one:
// the softmax's denominator holds exp(sink), a key without a value (decode: in the first key range).
//
// Keys past the last one a block sees and rows past the tile's are computed on whatever the pages and the neighbouring
// query rows hold (finite everywhere) and masked, or not stored.  Every wait is bounded; one that runs out sets a status
// word (lily_latent_attention_tc_status), the roles leave their loops, copies in flight get a bounded wait and the block
// frees its tensor memory.
#include "common.cuh"
#include "tcgen05.cuh"

namespace lily {
namespace lt {

using namespace tc5;

constexpr int BQ = 128;                   // query rows per block
constexpr int BKV = 128;                  // keys per tile
constexpr int STAGE = 128 * 64 * 2;       // 16 KB: [128 keys][64 columns] of the rows, or [32 keys][256 columns] of the values
constexpr int BOX_K = 64 * 64 * 2;        // one TMA box of 64 keys
constexpr int VKEYS = 32, BOX_V = VKEYS * 64 * 2;
constexpr int MAX_STAGES = 8;
constexpr int MAX_COLUMNS = 256;          // value columns a block
constexpr int THREADS = 64 + BQ;
constexpr int SMEM_LIMIT = 227 * 1024;
constexpr int TAIL = 8 * (1 + 2 * MAX_STAGES + 6) + 16;     // mbarriers, tensor-memory base, abort flag
constexpr uint32_t SPIN_LIMIT = 1u << 24;
constexpr float GROW_LOG2 = 8.f;

__device__ int g_status = 0;              // 0 ok; else (code << 24 | block) of the first wait that gave up

struct Params {
    const int* block_table;
    const int* cu_seqlens;
    const int* prefix_lens;
    const int* tile_req;
    const int* tile_start;
    const int* seq_lens;                  // decode: [requests]; null: prompt portions
    float* part_o;                        // decode with key ranges
    float* part_ml;
    int splits;
    __nv_bfloat16* out;                   // [tokens, heads, rank]
    int bt_stride, tiles, tile_tokens, row_blocks, heads, row, rank, page_size, window;
    int chunks;                           // pieces of 64 columns of a row
    int col_blocks, cols;                 // column blocks and value columns of one (a multiple of 16)
    int stages, q_rows;                   // rows of the queries' box
    float scale_log2;
    const float* sinks;                   // [heads], or null
};

__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag, int code) {
    for (uint32_t i = 0; i < SPIN_LIMIT; ++i) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((i & 1023u) == 1023u && *abort_flag) return false;
    }
    *abort_flag = 1;
    atomicCAS(&g_status, 0, (code << 24) | (int)(blockIdx.x & 0xFFFFFF));
    return false;
}

// The same for a whole warp, which leaves with one answer.
__device__ __forceinline__ bool warp_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag, int code) {
    for (uint32_t i = 0; i < SPIN_LIMIT; ++i) {
        if (__all_sync(0xffffffffu, mbar_try_wait(bar, parity))) return true;
        if ((i & 1023u) == 1023u && __any_sync(0xffffffffu, *abort_flag)) return false;
    }
    *abort_flag = 1;
    atomicCAS(&g_status, 0, (code << 24) | (int)(blockIdx.x & 0xFFFFFF));
    return false;
}

__global__ void __launch_bounds__(THREADS, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                           const __grid_constant__ CUtensorMap map_v, const Params p) {
    extern __shared__ __align__(1024) unsigned char smem[];
    const int warp = uniform(threadIdx.x >> 5), lane = threadIdx.x & 31;
    if ((smem_u32(smem) & 1023u) != 0) {                        // the swizzled tiles need it; never seen, but checked
        if (threadIdx.x == 0) atomicCAS(&g_status, 0, (11 << 24) | (int)(blockIdx.x & 0xFFFFFF));
        pdl_wait();
        return;
    }
    const int NC = p.chunks, ST = p.stages;
    const uint32_t q_smem = smem_u32(smem), ring = q_smem + NC * STAGE;
    unsigned char* tail = smem + (size_t)(NC + ST) * STAGE;
    const uint32_t q_full = smem_u32(tail), full = q_full + 8, empty = full + 8 * MAX_STAGES, s_full = empty + 8 * MAX_STAGES,
                   p_full = s_full + 16, pv_done = p_full + 16;
    uint32_t& tmem_base_s = *reinterpret_cast<uint32_t*>(tail + 8 * (1 + 2 * MAX_STAGES + 6));
    int& abort_s = *reinterpret_cast<int*>(tail + 8 * (1 + 2 * MAX_STAGES + 6) + 4);
    if (threadIdx.x == 0) {
        abort_s = 0;
        mbar_init(q_full, 1);
        for (int s = 0; s < ST; ++s) {
            mbar_init(full + 8 * s, 1);
            mbar_init(empty + 8 * s, 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(s_full + 8 * b, 1);
            mbar_init(p_full + 8 * b, BQ);                      // one arrival per softmax thread
            mbar_init(pv_done + 8 * b, 1);
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&tmem_base_s)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = (uint32_t)uniform((int)tmem_base_s), tmem_o = tmem + 2 * BKV;     // S (then P) of tile j: columns 128 (j & 1)
    volatile int* abort_flag = &abort_s;

    // q and the cache come from the kernels before this one
    pdl_wait();
    pdl_launch_dependents();

    const int cb = blockIdx.x % p.col_blocks;
    int work = blockIdx.x / p.col_blocks;
    const int row0 = (work % p.row_blocks) * BQ;                    // this block's first row of the tile's
    work /= p.row_blocks;
    const bool decode = p.seq_lens != nullptr;
    int req, tok0, ntok, pos0, range = 0;
    if (decode) {
        range = work % p.splits;
        req = work / p.splits;
        tok0 = req;
        ntok = 1;
        pos0 = uniform(p.seq_lens[req]) - 1;
    } else {
        const int tile = p.tiles - 1 - work;                        // the last tiles, which see the most keys, go first
        req = uniform(p.tile_req[tile]);
        const int start = uniform(p.tile_start[tile]);
        tok0 = uniform(p.cu_seqlens[req]) + start;
        ntok = min(p.tile_tokens, uniform(p.cu_seqlens[req + 1]) - tok0);
        pos0 = uniform(p.prefix_lens[req]) + start;                 // position of the tile's first token
    }
    const int nrows = ntok * p.heads;
    const int rows_valid = min(BQ, nrows - row0);                   // >= 1: a tile of several tokens has one row block
    const int first_pos = pos0 + row0 / p.heads, last_pos = pos0 + (row0 + rows_valid - 1) / p.heads;
    int kv_end = last_pos + 1;
    const int k_lo = (p.window > 0 && first_pos + 1 > p.window) ? first_pos + 1 - p.window : 0;
    int jt0 = k_lo / BKV;
    int n = (kv_end - 1) / BKV - jt0 + 1;                           // key tiles of this block (>= 1, but for a range past the keys)
    if (decode && p.splits > 1) {
        const int per = (n + p.splits - 1) / p.splits;
        jt0 += range * per;
        n = min(per, n - range * per);
        kv_end = min(kv_end, (jt0 + per) * BKV);
    }
    const int v0 = cb * p.cols, nv = (p.cols + 63) / 64;            // first value column, boxes of 64 columns

    if (warp == 0) {
        const int* table = p.block_table + (size_t)req * p.bt_stride;
        if (elect_one()) {
            mbar_expect_tx(q_full, NC * p.q_rows * 128);
            for (int c = 0; c < NC; ++c) tma_load_2d(q_smem + c * STAGE, &map_q, q_full, c * 64, tok0 * p.heads + row0);
        }
        int it = 0, s = 0;                                          // pieces issued so far; the next one's stage
        uint32_t par = 1;                                           // parity of the stage's "empty" phase that frees it
        auto next = [&]() {
            ++it;
            if (++s == ST) { s = 0; par ^= 1; }
        };
        // the pages of a tile's two halves of 64 keys and the places in them: of the tile whose keys were issued last, and of
        // the one before it, whose values come next
        int page0 = 0, off0 = 0, page1 = 0, off1 = 0, vpage0, voff0, vpage1, voff1;
        bool ok = true;
        auto keys = [&](int j) {
            vpage0 = page0; voff0 = off0; vpage1 = page1; voff1 = off1;
            const int key = (jt0 + j) * BKV;                        // a tile holds at least one key that is seen
            page0 = uniform(table[key / p.page_size]);
            off0 = key % p.page_size;
            const bool held = key + 64 < kv_end;
            page1 = held ? uniform(table[(key + 64) / p.page_size]) : 0;
            off1 = held ? (key + 64) % p.page_size : 0;
            for (int c = 0; c < NC; ++c) {
                ok = warp_wait(empty + 8 * s, par, abort_flag, 1);
                if (!ok) return;
                if (elect_one()) {
                    const uint32_t dst = ring + s * STAGE, bar = full + 8 * s;
                    mbar_expect_tx(bar, STAGE);
                    tma_load_3d(dst, &map_k, bar, c * 64, off0, page0);
                    tma_load_3d(dst + BOX_K, &map_k, bar, c * 64, off1, page1);
                }
                next();
            }
        };
        if (n > 0) keys(0);
        for (int j = 0; j < n && ok; ++j) {
            if (j + 1 < n) {
                keys(j + 1);
            } else {
                vpage0 = page0; voff0 = off0; vpage1 = page1; voff1 = off1;
            }
            for (int g = 0; g < BKV / VKEYS && ok; ++g) {
                ok = warp_wait(empty + 8 * s, par, abort_flag, 2);
                if (!ok) break;
                if (elect_one()) {
                    const uint32_t dst = ring + s * STAGE, bar = full + 8 * s;
                    const int page = g < 2 ? vpage0 : vpage1, off = (g < 2 ? voff0 : voff1) + VKEYS * (g & 1);
                    mbar_expect_tx(bar, nv * BOX_V);
                    for (int v = 0; v < nv; ++v) tma_load_3d(dst + v * BOX_V, &map_v, bar, v0 + v * 64, off, page);
                }
                next();
            }
        }
        if (*abort_flag) {
            // copies already issued still land in this block's shared memory: give each a bounded wait
            for (uint32_t i = 0; i < (1u << 20) && !mbar_try_wait(q_full, 0); ++i) {}
            for (int k = max(0, it - ST); k < it; ++k)
                for (uint32_t i = 0; i < (1u << 20) && !mbar_try_wait(full + 8 * (k % ST), (uint32_t)((k / ST) & 1)); ++i) {}
        }
    } else if (warp == 1) {
        // kind::f16: float32 accumulator, bfloat16 a and b, m = 128; bit 16 makes b MN-major
        const uint32_t common = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BQ >> 4) << 24);
        const uint32_t idesc_s = common | ((uint32_t)(BKV >> 3) << 17);
        const uint32_t idesc_o = common | (1u << 16) | ((uint32_t)(p.cols >> 3) << 17);
        int s = 0;
        uint32_t par = 0;                                           // parity of the stage's "full" phase
        auto next = [&]() {
            if (++s == ST) { s = 0; par ^= 1; }
        };
        const uint64_t dq0 = desc_k_major(q_smem), dk0 = desc_k_major(ring), dv0 = desc_mn_major(ring, BOX_V);
        bool ok = warp_wait(q_full, 0, abort_flag, 3);
        auto scores = [&](int i) {                                  // S_i = Q K_i^T into accumulator i % 2
            const uint32_t acc = tmem + (uint32_t)(i & 1) * BKV;
            for (int c = 0; c < NC; ++c) {
                if (!warp_wait(full + 8 * s, par, abort_flag, 4)) return false;
                tc_fence_after();
                if (elect_one()) {
                    const uint64_t dq = dq0 + (uint64_t)(c * STAGE >> 4), dk = dk0 + (uint64_t)(s * STAGE >> 4);
                    const int steps = min(4, (p.row - c * 64 + 15) / 16);
                    if (steps == 4) {
#pragma unroll
                        for (int kk = 0; kk < 4; ++kk)
                            umma(acc, dq + (uint64_t)(kk * 32 >> 4), dk + (uint64_t)(kk * 32 >> 4), idesc_s, (c | kk) != 0 ? 1u : 0u);
                    } else {
                        for (int kk = 0; kk < steps; ++kk)
                            umma(acc, dq + (uint64_t)(kk * 32 >> 4), dk + (uint64_t)(kk * 32 >> 4), idesc_s, (c | kk) != 0 ? 1u : 0u);
                    }
                    umma_commit(empty + 8 * s);
                    if (c == NC - 1) umma_commit(s_full + 8 * (i & 1));
                }
                __syncwarp();
                next();
            }
            return true;
        };
        if (ok && n > 0) ok = scores(0);
        for (int j = 0; j < n && ok; ++j) {
            const int b = j & 1;
            if (j + 1 < n) {
                ok = scores(j + 1);
                if (!ok) break;
            }
            ok = warp_wait(p_full + 8 * b, (uint32_t)((j >> 1) & 1), abort_flag, 5);
            for (int g = 0; g < BKV / VKEYS && ok; ++g) {
                ok = warp_wait(full + 8 * s, par, abort_flag, 6);
                if (!ok) break;
                tc_fence_after();
                if (elect_one()) {
                    const uint64_t dv = dv0 + (uint64_t)(s * STAGE >> 4);
#pragma unroll
                    for (int kk = 0; kk < VKEYS / 16; ++kk)         // 16 keys of P are 8 columns of bfloat16 pairs in S's buffer
                        umma_ts(tmem_o, tmem + (uint32_t)(b * BKV + (g * 2 + kk) * 8), dv + (uint64_t)(kk * 2048 >> 4), idesc_o,
                                (j | g | kk) != 0 ? 1u : 0u);
                    umma_commit(empty + 8 * s);
                    if (g == BKV / VKEYS - 1) umma_commit(pv_done + 8 * b);
                }
                __syncwarp();
                next();
            }
        }
    } else {
        // a warp reads the quarter of tensor memory (32 lanes = 32 query rows) that its index modulo 4 names
        const int row = (warp & 3) * 32 + lane;
        const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
        const int pos = pos0 + (row0 + row) / p.heads;
        const uint32_t my_o = tmem_o + lane_addr;
        const int pieces = (p.cols + 31) / 32;
        const bool idle = (warp & 3) * 32 >= rows_valid;
        float m_used = -INFINITY, l = 0.f;
        const bool sunk = p.sinks != nullptr && range == 0;
        if (sunk) m_used = p.sinks[(row0 + row) % p.heads] * (1.4426950408889634f / p.scale_log2);
        bool ok = true;
        for (int j = 0; j < n && ok; ++j) {
            const int b = j & 1;
            const uint32_t my_s = tmem + lane_addr + (uint32_t)(b * BKV);
            ok = mbar_wait(s_full + 8 * b, (uint32_t)((j >> 1) & 1), abort_flag, 7);
            if (!ok) break;
            if (idle) {                                             // none of this warp's rows is stored: whatever P they have will do
                mbar_arrive(p_full + 8 * b);
                continue;
            }
            tc_fence_after();
            const int kb = (jt0 + j) * BKV;
            const bool need_mask = kb + BKV - 1 > first_pos || (p.window > 0 && kb <= last_pos - p.window);
            float s[BKV];
#pragma unroll
            for (int c = 0; c < BKV / 32; ++c) tmem_ld32(my_s + (uint32_t)(c * 32), s + c * 32);
            tmem_wait_ld();
            if (need_mask) {
#pragma unroll
                for (int e = 0; e < BKV; ++e) s[e] = kb + e <= pos && (p.window <= 0 || kb + e > pos - p.window) ? s[e] : -INFINITY;
            }
            float mx4[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
            for (int e = 4; e < BKV; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], s[e]);
            const float m_new = fmaxf(m_used, fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])));
            if (j == 0) {
                if (sunk) l = ex2((m_used - m_new) * p.scale_log2);
                m_used = m_new;
            } else {
                const bool grow = (m_new - m_used) * p.scale_log2 > GROW_LOG2;      // also when m_used is -inf
                if (__any_sync(0xffffffffu, grow)) {
                    // O must hold every product up to tile j - 1 before its rows are rescaled
                    ok = mbar_wait(pv_done + 8 * ((j - 1) & 1), (uint32_t)(((j - 1) >> 1) & 1), abort_flag, 8);
                    if (!ok) break;
                    tc_fence_after();
                    const float alpha = grow ? ex2((m_used - m_new) * p.scale_log2) : 1.f;
                    if (grow) m_used = m_new;
                    l *= alpha;
#pragma unroll 1
                    for (int c = 0; c < pieces; ++c) {
                        float o[32];
                        tmem_ld32(my_o + (uint32_t)(c * 32), o);
                        tmem_wait_ld();
#pragma unroll
                        for (int e = 0; e < 32; ++e) o[e] *= alpha;
                        tmem_st32(my_o + (uint32_t)(c * 32), o);
                    }
                    tmem_wait_st();
                }
            }
            // P over the first 64 columns of S
            const float mb = (m_used == -INFINITY ? 0.f : m_used) * p.scale_log2;
            float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < BKV / 64; ++c) {
                uint32_t packed[32];
#pragma unroll
                for (int e = 0; e < 32; ++e) {
                    const float x = ex2(fmaf(s[c * 64 + 2 * e], p.scale_log2, -mb)), y = ex2(fmaf(s[c * 64 + 2 * e + 1], p.scale_log2, -mb));
                    sum4[e & 1] += x;
                    sum4[2 + (e & 1)] += y;
                    packed[e] = pack2(x, y);
                }
                tmem_st32(my_s + (uint32_t)(c * 32), reinterpret_cast<const float*>(packed));
            }
            l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
            tmem_wait_st();
            tc_fence_before();
            mbar_arrive(p_full + 8 * b);
        }
        if (ok && n > 0) ok = mbar_wait(pv_done + 8 * ((n - 1) & 1), (uint32_t)(((n - 1) >> 1) & 1), abort_flag, 10);
        if (ok && !idle) {
            tc_fence_after();
            const bool partial = decode && p.splits > 1;
            const float inv = partial ? 1.f : (l > 0.f ? 1.f / l : 0.f);
            const int last = min(p.rank, v0 + p.cols);              // the rank is a multiple of 8: an eighth is in or out as a whole
            const size_t line = (size_t)tok0 * p.heads + row0 + row, slot = line * p.splits + range;
            __nv_bfloat16* dst = p.out + line * p.rank;
            float* dst_f = p.part_o + slot * p.rank;
            if (partial && cb == 0 && row < rows_valid) {
                p.part_ml[slot * 2] = m_used * (p.scale_log2 * 0.6931471805599453f);      // natural units of the scaled score
                p.part_ml[slot * 2 + 1] = l;
            }
#pragma unroll 1
            for (int c = 0; c < pieces; ++c) {
                float o[32];
                if (n > 0) {
                    tmem_ld32(my_o + (uint32_t)(c * 32), o);
                    tmem_wait_ld();
                } else {
#pragma unroll
                    for (int e = 0; e < 32; ++e) o[e] = 0.f;        // a range without keys
                }
                if (row < rows_valid) {
#pragma unroll
                    for (int v = 0; v < 4; ++v) {
                        const int col = v0 + c * 32 + v * 8;
                        if (col >= last) continue;
                        if (partial) {
                            *reinterpret_cast<float4*>(dst_f + col) = make_float4(o[v * 8], o[v * 8 + 1], o[v * 8 + 2], o[v * 8 + 3]);
                            *reinterpret_cast<float4*>(dst_f + col + 4) = make_float4(o[v * 8 + 4], o[v * 8 + 5], o[v * 8 + 6], o[v * 8 + 7]);
                        } else {
                            *reinterpret_cast<uint4*>(dst + col) =
                                make_uint4(pack2(o[v * 8] * inv, o[v * 8 + 1] * inv), pack2(o[v * 8 + 2] * inv, o[v * 8 + 3] * inv),
                                           pack2(o[v * 8 + 4] * inv, o[v * 8 + 5] * inv), pack2(o[v * 8 + 6] * inv, o[v * 8 + 7] * inv));
                        }
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(512) : "memory");
    }
}

static int ring_stages(int row) {
    const int rest = (SMEM_LIMIT - TAIL) / STAGE - (row + 63) / 64;
    return rest > MAX_STAGES ? MAX_STAGES : rest;
}

static bool encode(CUtensorMap* map, const void* base, int rank, const cuuint64_t* dims, const cuuint64_t* strides, const cuuint32_t* box) {
    const cuuint32_t elem[3] = {1, 1, 1};
    EncodeTiled enc = encoder();
    return enc && enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), dims, strides, box, elem,
                      CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                      CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace lt
}  // namespace lily

using namespace lily;

// Whether the kernel takes these sizes: rows and ranks of whole 16-byte pieces, rows that leave a ring of four stages and
// more beside the 128 query rows in shared memory, pages of a multiple of 64.
LILY_API int lily_latent_attention_tc_takes(int row, int rank, int page_size) {
    return row > 0 && rank > 0 && rank <= row && row % 8 == 0 && rank % 8 == 0 && rank <= 2 * lt::MAX_COLUMNS && page_size > 0 &&
           page_size % 64 == 0 && lt::ring_stages(row) >= 4;
}

// New tokens a tile holds for this many heads (a block takes 128 of the tile's (token, head) rows).
LILY_API int lily_latent_attention_tc_tile_tokens(int heads) { return heads >= lt::BQ ? 1 : lt::BQ / heads; }

// Column blocks the values of this rank are cut into (each forms the scores for itself).
LILY_API int lily_latent_attention_tc_col_blocks(int rank) { return (rank + lt::MAX_COLUMNS - 1) / lt::MAX_COLUMNS; }

namespace lily {
namespace lt {

// Fills in what both entries share, encodes the tensor maps and launches `units` (tile or request and range) blocks a row and column block.
static int launch(Params& p, long units, const void* q, const void* cache, int tokens, int num_pages, float scale, cudaStream_t stream) {
    LILY_REQUIRE(lily_latent_attention_tc_takes(p.row, p.rank, p.page_size), "latent_attention_tc: rows of %d with rank %d in pages of %d are not for this kernel", p.row, p.rank, p.page_size);
    LILY_REQUIRE(p.heads > 0 && tokens > 0 && num_pages > 0 && scale > 0.f, "latent_attention_tc: heads=%d tokens=%d pages=%d scale=%g", p.heads, tokens, num_pages, scale);
    LILY_REQUIRE(((uintptr_t)q % 16 == 0) && ((uintptr_t)cache % 16 == 0) && ((uintptr_t)p.out % 16 == 0) && ((uintptr_t)p.part_o % 16 == 0),
                 "latent_attention_tc: operands must be 16-byte aligned");
    const int tile_rows = p.tile_tokens * p.heads;
    p.row_blocks = (tile_rows + BQ - 1) / BQ;
    p.chunks = (p.row + 63) / 64;
    p.col_blocks = lily_latent_attention_tc_col_blocks(p.rank);
    p.cols = ((p.rank + p.col_blocks - 1) / p.col_blocks + 15) / 16 * 16;
    p.stages = ring_stages(p.row);
    p.q_rows = tile_rows >= BQ ? BQ : (tile_rows + 7) / 8 * 8;      // rows of a tile past its last are computed on whatever is there
    p.scale_log2 = scale * 1.4426950408889634f;
    CUtensorMap map_q, map_k, map_v;
    {
        const cuuint64_t dims[2] = {(cuuint64_t)p.row, (cuuint64_t)tokens * p.heads}, strides[1] = {(cuuint64_t)p.row * 2};
        const cuuint32_t box[2] = {64, (cuuint32_t)p.q_rows};
        LILY_REQUIRE(encode(&map_q, q, 2, dims, strides, box), "latent_attention_tc: the tensor map of the queries was refused");
    }
    {
        const cuuint64_t dims[3] = {(cuuint64_t)p.row, (cuuint64_t)p.page_size, (cuuint64_t)num_pages};
        const cuuint64_t strides[2] = {(cuuint64_t)p.row * 2, (cuuint64_t)p.page_size * p.row * 2};
        const cuuint32_t box_k[3] = {64, 64, 1}, box_v[3] = {64, (cuuint32_t)VKEYS, 1};
        LILY_REQUIRE(encode(&map_k, cache, 3, dims, strides, box_k) && encode(&map_v, cache, 3, dims, strides, box_v),
                     "latent_attention_tc: the tensor map of the cache was refused");
    }
    const size_t smem = (size_t)(p.chunks + p.stages) * STAGE + TAIL;
    static size_t granted = 0;
    if (smem > granted) {
        cudaError_t e = cudaFuncSetAttribute(latent_attention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { set_error("latent_attention_tc: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e)); return 2; }
        granted = smem;
    }
    const long blocks = units * p.row_blocks * p.col_blocks;
    LILY_REQUIRE(blocks < (1l << 31), "latent_attention_tc: %ld blocks", blocks);
    launch_pdl(latent_attention_tc_kernel, dim3((unsigned)blocks), dim3(THREADS), smem, stream, map_q, map_k, map_v, p);
    LILY_CHECK_LAUNCH("latent_attention_tc");
    return 0;
}

}  // namespace lt
}  // namespace lily

// Prompt portions: `tiles` of `tile_tokens` new tokens (request and offset); q and out have `tokens` rows in all.
LILY_API int lily_latent_attention_prefill_tc(const void* q, const void* cache, void* out, const int* block_table, int bt_stride,
                                              const int* cu_seqlens, const int* prefix_lens, const int* tile_req, const int* tile_start,
                                              int tiles, int tile_tokens, int heads, int row, int rank, int page_size, int window,
                                              float scale, int tokens, int num_pages, const float* sinks, cudaStream_t stream) {
    if (tiles == 0) return 0;
    LILY_REQUIRE(tile_tokens > 0 && (tile_tokens == 1 || tile_tokens * heads <= lt::BQ), "latent_attention_tc: tiles of %d tokens of %d heads", tile_tokens, heads);
    lt::Params p{};
    p.block_table = block_table; p.cu_seqlens = cu_seqlens; p.prefix_lens = prefix_lens; p.tile_req = tile_req; p.tile_start = tile_start;
    p.out = (__nv_bfloat16*)out; p.bt_stride = bt_stride; p.tiles = tiles; p.tile_tokens = tile_tokens; p.heads = heads; p.row = row;
    p.rank = rank; p.page_size = page_size; p.window = window; p.splits = 1; p.sinks = sinks;
    return lt::launch(p, tiles, q, cache, tokens, num_pages, scale, stream);
}

// One new token a request: q [requests, heads, row], out [requests, heads, rank]; with more than one key range the ranges'
// results go to scratch, ahead of lily_attention_combine.
LILY_API int lily_latent_attention_decode_tc(const void* q, const void* cache, void* out, const int* block_table, int bt_stride,
                                             const int* seq_lens, float* scratch, int requests, int splits, int heads, int row, int rank,
                                             int page_size, int window, float scale, int num_pages, const float* sinks, cudaStream_t stream) {
    if (requests == 0) return 0;
    LILY_REQUIRE(seq_lens && splits >= 1 && (splits == 1 || scratch), "latent_attention_tc: %d key ranges need scratch", splits);
    lt::Params p{};
    p.block_table = block_table; p.seq_lens = seq_lens; p.splits = splits; p.out = (__nv_bfloat16*)out; p.bt_stride = bt_stride;
    p.tiles = requests; p.tile_tokens = 1; p.heads = heads; p.row = row; p.rank = rank; p.page_size = page_size; p.window = window; p.sinks = sinks;
    p.part_o = splits > 1 ? scratch : nullptr;
    p.part_ml = splits > 1 ? scratch + (size_t)requests * heads * splits * rank : nullptr;
    return lt::launch(p, (long)requests * splits, q, cache, requests, num_pages, scale, stream);
}

// 0 while no wait has given up since the last call; else (code << 24 | block).  Codes: 1, 2 the loader waiting for a free
// stage; 3 the mma thread waiting for the queries, 4, 6 for a stage, 5 for P; 7 the softmax waiting for scores, 8 and 10 for a
// product into O.  Synchronises the device.  Reading clears it.
LILY_API int lily_latent_attention_tc_status() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, lt::g_status, sizeof(int)) != cudaSuccess) return -1;
    if (v != 0) cudaMemcpyToSymbol(lt::g_status, &zero, sizeof(int));
    return v;
}
