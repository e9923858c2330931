// The matrix-memory recurrence (see mlstm.cu) over long portions in bfloat16: chunks of a portion side by side, their sums as
// matrix products on the tensor cores (mma.sync m16n8k16, float32 accumulation).
//
// Within a chunk that starts from (S_0, n_0, m_0), with b_t the sum of the log forget gates up to and with token t:
//
//     g_t = max_(s <= t) (i_s - b_s),    m_t = b_t + max(m_0, g_t)                        (the running maximum)
//     S_t^T q_t = e^(b_t + m_0 - m_t) S_0^T q_t + sum_(s <= t) e^(b_t - b_s + i_s - m_t) (q_t . k_s) v_s
//     S_end     = e^(b + m_0 - m) S_0 + e^(b + g - m) D,   D = sum_s e^(i_s - b_s - g) k_s v_s^T       (b, g, m of the last token)
//
// and n likewise with v_s = 1.  Four launches:
//   mlstm_chunk_gates    a warp a (chunk, head): i_t, b_t and g_t of every token, b and b + g of the chunk
//   mlstm_chunk_write    D and its vector for n: a block a tile of 64 value columns by 128 keys of a (chunk, head)
//   mlstm_chunk_combine  walks the chunks of a portion in order: leaves each chunk's starting state in the workspace and the last
//                        one in the slot (the slot's m is written by mlstm_out)
//   mlstm_chunk_read     the outputs: a block 64 tokens by 128 value columns of a head
//
// The state, everything that scales it and every sum are float32.  What meets the tensor cores as float32 (a weighted value,
// a decayed score, an entry of the starting state) is cut into the sum of two bfloat16 numbers and multiplied twice, so that
// 16 bits of it count; q, k and v are the projection's own bfloat16 numbers.
#include "common.cuh"
#include "mma.cuh"
#include "operand.cuh"

namespace lily {
namespace mlc {

using namespace mma16;

constexpr int THREADS = 128;
constexpr int TOK = 64;                    // tokens of a tile
constexpr int WV = 64, WD = 128, WT = 128; // value columns, keys and tokens of a turn of a block of the write kernel
constexpr int RV = 128, RD = 64;           // value columns of a block of the read kernel, keys of a staged piece of the state
constexpr int PAD = 8;                     // an odd number of 16-byte pieces a row: ldmatrix without bank conflicts

struct Args {
    const __nv_bfloat16* proj;             // [tokens, ld]
    int ld, q_col, k_col, v_col;
    Operand gates;
    int gates_ld, i_col, f_col;
    const float* i_bias;
    const float* f_bias;
    float cap, q_scale;
    const int* cu_seqlens;
    const int* slots;
    const int* item_req;                   // [items]: chunk -> request, first token in its portion, tokens
    const int* item_start;
    const int* item_len;
    const int* long_req;                   // [longs]: portion -> request, first chunk, chunks
    const int* long_first;
    const int* long_count;
    const int* tile_item;                  // [tiles]: tile of 64 tokens -> chunk, first token in the chunk
    const int* tile_start;
    float* gate_i;                         // [tokens, heads] each
    float* gate_b;
    float* gate_g;
    float* item_b;                         // [items, heads]: b and b + g of the chunk, m it starts from
    float* item_g;
    float* item_m;
    float* wrote;                          // [items, heads, dv + 1, d]: D, then its vector for n
    __nv_bfloat16* start_hi;               // [items, heads, dv, d]: the starting state as a sum of two
    __nv_bfloat16* start_lo;
    float* start_n;                        // [items, heads, d]
    float* state;
    size_t state_stride;
    float* y;                              // [tokens, heads * dv]
    float* nq;                             // [tokens, heads]
    float* m;
    int heads, d, dv;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// grid (chunks, ceil(heads / 4)), block 128: a warp a (chunk, head).
__global__ void __launch_bounds__(THREADS) gates_kernel(const Args a) {
    pdl_enter_small();
    const int item = blockIdx.x, head = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (head >= a.heads) return;
    const int len = a.item_len[item];
    const size_t tok0 = a.cu_seqlens[a.item_req[item]] + a.item_start[item];
    const float bi = a.i_bias[head], bf = a.f_bias[head];
    float b0 = 0.f, g0 = -INFINITY;                              // carried from the 32 tokens before
    for (int t0 = 0; t0 < len; t0 += 32) {
        const bool in = t0 + lane < len;
        const size_t tok = tok0 + (in ? t0 + lane : 0), row = tok * a.gates_ld + head;
        const float i = a.cap * tanhf((a.gates(row + a.i_col) + bi) / a.cap);
        float b = in ? log_sigmoid(a.cap * tanhf((a.gates(row + a.f_col) + bf) / a.cap)) : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float left = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) b += left;
        }
        b += b0;
        float g = in ? i - b : -INFINITY;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float left = __shfl_up_sync(0xffffffffu, g, o);
            if (lane >= o) g = fmaxf(g, left);
        }
        g = fmaxf(g, g0);
        if (in) {
            a.gate_i[tok * a.heads + head] = i;
            a.gate_b[tok * a.heads + head] = b;
            a.gate_g[tok * a.heads + head] = g;
        }
        b0 = __shfl_sync(0xffffffffu, b, 31);
        g0 = __shfl_sync(0xffffffffu, g, 31);
    }
    if (lane == 0) {
        a.item_b[(size_t)item * a.heads + head] = b0;
        a.item_g[(size_t)item * a.heads + head] = g0;
    }
}

// Rows [0, rows) of `cols` bfloat16 from `src` (rows `ld` apart) into rows `stride` apart in shared memory, 16 bytes a copy; what
// lies outside is zero.  cols is a multiple of 8; `have` columns exist.
__device__ __forceinline__ void stage_rows(__nv_bfloat16* dst, int stride, const __nv_bfloat16* src, size_t ld, int rows, int total_rows,
                                           int cols, int have) {
    const int per = cols / 8;
    for (int e = threadIdx.x; e < total_rows * per; e += THREADS) {
        const int r = e / per, c = (e % per) * 8;
        const bool in = r < rows && c < have;
        cp_async16(smem_u32(dst + r * stride + c), src + (in ? (size_t)r * ld + c : 0), in);
    }
}

// grid (chunks, heads, ceil(dv / WV) * ceil(d / WD)), block 128: warp w has the 16 value columns w of the block's 64.  WT tokens at a
// time: a chunk of the usual length is one turn, whose loads are all in flight together.
struct WriteTile {
    __nv_bfloat16 k[WT][WD + PAD], vh[WT][WV + PAD], vl[WT][WV + PAD];
    float w[WT];
};

__global__ void __launch_bounds__(THREADS) write_kernel(const Args a) {
    extern __shared__ __align__(16) unsigned char smem[];
    WriteTile& s = *reinterpret_cast<WriteTile*>(smem);
    pdl_wait();
    pdl_launch_dependents();
    const int item = blockIdx.x, head = blockIdx.y, dtiles = (a.d + WD - 1) / WD;
    const int v0 = (int)blockIdx.z / dtiles * WV, d0 = (int)blockIdx.z % dtiles * WD;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
    const int len = a.item_len[item];
    const size_t tok0 = a.cu_seqlens[a.item_req[item]] + a.item_start[item];
    const float gmax = a.item_g[(size_t)item * a.heads + head];
    float acc[WD / 8][4];
#pragma unroll
    for (int j = 0; j < WD / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    float n_sum = 0.f;
    static_assert(WT == THREADS, "a thread a token's weight");
    constexpr int VPER = WT * (WV / 8) / THREADS;                // 16-byte pieces of values a thread scales
    for (int t0 = 0; t0 < len; t0 += WT) {
        const int n = min(WT, len - t0);
        __syncthreads();
        stage_rows(&s.k[0][0], WD + PAD, a.proj + (tok0 + t0) * a.ld + a.k_col + (size_t)head * a.d + d0, a.ld, n, WT, WD, a.d - d0);
        cp_async_commit();
        const __nv_bfloat16* vsrc = a.proj + (tok0 + t0) * a.ld + a.v_col + (size_t)head * a.dv + v0;
        uint4 raw[VPER];
#pragma unroll
        for (int k = 0; k < VPER; ++k) {
            const int e = k * THREADS + tid, t = e / (WV / 8), col = (e % (WV / 8)) * 8;
            raw[k] = t < n && v0 + col < a.dv ? *reinterpret_cast<const uint4*>(vsrc + (size_t)t * a.ld + col) : make_uint4(0, 0, 0, 0);
        }
        {
            const size_t at = (tok0 + t0 + (tid < n ? tid : 0)) * a.heads + head;
            s.w[tid] = tid < n ? expf(a.gate_i[at] - a.gate_b[at] - gmax) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < VPER; ++k) {
            const int e = k * THREADS + tid, t = e / (WV / 8), col = (e % (WV / 8)) * 8;
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw[k]);
            uint4 hi, lo;
            const float w = s.w[t];
            const float2 f0 = __bfloat1622float2(p[0]), f1 = __bfloat1622float2(p[1]), f2 = __bfloat1622float2(p[2]), f3 = __bfloat1622float2(p[3]);
            split2(f0.x * w, f0.y * w, hi.x, lo.x);
            split2(f1.x * w, f1.y * w, hi.y, lo.y);
            split2(f2.x * w, f2.y * w, hi.z, lo.z);
            split2(f3.x * w, f3.y * w, hi.w, lo.w);
            *reinterpret_cast<uint4*>(&s.vh[t][col]) = hi;
            *reinterpret_cast<uint4*>(&s.vl[t][col]) = lo;
        }
        cp_async_wait<0>();
        __syncthreads();
        if (v0 == 0)
            for (int t = 0; t < n; ++t) n_sum = fmaf(s.w[t], __bfloat162float(s.k[t][tid]), n_sum);
        const int steps = (n + 15) / 16;
        for (int k16 = 0; k16 < steps; ++k16) {
            uint32_t ah[4], al[4];
            const int ar = k16 * 16 + (lane & 7) + ((lane >> 4) << 3), ac = warp * 16 + (((lane >> 3) & 1) << 3);
            ldmatrix_x4_trans(smem_u32(&s.vh[ar][ac]), ah[0], ah[1], ah[2], ah[3]);
            ldmatrix_x4_trans(smem_u32(&s.vl[ar][ac]), al[0], al[1], al[2], al[3]);
            // the two parts of a sum are a run of products apart, so that no product waits for the one before it
#pragma unroll
            for (int half = 0; half < WD / 64; ++half) {
                uint32_t b[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    ldmatrix_x4_trans(smem_u32(&s.k[k16 * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)][half * 64 + u * 16 + ((lane >> 4) << 3)]),
                                      b[u][0], b[u][1], b[u][2], b[u][3]);
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    mma_bf16(acc[half * 8 + 2 * u], ah, b[u][0], b[u][1]);
                    mma_bf16(acc[half * 8 + 2 * u + 1], ah, b[u][2], b[u][3]);
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    mma_bf16(acc[half * 8 + 2 * u], al, b[u][0], b[u][1]);
                    mma_bf16(acc[half * 8 + 2 * u + 1], al, b[u][2], b[u][3]);
                }
            }
        }
    }
    float* dst = a.wrote + ((size_t)item * a.heads + head) * (a.dv + 1) * a.d;
    const int r_lo = v0 + warp * 16 + g, r_hi = r_lo + 8;
#pragma unroll
    for (int j = 0; j < WD / 8; ++j) {
        const int col = d0 + j * 8 + 2 * c;
        if (col >= a.d) continue;
        if (r_lo < a.dv) *reinterpret_cast<float2*>(dst + (size_t)r_lo * a.d + col) = make_float2(acc[j][0], acc[j][1]);
        if (r_hi < a.dv) *reinterpret_cast<float2*>(dst + (size_t)r_hi * a.d + col) = make_float2(acc[j][2], acc[j][3]);
    }
    if (v0 == 0 && d0 + tid < a.d) dst[(size_t)a.dv * a.d + d0 + tid] = n_sum;
}

// grid (ceil((dv + 1) d / 1024), heads, portions), block 256: a thread walks four neighbouring entries of a head's state.
__global__ void __launch_bounds__(256) combine_kernel(const Args a) {
    pdl_wait();
    pdl_launch_dependents();
    const int head = blockIdx.y, which = blockIdx.z, per = (a.dv + 1) * a.d;
    const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
    if (e >= per) return;
    float* slot = a.state + (size_t)a.slots[a.long_req[which]] * a.state_stride;
    float* st = slot + (size_t)head * per + e;
    float m = slot[(size_t)a.heads * per + head];
    float4 S = *reinterpret_cast<const float4*>(st);
    const int first = a.long_first[which], count = a.long_count[which];
    const bool vector = e >= a.dv * a.d;
    for (int c0 = 0; c0 < count; c0 += 4) {                          // four chunks' numbers asked for before the first is used
        float4 add[4];
        float bs[4], gs[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const size_t at = (size_t)(first + (c0 + j < count ? c0 + j : c0)) * a.heads + head;
            add[j] = *reinterpret_cast<const float4*>(a.wrote + at * per + e);
            bs[j] = a.item_b[at];
            gs[j] = a.item_g[at];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (c0 + j >= count) break;
            const size_t at = (size_t)(first + c0 + j) * a.heads + head;
            if (vector) {
                *reinterpret_cast<float4*>(a.start_n + at * a.d + (e - a.dv * a.d)) = S;
                if (e == a.dv * a.d) a.item_m[at] = m;
            } else {
                uint2 hi, lo;
                split2(S.x, S.y, hi.x, lo.x);
                split2(S.z, S.w, hi.y, lo.y);
                const size_t to = at * ((size_t)a.dv * a.d) + e;
                *reinterpret_cast<uint2*>(a.start_hi + to) = hi;
                *reinterpret_cast<uint2*>(a.start_lo + to) = lo;
            }
            const float next = bs[j] + fmaxf(m, gs[j]), keep = expf(bs[j] + m - next), put = expf(bs[j] + gs[j] - next);
            S.x = fmaf(keep, S.x, put * add[j].x);
            S.y = fmaf(keep, S.y, put * add[j].y);
            S.z = fmaf(keep, S.z, put * add[j].z);
            S.w = fmaf(keep, S.w, put * add[j].w);
            m = next;
        }
    }
    *reinterpret_cast<float4*>(st) = S;
}

// grid (tiles of 64 tokens, heads, ceil(dv / RV)), block 128: warp w has the tokens 16 w ... of the tile.  Shared memory: queries
// [64][d + PAD], then either pieces of the starting state (two stages of two of [RV][RD + PAD]) or keys [64][d + PAD] and values [64][RV + PAD].
__global__ void __launch_bounds__(THREADS) read_kernel(const Args a) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float row_b[TOK], row_m[TOK], key_s[TOK];
    pdl_wait();
    pdl_launch_dependents();
    const int d = a.d, dv = a.dv, qstride = d + PAD;
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* rest = q_s + TOK * qstride;
    __nv_bfloat16 *k_s = rest, *v_s = rest + TOK * qstride;
    const int tile = gridDim.x - 1 - blockIdx.x;                     // the last tiles of a chunk, which see the most keys, go first
    const int item = a.tile_item[tile], start = a.tile_start[tile], head = blockIdx.y, v0 = blockIdx.z * RV;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
    const int n = min(TOK, a.item_len[item] - start);
    const size_t tok0 = (size_t)a.cu_seqlens[a.item_req[item]] + a.item_start[item];       // the chunk's first token
    const size_t at = (size_t)item * a.heads + head;
    const float m0 = a.item_m[at];

    stage_rows(q_s, qstride, a.proj + (tok0 + start) * a.ld + a.q_col + (size_t)head * d, a.ld, n, TOK, d, d);
    cp_async_commit();
    if (tid < TOK) {
        const size_t row = (tok0 + start + (tid < n ? tid : 0)) * a.heads + head;
        row_b[tid] = a.gate_b[row];
        row_m[tid] = a.gate_b[row] + fmaxf(m0, a.gate_g[row]);
    }
    float o[RV / 8][4];
#pragma unroll
    for (int j = 0; j < RV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

    // ---- what the starting state answers
    const __nv_bfloat16* qrow = q_s + (warp * 16 + (lane & 15)) * qstride + ((lane >> 4) << 3);
    auto ask_piece = [&](int k) {                                    // the keys [k RD, (k + 1) RD) of the starting state, stage k % 2
        const size_t from = (at * dv + v0) * d + k * RD;
        __nv_bfloat16* to = rest + (k & 1) * 2 * RV * (RD + PAD);
        stage_rows(to, RD + PAD, a.start_hi + from, d, dv - v0, RV, RD, d - k * RD);
        stage_rows(to + RV * (RD + PAD), RD + PAD, a.start_lo + from, d, dv - v0, RV, RD, d - k * RD);
        cp_async_commit();
    };
    const int pieces = (d + RD - 1) / RD;
    ask_piece(0);
    for (int k = 0; k < pieces; ++k) {
        if (k + 1 < pieces) {
            ask_piece(k + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();                                             // piece k (and the queries) have landed
        const __nv_bfloat16 *hi_s = rest + (k & 1) * 2 * RV * (RD + PAD), *lo_s = hi_s + RV * (RD + PAD);
        const int d0 = k * RD, steps = min(RD, d - d0) / 16;
        for (int kk = 0; kk < steps; ++kk) {
            uint32_t q[4];
            ldmatrix_x4(smem_u32(qrow + d0 + kk * 16), q[0], q[1], q[2], q[3]);
            const int br = (lane & 7) + ((lane >> 4) << 3), bc = kk * 16 + (((lane >> 3) & 1) << 3);
            // the two parts of a sum are a run of products apart, so that no product waits for the one before it
#pragma unroll
            for (int part = 0; part < 4; ++part) {
                const __nv_bfloat16* from = (part & 1 ? lo_s : hi_s) + ((part >> 1) * 64 + br) * (RD + PAD) + bc;
                uint32_t b[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u) ldmatrix_x4(smem_u32(from + u * 16 * (RD + PAD)), b[u][0], b[u][1], b[u][2], b[u][3]);
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    mma_bf16(o[(part >> 1) * 8 + 2 * u], q, b[u][0], b[u][1]);
                    mma_bf16(o[(part >> 1) * 8 + 2 * u + 1], q, b[u][2], b[u][3]);
                }
            }
        }
        __syncthreads();                                             // everyone is done with its stage
    }
    const int r_lo = warp * 16 + g, r_hi = r_lo + 8;
    const float b_lo = row_b[r_lo], b_hi = row_b[r_hi], m_lo = row_m[r_lo], m_hi = row_m[r_hi];
    const float f_lo = a.q_scale * expf(b_lo + m0 - m_lo), f_hi = a.q_scale * expf(b_hi + m0 - m_hi);
#pragma unroll
    for (int j = 0; j < RV / 8; ++j) {
        o[j][0] *= f_lo;
        o[j][1] *= f_lo;
        o[j][2] *= f_hi;
        o[j][3] *= f_hi;
    }
    // n . q of this warp's rows over the starting vector: four lanes a row, as the products' rows lie
    float n_lo = 0.f, n_hi = 0.f;
    if (v0 == 0) {
        const float* n0 = a.start_n + at * d;
        for (int i = c; i < d; i += 4) {
            const float x = n0[i];
            n_lo = fmaf(x, __bfloat162float(q_s[r_lo * qstride + i]), n_lo);
            n_hi = fmaf(x, __bfloat162float(q_s[r_hi * qstride + i]), n_hi);
        }
        n_lo *= f_lo;
        n_hi *= f_hi;
    }

    // ---- what the chunk's own tokens answer
    for (int k0 = 0; k0 <= start; k0 += TOK) {
        const int nk = min(TOK, a.item_len[item] - k0);
        __syncthreads();
        stage_rows(k_s, qstride, a.proj + (tok0 + k0) * a.ld + a.k_col + (size_t)head * d, a.ld, nk, TOK, d, d);
        cp_async_commit();
        stage_rows(v_s, RV + PAD, a.proj + (tok0 + k0) * a.ld + a.v_col + (size_t)head * dv + v0, a.ld, nk, TOK, RV, dv - v0);
        cp_async_commit();
        if (tid < TOK) {
            const size_t row = (tok0 + k0 + (tid < nk ? tid : 0)) * a.heads + head;
            key_s[tid] = a.gate_i[row] - a.gate_b[row];
        }
        cp_async_wait<1>();
        __syncthreads();
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        for (int kk = 0; kk < d / 16; ++kk) {
            uint32_t q[4];
            ldmatrix_x4(smem_u32(qrow + kk * 16), q[0], q[1], q[2], q[3]);
#pragma unroll
            for (int jp = 0; jp < 4; ++jp) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(smem_u32(k_s + (jp * 16 + (lane & 7) + ((lane >> 4) << 3)) * qstride + kk * 16 + (((lane >> 3) & 1) << 3)), b0, b1, b2, b3);
                mma_bf16(s[2 * jp], q, b0, b1);
                mma_bf16(s[2 * jp + 1], q, b2, b3);
            }
        }
        const bool diagonal = k0 == start;
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = j * 8 + 2 * c + (e & 1), row = e < 2 ? r_lo : r_hi;
                const bool seen = !diagonal || key <= row;
                const float w = seen ? a.q_scale * expf((e < 2 ? b_lo - m_lo : b_hi - m_hi) + key_s[key]) : 0.f;
                s[j][e] *= w;
                if (e < 2) n_lo += s[j][e]; else n_hi += s[j][e];
            }
        cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int k16 = 0; k16 < TOK / 16; ++k16) {
            uint32_t ph[4], pl[4];
            split2(s[2 * k16][0], s[2 * k16][1], ph[0], pl[0]);
            split2(s[2 * k16][2], s[2 * k16][3], ph[1], pl[1]);
            split2(s[2 * k16 + 1][0], s[2 * k16 + 1][1], ph[2], pl[2]);
            split2(s[2 * k16 + 1][2], s[2 * k16 + 1][3], ph[3], pl[3]);
            const int vr = k16 * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int half = 0; half < RV / 64; ++half) {
                uint32_t b[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    ldmatrix_x4_trans(smem_u32(v_s + vr * (RV + PAD) + half * 64 + u * 16 + ((lane >> 4) << 3)), b[u][0], b[u][1], b[u][2], b[u][3]);
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    mma_bf16(o[half * 8 + 2 * u], ph, b[u][0], b[u][1]);
                    mma_bf16(o[half * 8 + 2 * u + 1], ph, b[u][2], b[u][3]);
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    mma_bf16(o[half * 8 + 2 * u], pl, b[u][0], b[u][1]);
                    mma_bf16(o[half * 8 + 2 * u + 1], pl, b[u][2], b[u][3]);
                }
            }
        }
    }

    // ---- results
    float* dst_lo = a.y + ((tok0 + start + r_lo) * a.heads + head) * dv;
    float* dst_hi = a.y + ((tok0 + start + r_hi) * a.heads + head) * dv;
#pragma unroll
    for (int j = 0; j < RV / 8; ++j) {
        const int col = v0 + j * 8 + 2 * c;
        if (col >= dv) continue;
        if (r_lo < n) *reinterpret_cast<float2*>(dst_lo + col) = make_float2(o[j][0], o[j][1]);
        if (r_hi < n) *reinterpret_cast<float2*>(dst_hi + col) = make_float2(o[j][2], o[j][3]);
    }
    if (v0 == 0) {
        n_lo += __shfl_xor_sync(0xffffffffu, n_lo, 1);
        n_lo += __shfl_xor_sync(0xffffffffu, n_lo, 2);
        n_hi += __shfl_xor_sync(0xffffffffu, n_hi, 1);
        n_hi += __shfl_xor_sync(0xffffffffu, n_hi, 2);
        if (c == 0) {
            const size_t lo = (tok0 + start + r_lo) * a.heads + head, hi = (tok0 + start + r_hi) * a.heads + head;
            if (r_lo < n) { a.nq[lo] = n_lo; a.m[lo] = m_lo; }
            if (r_hi < n) { a.nq[hi] = n_hi; a.m[hi] = m_hi; }
        }
    }
}

static size_t read_smem(int d) {
    const size_t q = (size_t)TOK * (d + PAD), pieces = 4 * (size_t)RV * (RD + PAD), tiles = (size_t)TOK * (d + PAD) + (size_t)TOK * (RV + PAD);
    return sizeof(__nv_bfloat16) * (q + (pieces > tiles ? pieces : tiles));
}

}  // namespace mlc
}  // namespace lily

using namespace lily;

// Whether the chunk kernels take these head sizes (bfloat16 rows whose heads start on 16-byte boundaries).
LILY_API int lily_mlstm_chunk_takes(int d, int dv) {
    return d > 0 && d % 16 == 0 && d <= 512 && dv > 0 && dv % 8 == 0 && mlc::read_smem(d) <= 220 * 1024;
}

// float32 entries of workspace for `items` chunks of `tokens` tokens in all: every piece starts on a 16-byte boundary.
static size_t up4(size_t n) { return (n + 3) / 4 * 4; }

LILY_API size_t lily_mlstm_chunk_floats(int items, int tokens, int heads, int d, int dv) {
    const size_t ih = (size_t)items * heads;
    return 3 * up4((size_t)tokens * heads) + 3 * up4(ih) + up4(ih * (dv + 1) * d) + up4(ih * dv * d) + up4(ih * d);
}

LILY_API int lily_mlstm_chunks(const void* proj, int ld, int q_col, int k_col, int v_col, const void* gates, int gates_dtype, int gates_splits,
                               size_t gates_stride, int gates_ld, int i_col, int f_col, const float* i_bias, const float* f_bias, float cap,
                               float q_scale, float* state, size_t state_stride, float* y, float* nq, float* m, const int* cu_seqlens,
                               const int* slots, const int* item_req, const int* item_start, const int* item_len, int items,
                               const int* long_req, const int* long_first, const int* long_count, int longs, const int* tile_item,
                               const int* tile_start, int tiles, float* workspace, int tokens, int heads, int d, int dv, cudaStream_t stream) {
    if (items == 0) return 0;
    LILY_REQUIRE(lily_mlstm_chunk_takes(d, dv), "mlstm_chunks: heads of %d x %d are not for these kernels", d, dv);
    LILY_REQUIRE(heads > 0 && heads <= 65535 && longs > 0 && longs <= 65535 && tiles > 0, "mlstm_chunks: %d heads, %d portions, %d tiles", heads, longs, tiles);
    LILY_REQUIRE(ld % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 && ((uintptr_t)proj & 15) == 0, "mlstm_chunks: rows of %d are not whole 16-byte pieces", ld);
    LILY_REQUIRE(state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0 && (size_t)heads * (dv + 1) * d + heads <= state_stride, "mlstm_chunks: state rows of %zu", state_stride);
    LILY_REQUIRE(workspace && ((uintptr_t)workspace & 15) == 0, "mlstm_chunks: a workspace is needed");
    LILY_REQUIRE(gates_splits >= 1 && (gates_splits == 1 || gates_dtype == kF32) && cap > 0.f, "mlstm_chunks: gates");
    mlc::Args a{};
    a.proj = (const __nv_bfloat16*)proj; a.ld = ld; a.q_col = q_col; a.k_col = k_col; a.v_col = v_col;
    a.gates = Operand{gates, gates_dtype == kBF16, gates_splits, gates_stride}; a.gates_ld = gates_ld; a.i_col = i_col; a.f_col = f_col;
    a.i_bias = i_bias; a.f_bias = f_bias; a.cap = cap; a.q_scale = q_scale; a.cu_seqlens = cu_seqlens; a.slots = slots;
    a.item_req = item_req; a.item_start = item_start; a.item_len = item_len; a.long_req = long_req; a.long_first = long_first; a.long_count = long_count;
    a.tile_item = tile_item; a.tile_start = tile_start; a.state = state; a.state_stride = state_stride; a.y = y; a.nq = nq; a.m = m;
    a.heads = heads; a.d = d; a.dv = dv;
    const size_t ih = (size_t)items * heads;
    float* at = workspace;
    auto take = [&](size_t n) { float* p = at; at += up4(n); return p; };
    a.gate_i = take((size_t)tokens * heads); a.gate_b = take((size_t)tokens * heads); a.gate_g = take((size_t)tokens * heads);
    a.item_b = take(ih); a.item_g = take(ih); a.item_m = take(ih);
    a.wrote = take(ih * (dv + 1) * d);
    a.start_hi = (__nv_bfloat16*)take(ih * dv * d);
    a.start_lo = a.start_hi + ih * dv * d;
    a.start_n = take(ih * d);
    launch_pdl(mlc::gates_kernel, dim3(items, (heads + 3) / 4), dim3(mlc::THREADS), 0, stream, a);
    LILY_CHECK_LAUNCH("mlstm_chunk_gates");
    const int wz = (dv + mlc::WV - 1) / mlc::WV * ((d + mlc::WD - 1) / mlc::WD);
    static bool room = false;
    if (!room) {
        cudaError_t e = cudaFuncSetAttribute(mlc::write_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(mlc::WriteTile));
        if (e != cudaSuccess) { set_error("mlstm_chunks: cannot get %zu bytes of shared memory: %s", sizeof(mlc::WriteTile), cudaGetErrorString(e)); return 2; }
        room = true;
    }
    launch_pdl(mlc::write_kernel, dim3(items, heads, wz), dim3(mlc::THREADS), sizeof(mlc::WriteTile), stream, a);
    LILY_CHECK_LAUNCH("mlstm_chunk_write");
    launch_pdl(mlc::combine_kernel, dim3(((dv + 1) * d + 1023) / 1024, heads, longs), dim3(256), 0, stream, a);
    LILY_CHECK_LAUNCH("mlstm_chunk_combine");
    const size_t smem = mlc::read_smem(d);
    static size_t granted = 40 * 1024;
    if (smem > granted) {
        cudaError_t e = cudaFuncSetAttribute(mlc::read_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { set_error("mlstm_chunks: cannot get %zu bytes of shared memory: %s", smem, cudaGetErrorString(e)); return 2; }
        granted = smem;
    }
    launch_pdl(mlc::read_kernel, dim3(tiles, heads, (dv + mlc::RV - 1) / mlc::RV), dim3(mlc::THREADS), smem, stream, a);
    LILY_CHECK_LAUNCH("mlstm_chunk_read");
    return 0;
}
