// A routed mixture of small feed-forward layers: router, grouping of the (token, choice) pairs by expert, the two
// grouped products, and the weighted sum.  Everything stays on the device (no count is read by the host), so a step
// can be captured in a CUDA graph.
//
//   route     z = W_router h (float32); s = softmax(z) over all router outputs, or sigmoid(z) one by one; the `top`
//             largest s (+ correction) are chosen; their weights are s, or s / (sum of the chosen s + 1e-20).  One more
//             row of the matrix may follow the outputs': the sigmoid of its product is the token's gate for a shared expert.
//             With groups (equal runs of neighbouring outputs) only outputs of the `keep` best groups can be chosen; a
//             group's score is the sum of its two largest choice scores
//   align     pairs (token, choice) whose expert has weights are grouped by expert: offsets, the pairs in grouped
//             order, each pair's place there, and the list of (expert, first row) tiles the products run over
//   gate/up   a[row, n] = g sigmoid(alpha g) (u + 1), g = min(W_gate x, limit), u = clamp(W_up x, -limit, limit), or
//             silu(g) u with g = W_gate x, u = W_up x; a weight that belongs to the expert's input multiplies g and u
//             ahead of the activation (both are linear in x).  An ungated expert has W_up alone: a = max(W_up x, 0)^2
//   down      y[row, :] = W_down a[row, :]                                  (float32)
//   combine   out[t] = sum over the token's choices of weight * (y of the pair, or the token's input itself where the
//             chosen router output is one of the last `identity` ones, which have no weights); without the weight where
//             it went into the input; plus gate * the shared expert's output where there is one
//
// Each output number of the products is summed over k in a fixed order, so a pair's result does not depend on what
// else is in the batch.  Router, softmax and the weighted sum are float32.
#include "common.cuh"
#include "operand.cuh"

namespace lily {

constexpr int ROUTE_MAX = 1024;       // router outputs
constexpr int ROUTE_TOP_MAX = 64;
constexpr int ROUTE_GROUPS_MAX = 128;

// Groups of router outputs: `count` equal runs of neighbours (0: none), of which the `keep` best can be chosen from.
struct RouteGroups {
    int count, keep;
};

// The two largest of a set, kept while numbers come in.
struct BestTwo {
    float first = -INFINITY, second = -INFINITY;
    __device__ __forceinline__ void add(float v) {
        if (v > first) { second = first; first = v; }
        else if (v > second) second = v;
    }
    // a set of one number scores that number
    __device__ __forceinline__ float sum() const { return second > -INFINITY ? first + second : first; }
};

// Scores and choice of token t by one warp.  s: the token's logits in shared memory (overwritten), `outputs` of them and, with
// `gate`, the shared gate's behind them; picked: room for `top` numbers.
__device__ __forceinline__ void choose_experts(float* s, int t, int outputs, const float* __restrict__ correction, int top, int sigmoid,
                                               int renormalise, RouteGroups groups, float* picked, int* __restrict__ chosen,
                                               float* __restrict__ weights, float* __restrict__ gate) {
    const int lane = threadIdx.x & 31, rows = outputs + (gate ? 1 : 0);
    float inv = 1.f;
    if (sigmoid) {
        for (int e = lane; e < rows; e += 32) {
            const float p = 1.f / (1.f + expf(-s[e]));
            s[e] = p;
            if (e == outputs) gate[t] = p;
        }
    } else {
        float mx = -INFINITY;
        for (int e = lane; e < outputs; e += 32) mx = fmaxf(mx, s[e]);
        mx = warp_max(mx);
        float sum = 0.f;
        for (int e = lane; e < outputs; e += 32) {
            const float p = expf(s[e] - mx);
            s[e] = p;
            sum += p;
        }
        sum = warp_sum(sum);
        inv = 1.f / sum;
        if (gate && lane == 0) gate[t] = 1.f / (1.f + expf(-s[outputs]));
    }
    __syncwarp();
    if (groups.count > 1) {
        // a lane a group and turn: its score, then its place among the groups (ties: the earlier one); the outputs of the
        // groups that are not kept are marked as taken
        const int size = outputs / groups.count;
        float score[ROUTE_GROUPS_MAX / 32];
#pragma unroll
        for (int r = 0; r < ROUTE_GROUPS_MAX / 32; ++r) {
            const int g = lane + 32 * r;
            score[r] = -INFINITY;
            if (g < groups.count) {
                BestTwo two;
                for (int e = g * size; e < (g + 1) * size; ++e) two.add(correction ? s[e] * inv + correction[e] : s[e] * inv);
                score[r] = two.sum();
            }
        }
        int ahead[ROUTE_GROUPS_MAX / 32] = {};
#pragma unroll
        for (int r = 0; r < ROUTE_GROUPS_MAX / 32; ++r) {
            if (32 * r >= groups.count) break;
            for (int l = 0; l < 32; ++l) {
                const float other = __shfl_sync(0xffffffffu, score[r], l);
                const int og = 32 * r + l;
                if (og >= groups.count) continue;
#pragma unroll
                for (int q = 0; q < ROUTE_GROUPS_MAX / 32; ++q)
                    ahead[q] += other > score[q] || (other == score[q] && og < lane + 32 * q);
            }
        }
        __syncwarp();
#pragma unroll
        for (int r = 0; r < ROUTE_GROUPS_MAX / 32; ++r) {
            const int g = lane + 32 * r;
            if (g < groups.count && ahead[r] >= groups.keep)
                for (int e = g * size; e < (g + 1) * size; ++e) s[e] = -1.f;
        }
        __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int at = outputs;
        for (int e = lane; e < outputs; e += 32) {
            const float p = s[e];
            if (p < 0.f) continue;                                // taken already, or in a group that is not kept
            const float c = correction ? p * inv + correction[e] : p * inv;
            if (c > best) { best = c; at = e; }
        }
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
        }
        if (at >= outputs) at = 0;                                // cannot happen while top <= outputs
        const float p = s[at] * inv;
        total += p;
        __syncwarp();
        if (lane == 0) {
            chosen[(size_t)t * top + k] = at;
            picked[k] = p;
            s[at] = -1.f;
        }
        __syncwarp();
    }
    const float norm = renormalise ? 1.f / (total + 1e-20f) : 1.f;
    for (int k = lane; k < top; k += 32) weights[(size_t)t * top + k] = picked[k] * norm;
    __syncwarp();
}

// The choice from logits that a product has left (finished rows or partial sums).  grid (ceil(tokens / 4)), block 128: a
// warp a token.
__global__ void moe_choose_kernel(const Operand logits, int ld, int tokens, const float* __restrict__ correction, int outputs, int top, int sigmoid,
                                  int renormalise, const RouteGroups groups, int* __restrict__ chosen, float* __restrict__ weights, float* __restrict__ gate) {
    __shared__ float picked[4][ROUTE_TOP_MAX];
    extern __shared__ __align__(16) float dyn[];             // [4][rows]
    pdl_enter_small();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp, rows = outputs + (gate ? 1 : 0);
    if (t >= tokens) return;
    float* s = dyn + warp * rows;
    for (int e = lane; e < rows; e += 32) s[e] = logits((size_t)t * ld + e);
    __syncwarp();
    choose_experts(s, t, outputs, correction, top, sigmoid, renormalise, groups, picked[warp], chosen, weights, gate);
}

// grid (ceil(tokens / TB)), block 128: a block takes TB tokens, so a number of the router matrix read once serves TB
// sums (one token a block rereads the matrix from L2 for every token: 50 us for 2,048 tokens of 2,048 columns).
// A token's logits are summed in the same order whatever TB is.
template <typename T, int TB>
__global__ void moe_route_kernel(const T* __restrict__ h, int tokens, int width, const float* __restrict__ router,
                                 const float* __restrict__ correction, int outputs, int top, int sigmoid, int renormalise,
                                 const RouteGroups groups, int* __restrict__ chosen, float* __restrict__ weights, float* __restrict__ gate) {
    __shared__ float picked[4][ROUTE_TOP_MAX];
    extern __shared__ __align__(16) float dyn[];             // [TB][width] the tokens' rows, then [TB][rows of the matrix] their scores
    const int rows = outputs + (gate ? 1 : 0);
    float* xs = dyn;
    float* sc = dyn + (size_t)TB * width;
    pdl_enter_small();
    const int t0 = blockIdx.x * TB, nt = min(TB, tokens - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    // the tokens' rows into shared memory as float32, 16 bytes a load where the rows allow (a plain loop of single
    // numbers waits for memory a hundred times over)
    const T* src = h + (size_t)t0 * width;
    constexpr int PER = 16 / (int)sizeof(T);
    if (width % PER == 0 && ((uintptr_t)h & 15) == 0) {
        for (int i = threadIdx.x * PER; i < TB * width; i += blockDim.x * PER) {
            float v[PER];
            if (i < nt * width) {
                const uint4 raw = *reinterpret_cast<const uint4*>(src + i);
                const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int u = 0; u < PER; ++u) v[u] = to_float(e[u]);
            } else {
#pragma unroll
                for (int u = 0; u < PER; ++u) v[u] = 0.f;
            }
#pragma unroll
            for (int u = 0; u < PER; u += 4) *reinterpret_cast<float4*>(xs + i + u) = make_float4(v[u], v[u + 1], v[u + 2], v[u + 3]);
        }
    } else {
        for (int i = threadIdx.x; i < TB * width; i += blockDim.x) xs[i] = i < nt * width ? to_float(src[i]) : 0.f;
    }
    __syncthreads();
    for (int e = warp; e < rows; e += nwarp) {
        const float* w = router + (size_t)e * width;
        float z[TB];
#pragma unroll
        for (int j = 0; j < TB; ++j) z[j] = 0.f;
        if ((width & 3) == 0) {
            // four columns a lane and turn, four turns' numbers of the matrix asked for ahead of their sums
            int c = lane * 4;
            for (; c + 3 * 128 < width; c += 4 * 128) {
                float4 wv[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) wv[u] = *reinterpret_cast<const float4*>(w + c + u * 128);
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int j = 0; j < TB; ++j) {
                        const float4 x0 = *reinterpret_cast<const float4*>(xs + j * width + c + u * 128);
                        z[j] = fmaf(x0.x, wv[u].x, fmaf(x0.y, wv[u].y, fmaf(x0.z, wv[u].z, fmaf(x0.w, wv[u].w, z[j]))));
                    }
                }
            }
            for (; c < width; c += 128) {
                const float4 w0 = *reinterpret_cast<const float4*>(w + c);
#pragma unroll
                for (int j = 0; j < TB; ++j) {
                    const float4 x0 = *reinterpret_cast<const float4*>(xs + j * width + c);
                    z[j] = fmaf(x0.x, w0.x, fmaf(x0.y, w0.y, fmaf(x0.z, w0.z, fmaf(x0.w, w0.w, z[j]))));
                }
            }
        } else {
            for (int c = lane; c < width; c += 32) {
                const float wv = w[c];
#pragma unroll
                for (int j = 0; j < TB; ++j) z[j] = fmaf(xs[j * width + c], wv, z[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < TB; ++j) {
            const float total = warp_sum(z[j]);
            if (lane == 0) sc[j * rows + e] = total;
        }
    }
    __syncthreads();
    for (int j = warp; j < nt; j += nwarp)
        choose_experts(sc + j * rows, t0 + j, outputs, correction, top, sigmoid, renormalise, groups, picked[warp], chosen, weights, gate);
}

// One block of 1024 threads.  chosen [pairs]; experts: router outputs that have weights (the rest are skipped here).
// offsets [experts + 1], order [pairs] (pairs grouped by expert; entries beyond offsets[experts] are unused),
// place [pairs] (where the pair stands in `order`, -1 without weights), tiles: tile_expert / tile_row [max_tiles]
// (first row of the tile in `order`), tile_count [1].
__global__ void moe_align_kernel(const int* __restrict__ chosen, int pairs, int experts, int rows_per_tile,
                                 int* __restrict__ offsets, int* __restrict__ order, int* __restrict__ place,
                                 int* __restrict__ tile_expert, int* __restrict__ tile_row, int* __restrict__ tile_count,
                                 int max_tiles) {
    extern __shared__ int sh[];            // counts [experts], cursor [experts], start [experts + 1]
    int* counts = sh;
    int* cursor = sh + experts;
    int* start = sh + 2 * experts;
    pdl_enter_small();
    for (int e = threadIdx.x; e < experts; e += blockDim.x) { counts[e] = 0; cursor[e] = 0; }
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int e = chosen[p];
        if (e < experts) atomicAdd(&counts[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int run = 0, tiles = 0;
        for (int e = 0; e < experts; ++e) {
            start[e] = run;
            offsets[e] = run;
            for (int r = 0; r < counts[e] && tiles < max_tiles; r += rows_per_tile) {
                tile_expert[tiles] = e;
                tile_row[tiles] = run + r;
                ++tiles;
            }
            run += counts[e];
        }
        start[experts] = run;
        offsets[experts] = run;
        tile_count[0] = tiles;
    }
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int e = chosen[p];
        if (e < experts) {
            const int at = start[e] + atomicAdd(&cursor[e], 1);
            order[at] = p;
            place[p] = at;
        } else {
            place[p] = -1;
        }
    }
}

// The grouped products.  grid (ceil(N / BN), max_tiles), block 256: tile `blockIdx.y` of the list holds up to BM rows
// of one expert.  MODE 0: A rows are the tokens of the pairs (pair / top), W = [gate rows | up rows] of the expert,
// the output is the activation in T.  MODE 1: A rows are the rows of `a` in grouped order, the output float32.  MODE 2: as
// mode 0 for ungated experts, W = the up rows alone.
constexpr int EBM = 32, EBN = 64, EBK = 16;

// act 0: the clamped gate; 1: silu(g) u
__device__ __forceinline__ float expert_gate(int act, float g, float u, float limit, float alpha) {
    if (act == 1) return (g / (1.f + expf(-g))) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return (g / (1.f + expf(-alpha * g))) * (u + 1.f);
}

__device__ __forceinline__ float squared_relu(float z) {
    const float r = fmaxf(z, 0.f);
    return r * r;
}

template <typename T, int MODE>
__global__ void __launch_bounds__(256)
moe_gemm_kernel(const T* __restrict__ A, int lda, const T* __restrict__ W, size_t w_expert, int N, int K,
                const int* __restrict__ offsets, const int* __restrict__ order, int top,
                const int* __restrict__ tile_expert, const int* __restrict__ tile_row, const int* __restrict__ tile_count,
                void* __restrict__ out, int act, float limit, float alpha, const float* __restrict__ in_weight) {
    __shared__ float As[EBK][EBM + 4];
    __shared__ float Ws[MODE == 0 ? 2 : 1][EBK][EBN + 4];
    __shared__ int arow[EBM];
    pdl_wait();
    if ((int)blockIdx.y >= tile_count[0]) return;
    const int e = tile_expert[blockIdx.y], row0 = tile_row[blockIdx.y];
    const int rows = min(EBM, offsets[e + 1] - row0);
    const int n0 = blockIdx.x * EBN;
    const T* We = W + (size_t)e * w_expert;
    if (threadIdx.x < EBM) {
        const int r = threadIdx.x;
        arow[r] = r < rows ? (MODE != 1 ? order[row0 + r] / top : row0 + r) : -1;
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;          // 4 columns, 2 rows a thread
    float acc[2][4] = {}, acc2[2][4] = {};
    for (int k0 = 0; k0 < K; k0 += EBK) {
        // A tile: 32 rows x 16 k = 512 numbers, two a thread; W tile(s): 64 rows x 16 k = 1024, four a thread
        for (int i = threadIdx.x; i < EBM * EBK; i += 256) {
            const int r = i / EBK, kk = i % EBK, src = arow[r];
            As[kk][r] = (src >= 0 && k0 + kk < K) ? to_float(A[(size_t)src * lda + k0 + kk]) : 0.f;
        }
        for (int i = threadIdx.x; i < EBN * EBK; i += 256) {
            const int r = i / EBK, kk = i % EBK, n = n0 + r;
            const bool ok = n < N && k0 + kk < K;
            Ws[0][kk][r] = ok ? to_float(We[(size_t)n * K + k0 + kk]) : 0.f;
            if (MODE == 0) Ws[1][kk][r] = ok ? to_float(We[(size_t)(N + n) * K + k0 + kk]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < EBK; ++kk) {
            float a[2], b[4], b2[4];
#pragma unroll
            for (int i = 0; i < 2; ++i) a[i] = As[kk][ty * 2 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                b[j] = Ws[0][kk][tx * 4 + j];
                if (MODE == 0) b2[j] = Ws[1][kk][tx * 4 + j];
            }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
                    if (MODE == 0) acc2[i][j] = fmaf(a[i], b2[j], acc2[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = ty * 2 + i;
        if (r >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            if (MODE == 0) {
                const float w = in_weight ? in_weight[order[row0 + r]] : 1.f;
                ((T*)out)[(size_t)(row0 + r) * N + n] = from_float<T>(expert_gate(act, w * acc[i][j], w * acc2[i][j], limit, alpha));
            } else if (MODE == 2) {
                const float w = in_weight ? in_weight[order[row0 + r]] : 1.f;
                ((T*)out)[(size_t)(row0 + r) * N + n] = from_float<T>(squared_relu(w * acc[i][j]));
            } else {
                ((float*)out)[(size_t)(row0 + r) * N + n] = acc[i][j];
            }
        }
    }
}

// out[t] = sum over the token's choices of weight * y[place] (the token's input h where the choice has no weights of its
// own), the weights left out where `weights` is null, plus gate[t] * shared[t] where `gate` is given.  y [pairs in
// grouped order, width] in T or float32, out [tokens, width] float32.  grid (tokens, ceil(width / (256 VEC))), block 256.
template <typename Y> __device__ __forceinline__ float4 four_of(const Y* p);
template <> __device__ __forceinline__ float4 four_of<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 four_of<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

template <typename Y, typename T, int VEC>
__global__ void moe_combine_kernel(const Y* __restrict__ y, const T* __restrict__ h, const int* __restrict__ place,
                                   const float* __restrict__ weights, int top, int width, const Operand shared,
                                   const float* __restrict__ gate, float* __restrict__ out) {
    pdl_wait();
    const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= width) return;
    const size_t at_out = (size_t)t * width + c;
    if (VEC == 4) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < top; ++k) {
            const int at = place[(size_t)t * top + k];
            const float w = weights ? weights[(size_t)t * top + k] : 1.f;
            const float4 v = at >= 0 ? four_of<Y>(y + (size_t)at * width + c) : four_of<T>(h + at_out);
            acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
        }
        if (gate) {
            const float g = gate[t];
            const float4 v = shared.four(at_out);
            acc.x = fmaf(g, v.x, acc.x); acc.y = fmaf(g, v.y, acc.y); acc.z = fmaf(g, v.z, acc.z); acc.w = fmaf(g, v.w, acc.w);
        }
        *reinterpret_cast<float4*>(out + at_out) = acc;
    } else {
        float acc = 0.f;
        for (int k = 0; k < top; ++k) {
            const int at = place[(size_t)t * top + k];
            const float w = weights ? weights[(size_t)t * top + k] : 1.f;
            const float v = at >= 0 ? to_float(y[(size_t)at * width + c]) : to_float(h[at_out]);
            acc = fmaf(w, v, acc);
        }
        if (gate) acc = fmaf(gate[t], shared(at_out), acc);
        out[at_out] = acc;
    }
}

// For the library's grouped product (bfloat16, many rows): the pairs' input rows in grouped order, and the activation
// over its gate/up result.  Rows of whole 16-byte pieces (width, ff multiples of 8).  grid (pairs); rows beyond
// offsets[experts] (pairs without weights) are zeroed so that the product reads nothing unwritten.
__global__ void moe_gather_kernel(const __nv_bfloat16* __restrict__ h, int width, const int* __restrict__ offsets, int experts,
                                  const int* __restrict__ order, int top, __nv_bfloat16* __restrict__ out) {
    pdl_wait();
    const int row = blockIdx.x;
    const bool live = row < offsets[experts];
    const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)(live ? order[row] / top : 0) * width);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)row * width);
    for (int c = threadIdx.x; c < width / 8; c += blockDim.x) dst[c] = live ? src[c] : make_uint4(0, 0, 0, 0);
}

// a[row] = max(u[row], 0)^2 with u[row] = the up product (ff), times the pair's weight first where it belongs to the input.
__global__ void moe_relu2_kernel(const __nv_bfloat16* __restrict__ u, int ff, __nv_bfloat16* __restrict__ a, const float* __restrict__ in_weight,
                                 const int* __restrict__ offsets, int experts, const int* __restrict__ order) {
    pdl_wait();
    const size_t row = blockIdx.x;
    const bool live = (int)row < offsets[experts];      // a row of no pair: the next product must not read what was never written
    const float w = live && in_weight ? in_weight[order[row]] : 1.f;
    for (int c = threadIdx.x; c < ff / 8; c += blockDim.x) {
        uint4 v = make_uint4(0, 0, 0, 0);
        if (live) {
            v = reinterpret_cast<const uint4*>(u + row * ff)[c];
            __nv_bfloat162* v2 = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 z = __bfloat1622float2(v2[k]);
                v2[k] = __floats2bfloat162_rn(squared_relu(w * z.x), squared_relu(w * z.y));
            }
        }
        reinterpret_cast<uint4*>(a + row * ff)[c] = v;
    }
}

// a[row] = gate(gu[row]) with gu[row] = [gate (ff) | up (ff)], both times the pair's weight first where it belongs to the input.
__global__ void moe_activation_kernel(const __nv_bfloat16* __restrict__ gu, int ff, __nv_bfloat16* __restrict__ a, int act, float limit,
                                      float alpha, const float* __restrict__ in_weight, const int* __restrict__ offsets,
                                      int experts, const int* __restrict__ order) {
    pdl_wait();
    const size_t row = blockIdx.x;
    if ((int)row >= offsets[experts]) {                // a row of no pair: the next product must not read what was never written
        for (int c = threadIdx.x; c < ff / 8; c += blockDim.x) reinterpret_cast<uint4*>(a + row * ff)[c] = make_uint4(0, 0, 0, 0);
        return;
    }
    const float w = in_weight ? in_weight[order[row]] : 1.f;
    const uint4* gs = reinterpret_cast<const uint4*>(gu + row * 2 * ff);
    const uint4* us = reinterpret_cast<const uint4*>(gu + row * 2 * ff + ff);
    for (int c = threadIdx.x; c < ff / 8; c += blockDim.x) {
        uint4 g4 = gs[c];
        const uint4 u4 = us[c];
        __nv_bfloat162* g2 = reinterpret_cast<__nv_bfloat162*>(&g4);
        const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&u4);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
            g2[k] = __floats2bfloat162_rn(expert_gate(act, w * g.x, w * u.x, limit, alpha), expert_gate(act, w * g.y, w * u.y, limit, alpha));
        }
        reinterpret_cast<uint4*>(a + row * ff)[c] = g4;
    }
}

}  // namespace lily

using namespace lily;

// router [outputs (+ 1 with `gate`), width]; correction [outputs] or null; sigmoid 0: softmax over the outputs, 1: each
// output's sigmoid; renormalise: the chosen scores over their sum; groups (0 or 1: none) and how many of them are kept.
static int check_groups(const char* name, int outputs, int top, int groups, int keep) {
    LILY_REQUIRE(groups >= 0 && groups <= ROUTE_GROUPS_MAX, "%s: %d groups (up to %d)", name, groups, ROUTE_GROUPS_MAX);
    LILY_REQUIRE(groups <= 1 || (outputs % groups == 0 && keep >= 1 && keep <= groups && top <= keep * (outputs / groups)),
                 "%s: top %d of the best %d of %d groups of %d outputs", name, top, keep, groups, outputs);
    return 0;
}

LILY_API int lily_moe_route(const void* h, int tokens, int width, const float* router, const float* correction, int outputs,
                            int top, int sigmoid, int renormalise, int group_count, int group_keep, int* chosen, float* weights, float* gate, int dtype,
                            cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(outputs >= 1 && outputs <= ROUTE_MAX, "moe_route: %d router outputs (up to %d)", outputs, ROUTE_MAX);
    LILY_REQUIRE(top >= 1 && top <= outputs && top <= ROUTE_TOP_MAX, "moe_route: top %d of %d", top, outputs);
    if (check_groups("moe_route", outputs, top, group_count, group_keep)) return 1;
    const RouteGroups groups{group_count, group_keep};
    const int rows = outputs + (gate ? 1 : 0);
    // four tokens a block once there are blocks enough for the device, and while their rows fit the shared memory
    const int tb = (tokens >= 1024 && (size_t)(4 * width + 4 * rows) * sizeof(float) <= 40 * 1024) ? 4 : 1;
    const size_t smem = (size_t)tb * (width + rows) * sizeof(float);
    LILY_REQUIRE(width > 0 && smem <= 44 * 1024, "moe_route: rows of %d numbers and %d outputs do not fit a block's shared memory", width, outputs);
    dim3 grid((tokens + tb - 1) / tb), block(128);
#define GO(T, TB)                                                                                                   \
    launch_pdl(moe_route_kernel<T, TB>, grid, block, smem, stream, (const T*)h, tokens, width, router, correction, outputs, \
               top, sigmoid, renormalise, groups, chosen, weights, gate)
    if (dtype == kBF16) { if (tb == 4) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
    else { if (tb == 4) GO(float, 4); else GO(float, 1); }
#undef GO
    LILY_CHECK_LAUNCH("moe_route");
    return 0;
}

// The same from the logits: rows `ld` apart, outputs (+ 1 with `gate`) of them read.
LILY_API int lily_moe_choose(const void* logits, int logits_dtype, int splits, size_t stride, int ld, int tokens, const float* correction, int outputs,
                             int top, int sigmoid, int renormalise, int group_count, int group_keep, int* chosen, float* weights, float* gate, cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(outputs >= 1 && outputs <= ROUTE_MAX, "moe_choose: %d router outputs (up to %d)", outputs, ROUTE_MAX);
    LILY_REQUIRE(top >= 1 && top <= outputs && top <= ROUTE_TOP_MAX, "moe_choose: top %d of %d", top, outputs);
    LILY_REQUIRE(splits >= 1 && logits_dtype == kF32 && ld >= outputs + (gate ? 1 : 0), "moe_choose: float32 logits in rows of %d", ld);
    if (check_groups("moe_choose", outputs, top, group_count, group_keep)) return 1;
    const RouteGroups groups{group_count, group_keep};
    const Operand x{logits, 0, splits, stride};
    launch_pdl(moe_choose_kernel, dim3((tokens + 3) / 4), dim3(128), (size_t)4 * (outputs + 1) * sizeof(float), stream, x, ld, tokens, correction,
               outputs, top, sigmoid, renormalise, groups, chosen, weights, gate);
    LILY_CHECK_LAUNCH("moe_choose");
    return 0;
}

LILY_API int lily_moe_tile_rows() { return EBM; }

LILY_API int lily_moe_align(const int* chosen, int pairs, int experts, int* offsets, int* order, int* place,
                            int* tile_expert, int* tile_row, int* tile_count, int max_tiles, cudaStream_t stream) {
    LILY_REQUIRE(experts >= 0 && experts <= 4000, "moe_align: %d experts", experts);
    LILY_REQUIRE(max_tiles >= (pairs + EBM - 1) / EBM + experts, "moe_align: room for %d tiles is too little", max_tiles);
    launch_pdl(moe_align_kernel, dim3(1), dim3(1024), (size_t)(3 * experts + 1) * sizeof(int), stream, chosen, pairs, experts,
               EBM, offsets, order, place, tile_expert, tile_row, tile_count, max_tiles);
    LILY_CHECK_LAUNCH("moe_align");
    return 0;
}

// mode 0: gate/up with the activation (W [experts, 2 N, K], out [pairs, N] in the activation dtype; in_weight: the pairs'
// weights where they belong to the input, else null); mode 1: down (W [experts, N, K], out [pairs, N] float32); mode 2: up with
// the squared relu (W [experts, N, K], out and in_weight as in mode 0).
LILY_API int lily_moe_gemm(int mode, const void* A, int lda, const void* W, int N, int K, const int* offsets,
                           const int* order, int top, const int* tile_expert, const int* tile_row, const int* tile_count,
                           int max_tiles, void* out, int act, float limit, float alpha, const float* in_weight, int dtype,
                           cudaStream_t stream) {
    if (max_tiles == 0 || N == 0) return 0;
    LILY_REQUIRE(K > 0 && lda >= K && mode >= 0 && mode <= 2, "moe_gemm: mode=%d N=%d K=%d lda=%d", mode, N, K, lda);
    LILY_REQUIRE(max_tiles <= 65535, "moe_gemm: %d tiles", max_tiles);
    dim3 grid((N + EBN - 1) / EBN, max_tiles), block(256);
    const size_t w_expert = (size_t)(mode == 0 ? 2 : 1) * N * K;
#define GO(T, MODE)                                                                                                \
    launch_pdl(moe_gemm_kernel<T, MODE>, grid, block, 0, stream, (const T*)A, lda, (const T*)W, w_expert, N, K, offsets, \
               order, top, tile_expert, tile_row, tile_count, out, act, limit, alpha, in_weight)
    if (dtype == kBF16) { if (mode == 0) GO(__nv_bfloat16, 0); else if (mode == 2) GO(__nv_bfloat16, 2); else GO(__nv_bfloat16, 1); }
    else { if (mode == 0) GO(float, 0); else if (mode == 2) GO(float, 2); else GO(float, 1); }
#undef GO
    LILY_CHECK_LAUNCH("moe_gemm");
    return 0;
}

// y_dtype: float32 (this file's product) or the activation dtype (the library's); weights null: the pairs' outputs as they
// are; gate null: no shared expert.
LILY_API int lily_moe_combine(const void* y, int y_dtype, const void* h, const int* place, const float* weights, int tokens, int top,
                              int width, const void* shared, int shared_dtype, int shared_splits, size_t shared_stride,
                              const float* gate, float* out, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(y_dtype == dtype || y_dtype == kF32, "moe_combine: outputs are the activation dtype or float32");
    LILY_REQUIRE(!gate || (shared && shared_splits >= 1 && (shared_splits == 1 || shared_dtype == kF32)), "moe_combine: the shared expert's output");
    const Operand sh{shared, shared_dtype == kBF16, shared_splits, shared_stride};
    const bool vec = width % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)h & 15) == 0 && ((uintptr_t)out & 15) == 0 && sh.vector_ok();
    const int per = vec ? 4 : 1;
    dim3 grid(tokens, (width + 256 * per - 1) / (256 * per)), block(256);
#define GO(Y, T)                                                                                                             \
    do {                                                                                                                     \
        if (vec) launch_pdl(moe_combine_kernel<Y, T, 4>, grid, block, 0, stream, (const Y*)y, (const T*)h, place, weights, top, width, sh, gate, out); \
        else launch_pdl(moe_combine_kernel<Y, T, 1>, grid, block, 0, stream, (const Y*)y, (const T*)h, place, weights, top, width, sh, gate, out);     \
    } while (0)
    if (dtype == kBF16) { if (y_dtype == kF32) GO(float, __nv_bfloat16); else GO(__nv_bfloat16, __nv_bfloat16); }
    else GO(float, float);
#undef GO
    LILY_CHECK_LAUNCH("moe_combine");
    return 0;
}

LILY_API int lily_moe_gather(const void* h, int width, const int* offsets, int experts, const int* order, int top, int pairs,
                             void* out, cudaStream_t stream) {
    if (pairs == 0) return 0;
    LILY_REQUIRE(width % 8 == 0 && ((uintptr_t)h & 15) == 0 && ((uintptr_t)out & 15) == 0, "moe_gather: rows of %d are not whole 16-byte pieces", width);
    launch_pdl(moe_gather_kernel, dim3(pairs), dim3(width >= 2048 ? 256 : 128), 0, stream, (const __nv_bfloat16*)h, width, offsets,
               experts, order, top, (__nv_bfloat16*)out);
    LILY_CHECK_LAUNCH("moe_gather");
    return 0;
}

LILY_API int lily_moe_activation(const void* gu, int ff, int rows, void* a, int act, float limit, float alpha, const float* in_weight,
                                 const int* offsets, int experts, const int* order, cudaStream_t stream) {
    if (rows == 0) return 0;
    LILY_REQUIRE(ff % 8 == 0 && ((uintptr_t)gu & 15) == 0 && ((uintptr_t)a & 15) == 0, "moe_activation: rows of %d are not whole 16-byte pieces", ff);
    launch_pdl(moe_activation_kernel, dim3(rows), dim3(ff >= 1024 ? 128 : (ff >= 512 ? 64 : 32)), 0, stream, (const __nv_bfloat16*)gu, ff,
               (__nv_bfloat16*)a, act, limit, alpha, in_weight, offsets, experts, order);
    LILY_CHECK_LAUNCH("moe_activation");
    return 0;
}

// The same for ungated experts: u [rows, ff] the up product, a = max(u, 0)^2.
LILY_API int lily_moe_relu2(const void* u, int ff, int rows, void* a, const float* in_weight, const int* offsets, int experts, const int* order,
                            cudaStream_t stream) {
    if (rows == 0) return 0;
    LILY_REQUIRE(ff % 8 == 0 && ((uintptr_t)u & 15) == 0 && ((uintptr_t)a & 15) == 0, "moe_relu2: rows of %d are not whole 16-byte pieces", ff);
    launch_pdl(moe_relu2_kernel, dim3(rows), dim3(ff >= 1024 ? 128 : (ff >= 512 ? 64 : 32)), 0, stream, (const __nv_bfloat16*)u, ff,
               (__nv_bfloat16*)a, in_weight, offsets, experts, order);
    LILY_CHECK_LAUNCH("moe_relu2");
    return 0;
}
