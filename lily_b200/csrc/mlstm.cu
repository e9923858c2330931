// The recurrence of the matrix-memory mixer with exponential gates (mLSTM), with its state in the request's slot.
//
// Per head, with S a d x dv matrix, n a vector of d and m a number that are all zero when the request starts, and log gates
// i_t = cap tanh(a_t / cap), f_t = logsigmoid(cap tanh(b_t / cap)) of the token's gate inputs a_t, b_t (bias included):
//
//     m_t = max(f_t + m, i_t);   S <- exp(f_t + m - m_t) S + exp(i_t - m_t) k_t v_t^T;   n likewise with k_t alone
//     o_t = S^T q_t / (max(|n . q_t|, exp(-m_t)) + floor)
//
// n is one more column of S whose value is always one, so a row of the state is [heads][dv + 1][d] (d fastest), then the
// heads' m.  The columns never meet in the recurrence.
//
//   mlstm_scan   raw sums S^T q_t [tokens, heads, dv], n . q_t [tokens, heads] and m_t [tokens, heads]: a block owns a few
//                columns of one head of one request and walks the request's new tokens in order
//                (long portions in bfloat16 run in chunks side by side instead: mlstm_chunk.cu)
//   mlstm_out    the division, each head's unit root mean square, gain and sigmoid gate; writes the last token's m into the
//                slot (every block of the scan reads the old one)
//
// Gates, m, the state and every sum over it are float32 whatever the activation dtype.
#include "common.cuh"
#include "operand.cuh"

namespace lily {

constexpr int ML_LANES = 8;                  // lanes that share a column, four neighbouring rows of it each a turn
constexpr int ML_THREADS = 128;
constexpr int ML_COLS = ML_THREADS / ML_LANES;

struct MlstmArgs {
    Operand proj;                            // [tokens, ld]: q (heads x d), k (heads x d), v (heads x dv) from their columns on
    int ld, q_col, k_col, v_col;
    Operand gates;                           // [tokens, gates_ld]: heads columns of either gate's input, without bias
    int gates_ld, i_col, f_col;
    const float* i_bias;                     // [heads]
    const float* f_bias;
    float cap, q_scale;
    float* state;
    size_t state_stride;
    float* y;                                // [tokens, heads * dv]
    float* nq;                               // [tokens, heads]
    float* m;                                // [tokens, heads]
    const int* cu_seqlens;
    const int* slots;
    const int* reqs;                         // the requests to run (null: all)
    int heads, d, dv;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

__device__ __forceinline__ float sum_over_column(float v) {
#pragma unroll
    for (int o = ML_LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// grid (requests, heads, ceil((dv + 1) / ML_COLS)), block ML_THREADS; d <= 32 R.  VEC: d, ld, columns and the state's rows are
// multiples of four and the bases aligned.
template <int R, int TT, bool VEC>
__global__ void __launch_bounds__(ML_THREADS) mlstm_scan_kernel(const MlstmArgs a) {
    constexpr int DP = 4 * ML_LANES * R;
    __shared__ __align__(16) float qs[TT][DP], ks[TT][DP];
    __shared__ float vs[TT][ML_COLS], os[TT][ML_COLS], keep_s[TT], write_s[TT], m_s[TT], gi[TT], gf[TT];
    pdl_enter_small();
    const int req = a.reqs ? a.reqs[blockIdx.x] : (int)blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * ML_COLS;
    const int tid = threadIdx.x, l = tid % ML_LANES, cg = tid / ML_LANES;
    const int d = a.d, dv = a.dv, j = col0 + cg;
    const bool col_ok = j <= dv;                                 // column dv is n
    const int tok0 = a.cu_seqlens[req], len = a.cu_seqlens[req + 1] - tok0;
    if (len <= 0) return;
    float* slot = a.state + (size_t)a.slots[req] * a.state_stride;
    float* st = slot + ((size_t)head * (dv + 1) + (col_ok ? j : 0)) * d;
    float m = slot[(size_t)a.heads * (dv + 1) * d + head];
    float4 S[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = (r * ML_LANES + l) * 4;
        if (VEC) {
            S[r] = col_ok && i < d ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            S[r].x = col_ok && i < d ? st[i] : 0.f;
            S[r].y = col_ok && i + 1 < d ? st[i + 1] : 0.f;
            S[r].z = col_ok && i + 2 < d ? st[i + 2] : 0.f;
            S[r].w = col_ok && i + 3 < d ? st[i + 3] : 0.f;
        }
    }
    for (int t0 = 0; t0 < len; t0 += TT) {
        const int n = min(TT, len - t0);
        __syncthreads();
        if (VEC) {
            for (int e = tid * 4; e < n * DP; e += ML_THREADS * 4) {
                const int t = e / DP, i = e % DP;
                const size_t row = (size_t)(tok0 + t0 + t) * a.ld + (size_t)head * d + i;
                float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
                if (i < d) {
                    q = a.proj.four(row + a.q_col);
                    k = a.proj.four(row + a.k_col);
                }
                *reinterpret_cast<float4*>(&qs[t][i]) = make_float4(q.x * a.q_scale, q.y * a.q_scale, q.z * a.q_scale, q.w * a.q_scale);
                *reinterpret_cast<float4*>(&ks[t][i]) = k;
            }
        } else {
            for (int e = tid; e < n * DP; e += ML_THREADS) {
                const int t = e / DP, i = e % DP;
                const size_t row = (size_t)(tok0 + t0 + t) * a.ld + (size_t)head * d + i;
                qs[t][i] = i < d ? a.proj(row + a.q_col) * a.q_scale : 0.f;
                ks[t][i] = i < d ? a.proj(row + a.k_col) : 0.f;
            }
        }
        for (int e = tid; e < n * ML_COLS; e += ML_THREADS) {
            const int t = e / ML_COLS, c = e % ML_COLS;
            vs[t][c] = col0 + c < dv ? a.proj((size_t)(tok0 + t0 + t) * a.ld + a.v_col + (size_t)head * dv + col0 + c) : (col0 + c == dv ? 1.f : 0.f);
        }
        if (tid < n) {
            const size_t row = (size_t)(tok0 + t0 + tid) * a.gates_ld + head;
            gi[tid] = soft_cap(a.gates(row + a.i_col) + a.i_bias[head], a.cap);
            gf[tid] = log_sigmoid(soft_cap(a.gates(row + a.f_col) + a.f_bias[head], a.cap));
        }
        __syncthreads();
        if (tid < 32) {                                          // the scale's own recurrence, the same in every lane
            float mine = m;
            for (int t = 0; t < n; ++t) {
                const float held = gf[t] + mine, next = fmaxf(held, gi[t]);
                if (tid == (t & 31)) {
                    keep_s[t] = expf(held - next);
                    write_s[t] = expf(gi[t] - next);
                    m_s[t] = next;
                }
                mine = next;
            }
        }
        __syncthreads();
        m = m_s[n - 1];
        for (int t = 0; t < n; ++t) {
            const float keep = keep_s[t], u = write_s[t] * vs[t][cg];
            float acc = 0.f;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float4 k = *reinterpret_cast<const float4*>(&ks[t][(r * ML_LANES + l) * 4]);
                const float4 q = *reinterpret_cast<const float4*>(&qs[t][(r * ML_LANES + l) * 4]);
                S[r].x = fmaf(u, k.x, keep * S[r].x);
                S[r].y = fmaf(u, k.y, keep * S[r].y);
                S[r].z = fmaf(u, k.z, keep * S[r].z);
                S[r].w = fmaf(u, k.w, keep * S[r].w);
                acc = fmaf(S[r].x, q.x, fmaf(S[r].y, q.y, fmaf(S[r].z, q.z, fmaf(S[r].w, q.w, acc))));
            }
            acc = sum_over_column(acc);
            if (l == 0) os[t][cg] = acc;
        }
        __syncthreads();
        for (int e = tid; e < n * ML_COLS; e += ML_THREADS) {
            const int t = e / ML_COLS, c = e % ML_COLS;
            const size_t at = (size_t)(tok0 + t0 + t) * a.heads + head;
            if (col0 + c < dv) a.y[at * dv + col0 + c] = os[t][c];
            else if (col0 + c == dv) {
                a.nq[at] = os[t][c];
                a.m[at] = m_s[t];
            }
        }
    }
    if (!col_ok) return;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = (r * ML_LANES + l) * 4;
        if (VEC) {
            if (i < d) *reinterpret_cast<float4*>(st + i) = S[r];
        } else {
            if (i < d) st[i] = S[r].x;
            if (i + 1 < d) st[i + 1] = S[r].y;
            if (i + 2 < d) st[i + 2] = S[r].z;
            if (i + 3 < d) st[i + 3] = S[r].w;
        }
    }
}

// out[t, c] = o / rms(o of the head) * gain[c] * sigmoid(gate[t, c]) with o = y / (max(|nq|, exp(-m)) + floor).
// VEC 4: dv a multiple of four, everything aligned.  WIDE 0: grid (tokens, ceil(heads / 4)), block 128, a warp a head of a token.
// WIDE 1 (a few tokens, VEC 4): grid (tokens, heads), block 128, four columns a thread and turn, so that a head's numbers
// are all asked for together.
template <typename T, int VEC, int WIDE>
__global__ void mlstm_out_kernel(const float* __restrict__ y, const float* __restrict__ nq, const float* __restrict__ m, const Operand gate,
                                 int gate_ld, int gate_col, const float* __restrict__ gain, float floor_, float eps, T* __restrict__ out,
                                 float* __restrict__ state, size_t state_stride, size_t m_off, const int* __restrict__ cu_seqlens,
                                 const int* __restrict__ token_req, const int* __restrict__ slots, int heads, int dv) {
    __shared__ float sums[4];
    pdl_enter_small();
    const int t = blockIdx.x, head = WIDE ? (int)blockIdx.y : blockIdx.y * 4 + (threadIdx.x >> 5), lane = WIDE ? threadIdx.x : threadIdx.x & 31;
    if (head >= heads) return;
    constexpr int STEP = (WIDE ? 128 : 32) * VEC;
    const size_t at = (size_t)t * heads + head;
    const float* yr = y + at * dv;
    const size_t g0 = (size_t)t * gate_ld + gate_col + (size_t)head * dv;
    const float* gn = gain + (size_t)head * dv;
    T* dst = out + at * dv;
    const float4 nil = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v0 = nil, z0 = nil, w0 = nil;
    if (WIDE && lane * 4 < dv) {
        v0 = *reinterpret_cast<const float4*>(yr + lane * 4);
        z0 = gate.four(g0 + lane * 4);
        w0 = *reinterpret_cast<const float4*>(gn + lane * 4);
    }
    const float mt = m[at];
    const int r = token_req[t];
    const float inv_den = 1.f / (fmaxf(fabsf(nq[at]), expf(-mt)) + floor_);
    auto square = [&](const float4& u) {
        const float x0 = u.x * inv_den, x1 = u.y * inv_den, x2 = u.z * inv_den, x3 = u.w * inv_den;
        return x0 * x0 + x1 * x1 + x2 * x2 + x3 * x3;
    };
    float ssq = 0.f;
    if (VEC == 4) {
        if (WIDE) ssq = square(v0);
        for (int c = lane * 4 + (WIDE ? STEP : 0); c < dv; c += STEP) ssq += square(*reinterpret_cast<const float4*>(yr + c));
    } else {
        for (int c = lane; c < dv; c += 32) {
            const float x = yr[c] * inv_den;
            ssq = fmaf(x, x, ssq);
        }
    }
    ssq = warp_sum(ssq);
    if (WIDE) {
        if ((threadIdx.x & 31) == 0) sums[threadIdx.x >> 5] = ssq;
        __syncthreads();
        ssq = (sums[0] + sums[1]) + (sums[2] + sums[3]);
    }
    const float f = inv_den * rsqrtf(ssq / (float)dv + eps);
    auto finish = [&](int c, const float4& u, const float4& z, const float4& x) {
        const float o0 = u.x * f * x.x / (1.f + expf(-z.x)), o1 = u.y * f * x.y / (1.f + expf(-z.y));
        const float o2 = u.z * f * x.z / (1.f + expf(-z.z)), o3 = u.w * f * x.w / (1.f + expf(-z.w));
        if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(dst + c) = make_float4(o0, o1, o2, o3);
        } else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(o0, o1), hi = __floats2bfloat162_rn(o2, o3);
            *reinterpret_cast<uint2*>(dst + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    };
    if (VEC == 4) {
        if (WIDE && lane * 4 < dv) finish(lane * 4, v0, z0, w0);
        for (int c = lane * 4 + (WIDE ? STEP : 0); c < dv; c += STEP)
            finish(c, *reinterpret_cast<const float4*>(yr + c), gate.four(g0 + c), *reinterpret_cast<const float4*>(gn + c));
    } else {
        for (int c = lane; c < dv; c += 32) dst[c] = from_float<T>(yr[c] * f * gn[c] / (1.f + expf(-gate(g0 + c))));
    }
    if (lane == 0 && t == cu_seqlens[r + 1] - 1) state[(size_t)slots[r] * state_stride + m_off + head] = mt;
}

}  // namespace lily

using namespace lily;

LILY_API int lily_mlstm_max_head_dim() { return 512; }

// Rows of the state: heads * (dv + 1) * d numbers, then the heads' m.
LILY_API int lily_mlstm_scan(const void* proj, int proj_dtype, int proj_splits, size_t proj_stride, int ld, int q_col, int k_col, int v_col,
                             const void* gates, int gates_dtype, int gates_splits, size_t gates_stride, int gates_ld, int i_col, int f_col,
                             const float* i_bias, const float* f_bias, float cap, float q_scale, float* state, size_t state_stride, float* y,
                             float* nq, float* m, const int* cu_seqlens, const int* slots, const int* reqs, int requests, int heads, int d,
                             int dv, cudaStream_t stream) {
    if (requests == 0) return 0;
    LILY_REQUIRE(heads > 0 && heads <= 65535 && d > 0 && d <= 512 && dv > 0, "mlstm_scan: %d heads of %d x %d (keys up to 512)", heads, d, dv);
    LILY_REQUIRE((size_t)heads * (dv + 1) * d + heads <= state_stride, "mlstm_scan: the state row is shorter than %d matrices of %d x %d", heads, d, dv + 1);
    LILY_REQUIRE(cap > 0.f, "mlstm_scan: gate cap %g", cap);
    LILY_REQUIRE(proj_splits >= 1 && (proj_splits == 1 || proj_dtype == kF32) && gates_splits >= 1 && (gates_splits == 1 || gates_dtype == kF32),
                 "mlstm_scan: only float32 partial sums come in several splits");
    MlstmArgs a{};
    a.proj = Operand{proj, proj_dtype == kBF16, proj_splits, proj_stride}; a.ld = ld; a.q_col = q_col; a.k_col = k_col; a.v_col = v_col;
    a.gates = Operand{gates, gates_dtype == kBF16, gates_splits, gates_stride}; a.gates_ld = gates_ld; a.i_col = i_col; a.f_col = f_col;
    a.i_bias = i_bias; a.f_bias = f_bias; a.cap = cap; a.q_scale = q_scale; a.state = state; a.state_stride = state_stride;
    a.y = y; a.nq = nq; a.m = m; a.cu_seqlens = cu_seqlens; a.slots = slots; a.reqs = reqs; a.heads = heads; a.d = d; a.dv = dv;
    dim3 grid(requests, heads, dv / ML_COLS + 1), block(ML_THREADS);
    LILY_REQUIRE(grid.z <= 65535, "mlstm_scan: %d value columns", dv);
    const bool vec = d % 4 == 0 && ld % 4 == 0 && q_col % 4 == 0 && k_col % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0 &&
                     a.proj.vector_ok();
    const int turns = (d + 4 * ML_LANES - 1) / (4 * ML_LANES);
#define GO(R, TT)                                                                           \
    do {                                                                                    \
        if (vec) launch_pdl(mlstm_scan_kernel<R, TT, true>, grid, block, 0, stream, a);     \
        else launch_pdl(mlstm_scan_kernel<R, TT, false>, grid, block, 0, stream, a);        \
    } while (0)
    if (turns <= 1) GO(1, 16);
    else if (turns <= 2) GO(2, 16);
    else if (turns <= 4) GO(4, 16);
    else if (turns <= 8) GO(8, 16);
    else GO(16, 8);
#undef GO
    LILY_CHECK_LAUNCH("mlstm_scan");
    return 0;
}

LILY_API int lily_mlstm_out(const float* y, const float* nq, const float* m, const void* gate, int gate_dtype, int gate_splits, size_t gate_stride,
                            int gate_ld, int gate_col, const float* gain, float floor_, float eps, void* out, int out_dtype, float* state,
                            size_t state_stride, size_t m_off, const int* cu_seqlens, const int* token_req, const int* slots, int tokens,
                            int heads, int dv, cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(heads > 0 && dv > 0 && (heads + 3) / 4 <= 65535, "mlstm_out: %d heads of %d columns", heads, dv);
    LILY_REQUIRE(gate_splits >= 1 && (gate_splits == 1 || gate_dtype == kF32), "mlstm_out: only float32 partial sums come in several splits");
    LILY_REQUIRE(m_off + heads <= state_stride, "mlstm_out: the state row has no room for the scales");
    const Operand g{gate, gate_dtype == kBF16, gate_splits, gate_stride};
    const bool vec = dv % 4 == 0 && gate_ld % 4 == 0 && gate_col % 4 == 0 && g.vector_ok() && ((uintptr_t)y & 15) == 0 &&
                     ((uintptr_t)gain & 15) == 0 && ((uintptr_t)out & 15) == 0;
    const bool wide = vec && tokens <= 64 && heads <= 65535;
    dim3 grid(tokens, wide ? heads : (heads + 3) / 4), block(128);
#define GO(T, V, W)                                                                                                                    \
    launch_pdl(mlstm_out_kernel<T, V, W>, grid, block, 0, stream, y, nq, m, g, gate_ld, gate_col, gain, floor_, eps, (T*)out, state, state_stride, \
               m_off, cu_seqlens, token_req, slots, heads, dv)
    if (out_dtype == kBF16) { if (wide) GO(__nv_bfloat16, 4, 1); else if (vec) GO(__nv_bfloat16, 4, 0); else GO(__nv_bfloat16, 1, 0); }
    else { if (wide) GO(float, 4, 1); else if (vec) GO(float, 4, 0); else GO(float, 1, 0); }
#undef GO
    LILY_CHECK_LAUNCH("mlstm_out");
    return 0;
}
