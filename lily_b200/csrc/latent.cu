// Attention over a low-rank latent of keys and values: what comes before and after the attention kernel itself.
//
// A token's cache row is [latent (rank) | rotated key part (rot)]: one row for all heads, in pages
// [page_size, rank + rot] of a layer [pages, page_size * (rank + rot)].  Per head the unrotated key is W_uk latent
// and the value W_uv latent, so with q' = W_uk^T q_unrotated the score is q' . latent + q_rotated . k_rotated, and
// the head's output is W_uv (sum_j p_j latent_j): the attention kernel runs over the rows as they are cached, all
// heads sharing them, and reads its values out of the first `rank` columns of the key rows.
//
//   latent_prepare  down-projection row -> RMS-normed query latent (none when the queries have no latent of their own); RMS-normed key/value latent and the rotated
//                   key part into the token's cache row
//   latent_query    the rotated part of every head's query, beside the part the per-head product has put in place
//   head_gate       per-head outputs times sigmoid(gate of the head) -> the rows the output projection takes
//
// Norms, angles and the sigmoid are float32.
#include "common.cuh"
#include "operand.cuh"

namespace lily {

// One block per token.  `in` is the token's row of the stacked down-projection (row stride `ld`; finished, or the
// partial sums of a split-k product): the query latent at column q0 (q_rank columns), the key/value latent at kv0
// (rank columns) followed by the part to rotate (rot columns, of which the first rd are rotated in halves and the
// rest pass).  The row is read once: what the norms need again stands in shared memory.
template <typename T> __device__ __forceinline__ void put_four(T* dst, float a, float b, float c, float d);
template <> __device__ __forceinline__ void put_four<float>(float* dst, float a, float b, float c, float d) { *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d); }
template <> __device__ __forceinline__ void put_four<__nv_bfloat16>(__nv_bfloat16* dst, float a, float b, float c, float d) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// VEC 4: columns, sizes and rows of whole pieces of four numbers, bases aligned to them.
template <typename T, int VEC>
__global__ void latent_prepare_kernel(const Operand in, int ld, int q0, int q_rank, int kv0, int rank, int rot,
                                      int rd, const float* __restrict__ q_gain, const float* __restrict__ kv_gain,
                                      float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                      const int* __restrict__ positions, const int* __restrict__ token_req,
                                      const int* __restrict__ block_table, int bt_stride, T* __restrict__ layer,
                                      int page_size, int write_kv, T* __restrict__ cq) {
    extern __shared__ __align__(16) float held[];       // [q_rank | rank + rot] of the token's row
    __shared__ float sums[2][32];
    pdl_enter_small();
    const int t = blockIdx.x, warps = blockDim.x >> 5;
    const size_t row = (size_t)t * ld;
    float* kv = held + q_rank;
    float ssq = 0.f, ssk = 0.f;
    if (VEC == 4) {
        for (int c = threadIdx.x * 4; c < q_rank; c += blockDim.x * 4) {
            const float4 x = in.four(row + q0 + c);
            *reinterpret_cast<float4*>(held + c) = x;
            ssq += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
        }
        if (write_kv)
            for (int c = threadIdx.x * 4; c < rank + rot; c += blockDim.x * 4) {
                const float4 x = in.four(row + kv0 + c);
                *reinterpret_cast<float4*>(kv + c) = x;
                if (c < rank) ssk += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
            }
    } else {
        for (int c = threadIdx.x; c < q_rank; c += blockDim.x) {
            const float x = in(row + q0 + c);
            held[c] = x;
            ssq = fmaf(x, x, ssq);
        }
    }
    if (VEC == 1 && write_kv)
        for (int c = threadIdx.x; c < rank + rot; c += blockDim.x) {
            const float x = in(row + kv0 + c);
            kv[c] = x;
            if (c < rank) ssk = fmaf(x, x, ssk);
        }
    ssq = warp_sum(ssq);
    ssk = warp_sum(ssk);
    if ((threadIdx.x & 31) == 0) {
        sums[0][threadIdx.x >> 5] = ssq;
        sums[1][threadIdx.x >> 5] = ssk;
    }
    __syncthreads();
    ssq = ssk = 0.f;
    for (int w = 0; w < warps; ++w) {
        ssq += sums[0][w];
        ssk += sums[1][w];
    }
    const float inv_q = rsqrtf(ssq / (float)max(q_rank, 1) + eps);
    if (VEC == 4)
        for (int c = threadIdx.x * 4; c < q_rank; c += blockDim.x * 4) {
            const float4 x = *reinterpret_cast<const float4*>(held + c), g = *reinterpret_cast<const float4*>(q_gain + c);
            put_four<T>(cq + (size_t)t * q_rank + c, x.x * inv_q * g.x, x.y * inv_q * g.y, x.z * inv_q * g.z, x.w * inv_q * g.w);
        }
    else
        for (int c = threadIdx.x; c < q_rank; c += blockDim.x) cq[(size_t)t * q_rank + c] = from_float<T>((held[c] * inv_q) * q_gain[c]);
    if (!write_kv) return;
    const float inv_kv = rsqrtf(ssk / (float)rank + eps);
    const int pos = positions[t];
    const int page = block_table[(size_t)token_req[t] * bt_stride + pos / page_size];
    const int width = rank + rot;
    T* dst = layer + ((size_t)page * page_size + pos % page_size) * width;
    if (VEC == 4)
        for (int c = threadIdx.x * 4; c < rank; c += blockDim.x * 4) {
            const float4 x = *reinterpret_cast<const float4*>(kv + c), g = *reinterpret_cast<const float4*>(kv_gain + c);
            put_four<T>(dst + c, x.x * inv_kv * g.x, x.y * inv_kv * g.y, x.z * inv_kv * g.z, x.w * inv_kv * g.w);
        }
    else
        for (int c = threadIdx.x; c < rank; c += blockDim.x)
            dst[c] = from_float<T>((kv[c] * inv_kv) * kv_gain[c]);
    const int half = rd / 2;
    const float* kr = kv + rank;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float u = kr[i], v = kr[i + half];
        const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
        dst[rank + i] = from_float<T>(u * c - v * s);
        dst[rank + i + half] = from_float<T>(v * c + u * s);
    }
    for (int i = rd + threadIdx.x; i < rot; i += blockDim.x) dst[rank + i] = from_float<T>(kr[i]);
}

// One block per token.  q [tokens, heads, d + rot]: the up-projected queries, of which the last rot columns of a head are
// rotated into the last rot columns of the head's row of out [tokens, heads, rank + rot] (the first rank are the
// unrotated part carried into the latent's space, which the per-head product has written).
// VEC 2 (bfloat16): two neighbouring pairs a thread.
template <typename T, int VEC>
__global__ void latent_query_kernel(const T* __restrict__ q, int heads, int d, int rank, int rot, int rd,
                                    const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                    const int* __restrict__ positions, T* __restrict__ out) {
    pdl_enter_small();
    const int t = blockIdx.x, pos = positions[t], half = rd / 2, rest = rot - rd;
    const T* src = q + (size_t)t * heads * (d + rot) + d;
    T* dst = out + (size_t)t * heads * (rank + rot) + rank;
    if (VEC == 2) {
        const int pairs = half / 2;
        for (int n = threadIdx.x; n < heads * pairs; n += blockDim.x) {
            const int h = n / pairs, i = n % pairs * 2;
            const __nv_bfloat16* qr = reinterpret_cast<const __nv_bfloat16*>(src) + (size_t)h * (d + rot) + i;
            __nv_bfloat16* to = reinterpret_cast<__nv_bfloat16*>(dst) + (size_t)h * (rank + rot) + i;
            const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(qr));
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(qr + half));
            const float2 c = *reinterpret_cast<const float2*>(cos_t + (size_t)pos * half + i);
            const float2 s = *reinterpret_cast<const float2*>(sin_t + (size_t)pos * half + i);
            *reinterpret_cast<__nv_bfloat162*>(to) = __floats2bfloat162_rn(u.x * c.x - v.x * s.x, u.y * c.y - v.y * s.y);
            *reinterpret_cast<__nv_bfloat162*>(to + half) = __floats2bfloat162_rn(v.x * c.x + u.x * s.x, v.y * c.y + u.y * s.y);
        }
    } else for (int n = threadIdx.x; n < heads * half; n += blockDim.x) {
        const int h = n / half, i = n % half;
        const T* qr = src + (size_t)h * (d + rot);
        T* to = dst + (size_t)h * (rank + rot);
        const float u = to_float(qr[i]), v = to_float(qr[i + half]);
        const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
        to[i] = from_float<T>(u * c - v * s);
        to[i + half] = from_float<T>(v * c + u * s);
    }
    for (int n = threadIdx.x; n < heads * rest; n += blockDim.x) {
        const int h = n / rest, i = rd + n % rest;
        dst[(size_t)h * (rank + rot) + i] = src[(size_t)h * (d + rot) + i];
    }
}

// grid (tokens, heads).  ov [heads, tokens, dv] (T or float32); gate: column g0 + head of the token's row of the
// stacked down-projection (row stride ld).  out [tokens, heads * dv] = ov * sigmoid(gate).
template <typename T, typename OV>
__global__ void head_gate_kernel(const OV* __restrict__ ov, const Operand gate, int ld, int g0, int tokens,
                                 int heads, int dv, T* __restrict__ out) {
    pdl_enter_small();
    const int t = blockIdx.x, h = blockIdx.y;
    const float g = 1.f / (1.f + expf(-gate((size_t)t * ld + g0 + h)));
    const OV* src = ov + ((size_t)h * tokens + t) * dv;
    T* dst = out + ((size_t)t * heads + h) * dv;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) dst[c] = from_float<T>(to_float(src[c]) * g);
}

}  // namespace lily

using namespace lily;

LILY_API int lily_latent_prepare(const void* in, int in_dtype, int in_splits, size_t in_stride, int ld, int q0, int q_rank,
                                 int kv0, int rank, int rot, int rd, const float* q_gain, const float* kv_gain, float eps,
                                 const float* cos_t, const float* sin_t, const int* positions, const int* token_req,
                                 const int* block_table, int bt_stride, void* layer, int page_size, int write_kv, void* cq,
                                 int tokens, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(q_rank >= 0 && rank > 0 && rot >= 0 && rd >= 0 && rd <= rot && rd % 2 == 0,
                 "latent_prepare: q_rank=%d rank=%d rot=%d rotated=%d", q_rank, rank, rot, rd);
    LILY_REQUIRE(rd == 0 || !write_kv || (cos_t && sin_t), "latent_prepare: rotation needs its tables");
    LILY_REQUIRE(in_splits >= 1 && (in_splits == 1 || in_dtype == kF32), "latent_prepare: only float32 partial sums come in several splits");
    const Operand x{in, in_dtype == kBF16, in_splits, in_stride};
    const size_t smem = sizeof(float) * (size_t)(q_rank + rank + rot);
    LILY_REQUIRE(smem <= 47 * 1024, "latent_prepare: latents of %d and %d columns do not fit a block's shared memory", q_rank, rank + rot);
    const int widest = q_rank > rank + rot ? q_rank : rank + rot;
    dim3 grid(tokens), block(tokens <= 64 && widest > 512 ? 512 : 128);
    const bool vec = q_rank % 4 == 0 && rank % 4 == 0 && rot % 4 == 0 && q0 % 4 == 0 && kv0 % 4 == 0 && ld % 4 == 0 && x.vector_ok() &&
                     ((uintptr_t)cq & 15) == 0 && ((uintptr_t)layer & 15) == 0 && ((uintptr_t)q_gain & 15) == 0 && ((uintptr_t)kv_gain & 15) == 0;
#define GO(T, V)                                                                                                                \
    launch_pdl(latent_prepare_kernel<T, V>, grid, block, smem, stream, x, ld, q0, q_rank, kv0, rank, rot, rd, q_gain, kv_gain, eps, \
               cos_t, sin_t, positions, token_req, block_table, bt_stride, (T*)layer, page_size, write_kv, (T*)cq)
    if (dtype == kBF16) { if (vec) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
    else { if (vec) GO(float, 4); else GO(float, 1); }
#undef GO
    LILY_CHECK_LAUNCH("latent_prepare");
    return 0;
}

LILY_API int lily_latent_query(const void* q, int tokens, int heads, int d, int rank, int rot, int rd, const float* cos_t,
                               const float* sin_t, const int* positions, void* out, int dtype, cudaStream_t stream) {
    if (tokens == 0 || rot == 0) return 0;
    LILY_REQUIRE(heads > 0 && rank > 0 && rot > 0 && rd <= rot && rd % 2 == 0, "latent_query: heads=%d rank=%d rot=%d", heads, rank, rot);
    LILY_REQUIRE(rd == 0 || (cos_t && sin_t), "latent_query: rotation needs its tables");
    const int work = heads * (rd / 2 > rot - rd ? rd / 2 : rot - rd);
    dim3 grid(tokens), block(work >= 512 ? 512 : (work >= 128 ? 128 : 32));
    const bool two = dtype == kBF16 && rd % 4 == 0 && rd > 0 && d % 2 == 0 && rot % 2 == 0 && rank % 2 == 0 && ((uintptr_t)q & 3) == 0 &&
                     ((uintptr_t)out & 3) == 0 && ((uintptr_t)cos_t & 7) == 0 && ((uintptr_t)sin_t & 7) == 0;
    if (two)
        launch_pdl(latent_query_kernel<__nv_bfloat16, 2>, grid, block, 0, stream, (const __nv_bfloat16*)q, heads, d, rank, rot, rd, cos_t,
                   sin_t, positions, (__nv_bfloat16*)out);
    else if (dtype == kBF16)
        launch_pdl(latent_query_kernel<__nv_bfloat16, 1>, grid, block, 0, stream, (const __nv_bfloat16*)q, heads, d, rank, rot, rd, cos_t,
                   sin_t, positions, (__nv_bfloat16*)out);
    else
        launch_pdl(latent_query_kernel<float, 1>, grid, block, 0, stream, (const float*)q, heads, d, rank, rot, rd, cos_t, sin_t, positions,
                   (float*)out);
    LILY_CHECK_LAUNCH("latent_query");
    return 0;
}

LILY_API int lily_head_gate(const void* ov, int ov_dtype, const void* gate, int gate_dtype, int gate_splits, size_t gate_stride,
                            int ld, int g0, int tokens, int heads, int dv, void* out, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    LILY_REQUIRE(heads > 0 && heads <= 65535 && dv > 0, "head_gate: heads=%d dv=%d", heads, dv);
    LILY_REQUIRE((ov_dtype == dtype || ov_dtype == kF32) && gate_splits >= 1 && (gate_splits == 1 || gate_dtype == kF32),
                 "head_gate: inputs are the activation dtype or float32; only float32 partial sums come in several splits");
    const Operand g{gate, gate_dtype == kBF16, gate_splits, gate_stride};
    dim3 grid(tokens, heads), block(dv >= 128 ? 128 : (dv >= 64 ? 64 : 32));
    if (dtype != kBF16)
        launch_pdl(head_gate_kernel<float, float>, grid, block, 0, stream, (const float*)ov, g, ld, g0, tokens, heads, dv, (float*)out);
    else if (ov_dtype == kF32)
        launch_pdl(head_gate_kernel<__nv_bfloat16, float>, grid, block, 0, stream, (const float*)ov, g, ld, g0, tokens, heads, dv,
                   (__nv_bfloat16*)out);
    else
        launch_pdl(head_gate_kernel<__nv_bfloat16, __nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)ov, g, ld, g0, tokens,
                   heads, dv, (__nv_bfloat16*)out);
    LILY_CHECK_LAUNCH("head_gate");
    return 0;
}
