// Row-wise operations of layer stacks with dense weights: norms, gated residual, short convolution over time, latent
// norms with the cache append.  One row = one position of one sequence.  T is the operand type of the matrix products
// (BF16 or FP32); norms, the residual stream, the convolution's state and all sums are FP32 whatever T is.
#pragma once
#include <cuda_bf16.h>

#include "attn.cuh"
#include "common.cuh"

namespace juno {

enum StackDtype { DT_BF16 = 0, DT_F32 = 1 };
inline int dt_bytes(int dt) { return dt == DT_F32 ? 4 : 2; }
inline int pad16(int n) { return (n + 15) / 16 * 16; }
inline int pad64(int n) { return (n + 63) / 64 * 64; }

// The rows of one pass.  one_seq: consecutive positions of one sequence (a portion of a prompt); otherwise row i is the next
// position of its own sequence.  Device pointers; positions[i] + 1 == lens[i].
struct RowSet {
    int n = 0;
    bool one_seq = false;
    const int32_t *tokens = nullptr, *positions = nullptr, *slots = nullptr, *lens = nullptr;
};

// x[r] = rms(embed[token]) * g
int launch_embed_norm(juno_ctx *c, int dt, const void *embed, int ld_embed, int width, int vocab, float g, float eps, const RowSet &rows,
                      float *x, int ldx, cudaStream_t st);

// x += rms(z) * g_z (z null: no sublayer result), then, with s = g_next / rms(x): h = x * s as operand, row_scale[r] = s.
struct ResidNormArgs {
    float *x;
    int ldx, width, n;
    const void *z = nullptr;
    int ldz = 0;
    float g_z = 0.f;
    float g_next = 0.f, eps = 0.f;
    void *h = nullptr;  // null: the residual update alone
    int ldh = 0;
    float *row_scale = nullptr;
};
int launch_resid_norm(juno_ctx *c, int dt, const ResidNormArgs &a, cudaStream_t st);

// out[i] = rms(x[row_idx[i]]) * g as operand (row_idx null: row i)
int launch_gather_norm(juno_ctx *c, int dt, const float *x, int ldx, int width, const int32_t *row_idx, int n, float g, float eps, void *out,
                       int ldo, cudaStream_t st);

// hc = h + conv(h), h = x * row_scale recomputed in FP32; conv(h)_t = sum_j w[j] h_(t - taps + 1 + j).  Inputs before this
// pass come from the pool's state, which receives this pass's inputs (a second launch when rows are a portion of a prompt).
struct ConvArgs {
    const float *x;
    int ldx, width;
    const float *row_scale;
    const void *w;  // [taps][ldx], type T
    int taps;
    const juno_kvpool *pool;
    int layer;
    void *out;
    int ldo;
};
int launch_conv(juno_ctx *c, int dt, const ConvArgs &a, const RowSet &rows, cudaStream_t st);

// u [n][ldu] FP32 holds, side by side, the two down projections of latent attention: queries at column 0 (q_rank), the
// key/value latent at column kv_col (kv_rank).  cq = rms(.) * wq as operand; the key/value latent is normed with wkv and
// appended to the sequence's pages.
struct LatentNormArgs {
    const float *u;
    int ldu, q_rank, kv_col, kv_rank;
    const float *wq, *wkv;
    float eps;
    void *cq;
    int ldq;
    const juno_kvpool *pool;
    int layer;
};
int launch_latent_norm(juno_ctx *c, int dt, const LatentNormArgs &a, const RowSet &rows, cudaStream_t st);

#if defined(__CUDACC__)
template <typename T>
struct Num;
template <>
struct Num<float> {
    static __device__ __forceinline__ float get(float v) { return v; }
    static __device__ __forceinline__ float put(float v) { return v; }
};
template <>
struct Num<__nv_bfloat16> {
    static __device__ __forceinline__ float get(__nv_bfloat16 v) { return __bfloat162float(v); }
    static __device__ __forceinline__ __nv_bfloat16 put(float v) { return __float2bfloat16_rn(v); }
};
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }
// 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), written as z * sigmoid(2 sqrt(2/pi) (...)): no cancellation for z << 0
__device__ __forceinline__ float gelu_tanh(float z) { return z * sigmoid_f32(1.5957691216057308f * fmaf(0.044715f * z * z, z, z)); }

// Four consecutive elements (16-byte aligned for FP32, 8-byte for BF16).
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p) {
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t *>(&a);
    u.y = *reinterpret_cast<const uint32_t *>(&b);
    *reinterpret_cast<uint2 *>(p) = u;
}
// Sum over a block of at most 1024 threads; every thread gets the result.  `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float *red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nw ? red[lane] : 0.f;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
        if (lane == 0) red[32] = t;
    }
    __syncthreads();
    return red[32];
}
// Row of a sequence's latent pages.
template <typename T>
__device__ __forceinline__ T *latent_row(T *plane, const int32_t *table_row, int width, int pos) {
    return plane + ((size_t)table_row[pos >> 4] * kPageTokens + (pos & (kPageTokens - 1))) * width;
}
#endif

}  // namespace juno
