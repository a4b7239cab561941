// Row kernels of hyper-connections (see streams.cuh).  They stream every row once; the sublayer's input stays in shared memory
// between the pass that sums its squares and the pass that scales it.
#include "streams.cuh"

namespace juno {

using bf16 = __nv_bfloat16;
constexpr int kStThreads = 256;

__device__ __forceinline__ float4 fma4(float s, float4 a, float4 b) {
    return make_float4(fmaf(s, a.x, b.x), fmaf(s, a.y, b.y), fmaf(s, a.z, b.z), fmaf(s, a.w, b.w));
}
__device__ __forceinline__ float4 mul4(float s, float4 a) { return make_float4(s * a.x, s * a.y, s * a.z, s * a.w); }
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

template <typename T>
__global__ void __launch_bounds__(kStThreads) stream_embed_kernel(const T *embed, int ld_embed, int vocab, int streams, const int32_t *tokens, float *x, int ldx) {
    const int r = blockIdx.x;
    const T *e = embed + (size_t)max(0, min(tokens[r], vocab - 1)) * ld_embed;
    float *row = x + (size_t)r * streams * ldx;
    for (int i = threadIdx.x * 4; i < ldx; i += kStThreads * 4) {
        const float4 v = load4(e + i);
        for (int s = 0; s < streams; s++) store4(row + (size_t)s * ldx + i, v);
    }
}

// S: the number of streams when it is a common one (the old streams stay in registers), else 0
template <typename T, int S>
__global__ void __launch_bounds__(kStThreads) stream_step_kernel(const StreamStepArgs a) {
    extern __shared__ __align__(16) float row[];  // the sublayer's input
    __shared__ float red[33], mix[kMaxStreams * kMaxStreams], out[kMaxStreams], in[kMaxStreams];
    const int r = blockIdx.x, ns = S ? S : a.streams, tid = threadIdx.x;
    if (tid < ns * ns) mix[tid] = a.z ? a.mix[tid] : 0.f;
    if (tid < ns) {
        out[tid] = a.z ? a.out[tid] : 0.f;
        in[tid] = a.h ? a.in[tid] : 0.f;
    }
    __syncthreads();
    float *x = a.x + (size_t)r * ns * a.ldx;
    const T *z = a.z ? static_cast<const T *>(a.z) + (size_t)r * a.ldz : nullptr;
    float sx = 0.f;
    for (int i = tid * 4; i < a.ldx; i += kStThreads * 4) {
        constexpr int N = S ? S : kMaxStreams;
        float4 old[N];
#pragma unroll
        for (int s = 0; s < N; s++)
            if (S || s < ns) old[s] = load4(x + (size_t)s * a.ldx + i);
        float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
        if (z) {
            const float4 y = load4(z + i);
#pragma unroll
            for (int t = 0; t < N; t++)
                if (S || t < ns) {
                    float4 v = mul4(out[t], y);
#pragma unroll
                    for (int s = 0; s < N; s++)
                        if (S || s < ns) v = fma4(mix[s * ns + t], old[s], v);
                    store4(x + (size_t)t * a.ldx + i, v);
                    u = fma4(in[t], v, u);
                }
        } else {
#pragma unroll
            for (int s = 0; s < N; s++)
                if (S || s < ns) u = fma4(in[s], old[s], u);
        }
        if (a.h) store4(row + i, u);
        sx += sq4(u);
    }
    if (!a.h) return;
    sx = block_sum(sx, red);
    const float k = 1.f / sqrtf(sx / (float)a.width + a.eps);
    T *h = static_cast<T *>(a.h) + (size_t)r * a.ldh;
    for (int i = tid * 4; i < a.ldx; i += kStThreads * 4) {
        const float4 v = load4(row + i), w = load4(a.w + i);
        store4(h + i, make_float4(v.x * k * w.x, v.y * k * w.y, v.z * k * w.z, v.w * k * w.w));
    }
}

template <typename T>
__global__ void __launch_bounds__(kStThreads) stream_gather_kernel(const float *x, int streams, int ldx, int width, const int32_t *row_idx, const float *w, float eps,
                                                                   T *out, float *sum, int ldo) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const int i0 = blockIdx.x, r = row_idx ? row_idx[i0] : i0;
    const float *xr = x + (size_t)r * streams * ldx;
    float sx = 0.f;
    for (int i = threadIdx.x * 4; i < ldx; i += kStThreads * 4) {
        float4 u = load4(xr + i);
        for (int s = 1; s < streams; s++) u = fma4(1.f, load4(xr + (size_t)s * ldx + i), u);
        if (sum)
            store4(sum + (size_t)i0 * ldo + i, u);
        else
            store4(row + i, u);
        sx += sq4(u);
    }
    if (sum) return;
    const float k = 1.f / sqrtf(block_sum(sx, red) / (float)width + eps);
    for (int i = threadIdx.x * 4; i < ldx; i += kStThreads * 4) {
        const float4 v = load4(row + i), g = load4(w + i);
        store4(out + (size_t)i0 * ldo + i, make_float4(v.x * k * g.x, v.y * k * g.y, v.z * k * g.z, v.w * k * g.w));
    }
}

// ───────────────────────────── launches ───────────────────────────────────────────────────
static bool streams_ok(int streams, int ldx, int width) { return streams >= 1 && streams <= kMaxStreams && ldx % 16 == 0 && width > 0 && width <= ldx && ldx <= 49152; }

template <typename K>
static int row_smem(K kernel, size_t bytes) {
    if (bytes > 48 * 1024) JUNO_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    return JUNO_OK;
}

int launch_stream_embed(juno_ctx *c, int dt, const void *embed, int ld_embed, int width, int vocab, int streams, const RowSet &rows, float *x, int ldx,
                        cudaStream_t st) {
    JUNO_REQUIRE(rows.n > 0 && streams_ok(streams, ldx, width) && ld_embed == ldx, "embedding of streams: bad arguments");
    ProfScope prof(c, st, PROF_ROWOPS, (double)rows.n * width * (dt_bytes(dt) + 4 * streams));
    if (dt == DT_F32)
        stream_embed_kernel<float><<<rows.n, kStThreads, 0, st>>>(static_cast<const float *>(embed), ld_embed, vocab, streams, rows.tokens, x, ldx);
    else
        stream_embed_kernel<bf16><<<rows.n, kStThreads, 0, st>>>(static_cast<const bf16 *>(embed), ld_embed, vocab, streams, rows.tokens, x, ldx);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

template <typename T, int S>
static int step_inst(const StreamStepArgs &a, cudaStream_t st) {
    const size_t smem = (size_t)a.ldx * 4;
    JUNO_TRY(row_smem(stream_step_kernel<T, S>, smem));
    stream_step_kernel<T, S><<<a.n, kStThreads, smem, st>>>(a);
    return JUNO_OK;
}
template <typename T>
static int step_streams(const StreamStepArgs &a, cudaStream_t st) {
    switch (a.streams) {
    case 1: return step_inst<T, 1>(a, st);
    case 2: return step_inst<T, 2>(a, st);
    case 3: return step_inst<T, 3>(a, st);
    case 4: return step_inst<T, 4>(a, st);
    default: return step_inst<T, 0>(a, st);
    }
}
int launch_stream_step(juno_ctx *c, int dt, const StreamStepArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.n > 0 && a.x && streams_ok(a.streams, a.ldx, a.width) && (!a.z || (a.ldz >= a.ldx && a.mix && a.out)) && (!a.h || (a.ldh >= a.ldx && a.in && a.w)),
                 "stream step: bad arguments");
    const double es = dt_bytes(dt);
    ProfScope prof(c, st, PROF_ROWOPS, (double)a.n * a.width * (a.streams * (a.z ? 8.0 : 4.0) + (a.z ? es : 0) + (a.h ? es : 0)));
    JUNO_TRY(dt == DT_F32 ? step_streams<float>(a, st) : step_streams<bf16>(a, st));
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_stream_gather(juno_ctx *c, int dt, const float *x, int streams, int ldx, int width, const int32_t *row_idx, int n, const float *w, float eps,
                         void *out, int ldo, cudaStream_t st) {
    JUNO_REQUIRE(n > 0 && streams_ok(streams, ldx, width) && ldo >= ldx, "stream norm: bad arguments");
    float *sum = w ? nullptr : static_cast<float *>(out);
    const size_t smem = sum ? 0 : (size_t)ldx * 4;
    ProfScope prof(c, st, PROF_ROWOPS, (double)n * width * (4 * streams + dt_bytes(dt)));
    if (dt == DT_F32 || sum) {
        JUNO_TRY(row_smem(stream_gather_kernel<float>, smem));
        stream_gather_kernel<float><<<n, kStThreads, smem, st>>>(x, streams, ldx, width, row_idx, w, eps, static_cast<float *>(out), sum, ldo);
    } else {
        JUNO_TRY(row_smem(stream_gather_kernel<bf16>, smem));
        stream_gather_kernel<bf16><<<n, kStThreads, smem, st>>>(x, streams, ldx, width, row_idx, w, eps, static_cast<bf16 *>(out), sum, ldo);
    }
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

}  // namespace juno
