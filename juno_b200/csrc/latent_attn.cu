// Attention over latent pages (see latent_attn.cuh).
#include "latent_attn.cuh"

#include <algorithm>

namespace juno {

using bf16 = __nv_bfloat16;

constexpr int kLaHeads = 4, kLaKeys = 64, kLaThreads = 256, kLaCols = 8;  // columns per thread: rank <= 2048

struct LatentSimtParams {
    const void *plane;
    const int32_t *table, *positions, *slots;
    int max_pages, heads, rank;
    float scale;
    const void *q;
    void *o;
};

// Scores by warps (a warp takes a key, its lanes the rank), online softmax per head, then one thread per latent column.
template <typename T>
__global__ void __launch_bounds__(kLaThreads) latent_attn_simt_kernel(const LatentSimtParams p) {
    extern __shared__ __align__(16) float qs[];  // [kLaHeads][rank]
    __shared__ float sc[kLaHeads][kLaKeys], run_max[kLaHeads], run_sum[kLaHeads], fac[kLaHeads];
    const int row = blockIdx.y, h0 = blockIdx.x * kLaHeads, nh = min(kLaHeads, p.heads - h0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, R = p.rank;
    const int32_t *table = p.table + (size_t)p.slots[row] * p.max_pages;
    const T *plane = static_cast<const T *>(p.plane);
    const int len = p.positions[row] + 1;
    const T *q = static_cast<const T *>(p.q) + ((size_t)row * p.heads + h0) * R;
    for (int i = tid; i < kLaHeads * R; i += kLaThreads) qs[i] = i < nh * R ? Num<T>::get(q[i]) * p.scale : 0.f;
    if (tid < kLaHeads) {
        run_max[tid] = -INFINITY;
        run_sum[tid] = 0.f;
    }
    float acc[kLaHeads][kLaCols];
#pragma unroll
    for (int h = 0; h < kLaHeads; h++)
#pragma unroll
        for (int k = 0; k < kLaCols; k++) acc[h][k] = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 < len; j0 += kLaKeys) {
        const int nj = min(kLaKeys, len - j0);
        for (int j = warp; j < nj; j += kLaThreads / 32) {
            const T *c = latent_row(plane, table, R, j0 + j);
            float d[kLaHeads] = {};
            for (int i = lane; i < R; i += 32) {
                const float v = Num<T>::get(c[i]);
#pragma unroll
                for (int h = 0; h < kLaHeads; h++) d[h] = fmaf(v, qs[h * R + i], d[h]);
            }
#pragma unroll
            for (int h = 0; h < kLaHeads; h++) {
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) d[h] += __shfl_xor_sync(0xffffffffu, d[h], o);
                if (lane == 0) sc[h][j] = d[h];
            }
        }
        __syncthreads();
        if (warp < kLaHeads) {
            const float a0 = lane < nj ? sc[warp][lane] : -INFINITY, a1 = lane + 32 < nj ? sc[warp][lane + 32] : -INFINITY;
            float m = fmaxf(a0, a1);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
            m = fmaxf(m, run_max[warp]);
            const float e0 = expf(a0 - m), e1 = expf(a1 - m);
            float s = e0 + e1;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            sc[warp][lane] = e0;
            sc[warp][lane + 32] = e1;
            if (lane == 0) {
                const float f = expf(run_max[warp] - m);
                fac[warp] = f;
                run_sum[warp] = run_sum[warp] * f + s;
                run_max[warp] = m;
            }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kLaCols; k++) {
            const int col = tid + k * kLaThreads;
            if (col < R) {
#pragma unroll
                for (int h = 0; h < kLaHeads; h++) acc[h][k] *= fac[h];
                for (int j = 0; j < nj; j++) {
                    const float v = Num<T>::get(latent_row(plane, table, R, j0 + j)[col]);
#pragma unroll
                    for (int h = 0; h < kLaHeads; h++) acc[h][k] = fmaf(sc[h][j], v, acc[h][k]);
                }
            }
        }
        __syncthreads();
    }
    T *o = static_cast<T *>(p.o) + ((size_t)row * p.heads + h0) * R;
#pragma unroll
    for (int k = 0; k < kLaCols; k++) {
        const int col = tid + k * kLaThreads;
        if (col < R)
#pragma unroll
            for (int h = 0; h < kLaHeads; h++)
                if (h < nh) o[(size_t)h * R + col] = Num<T>::put(acc[h][k] / run_sum[h]);
    }
}

int launch_latent_attn_simt(juno_ctx *c, int dt, const LatentAttnArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.rows.n > 0 && a.heads > 0 && a.rank > 0 && a.rank % 16 == 0 && a.pool->latent && a.pool->row_width[a.layer] == a.rank, "latent attention: bad arguments");
    JUNO_REQUIRE(a.rank <= kLaThreads * kLaCols, "latent attention: a latent of %d is wider than %d", a.rank, kLaThreads * kLaCols);
    LatentSimtParams p;
    p.plane = static_cast<const uint8_t *>(a.pool->k) + a.pool->row_off[a.layer] * a.pool->elem_bytes;
    p.table = a.pool->d_table;
    p.positions = a.rows.positions;
    p.slots = a.rows.slots;
    p.max_pages = a.pool->max_pages_per_seq;
    p.heads = a.heads;
    p.rank = a.rank;
    p.scale = a.scale;
    p.q = a.q_lat;
    p.o = a.o_lat;
    const dim3 grid((unsigned)((a.heads + kLaHeads - 1) / kLaHeads), (unsigned)a.rows.n);
    const size_t smem = (size_t)kLaHeads * a.rank * 4;
    ProfScope prof(c, st, PROF_ATTN, 0);
    if (dt == DT_F32)
        latent_attn_simt_kernel<float><<<grid, kLaThreads, smem, st>>>(p);
    else
        latent_attn_simt_kernel<bf16><<<grid, kLaThreads, smem, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

}  // namespace juno
