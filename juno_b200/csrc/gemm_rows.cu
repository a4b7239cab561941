// Matrix products of many rows.  BF16 runs on the tensor cores (gemm_rows_tc.cu); FP32 runs on the FMA units in true 32-bit (no reduced-precision matrix mode).
#include "gemm_rows.cuh"

#include <algorithm>

namespace juno {

constexpr int kSimtTile = 64, kSimtK = 16;

template <typename T>
__device__ __forceinline__ void simt_epilogue(const GemmArgs &p, int z, int m, int n, float v) {
    const size_t o = (size_t)m * p.ldo + (size_t)z * p.o_step + n;
    if (p.epi == GE_F32) {
        static_cast<float *>(p.out)[o] = p.bias ? v + p.bias[n] : v;
        return;
    }
    if (p.epi == GE_SIGMOID) v = sigmoid_f32(v + p.bias[n]);
    if (p.epi == GE_RELU2) {
        v = fmaxf(v, 0.f);
        v *= v;
    }
    if (p.epi == GE_MUL) v *= Num<T>::get(static_cast<const T *>(p.aux)[(size_t)m * p.ldaux + n]);
    if (p.epi == GE_GROUP_GATE) v *= sigmoid_f32(static_cast<const float *>(p.aux)[(size_t)m * p.ldaux + z]);
    static_cast<T *>(p.out)[o] = Num<T>::put(v);
}

// 64 x 64 tile, 4 x 4 outputs per thread.
template <typename T>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const GemmArgs p) {
    __shared__ __align__(16) float as[kSimtK][kSimtTile + 4], ws[kSimtK][kSimtTile + 4];
    const int z = blockIdx.z, m0 = blockIdx.y * kSimtTile, n0 = blockIdx.x * kSimtTile;
    const T *a = static_cast<const T *>(p.a) + (size_t)z * p.a_step;
    const T *w = static_cast<const T *>(p.w) + (size_t)z * p.w_step * p.ldw;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int lr = tid >> 2, lk = (tid & 3) * 4;  // loader: row, first of four k
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += kSimtK) {
        float4 av = make_float4(0.f, 0.f, 0.f, 0.f), wv = av;
        if (m0 + lr < p.M) av = load4(a + (size_t)(m0 + lr) * p.lda + k0 + lk);
        if (n0 + lr < p.N) wv = load4(w + (size_t)(n0 + lr) * p.ldw + k0 + lk);
        __syncthreads();
        as[lk][lr] = av.x, as[lk + 1][lr] = av.y, as[lk + 2][lr] = av.z, as[lk + 3][lr] = av.w;
        ws[lk][lr] = wv.x, ws[lk + 1][lr] = wv.y, ws[lk + 2][lr] = wv.z, ws[lk + 3][lr] = wv.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kSimtK; k++) {
            const float4 x = *reinterpret_cast<const float4 *>(&as[k][ty * 4]), y = *reinterpret_cast<const float4 *>(&ws[k][tx * 4]);
            const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], yv[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (p.epi == GE_GEGLU) {  // the value of column n is eight columns on: two threads further
                const float value = __shfl_down_sync(0xffffffffu, acc[i][j], 2);
                if (m < p.M && n < p.N && !(n & 8))
                    static_cast<T *>(p.out)[(size_t)m * p.ldo + (n >> 4) * 8 + (n & 7)] = Num<T>::put(gelu_tanh(acc[i][j]) * value);
                continue;
            }
            if (m < p.M && n < p.N) simt_epilogue<T>(p, z, m, n, acc[i][j]);
        }
}

int launch_gemm_rows(juno_ctx *c, int dt, const GemmArgs &a, unsigned *err, cudaStream_t st) {
    JUNO_REQUIRE(a.a && a.w && a.out && a.M > 0 && a.N > 0 && a.K > 0 && a.K % 16 == 0 && a.lda % 16 == 0 && a.ldw % 16 == 0 && a.a_step % 16 == 0 && a.groups >= 1 &&
                     (a.epi != GE_GEGLU || (a.N % 16 == 0 && a.groups == 1)),
                 "matrix product: bad arguments (M %d, N %d, K %d)", a.M, a.N, a.K);
    const double es = dt_bytes(dt);
    const double algo = a.groups * ((double)a.M * a.K + (double)a.N * a.K) * es + (double)a.groups * a.M * a.N * (a.epi == GE_F32 ? 4.0 : es);
    ProfScope prof(c, st, PROF_GEMM_ROWS, algo);
    if (dt == DT_BF16) return launch_gemm_rows_tc(c, a, err, st);
    const dim3 grid((unsigned)((a.N + kSimtTile - 1) / kSimtTile), (unsigned)((a.M + kSimtTile - 1) / kSimtTile), (unsigned)a.groups);
    gemm_simt_kernel<float><<<grid, 256, 0, st>>>(a);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

}  // namespace juno
