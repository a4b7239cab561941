// BF16 matrix products of many rows on the 5th-generation tensor cores.
//
// A persistent CTA walks 128 x BN output tiles.  One warp streams both operands with TMA (64 K values = 128-byte rows, 128-byte
// swizzle) through a ring of shared-memory stages; one thread issues tcgen05.mma into one of two TMEM accumulators and commits
// each stage back to the ring; four warps drain the other accumulator with tcgen05.ld and apply the epilogue while the next tile
// is multiplied.  Rows, columns and K tails come from the tensor maps (out-of-range elements load as zero) and from guarded
// stores, so sizes need only be multiples of 16.  Every wait is bounded; a wait that runs out marks the launch as failed, the
// copies in flight are waited for, TMEM is freed, and the host reports it after the step.
#include <cuda.h>

#include <algorithm>
#include <cstring>
#include <mutex>

#include "gemm_rows.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

constexpr int kBM = 128, kBK = 64, kTileThreads = 192;
constexpr int kMaxStages = 8;
constexpr long long kWaitClocks = 400000000ll;  // about 0.2 s

struct GemmTcParams {
    CUtensorMap ta, tw;
    GemmArgs g;
    int m_tiles, n_tiles, n_work, k_steps, stages;
    unsigned *err;
};

__device__ __forceinline__ uint32_t s_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ bool bar_test(uint32_t bar, unsigned parity) {
    unsigned ok;
    asm volatile(
        "{\n.reg .pred p;\n"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
        "selp.u32 %0, 1, 0, p;\n}\n"
        : "=r"(ok)
        : "r"(bar), "r"(parity)
        : "memory");
    return ok != 0;
}
__device__ __forceinline__ bool bar_wait(uint32_t bar, unsigned parity, volatile unsigned *fail) {
    if (bar_test(bar, parity)) return true;
    const long long t0 = clock64();
    for (;;) {
        if (bar_test(bar, parity)) return true;
        if (*fail) return false;
        if (clock64() - t0 > kWaitClocks) break;
    }
    *fail = 1u;
    return false;
}
__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cta.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
                 "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(bar)
                 : "memory");
}
// K-major operand with 128-byte swizzle: rows of 128 bytes, groups of eight rows 1024 bytes apart.
__device__ __forceinline__ uint64_t sw128_desc(uint32_t saddr) {
    return (uint64_t)((saddr >> 4) & 0x3FFFu) | (uint64_t)1 << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}
__device__ __forceinline__ void mma_bf16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
    asm volatile(
        "{\n.reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}\n" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"(acc)
        : "memory");
}
__device__ __forceinline__ void mma_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,"
        "%29,%30,%31}, [%32];\n"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
          "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]),
          "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}

__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float fast_geglu(float z, float v) { return z * v * fast_sigmoid(1.5957691216057308f * fmaf(0.044715f * z * z, z, z)); }

// 32 columns of one output row.  nv = columns that exist (0..32).
template <int EPI>
__device__ __forceinline__ void store_row(const GemmArgs &g, int z, int m, int n, int nv, const uint32_t (&r)[32]) {
    const size_t o = (size_t)m * g.ldo + (size_t)z * g.o_step + n;
    if (EPI == GE_F32) {
        float *out = static_cast<float *>(g.out) + o;
        if (g.bias) {  // nv is a multiple of 16 then
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                if (j >= nv) break;
                const float4 b = *reinterpret_cast<const float4 *>(g.bias + n + j);
                *reinterpret_cast<float4 *>(out + j) =
                    make_float4(__uint_as_float(r[j]) + b.x, __uint_as_float(r[j + 1]) + b.y, __uint_as_float(r[j + 2]) + b.z, __uint_as_float(r[j + 3]) + b.w);
            }
        } else if (nv == 32 && (g.ldo & 3) == 0 && (g.o_step & 3) == 0) {
#pragma unroll
            for (int j = 0; j < 32; j += 4)
                *reinterpret_cast<float4 *>(out + j) = make_float4(__uint_as_float(r[j]), __uint_as_float(r[j + 1]), __uint_as_float(r[j + 2]), __uint_as_float(r[j + 3]));
        } else {
#pragma unroll
            for (int j = 0; j < 32; j++)
                if (j < nv) out[j] = __uint_as_float(r[j]);
        }
        return;
    }
    if (EPI == GE_GEGLU) {
        bf16 *act = static_cast<bf16 *>(g.out) + (size_t)m * g.ldo + (n >> 1);
#pragma unroll
        for (int j = 0; j < 32; j += 16) {
            if (j >= nv) break;
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; e++) v[e] = fast_geglu(__uint_as_float(r[j + e]), __uint_as_float(r[j + 8 + e]));
            store4(act + j / 2, make_float4(v[0], v[1], v[2], v[3]));
            store4(act + j / 2 + 4, make_float4(v[4], v[5], v[6], v[7]));
        }
        return;
    }
    float gate = 1.f;
    if (EPI == GE_GROUP_GATE) gate = fast_sigmoid(static_cast<const float *>(g.aux)[(size_t)m * g.ldaux + z]);
    bf16 *out = static_cast<bf16 *>(g.out) + o;
    const bf16 *aux = EPI == GE_MUL ? static_cast<const bf16 *>(g.aux) + (size_t)m * g.ldaux + n : nullptr;
#pragma unroll
    for (int j = 0; j < 32; j += 4) {
        if (j >= nv) break;  // nv is a multiple of 16 on these outputs
        float4 v = make_float4(__uint_as_float(r[j]), __uint_as_float(r[j + 1]), __uint_as_float(r[j + 2]), __uint_as_float(r[j + 3]));
        if (EPI == GE_SIGMOID) {
            const float4 b = *reinterpret_cast<const float4 *>(g.bias + n + j);
            v = make_float4(fast_sigmoid(v.x + b.x), fast_sigmoid(v.y + b.y), fast_sigmoid(v.z + b.z), fast_sigmoid(v.w + b.w));
        } else if (EPI == GE_RELU2) {
            v = make_float4(fmaxf(v.x, 0.f), fmaxf(v.y, 0.f), fmaxf(v.z, 0.f), fmaxf(v.w, 0.f));
            v = make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w);
        } else if (EPI == GE_MUL) {
            const float4 b = load4(aux + j);
            v = make_float4(v.x * b.x, v.y * b.y, v.z * b.z, v.w * b.w);
        } else if (EPI == GE_GROUP_GATE) {
            v = make_float4(v.x * gate, v.y * gate, v.z * gate, v.w * gate);
        }
        store4(out + j, v);
    }
}

template <int BN, int EPI>
__global__ void __launch_bounds__(kTileThreads, 1) gemm_rows_tc_kernel(const __grid_constant__ GemmTcParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bars[2 * kMaxStages + 4];  // full[stages], empty[stages], acc_full[2], acc_empty[2]
    __shared__ uint32_t tmem_slot;
    __shared__ unsigned fail_s;
    volatile unsigned *fail = &fail_s;
    const uint32_t stage0 = (s_u32(smem_raw) + 1023u) & ~1023u;
    constexpr uint32_t kABytes = kBM * kBK * 2, kBBytes = BN * kBK * 2, kStageBytes = kABytes + kBBytes;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, S = p.stages;
    const uint32_t full0 = s_u32(bars), empty0 = full0 + 8 * kMaxStages, accf0 = empty0 + 8 * kMaxStages, acce0 = accf0 + 16;
    if (threadIdx.x == 0) {
        for (int s = 0; s < S; s++) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(full0 + 8 * s) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(empty0 + 8 * s) : "memory");
        }
        for (int s = 0; s < 2; s++) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(accf0 + 8 * s) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 4;" ::"r"(acce0 + 8 * s) : "memory");
        }
        fail_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    constexpr int kTmemCols = 2 * BN < 32 ? 32 : 2 * BN;
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(s_u32(&tmem_slot)), "r"(kTmemCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);
    const GemmArgs &g = p.g;
    pdl_wait();
    pdl_launch_dependents();

    if (warp == 0) {
        if (lane == 0) {
            unsigned it = 0;
            bool ok = true;
            for (int work = blockIdx.x; ok && work < p.n_work; work += gridDim.x) {
                const int mt = work % p.m_tiles, t = work / p.m_tiles, nt = t % p.n_tiles, z = t / p.n_tiles;
                for (int k = 0; k < p.k_steps; k++, it++) {
                    const unsigned s = it % S, use = it / S;
                    if (!(ok = bar_wait(empty0 + 8 * s, (use & 1u) ^ 1u, fail))) break;
                    const uint32_t bar = full0 + 8 * s, a_s = stage0 + s * kStageBytes;
                    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(kStageBytes) : "memory");
                    tma_2d(a_s, &p.ta, z * g.a_step + k * kBK, mt * kBM, bar);
                    tma_2d(a_s + kABytes, &p.tw, k * kBK, z * g.w_step + nt * BN, bar);
                }
            }
            // the last copies of every stage: nothing may be in flight when the CTA leaves
            for (int b = 0; b < S && b < (int)it; b++) {
                const unsigned j = it - 1 - b, s = j % S;
                const long long t0 = clock64();
                while (!bar_test(full0 + 8 * s, (j / S) & 1u) && clock64() - t0 < kWaitClocks) {
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // D FP32, A and B BF16, both K-major
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kBM >> 4) << 24);
            unsigned it = 0, tile = 0;
            bool ok = true;
            for (int work = blockIdx.x; ok && work < p.n_work; work += gridDim.x, tile++) {
                const unsigned acc = tile & 1u;
                if (!(ok = bar_wait(acce0 + 8 * acc, ((tile >> 1) & 1u) ^ 1u, fail))) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t d = tmem + acc * BN;
                for (int k = 0; k < p.k_steps; k++, it++) {
                    const unsigned s = it % S, use = it / S;
                    if (!(ok = bar_wait(full0 + 8 * s, use & 1u, fail))) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t ad = sw128_desc(stage0 + s * kStageBytes), bd = sw128_desc(stage0 + s * kStageBytes + kABytes);
#pragma unroll
                    for (int j = 0; j < kBK / 16; j++) mma_bf16(d, ad + 2 * j, bd + 2 * j, idesc, (k > 0 || j > 0) ? 1u : 0u);
                    mma_commit(empty0 + 8 * s);
                }
                if (ok) mma_commit(accf0 + 8 * acc);
            }
        }
    } else {
        const int quad = warp & 3;  // TMEM lanes a warp can read: 32 * (warp % 4) ..
        unsigned tile = 0;
        for (int work = blockIdx.x; work < p.n_work; work += gridDim.x, tile++) {
            const int mt = work % p.m_tiles, t = work / p.m_tiles, nt = t % p.n_tiles, z = t / p.n_tiles;
            const unsigned acc = tile & 1u;
            int ok = 0;
            if (lane == 0) ok = bar_wait(accf0 + 8 * acc, (tile >> 1) & 1u, fail) ? 1 : 0;
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int m = mt * kBM + quad * 32 + lane;
#pragma unroll 1
            for (int c0 = 0; c0 < BN; c0 += 32) {
                const int n = nt * BN + c0, nv = min(32, g.N - n);
                if (nv <= 0) break;
                uint32_t r[32];
                tmem_ld32(tmem + ((uint32_t)(quad * 32) << 16) + acc * BN + (uint32_t)c0, r);
                if (m < g.M) store_row<EPI>(g, z, m, n, nv, r);
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(acce0 + 8 * acc) : "memory");
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (*fail) {  // MMAs that were issued before the failure still write TMEM: let them finish (bounded) before it is freed
            const long long t0 = clock64();
            while (clock64() - t0 < 4000000ll) {
            }
            if (lane == 0) atomicCAS(p.err, 0u, kErrStackWait | (1u << 8) | (blockIdx.x << 16));
        }
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols) : "memory");
    }
}

// ───────────────────────────── host ───────────────────────────────────────────────────────
typedef CUresult (*EncodeTiled)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                                const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiled encode_tiled() {
    static EncodeTiled fn = [] {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) p = nullptr;
        return reinterpret_cast<EncodeTiled>(p);
    }();
    return fn;
}

// Row-major BF16 matrix [rows][cols] with pitch ld, boxes of box_rows x 64 columns.
int tensor_map_bf16(CUtensorMap *map, const void *base, int64_t rows, int64_t cols, int64_t ld, int box_rows) {
    EncodeTiled enc = encode_tiled();
    JUNO_REQUIRE(enc, "the driver has no cuTensorMapEncodeTiled");
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kBK, (cuuint32_t)box_rows}, es[2] = {1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    JUNO_REQUIRE(r == CUDA_SUCCESS, "cuTensorMapEncodeTiled failed: rc=%d (%lld x %lld, pitch %lld)", (int)r, (long long)rows, (long long)cols, (long long)ld);
    return JUNO_OK;
}

template <int BN, int EPI>
static int gemm_tc_inst(juno_ctx *c, const GemmTcParams &p, cudaStream_t st) {
    const size_t smem = (size_t)p.stages * (kBM + BN) * kBK * 2 + 1024;
    static std::mutex mu;
    static bool configured[16] = {false};
    {
        std::lock_guard<std::mutex> lk(mu);
        if (!configured[c->device & 15]) {
            JUNO_CUDA_TRY(cudaFuncSetAttribute(gemm_rows_tc_kernel<BN, EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
            configured[c->device & 15] = true;
        }
    }
    JUNO_CUDA_TRY(launch_pdl(gemm_rows_tc_kernel<BN, EPI>, dim3((unsigned)std::min(p.n_work, c->sm_count)), dim3(kTileThreads), smem, st, p));
    c->kernel_launches++;
    return JUNO_OK;
}
template <int BN>
static int gemm_tc_epi(juno_ctx *c, const GemmTcParams &p, cudaStream_t st) {
    switch (p.g.epi) {
    case GE_F32: return gemm_tc_inst<BN, GE_F32>(c, p, st);
    case GE_OP: return gemm_tc_inst<BN, GE_OP>(c, p, st);
    case GE_SIGMOID: return gemm_tc_inst<BN, GE_SIGMOID>(c, p, st);
    case GE_RELU2: return gemm_tc_inst<BN, GE_RELU2>(c, p, st);
    case GE_MUL: return gemm_tc_inst<BN, GE_MUL>(c, p, st);
    case GE_GEGLU: return gemm_tc_inst<BN, GE_GEGLU>(c, p, st);
    default: return gemm_tc_inst<BN, GE_GROUP_GATE>(c, p, st);
    }
}

int launch_gemm_rows_tc(juno_ctx *c, const GemmArgs &a, unsigned *err, cudaStream_t st) {
    GemmTcParams p;
    memset(&p, 0, sizeof(p));
    p.g = a;
    p.err = err;
    p.m_tiles = (a.M + kBM - 1) / kBM;
    p.k_steps = (a.K + kBK - 1) / kBK;
    // tile width: rounds of tiles over the SMs, each as long as its columns and a fixed share (operand A, start-up, epilogue)
    int bn = 32;
    double best = 1e30;
    for (int w = 256; w >= 32; w /= 2) {
        if (w > 32 && w / 2 >= a.N) continue;
        const long long tiles = (long long)p.m_tiles * ((a.N + w - 1) / w) * a.groups;
        const double cost = (double)((tiles + c->sm_count - 1) / c->sm_count) * (w + 40);
        if (cost < best) {
            best = cost;
            bn = w;
        }
    }
    p.n_tiles = (a.N + bn - 1) / bn;
    p.n_work = p.m_tiles * p.n_tiles * a.groups;
    p.stages = std::min(kMaxStages, 192 * 1024 / ((kBM + bn) * kBK * 2));
    const int a_cols = a.groups > 1 ? a.a_step * (a.groups - 1) + a.K : a.K;
    const int w_rows = a.w_rows ? a.w_rows : a.groups > 1 ? a.w_step * (a.groups - 1) + a.N : a.N;
    JUNO_TRY(tensor_map_bf16(&p.ta, a.a, a.M, a_cols, a.lda, kBM));
    JUNO_TRY(tensor_map_bf16(&p.tw, a.w, w_rows, a.K, a.ldw, bn));
    switch (bn) {
    case 256: return gemm_tc_epi<256>(c, p, st);
    case 128: return gemm_tc_epi<128>(c, p, st);
    case 64: return gemm_tc_epi<64>(c, p, st);
    default: return gemm_tc_epi<32>(c, p, st);
    }
}

}  // namespace juno
