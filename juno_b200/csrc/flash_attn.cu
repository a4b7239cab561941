// Causal flash attention of many rows of one sequence (see flash_attn.cuh), BF16 operands on mma.sync.
#include <algorithm>
#include <cstring>
#include <mutex>

#include "flash_attn.cuh"
#include "mma_bf16.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

// 64 * MT query rows of one head per CTA, four warps of MT 16-row tiles; 64 keys per step, keys and values double-buffered.
constexpr int kFlKeys = 64, kFlThreads = 128;
struct FlashParams {
    FlashArgs a;
    float scale_log2;
    const bf16 *plane;     // paged form
    const int32_t *table;
    int max_pages, row_width;
};
// D: most dimensions per head; MT: 16-row tiles per warp; PAGED: keys and values from the sequence's pages, with key spans,
// distance slopes and sinks (scores are kept in the log2 domain then); EXACT: query, key and value size are D
template <int D, int MT, bool PAGED, bool EXACT>
__global__ void __launch_bounds__(kFlThreads, D <= 128 ? 2 : 1) flash_prefill_kernel(const FlashParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    constexpr int BR = 64 * MT, NK = D / 16, NV = D / 16;
    const FlashArgs &a = p.a;
    const int dp = EXACT ? D : a.dim, vp = EXACT ? D : a.vdim, kp = dp + 8, vpitch = vp + 8, nk = dp >> 4, nv = vp >> 4;
    bf16 *qs = reinterpret_cast<bf16 *>(sm);
    bf16 *ks = qs + BR * kp;                 // [2][64][kp]
    bf16 *vs = ks + 2 * kFlKeys * kp;        // [2][64][vpitch]
    const int h = blockIdx.x, r0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * BR;  // long rows first
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bf16 *q = static_cast<const bf16 *>(a.q) + (size_t)h * dp;
    const bf16 *kv = static_cast<const bf16 *>(a.kv);
    const int G = a.kv_heads, kvh = PAGED ? h / (a.heads / G) : h;
    const int32_t *table = PAGED ? p.table + (size_t)*a.slot * p.max_pages : nullptr;
    const int ldq = a.heads * dp, rows = min(BR, a.n - r0), len = a.pos0 + r0 + rows;  // keys any row of the tile sees
    const int kc = dp >> 3, vc = vp >> 3;
    // this thread's first (row, 16-byte piece) of a tile and the step to its next, for keys and values
    const int kr0 = tid / kc, kch0 = tid - kr0 * kc, krs = kFlThreads / kc, kcs = kFlThreads - krs * kc;
    const int vr0 = tid / vc, vch0 = tid - vr0 * vc, vrs = kFlThreads / vc, vcs = kFlThreads - vrs * vc;
    const int first = PAGED ? a.span.first(a.pos0 + r0) : 0;  // first key any row of the tile sees
    auto load_rows = [&](const bf16 *src, uint32_t dst, int pitch, int j, int r, int ch, int rs, int chs, int nch) {
        while (r < kFlKeys) {
            const bool ok = j + r < len && (!PAGED || j + r >= first);
            const bf16 *s = src + ch * 8;
            if (PAGED)
                s += ok ? ((size_t)table[(j + r) >> 4] * kPageTokens + ((j + r) & (kPageTokens - 1))) * p.row_width : 0;
            else
                s += (size_t)(ok ? j + r : 0) * a.ldkv;
            cp16(dst + (uint32_t)(r * pitch + ch * 8) * 2, s, ok);
            ch += chs;
            r += rs;
            if (ch >= nch) {
                ch -= nch;
                r++;
            }
        }
    };
    auto load_kv = [&](int j, int buf) {
        const bf16 *base = PAGED ? p.plane : kv;
        if (EXACT && j >= first && j + kFlKeys <= len) {  // every row exists: a thread's pieces lie in one column of them
            constexpr int RS = kFlThreads / (D / 8);  // rows between them
            const bf16 *ksrc = base + kvh * dp + kch0 * 8, *vsrc = base + G * dp + kvh * vp + kch0 * 8;
            const uint32_t kd = smem_addr(ks + ((size_t)buf * kFlKeys + kr0) * kp + kch0 * 8), vd = smem_addr(vs + ((size_t)buf * kFlKeys + kr0) * vpitch + kch0 * 8);
            const size_t step = PAGED ? (size_t)p.row_width : (size_t)a.ldkv;
#pragma unroll
            for (int pg = 0; pg < kFlKeys / kPageTokens; pg++) {
                const size_t row0 = PAGED ? (size_t)table[(j >> 4) + pg] * kPageTokens : (size_t)j + pg * kPageTokens;
                size_t off = (row0 + kr0) * step;
#pragma unroll
                for (int r = 0; r < kPageTokens; r += RS, off += RS * step) {
                    const uint32_t d = (uint32_t)((pg * kPageTokens + r) * kp) * 2;  // kp == vpitch
                    cp16(kd + d, ksrc + off, true);
                    cp16(vd + d, vsrc + off, true);
                }
            }
            cp_commit();
            return;
        }
        load_rows(base + kvh * dp, smem_addr(ks + (size_t)buf * kFlKeys * kp), kp, j, kr0, kch0, krs, kcs, kc);
        load_rows(base + G * dp + kvh * vp, smem_addr(vs + (size_t)buf * kFlKeys * vpitch), vpitch, j, vr0, vch0, vrs, vcs, vc);
        cp_commit();
    };
    for (int i = tid; i < BR * kc; i += kFlThreads) {
        const int r = i / kc, ch = i - r * kc;
        const bool ok = r < rows;
        cp16(smem_addr(qs + r * kp + ch * 8), q + (size_t)(ok ? r0 + r : r0) * ldq + ch * 8, ok);
    }
    const int j0 = first & ~(kFlKeys - 1);
    load_kv(j0, 0);
    const int lr = lane & 15, lc = (lane >> 4) * 8, br = (lane & 7) + (lane >> 4) * 8, bc = ((lane >> 3) & 1) * 8;
    const int g = lane >> 2, t = lane & 3, wrow = warp * 16 * MT;
    float o[MT][NV][2][4], mx[MT][2], ls[MT][2];
    int lo[MT][2];  // first key of the rows g and g + 8 (paged form)
    const float slope = PAGED && a.slopes ? a.slopes[h] * kLog2e : 0.f;
    const bool sink = PAGED && a.sinks;  // the sink is one more key, seen first, without a value
    const float sink_l2 = sink ? a.sinks[h] * kLog2e : -INFINITY;
    const int wlo = PAGED ? a.span.first(a.pos0 + r0 + wrow) : 0;
#pragma unroll
    for (int m = 0; m < MT; m++) {
        mx[m][0] = mx[m][1] = sink_l2;
        ls[m][0] = ls[m][1] = sink && t == 0 ? 1.f : 0.f;
        lo[m][0] = PAGED ? a.span.first(a.pos0 + r0 + wrow + m * 16 + g) : 0;
        lo[m][1] = PAGED ? a.span.first(a.pos0 + r0 + wrow + m * 16 + g + 8) : 0;
#pragma unroll
        for (int i = 0; i < NV; i++)
#pragma unroll
            for (int k = 0; k < 2; k++)
#pragma unroll
                for (int e = 0; e < 4; e++) o[m][i][k][e] = 0.f;
    }
    int buf = 0;
    for (int j = j0; j < len; j += kFlKeys, buf ^= 1) {
        cp_wait<0>();
        __syncthreads();
        if (j + kFlKeys < len) load_kv(j + kFlKeys, buf ^ 1);
        if (j > a.pos0 + r0 + wrow + 16 * MT - 1) continue;  // every key of the tile lies behind this warp's rows
        if (PAGED && j + kFlKeys <= wlo) continue;                // or before the first that they see
        const bf16 *kt = ks + (size_t)buf * kFlKeys * kp, *vt = vs + (size_t)buf * kFlKeys * vpitch;
        float s[MT][kFlKeys / 8][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int i = 0; i < kFlKeys / 8; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[m][i][e] = 0.f;
#pragma unroll
        for (int k = 0; k < NK; k++) {
            if (k < nk) {
                uint32_t qa[MT][4];
#pragma unroll
                for (int m = 0; m < MT; m++) ldsm4(qa[m], smem_addr(qs + (wrow + m * 16 + lr) * kp + k * 16 + lc));
#pragma unroll
                for (int i = 0; i < kFlKeys / 16; i++) {
                    uint32_t b[4];
                    ldsm4(b, smem_addr(kt + (i * 16 + br) * kp + k * 16 + bc));
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        mma16816(s[m][2 * i], qa[m], b[0], b[1]);
                        mma16816(s[m][2 * i + 1], qa[m], b[2], b[3]);
                    }
                }
            }
        }
        uint32_t pa[MT][kFlKeys / 16][4];
#pragma unroll
        for (int m = 0; m < MT; m++) {
#pragma unroll
            for (int e2 = 0; e2 < 2; e2++) {  // rows g and g + 8
                const int pos = a.pos0 + r0 + wrow + m * 16 + g + e2 * 8;
                float mv = mx[m][e2];
                if (PAGED && a.slopes) {
                    const float b0 = (float)(j + 2 * t - pos) * slope;
#pragma unroll
                    for (int i = 0; i < kFlKeys / 8; i++)
#pragma unroll
                        for (int e = 0; e < 2; e++) s[m][i][e2 * 2 + e] = fmaf(s[m][i][e2 * 2 + e], p.scale_log2, fmaf((float)(i * 8 + e), slope, b0));
                } else if (PAGED) {
#pragma unroll
                    for (int i = 0; i < kFlKeys / 8; i++)
#pragma unroll
                        for (int e = 0; e < 2; e++) s[m][i][e2 * 2 + e] *= p.scale_log2;
                }
                if (j + kFlKeys - 1 > pos || (PAGED && j < lo[m][e2])) {
#pragma unroll
                    for (int i = 0; i < kFlKeys / 8; i++)
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            const int key = j + i * 8 + 2 * t + e;
                            if (key > pos || (PAGED && key < lo[m][e2])) s[m][i][e2 * 2 + e] = -INFINITY;
                        }
                }
#pragma unroll
                for (int i = 0; i < kFlKeys / 8; i++) mv = fmaxf(mv, fmaxf(s[m][i][e2 * 2], s[m][i][e2 * 2 + 1]));
                mv = fmaxf(mv, __shfl_xor_sync(0xffffffffu, mv, 1));
                mv = fmaxf(mv, __shfl_xor_sync(0xffffffffu, mv, 2));
                const float unit = PAGED ? 1.f : p.scale_log2;
                const float base = mv == -INFINITY ? 0.f : mv * unit;
                const float f = ex2(mx[m][e2] * unit - base);
                mx[m][e2] = mv;
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < kFlKeys / 8; i++)
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const float v = PAGED ? ex2(s[m][i][e2 * 2 + e] - base) : ex2(fmaf(s[m][i][e2 * 2 + e], p.scale_log2, -base));
                        s[m][i][e2 * 2 + e] = v;
                        sum += v;
                    }
                ls[m][e2] = ls[m][e2] * f + sum;
#pragma unroll
                for (int i = 0; i < NV; i++)
#pragma unroll
                    for (int k = 0; k < 2; k++) {
                        o[m][i][k][e2 * 2] *= f;
                        o[m][i][k][e2 * 2 + 1] *= f;
                    }
            }
#pragma unroll
            for (int i = 0; i < kFlKeys / 16; i++) {
                pa[m][i][0] = pack_bf16(s[m][2 * i][0], s[m][2 * i][1]);
                pa[m][i][1] = pack_bf16(s[m][2 * i][2], s[m][2 * i][3]);
                pa[m][i][2] = pack_bf16(s[m][2 * i + 1][0], s[m][2 * i + 1][1]);
                pa[m][i][3] = pack_bf16(s[m][2 * i + 1][2], s[m][2 * i + 1][3]);
            }
        }
#pragma unroll
        for (int kk = 0; kk < kFlKeys / 16; kk++)
#pragma unroll
            for (int i = 0; i < NV; i++) {
                if (i < nv) {
                    uint32_t b[4];
                    ldsm4_trans(b, smem_addr(vt + (kk * 16 + lr) * vpitch + i * 16 + lc));
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        mma16816(o[m][i][0], pa[m][kk], b[0], b[1]);
                        mma16816(o[m][i][1], pa[m][kk], b[2], b[3]);
                    }
                }
            }
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int e2 = 0; e2 < 2; e2++) {
            float l = ls[m][e2];
            l += __shfl_xor_sync(0xffffffffu, l, 1);
            l += __shfl_xor_sync(0xffffffffu, l, 2);
            const int r = wrow + m * 16 + g + e2 * 8;
            if (r >= rows) continue;
            float f = 1.f / l;
            if (a.gate) f *= sigmoid_f32(a.gate[(size_t)(r0 + r) * a.ld_gate + h]);
            bf16 *out = static_cast<bf16 *>(a.out) + (size_t)(r0 + r) * a.heads * vp + h * vp;
#pragma unroll
            for (int i = 0; i < NV; i++)
                if (i < nv)
#pragma unroll
                    for (int k = 0; k < 2; k++)
                        *reinterpret_cast<uint32_t *>(out + i * 16 + k * 8 + 2 * t) = pack_bf16(o[m][i][k][e2 * 2] * f, o[m][i][k][e2 * 2 + 1] * f);
        }
}

// ───────────────────────────── launches ───────────────────────────────────────────────────
template <int D, int MT, bool PAGED, bool EXACT>
static int flash_inst(juno_ctx *c, const FlashParams &p, cudaStream_t st) {
    constexpr int BR = 64 * MT;
    const size_t smem = ((size_t)(BR + 2 * kFlKeys) * (p.a.dim + 8) + (size_t)2 * kFlKeys * (p.a.vdim + 8)) * 2;
    static std::mutex mu;
    static size_t have[16] = {0};
    {
        std::lock_guard<std::mutex> lk(mu);
        if (smem > have[c->device & 15]) {
            JUNO_CUDA_TRY(cudaFuncSetAttribute(flash_prefill_kernel<D, MT, PAGED, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            have[c->device & 15] = smem;
        }
    }
    flash_prefill_kernel<D, MT, PAGED, EXACT><<<dim3((unsigned)p.a.heads, (unsigned)((p.a.n + BR - 1) / BR)), kFlThreads, smem, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

template <int D, int MT, bool PAGED>
static int flash_launch(juno_ctx *c, const FlashParams &p, cudaStream_t st) {
    return p.a.dim == D && p.a.vdim == D ? flash_inst<D, MT, PAGED, true>(c, p, st) : flash_inst<D, MT, PAGED, false>(c, p, st);
}

int launch_flash_prefill(juno_ctx *c, const FlashArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.n > 0 && a.pos0 >= 0 && a.heads > 0 && a.dim % 16 == 0 && a.vdim % 16 == 0 && a.dim <= kFlashMaxDim && a.vdim <= kFlashMaxDim &&
                     (a.pool ? a.slot != nullptr : a.kv && a.ldkv % 8 == 0),
                 "prompt attention: bad arguments (dim %d, vdim %d)", a.dim, a.vdim);
    FlashParams p;
    memset((void *)&p, 0, sizeof(p));
    p.a = a;
    if (p.a.kv_heads == 0) p.a.kv_heads = a.heads;
    JUNO_REQUIRE(a.heads % p.a.kv_heads == 0 && (a.pool || (p.a.kv_heads == a.heads && !a.slopes && !a.sinks && !a.span.window && !a.span.chunk)),
                 "prompt attention: %d heads over %d key/value heads", a.heads, p.a.kv_heads);
    p.scale_log2 = a.scale * kLog2e;
    double pairs = (double)a.n * a.pos0 + (double)a.n * (a.n + 1) / 2;
    const int d = std::max(a.dim, a.vdim);
    if (!a.pool) {
        ProfScope prof(c, st, PROF_ATTN, pairs * 2);
        if (d <= 64) return flash_launch<64, 2, false>(c, p, st);
        if (d <= 128) return flash_launch<128, 2, false>(c, p, st);
        return flash_launch<256, 1, false>(c, p, st);
    }
    p.row_width = a.pool->row_width[a.layer];
    JUNO_REQUIRE(a.pool->latent && a.pool->dtype == 2 && p.row_width == p.a.kv_heads * (a.dim + a.vdim), "prompt attention: pages of another layout");
    p.plane = reinterpret_cast<const bf16 *>(static_cast<const uint8_t *>(a.pool->k) + a.pool->row_off[a.layer] * 2);
    p.table = a.pool->d_table;
    p.max_pages = a.pool->max_pages_per_seq;
    ProfScope prof(c, st, PROF_ATTN, pairs * 2);
    if (d <= 64) return flash_launch<64, 2, true>(c, p, st);
    if (d <= 128) return flash_launch<128, 2, true>(c, p, st);
    return flash_launch<256, 1, true>(c, p, st);
}

}  // namespace juno
