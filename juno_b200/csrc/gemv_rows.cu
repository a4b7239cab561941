// Fused BF16 matrix-vector products of a decode step (see gemv_rows.cuh).
//
// A CTA (sixteen warps, one per SM) owns a contiguous range of 16-row tiles; the (row tile, 64-column block) items of a chunk
// of at most sixteen tiles are one flat sequence that the warps share evenly (qsplit.cuh, as in the quantised GEMV).  A lane
// reads 16 consecutive bytes of rows g and g + 8; the order of K inside an MMA is free as long as both operands use it, so
// those bytes ARE the A fragments of two mma.sync.m16n8k16 and no repacked copy of the weights is needed (the row products of
// gemm_rows_tc.cu read the same row-major matrix).  Columns of B are the sequences.  The first items are requested before the
// dependency wait; four are in flight per lane after that.
#include <algorithm>
#include <cstring>
#include <mutex>

#include "gemv_rows.cuh"
#include "mma_bf16.cuh"
#include "qsplit.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

constexpr int kGvThreads = 512, kGvWarps = 16, kGvDepth = 4;
static_assert(kGvDepth == 4, "the rotation below is written for four items");
constexpr int kGvRedFloats = kGvWarps * 2 * 128;  // partial sums of a chunk: [warp][first / last tile][16 rows][8 sequences]

struct GvParams {
    GvArgs a;
    int nkb, total_rt, pitch;  // 64-column blocks of K; row tiles; operand row pitch in bytes
    int seg_rt[3];             // first row tile of each segment
    int n_op;                  // operand images in shared memory
};

__host__ __device__ inline int gv_pitch(int cols) { return (cols * 2 + 127) / 128 * 128 + 64; }

__device__ __forceinline__ uint64_t evict_first_policy() {
    uint64_t p;
    asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(p));
    return p;
}
__device__ __forceinline__ uint4 ld_weights(const bf16 *ptr, uint64_t pol) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.L2::cache_hint.v4.u32 {%0,%1,%2,%3}, [%4], %5;"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(ptr), "l"(pol));
    return v;
}

// Walks the items of one warp over all chunks of its CTA.
struct GvCursor {
    int k, f, f1;    // chunk, next item, end of the warp's share in this chunk
    int rt, kb;      // row tile (of the launch) and 64-column block of item f
};
struct GvWalk {
    int rt0, rtc, n_chunks, nkb, warp;
    __device__ __forceinline__ int lo(int k) const { return qsplit_chunk_lo(rt0, rtc, n_chunks, k); }
    __device__ __forceinline__ void seek(GvCursor &c, int k) const {
        for (; k < n_chunks; k++) {
            const int l = lo(k), T = (lo(k + 1) - l) * nkb;
            int f0, f1;
            qsplit_warp(warp, T, f0, f1);
            if (f0 < f1) {
                c.k = k;
                c.f = f0;
                c.f1 = f1;
                c.rt = l + f0 / nkb;
                c.kb = f0 % nkb;
                return;
            }
        }
        c.k = n_chunks;
    }
    __device__ __forceinline__ bool done(const GvCursor &c) const { return c.k >= n_chunks; }
};

// COLS: groups of four columns a thread holds of a residual row (its width is at most 2048 * COLS).
template <int PRO, int COLS>
__global__ void __launch_bounds__(kGvThreads, 1) gemv_rows_kernel(const __grid_constant__ GvParams p) {
    extern __shared__ __align__(128) uint8_t sm[];
    __shared__ float red_s[33], coef_s[kMaxStreams + 1];
    const GvArgs &a = p.a;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    float *red = reinterpret_cast<float *>(sm);           // [2][kGvRedFloats]
    uint8_t *ops = sm + 2 * kGvRedFloats * 4;             // [n_op][n][pitch]
    GvWalk walk;
    qsplit_cta((int)blockIdx.x, (int)gridDim.x, p.total_rt, walk.rt0, walk.rtc);
    walk.n_chunks = qsplit_chunks(walk.rtc);
    walk.nkb = p.nkb;
    walk.warp = warp;
    const uint64_t pol = evict_first_policy();
    auto seg_of = [&](int rt) { return rt >= p.seg_rt[2] ? 2 : rt >= p.seg_rt[1] ? 1 : 0; };

    // weights in flight
    uint4 w[kGvDepth][4];
    GvCursor pc;
    const bf16 *wrow = nullptr;  // row g of the tile, this lane's 16 bytes of a 32-column half
    auto row_ptr = [&](int rt) {
        const int s = seg_of(rt);
        return a.seg[s].w + ((size_t)(rt - p.seg_rt[s]) * 16 + g) * a.K + t * 8;
    };
    auto fetch = [&](uint4 (&r)[4]) {
        const int col = pc.kb * 64;
        const bf16 *q = wrow + col;
        const bool v0 = col + t * 8 < a.K, v1 = col + 32 + t * 8 < a.K;
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
        r[0] = v0 ? ld_weights(q, pol) : zero;
        r[1] = v0 ? ld_weights(q + (size_t)8 * a.K, pol) : zero;
        r[2] = v1 ? ld_weights(q + 32, pol) : zero;
        r[3] = v1 ? ld_weights(q + (size_t)8 * a.K + 32, pol) : zero;
        if (++pc.f == pc.f1) {
            walk.seek(pc, pc.k + 1);
            if (!walk.done(pc)) wrow = row_ptr(pc.rt);
        } else if (++pc.kb == p.nkb) {
            pc.kb = 0;
            wrow = row_ptr(++pc.rt);
        }
    };
    walk.seek(pc, 0);
    if (!walk.done(pc)) wrow = row_ptr(pc.rt);
#pragma unroll
    for (int d = 0; d < kGvDepth; d++)
        if (!walk.done(pc)) fetch(w[d]);

    if (PRO == GVP_STREAMS && tid <= a.streams) {  // the sublayer's input as a sum over the old streams and the pending result
        float v = tid < a.streams && !a.z ? a.hc_in[tid] : 0.f;
        if (a.z)
            for (int t = 0; t < a.streams; t++) v = fmaf(tid < a.streams ? a.hc_mix[tid * a.streams + t] : a.hc_out[t], a.hc_in[t], v);
        coef_s[tid] = v;
    }

    pdl_wait();
    pdl_launch_dependents();

    // ── operand ──
    if (PRO == GVP_COPY) {
        const int per = a.in_cols >> 3;  // 16-byte pieces of a row
        for (int i = tid; i < a.n * per; i += kGvThreads) {
            const int b = i / per, ch = i - b * per;
            *reinterpret_cast<uint4 *>(ops + (size_t)b * p.pitch + ch * 16) = *reinterpret_cast<const uint4 *>(a.in + (size_t)b * a.ld_in + ch * 8);
        }
    } else if (PRO == GVP_LATENT) {
        for (int b = 0; b < a.n; b++) {
            const float *u = a.u + (size_t)b * a.ldu;
            float sq = 0.f;
            for (int i = tid; i < a.q_rank; i += kGvThreads) sq += u[i] * u[i];
            const float s = 1.f / sqrtf(block_sum(sq, red_s) / (float)a.q_rank + a.eps);
            bf16 *o = reinterpret_cast<bf16 *>(ops + (size_t)b * p.pitch);
            for (int i = tid; i < a.K; i += kGvThreads) o[i] = __float2bfloat16_rn(i < a.q_rank ? u[i] * s * a.wq[i] : 0.f);
            if ((int)blockIdx.x == (int)gridDim.x - 1 - b % (int)gridDim.x) {  // one CTA appends the key/value latent
                const float *c = u + a.kv_col;
                float sk = 0.f;
                for (int i = tid; i < a.kv_rank; i += kGvThreads) sk += c[i] * c[i];
                const float r = 1.f / sqrtf(block_sum(sk, red_s) / (float)a.kv_rank + a.eps);
                bf16 *dst = latent_row(a.plane, a.table + (size_t)a.slots[b] * a.max_pages, a.page_width, a.positions[b]);
                for (int i = tid; i < a.page_width; i += kGvThreads) dst[i] = __float2bfloat16_rn(i < a.kv_rank ? c[i] * r * a.wkv[i] : 0.f);
            }
        }
    } else if (PRO == GVP_STREAMS) {
        __syncthreads();
        const int S = a.streams;
        float4 nw[COLS];
#pragma unroll
        for (int i = 0; i < COLS; i++) {
            const int col = (i * kGvThreads + tid) * 4;
            if (col < a.K) nw[i] = load4(a.norm_w + col);
        }
        for (int b = 0; b < a.n; b++) {
            const float *x = a.x + (size_t)b * S * a.K, *z = a.z ? a.z + (size_t)b * a.K : nullptr;
            float4 u[COLS];
            float sx = 0.f;
#pragma unroll
            for (int i = 0; i < COLS; i++) {
                const int col = (i * kGvThreads + tid) * 4;
                u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (col >= a.K) continue;
                if (z) {
                    const float4 y = load4(z + col);
                    const float c = coef_s[S];
                    u[i] = make_float4(c * y.x, c * y.y, c * y.z, c * y.w);
                }
#pragma unroll 4
                for (int s = 0; s < S; s++) {
                    const float4 v = load4(x + (size_t)s * a.K + col);
                    const float c = coef_s[s];
                    u[i].x = fmaf(c, v.x, u[i].x);
                    u[i].y = fmaf(c, v.y, u[i].y);
                    u[i].z = fmaf(c, v.z, u[i].z);
                    u[i].w = fmaf(c, v.w, u[i].w);
                }
                sx += u[i].x * u[i].x + u[i].y * u[i].y + u[i].z * u[i].z + u[i].w * u[i].w;
            }
            const float k = 1.f / sqrtf(block_sum(sx, red_s) / (float)a.width + a.eps);
#pragma unroll
            for (int i = 0; i < COLS; i++) {
                const int col = (i * kGvThreads + tid) * 4;
                if (col < a.K)
                    store4(reinterpret_cast<bf16 *>(ops + (size_t)b * p.pitch) + col,
                           make_float4(u[i].x * k * nw[i].x, u[i].y * k * nw[i].y, u[i].z * k * nw[i].z, u[i].w * k * nw[i].w));
            }
        }
        if (a.z) {  // every CTA stores its share of the new streams
            const int groups = a.K >> 2, total = a.n * groups, per = (total + (int)gridDim.x - 1) / (int)gridDim.x;
            const int end = min(total, ((int)blockIdx.x + 1) * per);
            for (int e = (int)blockIdx.x * per + tid; e < end; e += kGvThreads) {
                const int b = e / groups, col = (e - b * groups) * 4;
                const float *x = a.x + (size_t)b * S * a.K + col;
                const float4 y = load4(a.z + (size_t)b * a.K + col);
                for (int t = 0; t < S; t++) {
                    const float o = a.hc_out[t];
                    float4 v = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll 4
                    for (int s = 0; s < S; s++) {
                        const float4 w4 = load4(x + (size_t)s * a.K);
                        const float m = a.hc_mix[s * S + t];
                        v.x = fmaf(m, w4.x, v.x);
                        v.y = fmaf(m, w4.y, v.y);
                        v.z = fmaf(m, w4.z, v.z);
                        v.w = fmaf(m, w4.w, v.w);
                    }
                    store4(a.x_store + ((size_t)b * S + t) * a.K + col, v);
                }
            }
        }
    } else {
        // which images this CTA's row tiles read
        const int s_first = seg_of(walk.rt0), s_last = seg_of(walk.rt0 + max(walk.rtc, 1) - 1);
        bool want_h = false, want_c = false;
        for (int s = s_first; s <= s_last; s++) (a.seg[s].operand ? want_c : want_h) = true;
        constexpr bool kAhead = COLS <= 2;  // the next sequence's row is requested early when the registers allow it
        float4 xv[COLS], zv[COLS], xn[kAhead ? COLS : 1], zn[kAhead ? COLS : 1];
        auto fetch_row = [&](int b, float4 *x, float4 *z) {
#pragma unroll
            for (int i = 0; i < COLS; i++) {
                const int col = (i * kGvThreads + tid) * 4;
                x[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (col < a.K) {
                    x[i] = load4(a.x + (size_t)b * a.K + col);
                    if (a.z) z[i] = load4(a.z + (size_t)b * a.K + col);
                }
            }
        };
        if (kAhead) fetch_row(0, xn, zn);
        for (int b = 0; b < a.n; b++) {
            if (kAhead) {
#pragma unroll
                for (int i = 0; i < COLS; i++) {
                    xv[i] = xn[kAhead ? i : 0];
                    zv[i] = zn[kAhead ? i : 0];
                }
                if (b + 1 < a.n) fetch_row(b + 1, xn, zn);
            } else {
                fetch_row(b, xv, zv);
            }
            if (a.z) {
                float sz = 0.f;
#pragma unroll
                for (int i = 0; i < COLS; i++) sz += zv[i].x * zv[i].x + zv[i].y * zv[i].y + zv[i].z * zv[i].z + zv[i].w * zv[i].w;
                const float kz = a.g_z / sqrtf(block_sum(sz, red_s) / (float)a.width + a.eps);
#pragma unroll
                for (int i = 0; i < COLS; i++) {
                    xv[i].x = fmaf(zv[i].x, kz, xv[i].x);
                    xv[i].y = fmaf(zv[i].y, kz, xv[i].y);
                    xv[i].z = fmaf(zv[i].z, kz, xv[i].z);
                    xv[i].w = fmaf(zv[i].w, kz, xv[i].w);
                }
            }
            float sx = 0.f;
#pragma unroll
            for (int i = 0; i < COLS; i++) sx += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
            const float s = a.g_next / sqrtf(block_sum(sx, red_s) / (float)a.width + a.eps);
            const bool keeper = (int)blockIdx.x == b % (int)gridDim.x;  // this CTA stores the sequence's new rows
            const int pos = a.conv_w ? a.positions[b] : 0;
            float *ring = a.state ? a.state + (size_t)a.slots[b] * a.slot_stride : nullptr;
#pragma unroll
            for (int i = 0; i < COLS; i++) {
                const int col = (i * kGvThreads + tid) * 4;
                if (col >= a.K) continue;
                const float4 h = make_float4(xv[i].x * s, xv[i].y * s, xv[i].z * s, xv[i].w * s);
                if (want_h) store4(reinterpret_cast<bf16 *>(ops + (size_t)b * p.pitch) + col, h);
                if (keeper) {
                    if (a.z) store4(a.x_store + (size_t)b * a.K + col, xv[i]);
                    if (ring) store4(ring + (size_t)(pos & a.ring_mask) * a.K + col, h);
                }
                if (want_c) {
                    float4 c = h;
                    for (int back = 0; back < a.taps && back <= pos; back++) {
                        const float4 v = back ? load4(ring + (size_t)((pos - back) & a.ring_mask) * a.K + col) : h;
                        const float4 cw = load4(a.conv_w + (size_t)(a.taps - 1 - back) * a.K + col);
                        c.x = fmaf(cw.x, v.x, c.x);
                        c.y = fmaf(cw.y, v.y, c.y);
                        c.z = fmaf(cw.z, v.z, c.z);
                        c.w = fmaf(cw.w, v.w, c.w);
                    }
                    store4(reinterpret_cast<bf16 *>(ops + (size_t)((p.n_op - 1) * a.n + b) * p.pitch) + col, c);
                }
            }
        }
    }
    __syncthreads();

    // ── products ──
    const bool live = g < a.n;  // column g of B is sequence g
    for (int k = 0; k < walk.n_chunks; k++) {
        const int lo = walk.lo(k), crt = walk.lo(k + 1) - lo, T = crt * p.nkb;
        int f0, f1;
        qsplit_warp(warp, T, f0, f1);
        float *cred = red + (k & 1) * kGvRedFloats;
        const int l_first = f0 / p.nkb;
        int l = l_first, kb = f0 - l_first * p.nkb;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        auto operand_of = [&](int rt) {
            const int s = seg_of(rt);
            size_t off = (size_t)((a.seg[s].operand && p.n_op > 1 ? a.n : 0) + g) * p.pitch + t * 16;
            if (a.group_rows) off += (size_t)((rt - p.seg_rt[s]) * 16 / a.group_rows) * a.K * 2;
            return ops + off;
        };
        const uint8_t *xrow = operand_of(lo + l);
        auto flush = [&]() {
            float *d = cred + (warp * 2 + (l == l_first ? 0 : 1)) * 128 + g * 8 + 2 * t;
            *reinterpret_cast<float2 *>(d) = make_float2(acc[0], acc[1]);
            *reinterpret_cast<float2 *>(d + 64) = make_float2(acc[2], acc[3]);
            acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
        };
        auto consume = [&](const uint4 (&r)[4]) {
            uint4 x0 = make_uint4(0u, 0u, 0u, 0u), x1 = x0;
            const int col = kb * 64 + t * 8;  // columns past K are zero in both operands
            if (live && col < a.K) x0 = *reinterpret_cast<const uint4 *>(xrow + kb * 128);
            if (live && col + 32 < a.K) x1 = *reinterpret_cast<const uint4 *>(xrow + kb * 128 + 64);
            {
                const uint32_t a0[4] = {r[0].x, r[1].x, r[0].y, r[1].y}, a1[4] = {r[0].z, r[1].z, r[0].w, r[1].w};
                mma16816(acc, a0, x0.x, x0.y);
                mma16816(acc, a1, x0.z, x0.w);
            }
            {
                const uint32_t a0[4] = {r[2].x, r[3].x, r[2].y, r[3].y}, a1[4] = {r[2].z, r[3].z, r[2].w, r[3].w};
                mma16816(acc, a0, x1.x, x1.y);
                mma16816(acc, a1, x1.z, x1.w);
            }
            if (++kb == p.nkb) {
                flush();
                kb = 0;
                l++;
                if (l < crt) xrow = operand_of(lo + l);
            }
        };
        // the ring of items in flight turns with the items, so its position is the same at the start of every chunk only if the
        // ring is realigned: shares need not be multiples of its depth
        int f = f0;
        for (; f + kGvDepth <= f1; f += kGvDepth) {
#pragma unroll
            for (int d = 0; d < kGvDepth; d++) {
                consume(w[d]);
                if (!walk.done(pc)) fetch(w[d]);
            }
        }
        const int rest = f1 - f;  // 0 .. depth - 1
        if (rest > 0) {
#pragma unroll
            for (int d = 0; d < kGvDepth - 1; d++)
                if (d < rest) {
                    consume(w[d]);
                    if (!walk.done(pc)) fetch(w[d]);
                }
            // rotate so that the oldest request is in w[0] again
            if (k + 1 < walk.n_chunks) {
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const uint4 o0 = w[0][i], o1 = w[1][i], o2 = w[2][i], o3 = w[3][i];
                    w[0][i] = rest == 1 ? o1 : rest == 2 ? o2 : o3;
                    w[1][i] = rest == 1 ? o2 : rest == 2 ? o3 : o0;
                    w[2][i] = rest == 1 ? o3 : rest == 2 ? o0 : o1;
                    w[3][i] = rest == 1 ? o0 : rest == 2 ? o1 : o2;
                }
            }
        }
        if (f0 < f1 && kb != 0) flush();
        __syncthreads();
        for (int o = tid; o < crt * 128; o += kGvThreads) {
            const int lt = o >> 7, r = (o >> 3) & 15, b = o & 7;
            if (b >= a.n) continue;
            int w_lo, w_hi;
            qsplit_row_tile_warps(lt, p.nkb, T, w_lo, w_hi);
            auto total = [&](int rr) {
                float v = 0.f;
                for (int x = w_lo; x <= w_hi; x++) {
                    int e0, e1;
                    qsplit_warp(x, T, e0, e1);
                    if (e0 < e1) v += cred[(x * 2 + (e0 / p.nkb == lt ? 0 : 1)) * 128 + rr * 8 + b];
                }
                return v;
            };
            const float v = total(r);
            const int rt = lo + lt, si = seg_of(rt), row = (rt - p.seg_rt[si]) * 16 + r;
            const GvSeg &sg = a.seg[si];
            if (sg.n_store && row >= sg.n_store) continue;
            const size_t idx = (size_t)b * sg.ldo + row;
            switch (sg.epi) {
            case GVE_F32: static_cast<float *>(sg.out)[idx] = sg.bias ? v + sg.bias[row] : v; break;
            case GVE_OP: static_cast<bf16 *>(sg.out)[idx] = __float2bfloat16_rn(v); break;
            case GVE_SIGMOID: static_cast<float *>(sg.out)[idx] = sigmoid_f32(v + sg.bias[row]); break;
            case GVE_RELU2: {
                const float y = fmaxf(v, 0.f);
                static_cast<bf16 *>(sg.out)[idx] = __float2bfloat16_rn(y * y);
                break;
            }
            case GVE_GEGLU:
                if (r < 8) static_cast<bf16 *>(sg.out)[(size_t)b * sg.ldo + (row >> 4) * 8 + r] = __float2bfloat16_rn(gelu_tanh(v) * total(r + 8));
                break;
            default: static_cast<float *>(sg.out)[idx] = v * sg.aux[(size_t)b * sg.ldaux + row];
            }
        }
    }
}

int gemv_rows_chunk(const juno_ctx *c, int cols, int operands, int n) {
    const size_t room = c->smem_optin - 2 * kGvRedFloats * 4 - 1024;
    const int fit = (int)(room / ((size_t)gv_pitch(cols) * operands));
    n = std::min(n, kGvMaxSeqs);
    if (fit <= 0) return 0;
    if (fit >= n) return n;
    const int passes = (n + fit - 1) / fit;  // passes of equal size
    return (n + passes - 1) / passes;
}

template <int PRO, int COLS>
static int launch_inst(juno_ctx *c, const GvParams &p, size_t smem, cudaStream_t st) {
    static std::mutex mu;
    static bool configured[16] = {false};
    {
        std::lock_guard<std::mutex> lk(mu);
        if (!configured[c->device & 15]) {
            JUNO_CUDA_TRY(cudaFuncSetAttribute(gemv_rows_kernel<PRO, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)c->smem_optin - 1024));
            configured[c->device & 15] = true;
        }
    }
    const dim3 grid((unsigned)std::min(p.total_rt, c->sm_count));
    if (p.a.early) {
        JUNO_CUDA_TRY(launch_pdl(gemv_rows_kernel<PRO, COLS>, grid, dim3(kGvThreads), smem, st, p));
    } else {
        gemv_rows_kernel<PRO, COLS><<<grid, kGvThreads, smem, st>>>(p);
        JUNO_CUDA_TRY(cudaGetLastError());
    }
    c->kernel_launches++;
    return JUNO_OK;
}

static int launch_one(juno_ctx *c, const GvArgs &a, cudaStream_t st) {
    GvParams p;
    memset((void *)&p, 0, sizeof(p));
    p.a = a;
    p.nkb = (a.K + 63) / 64;
    const int op_cols = a.prologue == GVP_COPY ? a.in_cols : a.K;
    p.pitch = gv_pitch(op_cols);
    p.n_op = a.prologue == GVP_RESIDUAL && a.conv_w ? 2 : 1;
    double bytes = 0;
    for (int s = 0; s < 3; s++) {
        p.seg_rt[s] = s < a.nseg ? p.total_rt : 1 << 30;
        if (s < a.nseg) {
            p.total_rt += a.seg[s].rows / 16;
            bytes += (double)a.seg[s].rows * a.K * 2 + (double)a.n * a.seg[s].rows * 4;
        }
    }
    bytes += (double)a.n * op_cols * 4;
    const size_t smem = 2 * kGvRedFloats * 4 + (size_t)p.n_op * a.n * p.pitch;
    JUNO_REQUIRE(smem <= c->smem_optin - 1024, "decode product: %zu bytes of shared memory needed", smem);
    ProfScope prof(c, st, PROF_GEMV_ROWS, bytes);
    if (a.prologue == GVP_COPY) return launch_inst<GVP_COPY, 1>(c, p, smem, st);
    if (a.prologue == GVP_LATENT) return launch_inst<GVP_LATENT, 1>(c, p, smem, st);
    if (a.prologue == GVP_STREAMS) return a.K <= 4096 ? launch_inst<GVP_STREAMS, 2>(c, p, smem, st) : launch_inst<GVP_STREAMS, 4>(c, p, smem, st);
    return a.K <= 4096 ? launch_inst<GVP_RESIDUAL, 2>(c, p, smem, st) : launch_inst<GVP_RESIDUAL, 4>(c, p, smem, st);
}

int launch_gemv_rows(juno_ctx *c, const GvArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.n >= 1 && a.n <= kGvMaxSeqs && a.K > 0 && a.K % 16 == 0 && a.nseg >= 1 && a.nseg <= 3, "decode product: bad arguments (n %d, K %d)", a.n, a.K);
    JUNO_REQUIRE(a.prologue != GVP_RESIDUAL || (a.K <= kGvMaxWidth && a.width <= a.K), "decode product: a residual row of %d is too wide", a.K);
    JUNO_REQUIRE(a.prologue != GVP_STREAMS || (a.K <= kGvMaxWidth && a.width <= a.K && a.streams >= 1 && a.streams <= kMaxStreams && a.x && a.hc_in && a.norm_w &&
                                               (!a.z || (a.hc_mix && a.hc_out && a.x_store && a.x_store != a.x))),
                 "decode product: bad streams");
    JUNO_REQUIRE(a.group_rows % 16 == 0, "decode product: groups of %d rows", a.group_rows);
    for (int s = 0; s < a.nseg; s++) JUNO_REQUIRE(a.seg[s].rows > 0 && a.seg[s].rows % 16 == 0 && a.seg[s].w && a.seg[s].out, "decode product: bad segment %d", s);
    const int n_op = a.prologue == GVP_RESIDUAL && a.conv_w ? 2 : 1;
    const int step = gemv_rows_chunk(c, a.prologue == GVP_COPY ? a.in_cols : a.K, n_op, a.n);
    JUNO_REQUIRE(step > 0, "decode product: rows of %d columns do not fit shared memory", a.K);
    for (int b = 0; b < a.n; b += step) {  // usually one pass
        GvArgs t = a;
        t.n = std::min(step, a.n - b);
        if (t.in) t.in += (size_t)b * t.ld_in;
        const size_t x_row = (size_t)t.K * std::max(t.streams, 1);
        if (t.x) t.x += b * x_row;
        if (t.z) t.z += (size_t)b * t.K;
        if (t.x_store) t.x_store += b * x_row;
        if (t.u) t.u += (size_t)b * t.ldu;
        if (t.positions) t.positions += b;
        if (t.slots) t.slots += b;
        for (int s = 0; s < t.nseg; s++) {
            GvSeg &g = t.seg[s];
            const size_t es = g.epi == GVE_OP || g.epi == GVE_RELU2 || g.epi == GVE_GEGLU ? 2 : 4;
            g.out = static_cast<uint8_t *>(g.out) + (size_t)b * g.ldo * es;
            if (g.aux) g.aux += (size_t)b * g.ldaux;
        }
        JUNO_TRY(launch_one(c, t, st));
    }
    return JUNO_OK;
}

}  // namespace juno
