// Row-wise kernels of layer stacks with dense weights (see rowops.cuh).  All of them stream their rows once; they are bound
// by memory traffic, so every value is read as a vector of four and the norms keep the row in shared memory between passes.
#include "rowops.cuh"

#include <algorithm>

namespace juno {

using bf16 = __nv_bfloat16;
constexpr int kRowThreads = 256;

static bool rows_ok(int ld, int width) { return ld % 16 == 0 && width > 0 && width <= ld && ld <= 49152; }

template <typename K>
static int row_smem(K kernel, size_t bytes) {
    if (bytes > 48 * 1024) JUNO_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    return JUNO_OK;
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads) embed_norm_kernel(const T *embed, int ld_embed, int width, int vocab, float g, float eps,
                                                                 const int32_t *tokens, float *x, int ldx) {
    __shared__ float red[33];
    const int r = blockIdx.x;
    const int tok = max(0, min(tokens[r], vocab - 1));
    const T *e = embed + (size_t)tok * ld_embed;
    float sq = 0.f;
    for (int i = threadIdx.x * 4; i < ldx; i += kRowThreads * 4) {
        const float4 v = load4(e + i);
        sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    sq = block_sum(sq, red);
    const float s = g / sqrtf(sq / (float)width + eps);
    for (int i = threadIdx.x * 4; i < ldx; i += kRowThreads * 4) {
        const float4 v = load4(e + i);
        store4(x + (size_t)r * ldx + i, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
    }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads) resid_norm_kernel(const ResidNormArgs a) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const int r = blockIdx.x;
    float *x = a.x + (size_t)r * a.ldx;
    const T *z = a.z ? static_cast<const T *>(a.z) + (size_t)r * a.ldz : nullptr;
    float sz = 0.f;
    if (z) {
        for (int i = threadIdx.x * 4; i < a.ldx; i += kRowThreads * 4) {
            const float4 v = load4(z + i);
            sz += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            store4(row + i, v);
        }
        sz = block_sum(sz, red);
    }
    const float kz = z ? a.g_z / sqrtf(sz / (float)a.width + a.eps) : 0.f;
    float sx = 0.f;
    for (int i = threadIdx.x * 4; i < a.ldx; i += kRowThreads * 4) {
        float4 v = load4(x + i);
        if (z) {
            const float4 w = load4(row + i);
            v.x = fmaf(w.x, kz, v.x);
            v.y = fmaf(w.y, kz, v.y);
            v.z = fmaf(w.z, kz, v.z);
            v.w = fmaf(w.w, kz, v.w);
            store4(x + i, v);
        }
        store4(row + i, v);
        sx += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    if (!a.h) return;
    sx = block_sum(sx, red);
    const float s = a.g_next / sqrtf(sx / (float)a.width + a.eps);
    if (threadIdx.x == 0 && a.row_scale) a.row_scale[r] = s;
    T *h = static_cast<T *>(a.h) + (size_t)r * a.ldh;
    for (int i = threadIdx.x * 4; i < a.ldx; i += kRowThreads * 4) {
        const float4 v = load4(row + i);
        store4(h + i, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
    }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads) gather_norm_kernel(const float *x, int ldx, int width, const int32_t *row_idx, float g,
                                                                  float eps, T *out, int ldo) {
    __shared__ float red[33];
    const int i0 = blockIdx.x, r = row_idx ? row_idx[i0] : i0;
    const float *xr = x + (size_t)r * ldx;
    float sx = 0.f;
    for (int i = threadIdx.x * 4; i < ldx; i += kRowThreads * 4) {
        const float4 v = load4(xr + i);
        sx += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    sx = block_sum(sx, red);
    const float s = g / sqrtf(sx / (float)width + eps);
    for (int i = threadIdx.x * 4; i < ldx; i += kRowThreads * 4) {
        const float4 v = load4(xr + i);
        store4(out + (size_t)i0 * ldo + i, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
    }
}

// Four channels per thread, kConvRows consecutive rows per block: a thread meets its own earlier inputs again in L1.
constexpr int kConvRows = 8;
struct ConvParams {
    const float *x;
    int ldx, n, taps, one_seq;
    const float *row_scale;
    const void *w;
    float *state;  // this layer's rows of slot 0
    size_t slot_stride;
    int ring_mask;
    const int32_t *positions, *slots;
    void *out;
    int ldo;
};
template <typename T>
__global__ void __launch_bounds__(128) conv_kernel(const ConvParams p) {
    const int col = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (col >= p.ldx) return;
    const T *w = static_cast<const T *>(p.w);
    const int r0 = blockIdx.y * kConvRows, r1 = min(p.n, r0 + kConvRows);
    for (int r = r0; r < r1; r++) {
        const int pos = p.positions[r];
        float *ring = p.state ? p.state + (size_t)p.slots[r] * p.slot_stride + col : nullptr;
        const float4 xv = load4(p.x + (size_t)r * p.ldx + col);
        const float s = p.row_scale[r];
        const float4 h = make_float4(xv.x * s, xv.y * s, xv.z * s, xv.w * s);
        float4 wv = load4(w + (size_t)(p.taps - 1) * p.ldx + col);
        float4 acc = make_float4(wv.x * h.x, wv.y * h.y, wv.z * h.z, wv.w * h.w);
        for (int back = 1; back < p.taps && back <= pos; back++) {
            float4 v;
            if (p.one_seq && back <= r) {
                v = load4(p.x + (size_t)(r - back) * p.ldx + col);
                const float sb = p.row_scale[r - back];
                v = make_float4(v.x * sb, v.y * sb, v.z * sb, v.w * sb);
            } else {
                v = load4(ring + (size_t)((pos - back) & p.ring_mask) * p.ldx);
            }
            wv = load4(w + (size_t)(p.taps - 1 - back) * p.ldx + col);
            acc.x = fmaf(wv.x, v.x, acc.x);
            acc.y = fmaf(wv.y, v.y, acc.y);
            acc.z = fmaf(wv.z, v.z, acc.z);
            acc.w = fmaf(wv.w, v.w, acc.w);
        }
        store4(static_cast<T *>(p.out) + (size_t)r * p.ldo + col, make_float4(h.x + acc.x, h.y + acc.y, h.z + acc.z, h.w + acc.w));
        // a sequence's own next position: the ring is longer than the taps, so no one else reads this entry now
        if (!p.one_seq && ring) store4(ring + (size_t)(pos & p.ring_mask) * p.ldx, h);
    }
}

// A portion of a prompt: the window of the last TAPS inputs stays in registers while a thread walks down its rows.
constexpr int kConvSeqRows = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_seq_kernel(const ConvParams p) {
    const int col = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (col >= p.ldx) return;
    const T *w = static_cast<const T *>(p.w);
    float4 wv[TAPS], win[TAPS];  // win[k]: the input k positions back
#pragma unroll
    for (int k = 0; k < TAPS; k++) wv[k] = load4(w + (size_t)(TAPS - 1 - k) * p.ldx + col);
    const int r0 = blockIdx.y * kConvSeqRows, r1 = min(p.n, r0 + kConvSeqRows);
    const int pos0 = p.positions[r0];
    auto input = [&](int r) {
        const float4 v = load4(p.x + (size_t)r * p.ldx + col);
        const float s = p.row_scale[r];
        return make_float4(v.x * s, v.y * s, v.z * s, v.w * s);
    };
#pragma unroll
    for (int k = 0; k < TAPS - 1; k++) {
        const int back = k + 1;  // before row r0
        win[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (back <= pos0)
            win[k] = back <= r0 ? input(r0 - back)
                                : load4(p.state + (size_t)p.slots[r0] * p.slot_stride + (size_t)((pos0 - back) & p.ring_mask) * p.ldx + col);
    }
#pragma unroll 4
    for (int r = r0; r < r1; r++) {
#pragma unroll
        for (int k = TAPS - 1; k > 0; k--) win[k] = win[k - 1];
        const float4 h = win[0] = input(r);
        float4 acc = h;
#pragma unroll
        for (int k = 0; k < TAPS; k++) {
            acc.x = fmaf(wv[k].x, win[k].x, acc.x);
            acc.y = fmaf(wv[k].y, win[k].y, acc.y);
            acc.z = fmaf(wv[k].z, win[k].z, acc.z);
            acc.w = fmaf(wv[k].w, win[k].w, acc.w);
        }
        store4(static_cast<T *>(p.out) + (size_t)r * p.ldo + col, acc);
    }
}

// After a portion: its last inputs into the state (a launch of its own, because the portion's first rows still read the
// entries that its last rows replace).
__global__ void __launch_bounds__(128) conv_state_kernel(const ConvParams p) {
    const int col = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (col >= p.ldx) return;
    const int r = p.n - 1 - (int)blockIdx.y;
    const float4 xv = load4(p.x + (size_t)r * p.ldx + col);
    const float s = p.row_scale[r];
    store4(p.state + (size_t)p.slots[r] * p.slot_stride + (size_t)(p.positions[r] & p.ring_mask) * p.ldx + col,
           make_float4(xv.x * s, xv.y * s, xv.z * s, xv.w * s));
}

struct LatentNormParams {
    LatentNormArgs a;
    const int32_t *positions, *slots, *table;
    int max_pages, row_width;
    void *plane;
};
template <typename T>
__global__ void __launch_bounds__(kRowThreads) latent_norm_kernel(const LatentNormParams p) {
    __shared__ float red[33];
    const int r = blockIdx.x, which = blockIdx.y;  // 0 = queries, 1 = key/value latent
    const LatentNormArgs &a = p.a;
    const float *u = a.u + (size_t)r * a.ldu + (which ? a.kv_col : 0);
    const int n = which ? a.kv_rank : a.q_rank;
    const float *w = which ? a.wkv : a.wq;
    T *dst;
    int ld;
    if (which) {
        dst = latent_row(static_cast<T *>(p.plane), p.table + (size_t)p.slots[r] * p.max_pages, p.row_width, p.positions[r]);
        ld = p.row_width;
    } else {
        dst = static_cast<T *>(a.cq) + (size_t)r * a.ldq;
        ld = a.ldq;
    }
    float sq = 0.f;
    for (int i = threadIdx.x; i < n; i += kRowThreads) sq += u[i] * u[i];
    sq = block_sum(sq, red);
    const float s = 1.f / sqrtf(sq / (float)n + a.eps);
    for (int i = threadIdx.x; i < ld; i += kRowThreads) dst[i] = Num<T>::put(i < n ? u[i] * s * w[i] : 0.f);
}

// ───────────────────────────── launches ───────────────────────────────────────────────────
int launch_embed_norm(juno_ctx *c, int dt, const void *embed, int ld_embed, int width, int vocab, float g, float eps, const RowSet &rows,
                      float *x, int ldx, cudaStream_t st) {
    JUNO_REQUIRE(rows.n > 0 && rows_ok(ldx, width) && ld_embed == ldx, "embed: bad arguments");
    ProfScope prof(c, st, PROF_ROWOPS, (double)rows.n * width * (dt_bytes(dt) + 4));
    if (dt == DT_F32)
        embed_norm_kernel<float><<<rows.n, kRowThreads, 0, st>>>(static_cast<const float *>(embed), ld_embed, width, vocab, g, eps, rows.tokens, x, ldx);
    else
        embed_norm_kernel<bf16><<<rows.n, kRowThreads, 0, st>>>(static_cast<const bf16 *>(embed), ld_embed, width, vocab, g, eps, rows.tokens, x, ldx);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_resid_norm(juno_ctx *c, int dt, const ResidNormArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.n > 0 && rows_ok(a.ldx, a.width) && (!a.z || a.ldz >= a.ldx) && (!a.h || a.ldh >= a.ldx), "residual norm: bad arguments");
    const size_t smem = (size_t)a.ldx * 4;
    ProfScope prof(c, st, PROF_ROWOPS, (double)a.n * a.width * ((a.z ? 8 + dt_bytes(dt) : 4) + (a.h ? dt_bytes(dt) : 0)));
    if (dt == DT_F32) {
        JUNO_TRY(row_smem(resid_norm_kernel<float>, smem));
        resid_norm_kernel<float><<<a.n, kRowThreads, smem, st>>>(a);
    } else {
        JUNO_TRY(row_smem(resid_norm_kernel<bf16>, smem));
        resid_norm_kernel<bf16><<<a.n, kRowThreads, smem, st>>>(a);
    }
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_gather_norm(juno_ctx *c, int dt, const float *x, int ldx, int width, const int32_t *row_idx, int n, float g, float eps, void *out,
                       int ldo, cudaStream_t st) {
    JUNO_REQUIRE(n > 0 && rows_ok(ldx, width) && ldo >= ldx, "row norm: bad arguments");
    ProfScope prof(c, st, PROF_ROWOPS, (double)n * width * (4 + dt_bytes(dt)));
    if (dt == DT_F32)
        gather_norm_kernel<float><<<n, kRowThreads, 0, st>>>(x, ldx, width, row_idx, g, eps, static_cast<float *>(out), ldo);
    else
        gather_norm_kernel<bf16><<<n, kRowThreads, 0, st>>>(x, ldx, width, row_idx, g, eps, static_cast<bf16 *>(out), ldo);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_conv(juno_ctx *c, int dt, const ConvArgs &a, const RowSet &rows, cudaStream_t st) {
    JUNO_REQUIRE(rows.n > 0 && rows_ok(a.ldx, a.width) && a.ldo >= a.ldx && a.taps >= 1, "convolution: bad arguments");
    JUNO_REQUIRE(a.taps == 1 || (a.pool->state && a.pool->state_width == a.ldx && a.pool->state_ring >= 2 * a.taps), "convolution: no state for %d taps", a.taps);
    ConvParams p;
    p.x = a.x;
    p.ldx = a.ldx;
    p.n = rows.n;
    p.taps = a.taps;
    p.one_seq = rows.one_seq ? 1 : 0;
    p.row_scale = a.row_scale;
    p.w = a.w;
    const juno_kvpool *pool = a.pool;
    p.state = pool->state ? pool->state + (size_t)a.layer * pool->state_ring * pool->state_width : nullptr;
    p.slot_stride = (size_t)pool->n_layers * pool->state_ring * pool->state_width;
    p.ring_mask = pool->state_ring - 1;
    p.positions = rows.positions;
    p.slots = rows.slots;
    p.out = a.out;
    p.ldo = a.ldo;
    const unsigned gx = (unsigned)((a.ldx + 511) / 512);
    const dim3 grid(gx, (unsigned)((rows.n + kConvRows - 1) / kConvRows));
    ProfScope prof(c, st, PROF_ROWOPS, (double)rows.n * a.width * (4 + dt_bytes(dt)));
    const dim3 sgrid(gx, (unsigned)((rows.n + kConvSeqRows - 1) / kConvSeqRows));
    if (dt == DT_F32)
        conv_kernel<float><<<grid, 128, 0, st>>>(p);
    else if (rows.one_seq && a.taps == 2)
        conv_seq_kernel<bf16, 2><<<sgrid, 128, 0, st>>>(p);
    else if (rows.one_seq && a.taps == 3)
        conv_seq_kernel<bf16, 3><<<sgrid, 128, 0, st>>>(p);
    else if (rows.one_seq && a.taps == 4)
        conv_seq_kernel<bf16, 4><<<sgrid, 128, 0, st>>>(p);
    else
        conv_kernel<bf16><<<grid, 128, 0, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    if (rows.one_seq && p.state) {
        conv_state_kernel<<<dim3(gx, (unsigned)std::min(rows.n, pool->state_ring)), 128, 0, st>>>(p);
        JUNO_CUDA_TRY(cudaGetLastError());
        c->kernel_launches++;
    }
    return JUNO_OK;
}

int launch_latent_norm(juno_ctx *c, int dt, const LatentNormArgs &a, const RowSet &rows, cudaStream_t st) {
    JUNO_REQUIRE(rows.n > 0 && a.pool->latent && a.pool->dtype == (dt == DT_F32 ? 1 : 2), "latent norm: bad arguments");
    LatentNormParams p;
    p.a = a;
    p.positions = rows.positions;
    p.slots = rows.slots;
    p.table = a.pool->d_table;
    p.max_pages = a.pool->max_pages_per_seq;
    p.row_width = a.pool->row_width[a.layer];
    p.plane = static_cast<uint8_t *>(a.pool->k) + a.pool->row_off[a.layer] * a.pool->elem_bytes;
    JUNO_REQUIRE(a.kv_rank <= p.row_width, "latent norm: rows of %d do not fit pages of %d", a.kv_rank, p.row_width);
    ProfScope prof(c, st, PROF_ROWOPS, (double)rows.n * (a.q_rank + a.kv_rank) * (4 + dt_bytes(dt)));
    if (dt == DT_F32)
        latent_norm_kernel<float><<<dim3(rows.n, 2), kRowThreads, 0, st>>>(p);
    else
        latent_norm_kernel<bf16><<<dim3(rows.n, 2), kRowThreads, 0, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

}  // namespace juno
