// Attention of grouped heads over row pages (see grouped_attn.cuh): the step from projections to queries, keys and values, the
// general kernel, and the tensor-core kernel of decode steps.  Prompts run on flash_attn.cu.
#include "grouped_attn.cuh"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <mutex>

#include "mma_bf16.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

struct GroupedParams {
    GroupedAttnArgs a;
    const int32_t *table;
    int max_pages, row_width;
    void *plane;
};

__device__ __forceinline__ float query_factor(const GroupedAttnArgs &a, int pos) {
    return a.temp_every > 0 ? fmaf(a.temp_coef, logf((float)((pos + 1) / a.temp_every) + 1.f), 1.f) : 1.f;
}

// One warp: a head of a projection -> norm, rotation, factor -> dst[0 .. dp), zeros past dim.
template <typename T>
__device__ __forceinline__ void put_head(const float *x, int dim, int dp, const float *w, float eps, const float2 *rot, int rot_dims, float factor, T *dst, int lane) {
    float k = 1.f;
    if (w) {
        float sq = 0.f;
        for (int i = lane; i < dim; i += 32) sq += x[i] * x[i];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        k = 1.f / sqrtf(sq / (float)dim + eps);
    }
    const int half = rot ? rot_dims >> 1 : 0;
    for (int i = lane; i < dp; i += 32) {
        float v = 0.f;
        if (i < dim) {
            v = w ? x[i] * k * w[i] : x[i];
            if (i < 2 * half) {
                const int j = i < half ? i + half : i - half;
                const float y = w ? x[j] * k * w[j] : x[j];
                const float2 cs = rot[i < half ? i : j];
                v = i < half ? v * cs.x - y * cs.y : v * cs.x + y * cs.y;
            }
            v *= factor;
        }
        dst[i] = Num<T>::put(v);
    }
}

constexpr int kPrepWarps = 8;
template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32) grouped_prep_kernel(const __grid_constant__ GroupedParams p) {
    const GroupedAttnArgs &a = p.a;
    const int r = blockIdx.x, unit = blockIdx.y * kPrepWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= a.heads + 2 * a.kv_heads) return;
    const int pos = a.rows.positions[r];
    const float *u = a.u + (size_t)r * a.ldu;
    const float2 *rot = a.rot ? a.rot + (size_t)pos * (a.rot_dims >> 1) : nullptr;
    if (unit < a.heads) {
        put_head(u + unit * a.dp, a.dim, a.dp, a.q_norm, a.eps, rot, a.rot_dims, query_factor(a, pos), static_cast<T *>(a.q) + ((size_t)r * a.heads + unit) * a.dp, lane);
        return;
    }
    T *row = latent_row(static_cast<T *>(p.plane), p.table + (size_t)a.rows.slots[r] * p.max_pages, p.row_width, pos);
    const int g = unit - a.heads;
    if (g < a.kv_heads) {
        put_head(u + (a.heads + g) * a.dp, a.dim, a.dp, a.k_norm, a.eps, rot, a.rot_dims, 1.f, row + g * a.dp, lane);
    } else {
        const float *v = u + (a.heads + a.kv_heads) * a.dp + (g - a.kv_heads) * a.vp;
        T *dst = row + a.kv_heads * a.dp + (g - a.kv_heads) * a.vp;
        for (int i = lane; i < a.vp; i += 32) dst[i] = Num<T>::put(v[i]);
    }
}

// ───────────────────────────── general kernel ─────────────────────────────────────────────
constexpr int kGsThreads = 128, kGsKeys = 64, kGsCols = kGroupedMaxVdim / kGsThreads;
template <typename T>
__global__ void __launch_bounds__(kGsThreads) grouped_simt_kernel(const __grid_constant__ GroupedParams p) {
    extern __shared__ __align__(16) float qs[];  // [dp]
    __shared__ float sc[kGsKeys], red[2];
    const GroupedAttnArgs &a = p.a;
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kvh = h / (a.heads / a.kv_heads), k_col = kvh * a.dp, v_col = a.kv_heads * a.dp + kvh * a.vp;
    const int32_t *table = p.table + (size_t)a.rows.slots[row] * p.max_pages;
    T *plane = static_cast<T *>(p.plane);
    const int pos = a.rows.positions[row], lo = a.span.first(pos);
    const float slope = a.slopes ? a.slopes[h] : 0.f;
    for (int i = tid; i < a.dp; i += kGsThreads) qs[i] = Num<T>::get(static_cast<const T *>(a.q)[((size_t)row * a.heads + h) * a.dp + i]);
    float acc[kGsCols];
#pragma unroll
    for (int k = 0; k < kGsCols; k++) acc[k] = 0.f;
    float run_m = a.sinks ? a.sinks[h] : -INFINITY, run_l = a.sinks ? 1.f : 0.f;  // every thread keeps the same pair
    __syncthreads();
    for (int j0 = lo; j0 <= pos; j0 += kGsKeys) {
        const int nj = min(kGsKeys, pos + 1 - j0);
        for (int j = warp; j < nj; j += kGsThreads / 32) {
            const T *k = latent_row(plane, table, p.row_width, j0 + j) + k_col;
            float d = 0.f;
            for (int i = lane; i < a.dp; i += 32) d = fmaf(Num<T>::get(k[i]), qs[i], d);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
            if (lane == 0) sc[j] = d * a.scale - slope * (float)(pos - j0 - j);
        }
        __syncthreads();
        if (warp == 0) {
            const float a0 = lane < nj ? sc[lane] : -INFINITY, a1 = lane + 32 < nj ? sc[lane + 32] : -INFINITY;
            float m = fmaxf(a0, a1);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
            m = fmaxf(m, run_m);
            const float e0 = expf(a0 - m), e1 = expf(a1 - m);
            float s = e0 + e1;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            sc[lane] = e0;
            sc[lane + 32] = e1;
            if (lane == 0) {
                red[0] = m;
                red[1] = s;
            }
        }
        __syncthreads();
        const float f = expf(run_m - red[0]);
        run_m = red[0];
        run_l = run_l * f + red[1];
#pragma unroll
        for (int k = 0; k < kGsCols; k++) {
            const int col = tid + k * kGsThreads;
            if (col < a.vp) {
                float v = acc[k] * f;
                for (int j = 0; j < nj; j++) v = fmaf(sc[j], Num<T>::get(latent_row(plane, table, p.row_width, j0 + j)[v_col + col]), v);
                acc[k] = v;
            }
        }
        __syncthreads();
    }
    T *o = static_cast<T *>(a.out) + ((size_t)row * a.heads + h) * a.vp;
#pragma unroll
    for (int k = 0; k < kGsCols; k++) {
        const int col = tid + k * kGsThreads;
        if (col < a.vp) o[col] = Num<T>::put(acc[k] / run_l);
    }
}

// ───────────────────────────── decode: splits of the span ─────────────────────────────────
// A CTA (four warps) takes a tile of at most sixteen query heads of one key/value head of one row and a range of page-sized key
// tiles; its warps take turns over the tiles, each with a ring of its own (cp.async, no barrier between warps) and its own
// online softmax on mma.sync.  The warps' states are merged through shared memory, the splits by whichever CTA arrives last.
constexpr int kGdThreads = 128, kGdWarps = 4, kGdStages = 3;
static_assert(kPageTokens == 16, "a key tile is a page");

struct GroupedSplitParams {
    GroupedParams g;
    int n_splits, head_tiles;
    float *part_o, *part_ml;
    unsigned *counters;
};

static size_t grouped_split_smem(int dp, int vp) {
    const size_t ring = (size_t)kGdWarps * kGdStages * 16 * (dp + vp + 16) * 2;
    const size_t merge = (size_t)kGdWarps * 16 * (vp + 4) * 4 + (size_t)kGdWarps * 16 * 2 * 4 + (size_t)16 * (kGroupedMaxSplits + 2) * 4;
    return (size_t)16 * (dp + 8) * 2 + std::max(ring, merge);
}

// ND: 16-column steps of a head at most; FUSED: queries, keys and values from the projections; DIM: query, key and value size
// of a head when they are equal and a common number (every offset and bound folds), else 0
template <int ND, bool FUSED, int DIM>
__global__ void __launch_bounds__(kGdThreads) grouped_split_kernel(const __grid_constant__ GroupedSplitParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    const GroupedAttnArgs &a = p.g.a;
    const int dp = DIM ? DIM : a.dp, vp = DIM ? DIM : a.vp, kp = dp + 8, vpitch = vp + 8, nk = dp >> 4, nv = vp >> 4;
    bf16 *qs = reinterpret_cast<bf16 *>(sm);  // [16][kp]
    uint8_t *pool_s = sm + 16 * kp * 2;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row = blockIdx.z, kvh = blockIdx.y / p.head_tiles, ht = blockIdx.y - kvh * p.head_tiles;
    const int group = a.heads / a.kv_heads, h0 = kvh * group + ht * 16, nh = min(16, group - ht * 16);
    if (!FUSED) pdl_wait();  // the appends of this step are the previous kernel's
    const int pos = a.rows.positions[row], lo = a.span.first(pos);
    const int32_t *table = p.g.table + (size_t)a.rows.slots[row] * p.g.max_pages;
    const int tile0 = lo >> 4, tiles = (pos >> 4) - tile0 + 1, per = (tiles + p.n_splits - 1) / p.n_splits;
    const int used = (tiles + per - 1) / per;  // splits that have tiles
    if ((int)blockIdx.x >= used) return;
    const int t_beg = tile0 + blockIdx.x * per, t_end = min(tile0 + tiles, t_beg + per);
    const bool newest = FUSED && t_end == tile0 + tiles;  // this CTA reads the position of this step
    bf16 *plane = static_cast<bf16 *>(p.g.plane);
    bf16 *ring = reinterpret_cast<bf16 *>(pool_s) + (size_t)warp * kGdStages * 16 * (kp + vpitch);
    const int kc = dp >> 3, vc = vp >> 3;
    const int kr0 = lane / kc, kch0 = lane - kr0 * kc, krs = 32 / kc, kcs = 32 - krs * kc;
    const int vr0 = lane / vc, vch0 = lane - vr0 * vc, vrs = 32 / vc, vcs = 32 - vrs * vc;
    auto load_part = [&](const bf16 *src, uint32_t dst, int pitch, int key0, int r, int ch, int rs, int chs, int nch) {
        if (DIM && key0 >= lo && key0 + 15 <= pos) {  // every row is seen: a lane's pieces lie in one column of them
            src += (size_t)r * p.g.row_width + ch * 8;
            dst += (uint32_t)(r * pitch + ch * 8) * 2;
#pragma unroll
            for (int i = 0; i < 16; i += 32 / (DIM ? DIM / 8 : 1)) {
                cp16(dst + (uint32_t)(i * pitch) * 2, src, true);
                src += (size_t)rs * p.g.row_width;
            }
            return;
        }
        while (r < 16) {
            const bool ok = key0 + r >= lo && key0 + r <= pos;
            cp16(dst + (uint32_t)(r * pitch + ch * 8) * 2, ok ? src + (size_t)r * p.g.row_width + ch * 8 : plane, ok);
            ch += chs;
            r += rs;
            if (ch >= nch) {
                ch -= nch;
                r++;
            }
        }
    };
    int page = t_beg + warp < t_end ? table[t_beg + warp] : 0;  // of the next tile to load
    auto load_tile = [&](int ti, int stage) {
        if (ti < t_end) {
            const bf16 *src = plane + (size_t)page * kPageTokens * p.g.row_width;
            bf16 *ks = ring + stage * 16 * (kp + vpitch);
            load_part(src + kvh * dp, smem_addr(ks), kp, ti * 16, kr0, kch0, krs, kcs, kc);
            load_part(src + a.kv_heads * dp + kvh * vp, smem_addr(ks + 16 * kp), vpitch, ti * 16, vr0, vch0, vrs, vcs, vc);
            if (ti + kGdWarps < t_end) page = table[ti + kGdWarps];
        }
        cp_commit();
    };
    auto first_tiles = [&]() {
#pragma unroll
        for (int s = 0; s < kGdStages - 1; s++) load_tile(t_beg + warp + s * kGdWarps, s);
    };
    if (FUSED) {
        if (!newest) first_tiles();  // pages that earlier steps have completed
        pdl_wait();
    }
    pdl_launch_dependents();
    if (FUSED) {
        const float *u = a.u + (size_t)row * a.ldu;
        const float2 *rot = a.rot ? a.rot + (size_t)pos * (a.rot_dims >> 1) : nullptr;
        const float f = query_factor(a, pos);
        for (int r = warp; r < 16; r += kGdWarps) {
            if (r < nh)
                put_head(u + (h0 + r) * dp, a.dim, dp, a.q_norm, a.eps, rot, a.rot_dims, f, qs + r * kp, lane);
            else
                for (int i = lane; i < dp; i += 32) qs[r * kp + i] = __float2bfloat16_rn(0.f);
        }
        if (newest) {  // the head tiles of a group append the same numbers
            bf16 *dst = latent_row(plane, table, p.g.row_width, pos);
            if (warp == kGdWarps - 1) {
                put_head(u + (a.heads + kvh) * dp, a.dim, dp, a.k_norm, a.eps, rot, a.rot_dims, 1.f, dst + kvh * dp, lane);
            } else if (warp == kGdWarps - 2) {
                const float *v = u + (a.heads + a.kv_heads) * dp + kvh * vp;
                bf16 *vd = dst + a.kv_heads * dp + kvh * vp;
                for (int i = lane; i < vp; i += 32) vd[i] = __float2bfloat16_rn(v[i]);
            }
        }
        __syncthreads();
        if (newest) first_tiles();
    } else {
        first_tiles();
        const bf16 *q = static_cast<const bf16 *>(a.q) + ((size_t)row * a.heads + h0) * dp;
        for (int i = tid; i < 16 * kc; i += kGdThreads) {
            const int r = i / kc, ch = i - r * kc;
            *reinterpret_cast<uint4 *>(qs + r * kp + ch * 8) = r < nh ? *reinterpret_cast<const uint4 *>(q + (size_t)r * dp + ch * 8) : make_uint4(0u, 0u, 0u, 0u);
        }
        __syncthreads();
    }
    const int lr = lane & 15, lc = (lane >> 4) * 8, br = (lane & 7) + (lane >> 4) * 8, bc = ((lane >> 3) & 1) * 8;
    uint32_t qa[ND][4];
#pragma unroll
    for (int k = 0; k < ND; k++)
        if (k < nk) ldsm4(qa[k], smem_addr(qs + lr * kp + k * 16 + lc));
    const float scale_l2 = a.scale * kLog2e;
    const float slope0 = a.slopes && g < nh ? a.slopes[h0 + g] * kLog2e : 0.f, slope1 = a.slopes && g + 8 < nh ? a.slopes[h0 + g + 8] * kLog2e : 0.f;
    float o[ND][2][4], mx[2] = {-INFINITY, -INFINITY}, ls[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < ND; i++)
#pragma unroll
        for (int k = 0; k < 2; k++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[i][k][e] = 0.f;
    int stage = 0;
    for (int ti = t_beg + warp; ti < t_end; ti += kGdWarps) {
        cp_wait<kGdStages - 2>();
        __syncwarp();
        load_tile(ti + (kGdStages - 1) * kGdWarps, stage == 0 ? kGdStages - 1 : stage - 1);
        const bf16 *ks = ring + stage * 16 * (kp + vpitch), *vs = ks + 16 * kp;
        stage = stage + 1 == kGdStages ? 0 : stage + 1;
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int k = 0; k < ND; k++)
            if (k < nk) {
                uint32_t b[4];
                ldsm4(b, smem_addr(ks + br * kp + k * 16 + bc));
                mma16816(s[0], qa[k], b[0], b[1]);
                mma16816(s[1], qa[k], b[2], b[3]);
            }
        float f[2];
        const bool whole = ti * 16 >= lo && ti * 16 + 15 <= pos;
#pragma unroll
        for (int e2 = 0; e2 < 2; e2++) {
            float m = mx[e2];
            const float slope = e2 ? slope1 : slope0;
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int key = ti * 16 + i * 8 + 2 * t + e;
                    float &v = s[i][e2 * 2 + e];
                    v *= scale_l2;
                    if (a.slopes) v = fmaf((float)(key - pos), slope, v);
                    if (!whole && (key < lo || key > pos)) v = -INFINITY;
                    m = fmaxf(m, v);
                }
            m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
            m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
            f[e2] = ex2(mx[e2] - m);  // every tile has a key that is seen: m is finite
            mx[e2] = m;
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const float v = ex2(s[i][e2 * 2 + e] - m);
                    s[i][e2 * 2 + e] = v;
                    sum += v;
                }
            ls[e2] = ls[e2] * f[e2] + sum;
        }
        const uint32_t pa[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
        if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {  // a maximum has moved
#pragma unroll
            for (int i = 0; i < ND; i++)
#pragma unroll
                for (int k = 0; k < 2; k++) {
                    o[i][k][0] *= f[0];
                    o[i][k][1] *= f[0];
                    o[i][k][2] *= f[1];
                    o[i][k][3] *= f[1];
                }
        }
#pragma unroll
        for (int i = 0; i < ND; i++)
            if (i < nv) {
                uint32_t b[4];
                ldsm4_trans(b, smem_addr(vs + lr * vpitch + i * 16 + lc));
                mma16816(o[i][0], pa, b[0], b[1]);
                mma16816(o[i][1], pa, b[2], b[3]);
            }
    }
    cp_wait<0>();
#pragma unroll
    for (int e2 = 0; e2 < 2; e2++) {
        ls[e2] += __shfl_xor_sync(0xffffffffu, ls[e2], 1);
        ls[e2] += __shfl_xor_sync(0xffffffffu, ls[e2], 2);
    }
    __syncthreads();  // the rings become the merge's buffers
    const int op = vp + 4;
    float *os = reinterpret_cast<float *>(pool_s);         // [warp][16][op]
    float *ml = os + kGdWarps * 16 * op;                   // [warp][16][2]
    float *wt = ml + kGdWarps * 16 * 2;                    // [16][kGroupedMaxSplits]: weights of the parts
    float *tot = wt + 16 * kGroupedMaxSplits;              // [16][2]: maximum and sum of this split
    if (t == 0) {
#pragma unroll
        for (int e2 = 0; e2 < 2; e2++) *reinterpret_cast<float2 *>(ml + (warp * 16 + g + e2 * 8) * 2) = make_float2(mx[e2], ls[e2]);
    }
#pragma unroll
    for (int i = 0; i < ND; i++)
        if (i < nv)
#pragma unroll
            for (int k = 0; k < 2; k++) {
                float *d = os + (warp * 16 + g) * op + i * 16 + k * 8 + 2 * t;
                *reinterpret_cast<float2 *>(d) = make_float2(o[i][k][0], o[i][k][1]);
                *reinterpret_cast<float2 *>(d + 8 * op) = make_float2(o[i][k][2], o[i][k][3]);
            }
    __syncthreads();
    const bool alone = used == 1;
    if (tid < nh) {
        float m = alone && a.sinks ? a.sinks[h0 + tid] * kLog2e : -INFINITY, l = 0.f;
        const float sink = m;
#pragma unroll
        for (int k = 0; k < kGdWarps; k++) m = fmaxf(m, ml[(k * 16 + tid) * 2]);
        if (alone && a.sinks) l = ex2(sink - m);
#pragma unroll
        for (int k = 0; k < kGdWarps; k++) l = fmaf(ml[(k * 16 + tid) * 2 + 1], ex2(ml[(k * 16 + tid) * 2] - m), l);
        const float norm = alone ? 1.f / l : 1.f;
#pragma unroll
        for (int k = 0; k < kGdWarps; k++) wt[tid * kGroupedMaxSplits + k] = ex2(ml[(k * 16 + tid) * 2] - m) * norm;
        tot[tid * 2] = m;
        tot[tid * 2 + 1] = l;
    }
    __syncthreads();
    bf16 *out = static_cast<bf16 *>(a.out) + ((size_t)row * a.heads + h0) * vp;
    const int cg = vp >> 2;  // groups of four columns
    const size_t part = ((size_t)row * a.heads + h0) * p.n_splits;
    for (int i = tid; i < nh * cg; i += kGdThreads) {
        const int r = i / cg, col = (i - r * cg) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < kGdWarps; k++) {
            const float w = wt[r * kGroupedMaxSplits + k];
            const float4 x = load4(os + (k * 16 + r) * op + col);
            v = make_float4(fmaf(w, x.x, v.x), fmaf(w, x.y, v.y), fmaf(w, x.z, v.z), fmaf(w, x.w, v.w));
        }
        if (alone)
            store4(out + (size_t)r * vp + col, v);
        else
            store4(p.part_o + (part + (size_t)r * p.n_splits + blockIdx.x) * vp + col, v);
    }
    if (alone) return;
    if (tid < nh) *reinterpret_cast<float2 *>(p.part_ml + (part + (size_t)tid * p.n_splits + blockIdx.x) * 2) = make_float2(tot[tid * 2], tot[tid * 2 + 1]);
    // the last split merges: its CTA sees every other CTA's stores, which were made visible before they were counted
    __shared__ bool last;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        unsigned *count = p.counters + (size_t)row * gridDim.y + blockIdx.y;
        last = atomicAdd(count, 1u) == (unsigned)used - 1u;
        if (last) *count = 0u;  // as the next launch expects it
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    for (int r = warp; r < nh; r += kGdWarps) {
        const float2 *e = reinterpret_cast<const float2 *>(p.part_ml) + part + (size_t)r * p.n_splits;
        const float2 none = make_float2(-INFINITY, 0.f), e0 = lane < used ? __ldcg(e + lane) : none, e1 = lane + 32 < used ? __ldcg(e + lane + 32) : none;
        const float sink = a.sinks ? a.sinks[h0 + r] * kLog2e : -INFINITY;
        float m = fmaxf(e0.x, e1.x);
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
        m = fmaxf(m, sink);
        const float f0 = ex2(e0.x - m), f1 = ex2(e1.x - m);
        float l = e0.y * f0 + e1.y * f1;
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
        const float norm = 1.f / (l + ex2(sink - m));
        wt[r * kGroupedMaxSplits + lane] = f0 * norm;
        wt[r * kGroupedMaxSplits + lane + 32] = f1 * norm;
    }
    __syncthreads();
    for (int i = tid; i < nh * cg; i += kGdThreads) {
        const int r = i / cg, col = (i - r * cg) * 4;
        const float *po = p.part_o + (part + (size_t)r * p.n_splits) * vp + col;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = 0; s < used; s++) {
            const float w = wt[r * kGroupedMaxSplits + s];
            const float4 x = __ldcg(reinterpret_cast<const float4 *>(po + (size_t)s * vp));
            v = make_float4(fmaf(w, x.x, v.x), fmaf(w, x.y, v.y), fmaf(w, x.z, v.z), fmaf(w, x.w, v.w));
        }
        store4(out + (size_t)r * vp + col, v);
    }
}

__global__ void rotation_table_kernel(int n, int half, double base, float2 *table) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)n * half) return;
    const int pos = (int)(i / half), k = (int)(i - (size_t)pos * half);
    double s, c;
    sincos((double)pos * pow(base, -(double)k / half), &s, &c);
    table[i] = make_float2((float)c, (float)s);
}

// ───────────────────────────── launches ───────────────────────────────────────────────────
static int grouped_params(int dt, const GroupedAttnArgs &a, GroupedParams *p) {
    JUNO_REQUIRE(a.rows.n > 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= a.dp && a.dp % 16 == 0 && a.vp % 16 == 0 && a.vp > 0,
                 "grouped attention: bad sizes (heads %d over %d, dim %d)", a.heads, a.kv_heads, a.dim);
    JUNO_REQUIRE(a.pool && a.pool->latent && a.pool->dtype == (dt == DT_F32 ? 1 : 2) && a.pool->row_width[a.layer] == a.kv_heads * (a.dp + a.vp),
                 "grouped attention: pages of another layout");
    JUNO_REQUIRE(!a.rot || (a.rot_dims % 2 == 0 && a.rot_dims <= a.dim), "grouped attention: %d rotated dimensions of %d", a.rot_dims, a.dim);
    memset((void *)p, 0, sizeof(*p));
    p->a = a;
    p->table = a.pool->d_table;
    p->max_pages = a.pool->max_pages_per_seq;
    p->row_width = a.pool->row_width[a.layer];
    p->plane = static_cast<uint8_t *>(a.pool->k) + a.pool->row_off[a.layer] * a.pool->elem_bytes;
    return JUNO_OK;
}

int launch_rotation_table(juno_ctx *c, int n, int dims, double base, float2 *table, cudaStream_t st) {
    const int half = dims / 2;
    const size_t total = (size_t)n * half;
    if (total == 0) return JUNO_OK;
    rotation_table_kernel<<<(unsigned)((total + 255) / 256), 256, 0, st>>>(n, half, base, table);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_grouped_prep(juno_ctx *c, int dt, const GroupedAttnArgs &a, cudaStream_t st) {
    GroupedParams p;
    JUNO_TRY(grouped_params(dt, a, &p));
    const int units = a.heads + 2 * a.kv_heads;
    const dim3 grid((unsigned)a.rows.n, (unsigned)((units + kPrepWarps - 1) / kPrepWarps));
    ProfScope prof(c, st, PROF_ROWOPS, (double)a.rows.n * (a.heads * a.dp + a.kv_heads * (a.dp + a.vp)) * (4 + dt_bytes(dt)));
    if (dt == DT_F32)
        grouped_prep_kernel<float><<<grid, kPrepWarps * 32, 0, st>>>(p);
    else
        grouped_prep_kernel<bf16><<<grid, kPrepWarps * 32, 0, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_grouped_simt(juno_ctx *c, int dt, const GroupedAttnArgs &a, cudaStream_t st) {
    GroupedParams p;
    JUNO_TRY(grouped_params(dt, a, &p));
    JUNO_REQUIRE(a.vp <= kGroupedMaxVdim && a.dp <= 8192 && a.rows.n <= 65535, "grouped attention: heads of %d / %d are too wide", a.dp, a.vp);
    const dim3 grid((unsigned)a.heads, (unsigned)a.rows.n);
    const size_t smem = (size_t)a.dp * 4;
    ProfScope prof(c, st, PROF_ATTN, 0);
    if (dt == DT_F32)
        grouped_simt_kernel<float><<<grid, kGsThreads, smem, st>>>(p);
    else
        grouped_simt_kernel<bf16><<<grid, kGsThreads, smem, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int grouped_pick_splits(const juno_ctx *c, int n, int heads, int kv_heads, int dim, int keys) {
    const int tiles = (keys + 15) / 16 + 1, rounds = (tiles + kGdWarps - 1) / kGdWarps;
    const long long ctas = (long long)n * kv_heads * ((heads / kv_heads + 15) / 16);
    const int slots = c->sm_count * (dim > 128 ? 1 : 2);
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= std::min(rounds, kGroupedMaxSplits); s++) {
        if (s > 1 && ctas * s > 4ll * c->sm_count) break;
        // rounds of CTAs over the SMs, each as long as a warp's tiles and a start-up; a merge costs its reader a little per part
        const double waves = (double)((ctas * s + slots - 1) / slots), cost = waves * ((rounds + s - 1) / s + 4) + (s > 1 ? 2 + 0.1 * s : 0);
        if (cost < best_cost) {
            best_cost = cost;
            best = s;
        }
    }
    return best;
}
size_t grouped_part_floats(const juno_ctx *c, int vp) { return (size_t)4 * c->sm_count * 16 * (vp + 2); }
size_t grouped_counters(const juno_ctx *c) { return (size_t)4 * c->sm_count; }

template <int ND, bool FUSED, int DIM = 0>
static int split_launch(juno_ctx *c, const GroupedSplitParams &p, dim3 grid, size_t smem, cudaStream_t st) {
    static std::mutex mu;
    static size_t have[16] = {0};
    {
        std::lock_guard<std::mutex> lk(mu);
        if (smem > have[c->device & 15]) {
            JUNO_CUDA_TRY(cudaFuncSetAttribute(grouped_split_kernel<ND, FUSED, DIM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            have[c->device & 15] = smem;
        }
    }
    if (FUSED)
        JUNO_CUDA_TRY(launch_pdl(grouped_split_kernel<ND, FUSED, DIM>, grid, dim3(kGdThreads), smem, st, p));
    else
        grouped_split_kernel<ND, FUSED, DIM><<<grid, kGdThreads, smem, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_grouped_split(juno_ctx *c, const GroupedAttnArgs &a, int n_splits, bool fused, float *part, size_t part_floats, unsigned *counters, cudaStream_t st) {
    GroupedSplitParams p;
    memset((void *)&p, 0, sizeof(p));
    JUNO_TRY(grouped_params(DT_BF16, a, &p.g));
    const int n = a.rows.n, d = std::max(a.dp, a.vp);
    JUNO_REQUIRE(d <= kGroupedMaxDim && n_splits >= 1 && n_splits <= kGroupedMaxSplits && n <= 65535 && (!fused || !a.rows.one_seq), "grouped attention (splits): bad arguments");
    p.head_tiles = (a.heads / a.kv_heads + 15) / 16;
    p.n_splits = n_splits;
    const long long ctas = (long long)n * a.kv_heads * p.head_tiles;
    if (n_splits > 1) {
        const size_t rows = (size_t)n * a.heads * n_splits;
        JUNO_REQUIRE(rows * (a.vp + 2) <= part_floats && ctas <= (long long)grouped_counters(c), "%d context splits of %d rows exceed the buffer", n_splits, n);
        p.part_o = part;
        p.part_ml = part + rows * a.vp;
        p.counters = counters;
    }
    const dim3 grid((unsigned)n_splits, (unsigned)(a.kv_heads * p.head_tiles), (unsigned)n);
    const size_t smem = grouped_split_smem(a.dp, a.vp);
    ProfScope prof(c, st, PROF_ATTN, 0);
    if (a.dp == 64 && a.vp == 64) return fused ? split_launch<4, true, 64>(c, p, grid, smem, st) : split_launch<4, false, 64>(c, p, grid, smem, st);
    if (a.dp == 128 && a.vp == 128) return fused ? split_launch<8, true, 128>(c, p, grid, smem, st) : split_launch<8, false, 128>(c, p, grid, smem, st);
    if (fused) {
        if (d <= 64) return split_launch<4, true>(c, p, grid, smem, st);
        if (d <= 128) return split_launch<8, true>(c, p, grid, smem, st);
        return split_launch<16, true>(c, p, grid, smem, st);
    }
    if (d <= 64) return split_launch<4, false>(c, p, grid, smem, st);
    if (d <= 128) return split_launch<8, false>(c, p, grid, smem, st);
    return split_launch<16, false>(c, p, grid, smem, st);
}

}  // namespace juno
