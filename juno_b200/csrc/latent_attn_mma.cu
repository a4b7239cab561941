// BF16 attention over latent pages on the tensor cores: the split kernel of decode steps with its merge (see latent_attn.cuh).
#include <algorithm>
#include <mutex>

#include "latent_attn.cuh"
#include "mma_bf16.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

// ───────────────────────────── decode: splits of the context ──────────────────────────────
// A CTA (sixteen warps, one per SM) takes a group of 16 * MT heads of one row and a range of positions, 32 at a time.  Scores:
// warp (16 positions, an eighth of the rank) multiplies its part of q_lat - A fragments it keeps in registers - with the tile,
// the eight parts are added in shared memory; online softmax by rows; O += P C: each warp owns a range of latent columns and
// reads the tile transposed.  The scores of tile i + 1 and the averages of tile i are one phase between barriers (their MMAs
// fill each other's latencies), while tile i + 2 is on its way.
constexpr int kSpThreads = 512, kSpWarps = 16;

struct SplitParams {
    const bf16 *plane;
    const int32_t *table, *positions, *slots;
    int max_pages, heads, rank, n_splits;
    float scale_log2;
    const bf16 *q;
    float *part_o, *part_ml;
};

__device__ __forceinline__ float warp_max(float v) {
    float r;
    asm("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
    return r;
}

constexpr int kSpKeys = 32, kSpParts = 8, kSpPitch = kSpKeys + 8;  // score rows 8 banks apart: the float2 stores of a warp meet no bank twice

template <int MT>
constexpr size_t split_smem(int rank) {
    return (size_t)3 * kSpKeys * (rank + 8) * 2 + (size_t)16 * MT * (kSpKeys + 8) * 2 + (size_t)kSpParts * 16 * MT * kSpPitch * 4 + (size_t)16 * MT * 4;
}

// NQ: 16-column steps of the rank a warp scores at most; NP: 16-column pairs of n-tiles a warp averages at most; RANK: the rank,
// when it is a common one (every offset and bound folds), else 0
template <int MT, int NQ, int NP, int RANK>
__global__ void __launch_bounds__(kSpThreads, 1) latent_split_kernel(const SplitParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    constexpr int HM = 16 * MT, SP = kSpPitch;
    const int R = RANK ? RANK : p.rank, pitch = R + 8;
    bf16 *cs = reinterpret_cast<bf16 *>(sm);          // [3][kSpKeys][pitch]
    bf16 *ps = cs + 3 * kSpKeys * pitch;              // [HM][kSpKeys + 8]
    float *ss = reinterpret_cast<float *>(ps + HM * (kSpKeys + 8));  // [kSpParts][HM][SP]
    float *fac = ss + kSpParts * HM * SP;
    const int split = blockIdx.x, h0 = blockIdx.y * HM, row = blockIdx.z, nh = min(HM, p.heads - h0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_launch_dependents();
    const int len = p.positions[row] + 1;
    const int tiles = (len + kSpKeys - 1) / kSpKeys, per = (tiles + p.n_splits - 1) / p.n_splits;
    const int j0 = split * per * kSpKeys, j1 = min(len, j0 + per * kSpKeys);
    const size_t part = ((size_t)row * p.heads + h0) * p.n_splits + split;  // + head * n_splits
    if (j0 >= j1) {
        if (tid < nh) {
            p.part_ml[(part + (size_t)tid * p.n_splits) * 2] = -INFINITY;
            p.part_ml[(part + (size_t)tid * p.n_splits) * 2 + 1] = 0.f;
        }
        return;
    }
    const int32_t *table = p.table + (size_t)p.slots[row] * p.max_pages;
    const int chunks = R >> 3;
    const int r0 = warp * 2;  // two consecutive rows per warp: they lie in one page, whose number is read a tile ahead
    auto page_of = [&](int j) { return j + r0 < j1 ? table[(j + r0) >> 4] : 0; };
    int page = page_of(j0);
    auto load_tile = [&](int j, int buf) {
        const bf16 *src = p.plane + ((size_t)page * kPageTokens + ((j + r0) & (kPageTokens - 1))) * R;
        page = page_of(j + kSpKeys);
        const uint32_t dst = smem_addr(cs + ((size_t)buf * kSpKeys + r0) * pitch);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const bool ok = j + r0 + i < j1;
            for (int ch = lane; ch < chunks; ch += 32) cp16(dst + (uint32_t)(i * pitch + ch * 8) * 2, ok ? src + (size_t)i * R + ch * 8 : p.plane, ok);
        }
        cp_commit();
    };
    load_tile(j0, 0);
    if (j0 + kSpKeys < j1)
        load_tile(j0 + kSpKeys, 1);
    else
        cp_commit();
    const int kg = warp & 1, rq = warp >> 1;                      // 16 positions, part of the rank
    const int ksteps = R >> 4, ks0 = ksteps * rq / kSpParts, nq = ksteps * (rq + 1) / kSpParts - ks0;
    const int pairs = R >> 4, pw = (pairs + kSpWarps - 1) / kSpWarps, c0 = warp * pw * 16;  // columns of O
    const int np = max(0, min(pw, pairs - warp * pw));
    uint32_t qa[NQ][MT][4];
#pragma unroll
    for (int k = 0; k < NQ; k++)
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = m * 16 + g + (e & 1) * 8, col = (ks0 + k) * 16 + 2 * t + (e >> 1) * 8;
                qa[k][m][e] = k < nq && r < nh ? *reinterpret_cast<const uint32_t *>(p.q + ((size_t)row * p.heads + h0 + r) * R + col) : 0u;
            }
    float o[MT][NP][2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int i = 0; i < NP; i++)
#pragma unroll
            for (int k = 0; k < 2; k++)
#pragma unroll
                for (int e = 0; e < 4; e++) o[m][i][k][e] = 0.f;
    const int lr = lane & 15, lc = (lane >> 4) * 8;   // ldmatrix x4: row, column offset (A operand; transposed B operand)
    const int br = (lane & 7) + (lane >> 4) * 8, bc = ((lane >> 3) & 1) * 8;  // B operand from rows of keys: two n-tiles at once
    const uint32_t p_a = smem_addr(ps + lr * (kSpKeys + 8) + lc);
    const uint32_t cs_a = smem_addr(cs), k_off = (uint32_t)((kg * 16 + br) * pitch + ks0 * 16 + bc) * 2, v_off = (uint32_t)(lr * pitch + c0 + lc) * 2;
    const uint32_t tile_bytes = (uint32_t)kSpKeys * pitch * 2;
    auto scores = [&](int buf) {
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int k = 0; k < 2; k++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[m][k][e] = 0.f;
#pragma unroll
        for (int k = 0; k < NQ; k++)
            if (k < nq) {
                uint32_t b[4];
                ldsm4(b, cs_a + buf * tile_bytes + k_off + k * 32);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma16816(s[m][0], qa[k][m], b[0], b[1]);
                    mma16816(s[m][1], qa[k][m], b[2], b[3]);
                }
            }
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int k = 0; k < 2; k++) {
                float *d = ss + (rq * HM + m * 16 + g) * SP + kg * 16 + k * 8 + 2 * t;
                *reinterpret_cast<float2 *>(d) = make_float2(s[m][k][0], s[m][k][1]);
                *reinterpret_cast<float2 *>(d + 8 * SP) = make_float2(s[m][k][2], s[m][k][3]);
            }
    };
    // a warp's MT rows are always the same ones: running maximum (the same in all lanes) and each lane's share of the sum
    float run_m[MT], run_l[MT];
#pragma unroll
    for (int i = 0; i < MT; i++) {
        run_m[i] = -INFINITY;
        run_l[i] = 0.f;
    }
    auto softmax = [&](int j) {
        float v[MT];
#pragma unroll
        for (int i = 0; i < MT; i++) v[i] = 0.f;
#pragma unroll
        for (int k = 0; k < kSpParts; k++)
#pragma unroll
            for (int i = 0; i < MT; i++) v[i] += ss[(k * HM + warp * MT + i) * SP + lane];
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int r = warp * MT + i;
            v[i] = j + lane < j1 ? v[i] * p.scale_log2 : -INFINITY;
            const float m = fmaxf(run_m[i], warp_max(v[i])), f = ex2(run_m[i] - m), e = ex2(v[i] - m);
            ps[r * (kSpKeys + 8) + lane] = __float2bfloat16_rn(e);
            if (lane == 0) fac[r] = f;
            run_l[i] = run_l[i] * f + e;
            run_m[i] = m;
        }
    };
    auto averages = [&](int buf) {
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const float f0 = fac[m * 16 + g], f1 = fac[m * 16 + g + 8];
            if (!__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) continue;  // no maximum has moved
#pragma unroll
            for (int i = 0; i < NP; i++)
#pragma unroll
                for (int k = 0; k < 2; k++) {
                    o[m][i][k][0] *= f0;
                    o[m][i][k][1] *= f0;
                    o[m][i][k][2] *= f1;
                    o[m][i][k][3] *= f1;
                }
        }
#pragma unroll
        for (int kk = 0; kk < kSpKeys / 16; kk++) {
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) ldsm4(a[m], p_a + (uint32_t)(m * 16 * (kSpKeys + 8) + kk * 16) * 2);
#pragma unroll
            for (int i = 0; i < NP; i++)
                if (i < np) {
                    uint32_t b[4];
                    ldsm4_trans(b, cs_a + buf * tile_bytes + v_off + (uint32_t)(kk * 16 * pitch + i * 16) * 2);
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        mma16816(o[m][i][0], a[m], b[0], b[1]);
                        mma16816(o[m][i][1], a[m], b[2], b[3]);
                    }
                }
        }
    };
    cp_wait<1>();
    __syncthreads();
    scores(0);
    __syncthreads();
    softmax(j0);
    int buf = 0;
    for (int j = j0; j < j1; j += kSpKeys) {  // tile j has its weights in ps
        const int b1 = buf == 2 ? 0 : buf + 1, b2 = b1 == 2 ? 0 : b1 + 1;
        cp_wait<0>();
        __syncthreads();
        if (j + 2 * kSpKeys < j1) load_tile(j + 2 * kSpKeys, b2);
        if (j + kSpKeys < j1) scores(b1);
        averages(buf);
        if (j + kSpKeys >= j1) break;
        __syncthreads();
        softmax(j + kSpKeys);
        buf = b1;
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int i = 0; i < NP; i++)
            if (i < np)
#pragma unroll
                for (int k = 0; k < 2; k++) {
                    const int col = c0 + i * 16 + k * 8 + 2 * t, ha = m * 16 + g, hb = ha + 8;
                    if (ha < nh) *reinterpret_cast<float2 *>(p.part_o + (part + (size_t)ha * p.n_splits) * R + col) = make_float2(o[m][i][k][0], o[m][i][k][1]);
                    if (hb < nh) *reinterpret_cast<float2 *>(p.part_o + (part + (size_t)hb * p.n_splits) * R + col) = make_float2(o[m][i][k][2], o[m][i][k][3]);
                }
#pragma unroll
    for (int i = 0; i < MT; i++) {
        const int r = warp * MT + i;
        float l = run_l[i];
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
        if (lane == 0 && r < nh) *reinterpret_cast<float2 *>(p.part_ml + (part + (size_t)r * p.n_splits) * 2) = make_float2(run_m[i], l);
    }
}

// ───────────────────────────── merge + value projection ───────────────────────────────────
// One block per (head, row, share of the value rows).  The threads form groups that add up different splits of the averaged
// latent; then every warp takes rows of W_uv.  Without w_uv the merged latent itself is the result (many rows: the value
// projection is a matrix product then).
constexpr int kMergeThreads = 512, kMaxSplits = 64;
struct MergeParams {
    LatentMergeArgs a;
    int rows_per;  // value rows of a block
};
__global__ void __launch_bounds__(kMergeThreads) latent_merge_kernel(const MergeParams p) {
    __shared__ __align__(16) float acc_s[kMergeThreads * 4];
    __shared__ __align__(16) float ol[kLatentSplitMaxRank];
    __shared__ float wsp[kMaxSplits];
    const LatentMergeArgs &a = p.a;
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int v0 = blockIdx.z * p.rows_per, v1 = min(a.vdim, v0 + p.rows_per);
    const bf16 *wuv = static_cast<const bf16 *>(a.w_uv);
    const size_t part = ((size_t)row * a.heads + h) * a.n_splits;
    if (warp == 0) {
        const bool h0 = lane < a.n_splits, h1 = lane + 32 < a.n_splits;
        const float2 z = make_float2(-INFINITY, 0.f), *ml = reinterpret_cast<const float2 *>(a.part_ml) + part;
        const float2 e0 = h0 ? ml[lane] : z, e1 = h1 ? ml[lane + 32] : z;
        float m = fmaxf(e0.x, e1.x);
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
        const float f0 = ex2(e0.x - m), f1 = ex2(e1.x - m);
        float l = e0.y * f0 + e1.y * f1;
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
        wsp[lane] = f0 / l;
        wsp[lane + 32] = f1 / l;
    }
    __syncthreads();
    const int nc = a.rank >> 2, ng = max(1, kMergeThreads / nc), gi = tid / nc, c = (tid - gi * nc) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (gi < ng) {
#pragma unroll 8
        for (int s = gi; s < a.n_splits; s += ng) {
            const float w = wsp[s];
            if (w != 0.f) {  // an empty split has written no rows
                const float4 x = load4(a.part_o + (part + s) * a.rank + c);
                v.x = fmaf(w, x.x, v.x);
                v.y = fmaf(w, x.y, v.y);
                v.z = fmaf(w, x.z, v.z);
                v.w = fmaf(w, x.w, v.w);
            }
        }
        store4(acc_s + tid * 4, v);
    }
    __syncthreads();
    if (gi == 0) {
        for (int k = 1; k < ng; k++) {
            const float4 x = load4(acc_s + (k * nc + tid) * 4);
            v.x += x.x;
            v.y += x.y;
            v.z += x.z;
            v.w += x.w;
        }
        if (!wuv)
            store4(static_cast<bf16 *>(a.out) + ((size_t)row * a.heads + h) * a.rank + c, v);
        else
            store4(ol + c, v);
    }
    if (!wuv) return;
    __syncthreads();
    const float gate = sigmoid_f32(a.gate[(size_t)row * a.ld_gate + h]);
    for (int r = v0 + warp; r < v1; r += kMergeThreads / 32) {
        const bf16 *w = wuv + ((size_t)h * a.vdim + r) * a.rank;
        float acc = 0.f;
#pragma unroll 4
        for (int k = lane * 4; k < a.rank; k += 128) {
            const float4 x = load4(w + k), y = load4(ol + k);
            acc = fmaf(x.x, y.x, acc);
            acc = fmaf(x.y, y.y, acc);
            acc = fmaf(x.z, y.z, acc);
            acc = fmaf(x.w, y.w, acc);
        }
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, d);
        if (lane == 0) static_cast<bf16 *>(a.out)[(size_t)row * a.heads * a.vdim + (size_t)h * a.vdim + r] = __float2bfloat16_rn(acc * gate);
    }
}

// ───────────────────────────── latents of a sequence, side by side ────────────────────────
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint8_t *plane, const int32_t *table, int max_pages, const int32_t *slot_of, int len,
                                                            int row_bytes, uint8_t *out) {
    const int per = row_bytes >> 4;
    const int32_t *row = table + (size_t)*slot_of * max_pages;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < (size_t)len * per; i += (size_t)gridDim.x * 256) {
        const int j = (int)(i / per), ch = (int)(i - (size_t)j * per);
        const uint4 v = *reinterpret_cast<const uint4 *>(plane + ((size_t)row[j >> 4] * kPageTokens + (j & (kPageTokens - 1))) * row_bytes + ch * 16);
        *reinterpret_cast<uint4 *>(out + (size_t)j * row_bytes + ch * 16) = v;
    }
}

// ───────────────────────────── launches ───────────────────────────────────────────────────
// Heads of a CTA: 32 (two tensor-core row tiles) when there are that many and the shared memory holds them.
static int head_tile(int heads, int rank) { return heads > 16 && rank <= 512 ? 32 : 16; }

int latent_pick_splits(const juno_ctx *c, int n, int heads, int rank, int len_bound) {
    const int ht = head_tile(heads, rank), ctas = n * ((heads + ht - 1) / ht), tiles = (len_bound + kSpKeys - 1) / kSpKeys;
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= std::min(tiles, kMaxSplits); s++) {
        // rounds of CTAs over the SMs, each as long as its tiles and a start-up; more splits cost the merge a little
        const double waves = ((long long)ctas * s + c->sm_count - 1) / c->sm_count, cost = waves * ((tiles + s - 1) / s + 3) + 0.04 * s;
        if (s > 1 && (long long)ctas * s > 2ll * c->sm_count + ctas) break;
        if (cost < best_cost) {
            best_cost = cost;
            best = s;
        }
    }
    return best;
}
size_t latent_part_floats(const juno_ctx *c, int n, int heads, int rank) {
    const int ht = head_tile(heads, rank);
    const long long groups = (long long)n * ((heads + ht - 1) / ht);
    return (size_t)std::min(groups * kMaxSplits, 2ll * c->sm_count + groups) * ht * (rank + 2);
}

template <int MT, int NQ, int NP, int RANK = 0>
static int split_launch(juno_ctx *c, const SplitParams &p, int n, cudaStream_t st) {
    constexpr int HM = 16 * MT;
    const size_t smem = split_smem<MT>(p.rank);
    static std::mutex mu;
    static size_t have[16] = {0};
    {
        std::lock_guard<std::mutex> lk(mu);
        if (smem > have[c->device & 15]) {
            JUNO_CUDA_TRY(cudaFuncSetAttribute(latent_split_kernel<MT, NQ, NP, RANK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            have[c->device & 15] = smem;
        }
    }
    JUNO_CUDA_TRY(launch_pdl(latent_split_kernel<MT, NQ, NP, RANK>, dim3((unsigned)p.n_splits, (unsigned)((p.heads + HM - 1) / HM), (unsigned)n), dim3(kSpThreads), smem, st, p));
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_latent_attn_split(juno_ctx *c, const LatentSplitArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.rows.n > 0 && a.heads > 0 && a.rank % 16 == 0 && a.rank <= kLatentSplitMaxRank && a.pool->latent && a.pool->dtype == 2 &&
                     a.pool->row_width[a.layer] == a.rank && a.n_splits >= 1 && a.n_splits <= kMaxSplits,
                 "latent attention (splits): bad arguments");
    SplitParams p;
    p.plane = reinterpret_cast<const bf16 *>(static_cast<const uint8_t *>(a.pool->k) + a.pool->row_off[a.layer] * 2);
    p.table = a.pool->d_table;
    p.positions = a.rows.positions;
    p.slots = a.rows.slots;
    p.max_pages = a.pool->max_pages_per_seq;
    p.heads = a.heads;
    p.rank = a.rank;
    p.n_splits = a.n_splits;
    p.scale_log2 = a.scale * kLog2e;
    p.q = static_cast<const bf16 *>(a.q_lat);
    p.part_o = a.part_o;
    p.part_ml = a.part_ml;
    ProfScope prof(c, st, PROF_ATTN, 0);
    const int n = a.rows.n;
    if (a.rank == 512) return a.heads <= 16 ? split_launch<1, 4, 2, 512>(c, p, n, st) : split_launch<2, 4, 2, 512>(c, p, n, st);
    if (a.rank > 512) return split_launch<1, 8, 4>(c, p, n, st);
    if (a.heads <= 16) return a.rank <= 256 ? split_launch<1, 2, 1>(c, p, n, st) : split_launch<1, 4, 2>(c, p, n, st);
    return a.rank <= 256 ? split_launch<2, 2, 1>(c, p, n, st) : split_launch<2, 4, 2>(c, p, n, st);
}

int launch_latent_merge(juno_ctx *c, const LatentMergeArgs &a, cudaStream_t st) {
    JUNO_REQUIRE(a.n > 0 && a.heads > 0 && a.rank % 16 == 0 && a.rank <= kLatentSplitMaxRank && a.n_splits >= 1 && a.n_splits <= kMaxSplits, "latent merge: bad arguments");
    MergeParams p;
    p.a = a;
    int parts = a.w_uv ? std::max(1, std::min((a.vdim + 15) / 16, (c->sm_count + a.n * a.heads - 1) / (a.n * a.heads))) : 1;
    p.rows_per = (a.vdim + parts - 1) / parts;
    parts = (a.vdim + p.rows_per - 1) / p.rows_per;
    ProfScope prof(c, st, PROF_ATTN, 0);
    // an ordinary launch: its many small blocks, made resident early by a programmatic dependent launch, measured 70 us per
    // layer slower at two and more sequences (they keep the large CTAs on both sides from their SMs)
    latent_merge_kernel<<<dim3((unsigned)a.heads, (unsigned)a.n, (unsigned)parts), kMergeThreads, 0, st>>>(p);
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

int launch_latent_gather(juno_ctx *c, const juno_kvpool *pool, int layer, const int32_t *slot_of, int len, void *out, cudaStream_t st) {
    JUNO_REQUIRE(pool->latent && len > 0, "latent gather: bad arguments");
    const int row_bytes = pool->row_width[layer] * pool->elem_bytes;
    const size_t n = (size_t)len * (row_bytes >> 4);
    ProfScope prof(c, st, PROF_ROWOPS, 2.0 * len * row_bytes);
    latent_gather_kernel<<<(unsigned)std::min<size_t>((n + 255) / 256, 4 * (size_t)c->sm_count), 256, 0, st>>>(
        static_cast<const uint8_t *>(pool->k) + pool->row_off[layer] * pool->elem_bytes, pool->d_table, pool->max_pages_per_seq, slot_of, len, row_bytes,
        static_cast<uint8_t *>(out));
    JUNO_CUDA_TRY(cudaGetLastError());
    c->kernel_launches++;
    return JUNO_OK;
}

}  // namespace juno
