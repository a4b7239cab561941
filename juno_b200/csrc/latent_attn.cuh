// Attention over latent pages: head h scores q_lat[h] . c_j and averages the same rows c_j, where c_j is the normed latent of
// position j and q_lat[h] = Wuk[h]^T q[h].  Keys and values are linear in c, so the pages hold one row per position for all
// heads, and the value projection Wuv[h] is applied to the averaged latent.
#pragma once
#include "rowops.cuh"

namespace juno {

struct LatentAttnArgs {
    const juno_kvpool *pool;
    int layer;
    RowSet rows;            // row i attends positions 0 .. positions[i] of its sequence
    int heads, rank;        // rank = row width of the pages (padded kv_rank)
    float scale;
    const void *q_lat;      // [n][heads * rank], operand type
    void *o_lat;            // [n][heads * rank], operand type
};
// One block per (row, up to four heads), true 32-bit arithmetic.
int launch_latent_attn_simt(juno_ctx *c, int dt, const LatentAttnArgs &a, cudaStream_t st);


// BF16, few rows over long caches (decode steps, short portions): the splits of a row's context run in parallel on the tensor
// cores, all heads of a group sharing every page that is read; part_o [n][heads][n_splits][rank], part_ml [n][heads][n_splits][2].
struct LatentSplitArgs {
    const juno_kvpool *pool;
    int layer;
    RowSet rows;
    int heads, rank, n_splits;
    float scale;
    const void *q_lat;
    float *part_o, *part_ml;
};
constexpr int kLatentSplitMaxRank = 1024;
int latent_pick_splits(const juno_ctx *c, int n, int heads, int rank, int len_bound);
size_t latent_part_floats(const juno_ctx *c, int n, int heads, int rank);  // enough for any split count latent_pick_splits returns
int launch_latent_attn_split(juno_ctx *c, const LatentSplitArgs &a, cudaStream_t st);
// Merges the splits and applies the value projection and the head gate: out[h] = W_uv[h] o_lat[h] * sigmoid(gate[h]); without
// w_uv the merged o_lat itself ([n][heads * rank]).
struct LatentMergeArgs {
    int n, heads, rank, vdim, n_splits;  // rank, vdim padded
    const float *part_o, *part_ml;
    const void *w_uv;    // [heads * vdim][rank] BF16, or null
    const float *gate;   // [n][ld_gate]
    int ld_gate;
    void *out;           // [n][heads * vdim] BF16
};
int launch_latent_merge(juno_ctx *c, const LatentMergeArgs &a, cudaStream_t st);

// out[j][rank] = the latent of position j of the sequence in `slot_of` (device, one word), j < len
int launch_latent_gather(juno_ctx *c, const juno_kvpool *pool, int layer, const int32_t *slot_of, int len, void *out, cudaStream_t st);

}  // namespace juno
