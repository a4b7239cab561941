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

}  // namespace juno
