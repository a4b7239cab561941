// Attention of grouped heads over row pages: a page row of a layer holds the keys of all key/value heads, then the values
// (kv_heads * (dim + vdim) numbers, padded sizes); query head h uses key/value head h / (heads / kv_heads).  What designs
// differ in are parameters: per-head norms, a rotation of the first dimensions, a temperature that grows with the position,
// the span of positions that are seen, a bias per distance, and sinks (scores that enter the softmax denominator alone).
// All of it is FP32 arithmetic; queries, keys and values are rounded to the operand type once, where they are stored.
#pragma once
#include "flash_attn.cuh"

namespace juno {

struct GroupedAttnArgs {
    const juno_kvpool *pool = nullptr;
    int layer = 0;
    RowSet rows;
    int heads = 0, kv_heads = 0, dim = 0, dp = 0, vp = 0;  // dim: real query/key size (norms divide by it); dp, vp: padded
    float scale = 1.f;
    KeySpan span;
    const float *slopes = nullptr;  // [heads] score -= slope * distance (null: none)
    const float *sinks = nullptr;   // [heads] (null: none)
    const float *u = nullptr;       // [n][ldu] projections: queries (heads * dp), keys (kv_heads * dp), values (kv_heads * vp)
    int ldu = 0;
    const float *q_norm = nullptr, *k_norm = nullptr;  // [dp] weights of per-head RMS norms (null: none)
    float eps = 0.f;
    const float2 *rot = nullptr;    // [position][rot_dims / 2] (cos, sin): dimension i turns with i + rot_dims / 2 (null: none)
    int rot_dims = 0;
    float temp_coef = 0.f;          // q *= 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1); temp_every 0: none
    int temp_every = 0;
    void *q = nullptr;              // [n][heads * dp], operand type
    void *out = nullptr;            // [n][heads * vp], operand type
};
// u -> q, and keys and values appended to the pages.
int launch_grouped_prep(juno_ctx *c, int dt, const GroupedAttnArgs &a, cudaStream_t st);
// One block per (head, row), true 32-bit arithmetic: FP32 models, and heads wider than the tensor-core kernels take.
constexpr int kGroupedMaxVdim = 2048;
int launch_grouped_simt(juno_ctx *c, int dt, const GroupedAttnArgs &a, cudaStream_t st);

// BF16, few rows (decode steps, short portions): the splits of a row's span run in parallel, the query heads of a key/value
// head share every page that is read, and the last split to finish merges them.  fused: q, k and v come straight from u (norms,
// rotation, temperature, append inside; every row is a sequence of its own); else launch_grouped_prep has run.
constexpr int kGroupedMaxDim = 256, kGroupedMaxSplits = 64;
int grouped_pick_splits(const juno_ctx *c, int n, int heads, int kv_heads, int dim, int keys);
size_t grouped_part_floats(const juno_ctx *c, int vp);   // enough for any split count grouped_pick_splits returns
size_t grouped_counters(const juno_ctx *c);              // words, zero between launches
int launch_grouped_split(juno_ctx *c, const GroupedAttnArgs &a, int n_splits, bool fused, float *part, size_t part_floats, unsigned *counters, cudaStream_t st);
// (cos, sin) of position * base^(-2 i / dims) for every position below n
int launch_rotation_table(juno_ctx *c, int n, int dims, double base, float2 *table, cudaStream_t st);

}  // namespace juno
