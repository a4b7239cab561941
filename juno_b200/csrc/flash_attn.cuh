// BF16 causal flash attention of many rows of one sequence (a prompt or a portion of one).
#pragma once
#include "attn_span.cuh"
#include "rowops.cuh"

namespace juno {

// Row r is position pos0 + r; query head h uses key/value head h / (heads / kv_heads).  Keys and values lie side by side in
// rows, keys of all key/value heads (kv_heads * dim), then values (kv_heads * vdim): rows of a plain buffer (kv, ldkv), or,
// when `pool` is set, the sequence's own pages of that layer.  out = softmax(q . k * scale - slope * distance) v; the span,
// the slopes and the sinks belong to the paged form.
struct FlashArgs {
    int n = 0, pos0 = 0, heads = 0, dim = 0, vdim = 0;  // padded sizes
    float scale = 1.f;
    const void *q = nullptr;      // [n][heads * dim]
    const void *kv = nullptr;
    int ldkv = 0;
    const float *gate = nullptr;  // [n][ld_gate], one per head, sigmoid taken here (null: none)
    int ld_gate = 0;
    void *out = nullptr;          // [n][heads * vdim]
    int kv_heads = 0;             // 0: one per query head
    const juno_kvpool *pool = nullptr;
    int layer = 0;
    const int32_t *slot = nullptr;   // device, one word
    KeySpan span;
    const float *slopes = nullptr;   // [heads], natural units (null: none)
    const float *sinks = nullptr;    // [heads] scores that enter the denominator alone (null: none)
};
constexpr int kFlashMaxDim = 256;
int launch_flash_prefill(juno_ctx *c, const FlashArgs &a, cudaStream_t st);

}  // namespace juno
