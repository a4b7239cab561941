// Layer stacks with dense (BF16 or FP32) weights: the description a model design is turned into, its weights in device
// memory, and the passes that run it.  A design (csrc/vosotar.cu, csrc/desilorn.cu) parses its configuration into a StackSpec and loads its
// tensors; everything below is shared between designs that use the same mechanisms.
#pragma once
#include <string>
#include <vector>

#include "gemm_rows.cuh"
#include "grouped_attn.cuh"
#include "latent_attn.cuh"
#include "rowops.cuh"
#include "safetensors.cuh"
#include "streams.cuh"

namespace juno {

// Latent attention without positions: queries through a normed latent of q_rank, keys and values through a normed latent of
// kv_rank that alone is cached; one sigmoid gate per head on the output.
struct LatentMixerSpec {
    int heads = 0, dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    float scale = 0.f;
    // padded sizes of the device layouts (multiples of 16: tensor-core steps and 32-byte rows)
    int qp() const { return pad16(q_rank); }
    int rp() const { return pad16(kv_rank); }
    int dp() const { return pad16(dim); }
    int vp() const { return pad16(vdim); }
    int kv_col() const { return qp(); }
    int gate_col() const { return qp() + rp(); }
    int down_rows() const { return qp() + rp() + pad16(heads); }
};

// Attention of grouped heads with biased projections (see grouped_attn.cuh); whatever is not set does not happen.
enum SinkKind { SINK_NONE = 0, SINK_LEARNED, SINK_ZERO };
struct GroupedMixerSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 0.f;
    KeySpan span;
    bool qk_norm = false, distance_bias = false;
    int sink = SINK_NONE;
    int rot_dims = 0;
    double rot_base = 0.;
    int temp_every = 0;
    float temp_coef = 0.f;
    int dp() const { return pad16(dim); }
    int vp() const { return pad16(vdim); }
    int qkv_rows() const { return (heads + kv_heads) * dp() + kv_heads * vp(); }
    int page_width() const { return kv_heads * (dp() + vp()); }
};

enum MixerKind { MIX_LATENT = 0, MIX_GROUPED };
enum FfKind { FF_RELU2 = 0 /* down(relu(up h)^2) */, FF_GEGLU /* down(gelu_tanh(gate h) * up h) */ };

struct StackLayerSpec {
    int mixer = MIX_LATENT;
    LatentMixerSpec mix;
    GroupedMixerSpec grouped;
    int ff = 0;            // 0: no feed-forward
    int ff_kind = FF_RELU2;
    int weights_of = -1;   // >= 0: this layer runs with that layer's weights
    int source = 0;        // index of the layer in the configuration, which its tensors are named after
    int page_width() const { return mixer == MIX_GROUPED ? grouped.page_width() : mix.rp(); }
};

struct StackSpec {
    int width = 0, vocab = 0, taps = 1;
    float eps = 0.f;
    // 0: one residual row; a sublayer's result is gated element by element, normed and added, its input is normed by one
    // number and convolved.  > 0: hyper-connections of that many residual streams, norms with a weight per column.
    int streams = 0;
    std::vector<StackLayerSpec> layers;  // in the order they run
    int wp() const { return pad16(width); }
    int weights(int layer) const {
        while (layers[layer].weights_of >= 0) layer = layers[layer].weights_of;
        return layer;
    }
};

struct StackMat {
    void *w = nullptr;
    int rows = 0, cols = 0;  // padded; cols is also the row pitch
};

struct HyperConnection {
    float *in = nullptr, *out = nullptr, *mix = nullptr;  // see streams.cuh
};

struct StackLayerWeights {
    float norm1 = 0, norm1b = 0, norm2 = 0, norm2b = 0;  // norms with one number
    StackMat down;    // W_dq | W_dkv | W_g, one product on the convolved input
    StackMat uq, ukt, ukv, o;  // ukt: per head W_uk transposed [rank][dim]; ukv: W_uk over W_uv
    StackMat rg1, rg2, up, mdown;
    float *dq_norm = nullptr, *dkv_norm = nullptr, *rg1_b = nullptr, *rg2_b = nullptr;
    void *conv = nullptr;  // [taps][wp]
    // grouped attention: W_q | W_k | W_v by padded heads; gated feed-forward: tiles of 8 rows of W_gate and 8 of W_up
    StackMat qkv, gu;
    float *qkv_b = nullptr, *q_norm = nullptr, *k_norm = nullptr, *sinks = nullptr, *slopes = nullptr;
    float *norm1_w = nullptr, *norm2_w = nullptr;  // norms with a weight per column
    HyperConnection hc1, hc2;
};

struct StackNet {
    StackSpec spec;
    int dt = DT_BF16;
    StackMat embed, head;
    float embed_norm = 0, final_norm = 0;
    float *final_w = nullptr, *ones = nullptr;  // streams: weights of the last norm; [kMaxStreams] ones
    std::vector<StackLayerWeights> layers;  // entries of layers with weights_of stay empty
    std::vector<void *> owned;              // every device allocation
    // buffers of a pass
    int cap = 0, lat_cap = 0, logit_cap = 0;
    float *x = nullptr, *u = nullptr, *row_scale = nullptr;
    float *x2 = nullptr;
    void *h = nullptr, *hc = nullptr, *gate = nullptr, *z = nullptr, *cq = nullptr, *q = nullptr, *qlat = nullptr, *olat = nullptr,
         *att = nullptr, *act = nullptr, *fin = nullptr;
    int ldu = 0, ldcq = 0, ldq = 0, ldlat = 0, ldatt = 0, ldact = 0;
    float *part_o = nullptr;  // partial results of the attention's context splits
    size_t part_floats = 0;
    unsigned *counters = nullptr;          // of the grouped attention's splits, zero between launches
    std::vector<const float2 *> rot;       // per layer: rotation table (null: none)
    float *hidden = nullptr;               // sum of the streams, when asked for
    size_t hidden_bytes = 0;
    void *ctx_lat = nullptr, *ctx_kv = nullptr;   // a prompt pass: the sequence's latents, and keys and values expanded from them
    size_t ctx_lat_bytes = 0, ctx_kv_bytes = 0;
    int32_t *row_idx = nullptr;  // device list of rows whose logits are wanted
    double weight_bytes = 0;     // bytes a one-token step reads
    // fused decode step: residual rows x / x2 in turn (last_x: which holds the newest), sublayer result not yet added to them
    float *dec_gate = nullptr, *dec_z = nullptr;
    int last_x = 0;
    bool pending = false;
    float pending_g = 0.f;
    const HyperConnection *pending_hc = nullptr;
};

// ── loading ──
// Host image of a padded matrix, filled block by block and uploaded once.
struct HostMat {
    int dt, rows, cols;
    std::vector<uint8_t> data;
    HostMat(int dtype, int r, int c) : dt(dtype), rows(r), cols(c), data((size_t)r * c * dt_bytes(dtype), 0) {}
    // dst[row + i][col + j] = src[r0 + i][c0 + j]
    void put(const juno_safetensors *f, const StTensor &t, int64_t r0, int64_t c0, int nr, int nc, int row, int col);
    // dst[row + j][col + i] = src[r0 + i][c0 + j]
    void put_transposed(const juno_safetensors *f, const StTensor &t, int64_t r0, int64_t c0, int nr, int nc, int row, int col);
};
int stack_upload(juno_ctx *c, StackNet *net, const HostMat &m, StackMat *out);
int stack_upload_f32(juno_ctx *c, StackNet *net, const std::vector<float> &v, float **out);
float st_value(const juno_safetensors *f, const StTensor &t, int64_t i);

// ── running ──
GroupedAttnArgs grouped_attn_args(const StackNet *net, const StackLayerWeights &L, const juno_kvpool *pool, int layer, const RowSet &rows);
int grouped_layer_splits(const juno_ctx *c, const GroupedMixerSpec &m, int n, int n_splits);  // of a step with n_splits at most
int stack_alloc(juno_ctx *c, StackNet *net, int max_batch, int max_rows, int logit_rows, int max_ctx);
void stack_free(StackNet *net);
// All layers for `rows`; `len_bound` bounds positions + 1 over the rows.  The residual stream ends in the net's x.
int stack_enqueue_layers(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, int len_bound, cudaStream_t st);
// logits[i] = head . norm(x[row_idx[i]]) (row_idx null: row i), n rows
int stack_enqueue_logits(juno_ctx *c, StackNet *net, const int32_t *row_idx, int n, float *logits, cudaStream_t st);
// The same for a decode step of few sequences, on fused products (stack_decode.cu).
bool stack_fused_ok(const juno_ctx *c, const StackNet *net, const RowSet &rows);
int stack_decode_hand_overs(const StackNet *net, int n);
int stack_enqueue_decode(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, cudaStream_t st);
int stack_enqueue_decode_logits(juno_ctx *c, StackNet *net, int n, float *logits, cudaStream_t st);
// One step of n sequences, logits included, on whichever of the two fits.
int stack_enqueue_step(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, int len_bound, float *logits, cudaStream_t st);
// A captured step has run: where its residual stream ended.
void stack_step_done(const juno_ctx *c, StackNet *net, int n);
// Residual stream of the first n rows of the last pass (the sum, when there are several streams), rows of wp() floats.
int stack_residual(juno_ctx *c, StackNet *net, int n, const float **out, cudaStream_t st);
int stack_pick_splits(const juno_ctx *c, const StackNet *net, int n, int len_bound);

// ── designs ──
struct Json;
int vosotar_spec(const Json &cfg, StackSpec *spec);
int vosotar_load(juno_ctx *c, const juno_safetensors *f, const StackSpec &spec, int dt, StackNet **out);
int desilorn_spec(const Json &cfg, StackSpec *spec);
int desilorn_load(juno_ctx *c, const juno_safetensors *f, const StackSpec &spec, int dt, StackNet **out);

}  // namespace juno
