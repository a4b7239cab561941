// The model object behind juno_model_*: one step function, cache and greedy loop for every model family.
#pragma once
#include <map>
#include <string>
#include <vector>

#include "attn.cuh"
#include "common.cuh"
#include "gemv.cuh"

namespace juno {
typedef struct ncclComm *NcclComm;
struct StackNet;
}  // namespace juno

// ───────────────────────────── model object ───────────────────────────────────────────────
struct JunoLayer {
    juno_qmat *w[12] = {nullptr};  // indexed by tensor kind (ATTN_Q .. FFN_DOWN); gate and up share w[FFN_GATE]
    std::vector<uint8_t> gate_host, up_host;  // row slices waiting for their partner
    int gate_type = -1, up_type = -1;
    float *attn_norm = nullptr, *ffn_norm = nullptr;
    float *bqkv = nullptr;  // optional attn_{q,k,v}.bias of this rank, laid out like a row of the q|k|v buffer
    int bias_seen = 0;      // bit per bias kind received
};

struct JunoGraph {
    cudaGraphExec_t exec = nullptr;
    int launches = 0;
    int seen = 0;
};

struct juno_model {
    uint32_t magic;
    juno_ctx *ctx;
    juno_model_cfg cfg;
    int hd, world, rank;
    int heads_loc, kv_loc, inter_loc, vocab_loc;  // this rank's share
    int qkv_ld;
    bool finalized = false;
    bool vocab_sharded = false;
    std::vector<JunoLayer> layers;
    juno_qmat *tok_embd = nullptr, *output = nullptr;
    bool output_is_embd = false, output_slice_of_embd = false;
    float *output_norm = nullptr;
    juno_kvpool *pool = nullptr;
    juno::NcclComm comm = nullptr;
    // activations
    float *x[2] = {nullptr, nullptr}, *qkv = nullptr, *att = nullptr, *proj = nullptr, *proj2 = nullptr;
    float *hdn = nullptr, *xsc = nullptr;  // batched path: silu(gate)*up rows; per-row factors of the three FP16 images
    uint8_t *img_h_tc = nullptr;            // batched path: the hidden-size activation again, chunk-major for the tcgen05 kernel
    unsigned *tc_err = nullptr;             // device word: a wait inside the tcgen05 kernel gave up
    bool tc_used = false;                   // the batched path ran since the word was last read
    uint8_t *img_h = nullptr, *img_att = nullptr, *img_i = nullptr;  // staged activations (K = hidden, local heads, local FFN)
    float *logits_loc = nullptr, *logits_gather = nullptr, *logits_full = nullptr;
    float *attn_scratch = nullptr;
    size_t attn_scratch_floats = 0;
    float2 *rope_cs = nullptr;
    int32_t *d_step = nullptr;  // tokens | positions | slots | seq_lens, max_batch each
    int32_t *d_argmax = nullptr, *d_pidx = nullptr, *d_out_ids = nullptr, *d_step_counter = nullptr;
    float *d_pval = nullptr;
    int out_ids_cap = 0;
    int32_t *h_step = nullptr;  // pinned mirror of d_step
    int last_n = 0, last_x = 0;
    double step_kv_bytes = 0;  // K+V bytes one layer's attention reads in the current step
    std::map<uint64_t, JunoGraph> graphs;
    bool use_graphs = true, mix_formats = true;  // JUNO_NO_GRAPH / JUNO_NO_MIXED
    // tensor parallelism without collective calls on the 1..8 sequence path: per-rank exchange buffer (flags + inbox
    // slots per row-parallel product), mapped into every peer (CUDA IPC), see enqueue_layers_q
    bool tp_push = false;
    uint8_t *tp_buf = nullptr;           // this rank's buffer
    uint8_t *tp_peer[8] = {nullptr};     // every rank's buffer as seen from here (tp_peer[rank] == tp_buf)
    size_t tp_inbox_off = 0, tp_pair_off = 0;
    int tp_bq = 0;                       // sequences an inbox slot holds
    unsigned *tp_failed = nullptr;       // device word: a wait for another rank ran out during this step
    float *tp_red = nullptr;             // [2 * n_layers][tp_bq][hidden] (value, step) pairs: the ranks' partials added by the first CTAs
    bool tp_reduce = false;              // consumers poll tp_red instead of every rank's inbox (four ranks and more)
    bool comm_failed = false;            // a collective timed out or NCCL reported an asynchronous error: no further steps
    unsigned *tp_epoch = nullptr;        // step number, incremented on the device at the start of every step
    // a layer stack with dense weights (csrc/stack.cuh) in place of the quantised LLaMA layers above
    juno::StackNet *stack = nullptr;
    std::string architecture = "llama";
    int step_cap = 0;    // rows the step buffers hold (max_batch; for a stack also the longest portion of a prompt)
    int logit_cap = 0;   // rows logits_loc holds
    int batched_from = 9;  // smallest batch on the FP16 one-pass kernels (JUNO_GEMM_MIN_BATCH, read when the model is created)
};

namespace juno {
// A finalized model around a loaded layer stack; takes ownership of `net` (also on failure).
int model_from_stack(juno_ctx *c, StackNet *net, const char *architecture, const juno_open_opts &opts, juno_model **out);
}  // namespace juno
