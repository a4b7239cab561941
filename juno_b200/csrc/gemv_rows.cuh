// Fused BF16 matrix-vector products of a decode step (one to eight sequences): the operand is built from FP32 rows inside the
// consuming product - residual sum or residual streams, norms, short convolution, latent norm - and the weights stream past it once.
#pragma once
#include "streams.cuh"

namespace juno {

constexpr int kGvMaxSeqs = 8;
constexpr int kGvMaxWidth = 8192;  // widest residual row the fused residual prologue takes

enum GvPrologue { GVP_COPY = 0, GVP_RESIDUAL, GVP_LATENT, GVP_STREAMS };
enum GvEpi {
    GVE_F32 = 0,  // v (+ bias when there is one), FP32
    GVE_OP,
    GVE_SIGMOID,  // sigmoid(v + bias), FP32
    GVE_RELU2,    // BF16
    GVE_MUL,      // v * aux, FP32
    GVE_GEGLU,    // rows in tiles of 8 gates and the 8 values they gate: gelu_tanh(gate) * value, BF16, half as many columns
};

struct GvSeg {
    const __nv_bfloat16 *w = nullptr;  // [rows][ldw], ldw = the launch's K padded to 16
    int rows = 0;                      // multiple of 16
    int n_store = 0;                   // rows that are stored (0: all)
    int operand = 0;                   // GVP_RESIDUAL: 0 = normed row, 1 = the same after the convolution
    int epi = GVE_F32;
    void *out = nullptr;
    int ldo = 0;
    const float *bias = nullptr;
    const float *aux = nullptr;
    int ldaux = 0;
};

struct GvArgs {
    int n = 0, K = 0;  // sequences; columns of every segment's matrix (multiple of 16)
    int nseg = 0;
    GvSeg seg[3];
    int prologue = GVP_COPY;
    bool early = true;  // may start while the kernel before it runs (programmatic dependent launch)
    // GVP_COPY: BF16 rows; group_rows > 0: rows group_rows * g .. of the matrix meet columns K * g .. of the operand
    const __nv_bfloat16 *in = nullptr;
    int ld_in = 0, in_cols = 0, group_rows = 0;
    // GVP_RESIDUAL: x += rms(z) * g_z (z null: nothing pending), operand = rms(x) * g_next; the sum goes to x_store
    const float *x = nullptr, *z = nullptr;
    float *x_store = nullptr;
    int width = 0;
    float g_z = 0, g_next = 0, eps = 0;
    const __nv_bfloat16 *conv_w = nullptr;  // [taps][K]; null: no convolution
    int taps = 1;
    float *state = nullptr;                 // this layer's state rows of slot 0
    size_t slot_stride = 0;
    int ring_mask = 0;
    // GVP_STREAMS (see streams.cuh): x [n][streams][K]; the pending result z [n][K] is mixed in with hc_mix and hc_out,
    // operand = rms(sum_s hc_in[s] x_s) * norm_w; the new streams go to x_store
    int streams = 0;
    const float *hc_mix = nullptr, *hc_out = nullptr, *hc_in = nullptr, *norm_w = nullptr;
    // GVP_LATENT: u [n][ldu]: operand = rms(u[0..q_rank)) * wq; u[kv_col..+kv_rank) is normed with wkv and appended to the pages
    const float *u = nullptr, *wq = nullptr, *wkv = nullptr;
    int ldu = 0, q_rank = 0, kv_col = 0, kv_rank = 0, page_width = 0, max_pages = 0;
    __nv_bfloat16 *plane = nullptr;
    const int32_t *table = nullptr;
    const int32_t *positions = nullptr, *slots = nullptr;
};
// Most sequences one launch takes (shared memory), at least 1 when the product fits at all, else 0.
int gemv_rows_chunk(const juno_ctx *c, int cols, int operands, int n);
int launch_gemv_rows(juno_ctx *c, const GvArgs &a, cudaStream_t st);

}  // namespace juno
