// Hyper-connections: the residual stream is `streams` parallel FP32 rows per position, x [n][streams][ldx].  A sublayer reads
// u = sum_s in[s] x_s; with its result z every stream becomes x_t <- sum_s mix[s][t] x_s + out[t] z, all from the old streams.
// One stream with in = mix = out = 1 is the plain residual sum.
#pragma once
#include "rowops.cuh"

namespace juno {

constexpr int kMaxStreams = 16;

// Every stream of row r = embed[token].
int launch_stream_embed(juno_ctx *c, int dt, const void *embed, int ld_embed, int width, int vocab, int streams, const RowSet &rows, float *x, int ldx,
                        cudaStream_t st);

// From one sublayer to the next: the streams take the result z of the one that ended (null: none), then
// h = rms(sum_s in[s] x_s) * w as operand of the one that follows (h null: the update alone).
struct StreamStepArgs {
    float *x = nullptr;
    int streams = 1, ldx = 0, width = 0, n = 0;
    const void *z = nullptr;
    int ldz = 0;
    const float *mix = nullptr, *out = nullptr;  // [from][to], [to]
    const float *in = nullptr, *w = nullptr;     // [streams], [ldx]
    float eps = 0.f;
    void *h = nullptr;
    int ldh = 0;
};
int launch_stream_step(juno_ctx *c, int dt, const StreamStepArgs &a, cudaStream_t st);

// out[i] = rms(sum_s x_s[row_idx[i]]) * w as operand (row_idx null: row i); w null: the sum itself, FP32 whatever dt.
int launch_stream_gather(juno_ctx *c, int dt, const float *x, int streams, int ldx, int width, const int32_t *row_idx, int n, const float *w, float eps,
                         void *out, int ldo, cudaStream_t st);

}  // namespace juno
