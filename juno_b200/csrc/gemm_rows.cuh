// Matrix products of layer stacks with dense weights: out[m][n] = epilogue(sum_k a[m][k] * w[n][k]), m = positions.
#pragma once
#include "rowops.cuh"

namespace juno {

enum GemmEpi {
    GE_F32 = 0,      // acc (+ bias[n] when there is one), FP32
    GE_OP,           // operand type
    GE_SIGMOID,      // sigmoid(acc + bias[n]), operand type
    GE_RELU2,        // max(acc, 0)^2, operand type
    GE_MUL,          // acc * aux[m][n] (operand type), operand type
    GE_GROUP_GATE,   // acc * sigmoid(gate[m][group]) (FP32), operand type
    GE_GEGLU,        // columns in tiles of 8 gates and the 8 values they gate: gelu_tanh(gate) * value, operand type, half as many columns
};

// `groups` > 1: a block-diagonal product (one block per attention head): group z multiplies columns a_step*z.. of `a` with rows
// w_step*z.. of `w` into columns o_step*z.. of `out`; N and K are a group's.
struct GemmArgs {
    const void *a = nullptr;
    int lda = 0;
    const void *w = nullptr;
    int ldw = 0;
    int M = 0, N = 0, K = 0;
    void *out = nullptr;
    int ldo = 0;
    int epi = GE_OP;
    const float *bias = nullptr;
    const void *aux = nullptr;
    int ldaux = 0;
    int groups = 1, a_step = 0, w_step = 0, o_step = 0;
    int w_rows = 0;  // rows of `w` in memory (0: N, or w_step * groups)
};
int launch_gemm_rows_tc(juno_ctx *c, const GemmArgs &a, unsigned *err, cudaStream_t st);  // BF16, tcgen05
int launch_gemm_rows(juno_ctx *c, int dt, const GemmArgs &a, unsigned *err, cudaStream_t st);

}  // namespace juno
