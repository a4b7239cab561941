// The decode step of a layer stack on the fused products (BF16, one to eight sequences): per layer
//   1  residual + norm + convolution -> gate | W_dq W_dkv W_g      5  merge of the splits + W_uv + head gate
//   2  latent norms, cache append    -> W_uq                       6  W_o, times the gate
//   3  per head W_uk^T q                                           7  residual + norm -> gate | W_up, squared ReLU
//   4  attention over the splits of the context                    8  W_down, times the gate
// The sublayer results travel un-normed (z); the product that follows norms them, adds them to the residual row and stores the
// sum once, so a layer has no launch that is not a product or attention.
#include <algorithm>

#include "gemv_rows.cuh"
#include "stack.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

bool stack_fused_ok(const juno_ctx *c, const StackNet *net, const RowSet &rows) {
    if (net->dt != DT_BF16 || rows.one_seq || rows.n > kGvMaxSeqs || net->spec.wp() > kGvMaxWidth) return false;
    int cols = net->ldact;
    for (const StackLayerSpec &L : net->spec.layers) {
        const LatentMixerSpec &m = L.mix;
        if (m.rp() > 1024) return false;
        cols = std::max(cols, std::max(m.qp(), m.heads * std::max(m.dp(), m.vp())));
    }
    // operands that need more than two passes over the weights: one pass on the row products is faster
    return 2 * gemv_rows_chunk(c, cols, 1, rows.n) >= rows.n && 2 * gemv_rows_chunk(c, net->spec.wp(), 2, rows.n) >= rows.n;
}

static GvSeg seg(const StackMat &w, int epi, void *out, int ldo) {
    GvSeg s;
    s.w = static_cast<const bf16 *>(w.w);
    s.rows = w.rows;
    s.epi = epi;
    s.out = out;
    s.ldo = ldo;
    return s;
}

// operand = norm of the residual row, the pending sublayer result added first
static GvArgs from_residual(StackNet *net, int n, float g_next) {
    GvArgs a;
    a.n = n;
    a.K = net->spec.wp();
    a.prologue = GVP_RESIDUAL;
    a.width = net->spec.width;
    a.eps = net->spec.eps;
    a.g_next = g_next;
    a.x = net->last_x ? net->x2 : net->x;
    if (net->pending) {
        a.z = net->dec_z;
        a.g_z = net->pending_g;
        net->last_x ^= 1;
        a.x_store = net->last_x ? net->x2 : net->x;
        net->pending = false;
    }
    return a;
}
static GvArgs from_rows(int n, const void *in, int ld, int cols, int K) {
    GvArgs a;
    a.n = n;
    a.K = K;
    a.in = static_cast<const bf16 *>(in);
    a.ld_in = ld;
    a.in_cols = cols;
    return a;
}

int stack_enqueue_decode(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    const int n = rows.n, wp = s.wp(), n_layers = (int)s.layers.size();
    net->last_x = 0;
    net->pending = false;
    JUNO_TRY(launch_embed_norm(c, net->dt, net->embed.w, net->embed.cols, s.width, s.vocab, net->embed_norm, s.eps, rows, net->x, wp, st));
    auto sublayer_out = [&](const void *in, int cols, const StackMat &w, float g) {
        GvArgs a = from_rows(n, in, cols, cols, cols);
        a.nseg = 1;
        a.seg[0] = seg(w, GVE_MUL, net->dec_z, wp);
        a.seg[0].aux = net->dec_gate;
        a.seg[0].ldaux = wp;
        net->pending = true;
        net->pending_g = g;
        return launch_gemv_rows(c, a, st);
    };
    for (int l = 0; l < n_layers; l++) {
        const StackLayerWeights &L = net->layers[s.weights(l)];
        const LatentMixerSpec &m = s.layers[l].mix;
        const int H = m.heads, rp = m.rp(), dp = m.dp(), vp = m.vp();
        {
            GvArgs a = from_residual(net, n, L.norm1);
            a.conv_w = static_cast<const bf16 *>(L.conv);
            a.taps = s.taps;
            if (pool->state) {
                a.state = pool->state + (size_t)l * pool->state_ring * pool->state_width;
                a.slot_stride = (size_t)pool->n_layers * pool->state_ring * pool->state_width;
                a.ring_mask = pool->state_ring - 1;
            }
            a.positions = rows.positions;
            a.slots = rows.slots;
            a.nseg = 2;
            a.seg[0] = seg(L.rg1, GVE_SIGMOID, net->dec_gate, wp);
            a.seg[0].bias = L.rg1_b;
            a.seg[1] = seg(L.down, GVE_F32, net->u, net->ldu);
            a.seg[1].operand = 1;
            JUNO_TRY(launch_gemv_rows(c, a, st));
        }
        {
            GvArgs a;
            a.n = n;
            a.K = m.qp();
            a.prologue = GVP_LATENT;
            a.eps = s.eps;
            a.u = net->u;
            a.ldu = net->ldu;
            a.q_rank = m.q_rank;
            a.kv_col = m.kv_col();
            a.kv_rank = m.kv_rank;
            a.wq = L.dq_norm;
            a.wkv = L.dkv_norm;
            a.plane = reinterpret_cast<bf16 *>(static_cast<uint8_t *>(pool->k) + pool->row_off[l] * 2);
            a.page_width = pool->row_width[l];
            a.table = pool->d_table;
            a.max_pages = pool->max_pages_per_seq;
            a.positions = rows.positions;
            a.slots = rows.slots;
            a.nseg = 1;
            a.seg[0] = seg(L.uq, GVE_OP, net->q, H * dp);
            JUNO_TRY(launch_gemv_rows(c, a, st));
        }
        {
            GvArgs a = from_rows(n, net->q, H * dp, H * dp, dp);
            a.group_rows = rp;
            a.nseg = 1;
            a.seg[0] = seg(L.ukt, GVE_OP, net->qlat, H * rp);
            JUNO_TRY(launch_gemv_rows(c, a, st));
        }
        const size_t ml = (size_t)n * H * n_splits * rp;
        JUNO_REQUIRE(ml + (size_t)n * H * n_splits * 2 <= net->part_floats, "%d context splits of %d rows exceed the buffer", n_splits, n);
        LatentSplitArgs sp{pool, l, rows, H, rp, n_splits, m.scale, net->qlat, net->part_o, net->part_o + ml};
        JUNO_TRY(launch_latent_attn_split(c, sp, st));
        LatentMergeArgs mg{n, H, rp, vp, n_splits, net->part_o, net->part_o + ml, static_cast<const bf16 *>(L.ukv.w) + (size_t)H * dp * rp,
                           net->u + m.gate_col(), net->ldu, net->att};
        JUNO_TRY(launch_latent_merge(c, mg, st));
        JUNO_TRY(sublayer_out(net->att, H * vp, L.o, L.norm1b));
        if (s.layers[l].ff == 0) continue;
        {
            GvArgs a = from_residual(net, n, L.norm2);
            a.nseg = 2;
            a.seg[0] = seg(L.rg2, GVE_SIGMOID, net->dec_gate, wp);
            a.seg[0].bias = L.rg2_b;
            a.seg[1] = seg(L.up, GVE_RELU2, net->act, L.mdown.cols);
            JUNO_TRY(launch_gemv_rows(c, a, st));
        }
        JUNO_TRY(sublayer_out(net->act, L.mdown.cols, L.mdown, L.norm2b));
    }
    return JUNO_OK;
}

int stack_enqueue_decode_logits(juno_ctx *c, StackNet *net, int n, float *logits, cudaStream_t st) {
    GvArgs a = from_residual(net, n, net->final_norm);
    a.nseg = 1;
    a.seg[0] = seg(net->head, GVE_F32, logits, net->spec.vocab);
    a.seg[0].n_store = net->spec.vocab;
    return launch_gemv_rows(c, a, st);
}

}  // namespace juno
