// The decode step of a layer stack on the fused products (BF16, one to eight sequences).  Latent attention, per layer
//   1  residual + norm + convolution -> gate | W_dq W_dkv W_g      5  merge of the splits + W_uv + head gate
//   2  latent norms, cache append    -> W_uq                       6  W_o, times the gate
//   3  per head W_uk^T q                                           7  residual + norm -> gate | W_up, squared ReLU
//   4  attention over the splits of the context                    8  W_down, times the gate
// grouped attention over residual streams
//   1  streams + norm -> W_q W_k W_v, biases                       4  streams + norm -> W_gate W_up, GELU(gate) * up
//   2  head norms, rotation, append, attention, merge              5  W_down
//   3  W_o
// The sublayer results travel as they are (z); the product that follows takes them into the residual rows and stores those
// once, so a layer has no launch that is not a product or attention.
#include <algorithm>

#include "gemv_rows.cuh"
#include "stack.cuh"

namespace juno {

using bf16 = __nv_bfloat16;

bool stack_fused_ok(const juno_ctx *c, const StackNet *net, const RowSet &rows) {
    if (net->dt != DT_BF16 || rows.one_seq || rows.n > kGvMaxSeqs || net->spec.wp() > kGvMaxWidth) return false;
    int cols = net->ldact;
    for (const StackLayerSpec &L : net->spec.layers) {
        if (L.mixer == MIX_GROUPED) {
            if (std::max(L.grouped.dp(), L.grouped.vp()) > kGroupedMaxDim) return false;
            cols = std::max(cols, L.grouped.heads * L.grouped.vp());
            continue;
        }
        const LatentMixerSpec &m = L.mix;
        if (m.rp() > 1024) return false;
        cols = std::max(cols, std::max(m.qp(), m.heads * std::max(m.dp(), m.vp())));
    }
    // operands that need more than two passes over the weights: one pass on the row products is faster
    const int images = net->spec.streams ? 1 : 2;
    return 2 * gemv_rows_chunk(c, cols, 1, rows.n) >= rows.n && 2 * gemv_rows_chunk(c, net->spec.wp(), images, rows.n) >= rows.n;
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

// Up to this many sequences every CTA of a product reads the streams itself; from there on that costs more than a launch that
// updates them and leaves the operand.
constexpr int kStreamsInProduct = 2;
static bool streams_in_product(const StackNet *net, int n) { return net->spec.streams > 0 && n <= kStreamsInProduct; }
int stack_decode_hand_overs(const StackNet *net, int n) {  // times the newest residual rows change between x and x2
    if (net->spec.streams && !streams_in_product(net, n)) return 0;
    int k = 0;
    for (const StackLayerSpec &L : net->spec.layers) k += L.ff ? 2 : 1;
    return k;
}

static GvArgs from_rows(int n, const void *in, int ld, int cols, int K);

// operand = norm of the residual, the pending sublayer result taken in first; what follows is a sublayer of `next`, or
// (null) the output
static int from_residual(juno_ctx *c, StackNet *net, int n, const StackLayerWeights *next, bool ff, GvArgs *out, cudaStream_t st) {
    const StackSpec &s = net->spec;
    const int wp = s.wp();
    GvArgs a;
    a.n = n;
    a.K = wp;
    a.width = s.width;
    a.eps = s.eps;
    a.x = net->last_x ? net->x2 : net->x;
    if (s.streams) {
        const float *in = next ? (ff ? next->hc2 : next->hc1).in : net->ones, *w = next ? (ff ? next->norm2_w : next->norm1_w) : net->final_w;
        if (!streams_in_product(net, n)) {
            StreamStepArgs t;
            t.x = net->x;
            t.streams = s.streams;
            t.ldx = wp;
            t.width = s.width;
            t.n = n;
            if (net->pending) {
                t.z = net->z;
                t.ldz = wp;
                t.mix = net->pending_hc->mix;
                t.out = net->pending_hc->out;
                net->pending = false;
            }
            t.in = in;
            t.w = w;
            t.eps = s.eps;
            t.h = net->h;
            t.ldh = wp;
            JUNO_TRY(launch_stream_step(c, net->dt, t, st));
            *out = from_rows(n, net->h, wp, wp, wp);
            return JUNO_OK;
        }
        a.prologue = GVP_STREAMS;
        a.streams = s.streams;
        a.hc_in = in;
        a.norm_w = w;
    } else {
        a.prologue = GVP_RESIDUAL;
        a.g_next = next ? (ff ? next->norm2 : next->norm1) : net->final_norm;
    }
    if (net->pending) {
        a.z = net->dec_z;
        if (s.streams) {
            a.hc_mix = net->pending_hc->mix;
            a.hc_out = net->pending_hc->out;
        } else {
            a.g_z = net->pending_g;
        }
        net->last_x ^= 1;
        a.x_store = net->last_x ? net->x2 : net->x;
        net->pending = false;
    }
    *out = a;
    return JUNO_OK;
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

// Latent attention, up to the heads' results in att; the mixer's gate goes to dec_gate.
static int latent_mixer(juno_ctx *c, StackNet *net, const juno_kvpool *pool, int l, const RowSet &rows, int n_splits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    const StackLayerWeights &L = net->layers[s.weights(l)];
    const LatentMixerSpec &m = s.layers[l].mix;
    const int n = rows.n, wp = s.wp(), H = m.heads, rp = m.rp(), dp = m.dp(), vp = m.vp();
    {
        GvArgs a;
        JUNO_TRY(from_residual(c, net, n, &L, false, &a, st));
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
    return launch_latent_merge(c, mg, st);
}

// Grouped attention: one product, one attention launch (norms, rotation, append and merge inside).
static int grouped_mixer(juno_ctx *c, StackNet *net, const juno_kvpool *pool, int l, const RowSet &rows, int n_splits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    const StackLayerWeights &L = net->layers[s.weights(l)];
    GvArgs a;
    JUNO_TRY(from_residual(c, net, rows.n, &L, false, &a, st));
    a.nseg = 1;
    a.seg[0] = seg(L.qkv, GVE_F32, net->u, L.qkv.rows);
    a.seg[0].bias = L.qkv_b;
    JUNO_TRY(launch_gemv_rows(c, a, st));
    const GroupedAttnArgs at = grouped_attn_args(net, L, pool, l, rows);
    return launch_grouped_split(c, at, grouped_layer_splits(c, s.layers[l].grouped, rows.n, n_splits), true, net->part_o, net->part_floats, net->counters, st);
}

int stack_enqueue_decode(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    const int n = rows.n, wp = s.wp(), n_layers = (int)s.layers.size();
    net->last_x = 0;
    net->pending = false;
    if (s.streams)
        JUNO_TRY(launch_stream_embed(c, net->dt, net->embed.w, net->embed.cols, s.width, s.vocab, s.streams, rows, net->x, wp, st));
    else
        JUNO_TRY(launch_embed_norm(c, net->dt, net->embed.w, net->embed.cols, s.width, s.vocab, net->embed_norm, s.eps, rows, net->x, wp, st));
    // the result of a sublayer stays pending: the next product takes it into the residual
    auto sublayer_out = [&](const void *in, const StackMat &w, float g, const HyperConnection &hc, bool early) {
        GvArgs a = from_rows(n, in, w.cols, w.cols, w.cols);
        a.early = early;
        a.nseg = 1;
        if (s.streams && !streams_in_product(net, n))
            a.seg[0] = seg(w, GVE_OP, net->z, wp);
        else
            a.seg[0] = seg(w, s.streams ? GVE_F32 : GVE_MUL, net->dec_z, wp);
        a.seg[0].aux = net->dec_gate;
        a.seg[0].ldaux = wp;
        net->pending = true;
        net->pending_g = g;
        net->pending_hc = &hc;
        return launch_gemv_rows(c, a, st);
    };
    for (int l = 0; l < n_layers; l++) {
        const StackLayerWeights &L = net->layers[s.weights(l)];
        const StackLayerSpec &spec = s.layers[l];
        JUNO_TRY(spec.mixer == MIX_GROUPED ? grouped_mixer(c, net, pool, l, rows, n_splits, st) : latent_mixer(c, net, pool, l, rows, n_splits, st));
        // started early, W_o's CTAs (each wants a whole SM) would wait among the small ones of the grouped attention, and the
        // product after it then ran at half its rate
        JUNO_TRY(sublayer_out(net->att, L.o, L.norm1b, L.hc1, spec.mixer != MIX_GROUPED));
        if (spec.ff == 0) continue;
        GvArgs a;
        JUNO_TRY(from_residual(c, net, n, &L, true, &a, st));
        if (!s.streams) {
            a.seg[a.nseg] = seg(L.rg2, GVE_SIGMOID, net->dec_gate, wp);
            a.seg[a.nseg++].bias = L.rg2_b;
        }
        a.seg[a.nseg++] = spec.ff_kind == FF_GEGLU ? seg(L.gu, GVE_GEGLU, net->act, L.mdown.cols) : seg(L.up, GVE_RELU2, net->act, L.mdown.cols);
        JUNO_TRY(launch_gemv_rows(c, a, st));
        JUNO_TRY(sublayer_out(net->act, L.mdown, L.norm2b, L.hc2, true));
    }
    return JUNO_OK;
}

int stack_enqueue_decode_logits(juno_ctx *c, StackNet *net, int n, float *logits, cudaStream_t st) {
    GvArgs a;
    JUNO_TRY(from_residual(c, net, n, nullptr, false, &a, st));
    a.nseg = 1;
    a.seg[0] = seg(net->head, GVE_F32, logits, net->spec.vocab);
    a.seg[0].n_store = net->spec.vocab;
    return launch_gemv_rows(c, a, st);
}

}  // namespace juno
