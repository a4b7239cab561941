// Layer stacks with dense weights: loading helpers, buffers, and the pass over many rows (portions of prompts, large decode
// batches, and every pass in 32-bit).
#include "gemv_rows.cuh"
#include "stack.cuh"

#include <algorithm>
#include <cstring>

namespace juno {

// ───────────────────────────── loading ────────────────────────────────────────────────────
static inline float bf16_to_f32(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}
static inline uint16_t f32_to_bf16(float f) {  // round to nearest even
    uint32_t u;
    memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return (uint16_t)((u >> 16) | 0x40u);
    return (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
}
float st_value(const juno_safetensors *f, const StTensor &t, int64_t i) {
    const uint8_t *p = f->base + t.offset;
    if (t.dtype == ST_BF16) {
        uint16_t v;
        memcpy(&v, p + 2 * i, 2);
        return bf16_to_f32(v);
    }
    float v;
    memcpy(&v, p + 4 * i, 4);
    return v;
}

void HostMat::put(const juno_safetensors *f, const StTensor &t, int64_t r0, int64_t c0, int nr, int nc, int row, int col) {
    const int64_t src_cols = t.shape.back();
    for (int i = 0; i < nr; i++) {
        const int64_t s = (r0 + i) * src_cols + c0;
        const size_t d = (size_t)(row + i) * cols + col;
        if (dt == DT_BF16 && t.dtype == ST_BF16) {
            memcpy(&data[d * 2], f->base + t.offset + s * 2, (size_t)nc * 2);
        } else if (dt == DT_F32 && t.dtype == ST_F32) {
            memcpy(&data[d * 4], f->base + t.offset + s * 4, (size_t)nc * 4);
        } else {
            for (int j = 0; j < nc; j++) {
                const float v = st_value(f, t, s + j);
                if (dt == DT_F32)
                    reinterpret_cast<float *>(data.data())[d + j] = v;
                else
                    reinterpret_cast<uint16_t *>(data.data())[d + j] = f32_to_bf16(v);
            }
        }
    }
}

void HostMat::put_transposed(const juno_safetensors *f, const StTensor &t, int64_t r0, int64_t c0, int nr, int nc, int row, int col) {
    const int64_t src_cols = t.shape.back();
    for (int i = 0; i < nr; i++)
        for (int j = 0; j < nc; j++) {
            const float v = st_value(f, t, (r0 + i) * src_cols + c0 + j);
            const size_t d = (size_t)(row + j) * cols + col + i;
            if (dt == DT_F32)
                reinterpret_cast<float *>(data.data())[d] = v;
            else
                reinterpret_cast<uint16_t *>(data.data())[d] = f32_to_bf16(v);
        }
}

static int net_alloc(StackNet *net, void **p, size_t bytes) {
    const cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
    if (e != cudaSuccess) {
        cudaGetLastError();
        set_error("cudaMalloc of %zu bytes failed: %s", bytes, cudaGetErrorString(e));
        return JUNO_ERR_OOM;
    }
    net->owned.push_back(*p);
    return JUNO_OK;
}

int stack_upload(juno_ctx *c, StackNet *net, const HostMat &m, StackMat *out) {
    JUNO_TRY(net_alloc(net, &out->w, m.data.size()));
    JUNO_CUDA_TRY(cudaMemcpyAsync(out->w, m.data.data(), m.data.size(), cudaMemcpyHostToDevice, c->stream));
    JUNO_CUDA_TRY(cudaStreamSynchronize(c->stream));
    c->h2d_bytes += (int64_t)m.data.size();
    out->rows = m.rows;
    out->cols = m.cols;
    return JUNO_OK;
}

int stack_upload_f32(juno_ctx *c, StackNet *net, const std::vector<float> &v, float **out) {
    JUNO_TRY(net_alloc(net, (void **)out, v.size() * 4));
    JUNO_CUDA_TRY(cudaMemcpyAsync(*out, v.data(), v.size() * 4, cudaMemcpyHostToDevice, c->stream));
    JUNO_CUDA_TRY(cudaStreamSynchronize(c->stream));
    c->h2d_bytes += (int64_t)v.size() * 4;
    return JUNO_OK;
}

// A portion of a prompt with at most this many positions attends with absorbed queries, like a decode step: expanding keys and
// values from the whole context would cost more than it saves.
constexpr int kAbsorbRows = 48;
constexpr int kMergeRows = 8;  // rows up to which the value projection is done by the merge of the context splits
static bool flash_fits(const LatentMixerSpec &m) { return m.dp() <= kFlashMaxDim && m.vp() <= kFlashMaxDim; }

// ───────────────────────────── buffers ────────────────────────────────────────────────────
int stack_alloc(juno_ctx *c, StackNet *net, int max_batch, int max_rows, int logit_rows) {
    const StackSpec &s = net->spec;
    const size_t es = dt_bytes(net->dt);
    const int cap = net->cap = std::max(max_batch, max_rows);
    net->logit_cap = logit_rows;
    // absorbed queries are kept for few rows only, unless some layer has to take the general kernel
    net->lat_cap = net->dt == DT_BF16 ? std::min(cap, std::max(max_batch, kAbsorbRows)) : cap;
    for (const StackLayerSpec &L : s.layers)
        if (!flash_fits(L.mix) || L.mix.rp() > kLatentSplitMaxRank) net->lat_cap = cap;
    const int wp = s.wp();
    int ff = 16;
    for (const StackLayerSpec &L : s.layers) {
        const LatentMixerSpec &m = L.mix;
        net->ldu = std::max(net->ldu, m.down_rows());
        net->ldcq = std::max(net->ldcq, m.qp());
        net->ldq = std::max(net->ldq, m.heads * m.dp());
        net->ldlat = std::max(net->ldlat, m.heads * m.rp());
        net->ldatt = std::max(net->ldatt, m.heads * m.vp());
        ff = std::max(ff, pad16(L.ff));
    }
    net->ldact = ff;
    net->weight_bytes = (double)net->head.rows * net->head.cols * es;
    for (size_t l = 0; l < s.layers.size(); l++) {
        const StackLayerWeights &L = net->layers[(size_t)s.weights((int)l)];
        for (const StackMat *m : {&L.down, &L.uq, &L.ukt, &L.o, &L.rg1, &L.rg2, &L.up, &L.mdown}) net->weight_bytes += (double)m->rows * m->cols * es;
        net->weight_bytes += (double)s.layers[l].mix.heads * s.layers[l].mix.vp() * s.layers[l].mix.rp() * es;  // W_uv
    }
    if (net->dt == DT_BF16) {
        for (const StackLayerSpec &L : s.layers)
            for (int n = 1; n <= net->lat_cap; n++) net->part_floats = std::max(net->part_floats, latent_part_floats(c, n, L.mix.heads, L.mix.rp()));
        JUNO_TRY(net_alloc(net, (void **)&net->part_o, net->part_floats * 4));
    }
    const struct { void **p; size_t bytes; } bufs[] = {
        {(void **)&net->x, (size_t)cap * wp * 4},
        {(void **)&net->u, (size_t)cap * net->ldu * 4},
        {(void **)&net->row_scale, (size_t)cap * 4},
        {&net->h, (size_t)cap * wp * es},
        {&net->hc, (size_t)cap * wp * es},
        {&net->gate, (size_t)cap * wp * es},
        {&net->z, (size_t)cap * wp * es},
        {&net->cq, (size_t)cap * net->ldcq * es},
        {&net->q, (size_t)cap * net->ldq * es},
        {&net->qlat, (size_t)net->lat_cap * net->ldlat * es},
        {&net->olat, (size_t)net->lat_cap * net->ldlat * es},
        {&net->att, (size_t)cap * net->ldatt * es},
        {&net->act, (size_t)cap * net->ldact * es},
        {&net->fin, (size_t)std::max(logit_rows, 1) * wp * es},
        {(void **)&net->row_idx, (size_t)cap * 4},
        {(void **)&net->x2, (size_t)std::min(cap, kGvMaxSeqs) * wp * 4},
        {(void **)&net->dec_gate, (size_t)std::min(cap, kGvMaxSeqs) * wp * 4},
        {(void **)&net->dec_z, (size_t)std::min(cap, kGvMaxSeqs) * wp * 4},
    };
    for (const auto &b : bufs) {
        JUNO_TRY(net_alloc(net, b.p, b.bytes));
        JUNO_CUDA_TRY(cudaMemsetAsync(*b.p, 0, b.bytes, c->stream));
    }
    JUNO_CUDA_TRY(cudaStreamSynchronize(c->stream));
    return JUNO_OK;
}

void stack_free(StackNet *net) {
    if (!net) return;
    for (void *p : net->owned) cudaFree(p);
    if (net->ctx_lat) cudaFree(net->ctx_lat);
    if (net->ctx_kv) cudaFree(net->ctx_kv);
    delete net;
}

int stack_enqueue_step(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, int len_bound, float *logits, cudaStream_t st) {
    if (stack_fused_ok(c, net, rows)) {
        JUNO_TRY(stack_enqueue_decode(c, net, pool, rows, n_splits, st));
        return stack_enqueue_decode_logits(c, net, rows.n, logits, st);
    }
    JUNO_TRY(stack_enqueue_layers(c, net, pool, rows, n_splits, len_bound, st));
    return stack_enqueue_logits(c, net, nullptr, rows.n, logits, st);
}

void stack_step_done(const juno_ctx *c, StackNet *net, int n) {
    RowSet rows;
    rows.n = n;
    net->last_x = 0;
    if (!stack_fused_ok(c, net, rows)) return;
    for (const StackLayerSpec &L : net->spec.layers) net->last_x ^= L.ff ? 0 : 1;  // one hand-over per sublayer
}

const float *stack_residual(const StackNet *net) { return net->last_x ? net->x2 : net->x; }

// One split count for all layers of a step (it is part of the captured step's key): the largest any layer's shape asks for
// that every layer's buffers and kernels take.
int stack_pick_splits(const juno_ctx *c, const StackNet *net, int n, int len_bound) {
    if (net->dt != DT_BF16) return 1;
    int best = 1, most = 1 << 30;
    for (const StackLayerSpec &L : net->spec.layers) {
        if (L.mix.rp() > kLatentSplitMaxRank) continue;
        best = std::max(best, latent_pick_splits(c, n, L.mix.heads, L.mix.rp(), len_bound));
        most = std::min<long long>(most, (long long)(net->part_floats / ((size_t)n * L.mix.heads * (L.mix.rp() + 2))));
    }
    return std::max(1, std::min(best, most));
}

// ───────────────────────────── attention of one layer ─────────────────────────────────────
// q -> att, the head gates applied.  Few rows: the queries are taken into the latent space (q_lat[h] = W_uk[h]^T q[h]) and
// attend the latent pages themselves.  Many rows of one sequence: keys and values are expanded once for the pass.
static int attention(juno_ctx *c, StackNet *net, const StackLayerWeights &L, const LatentMixerSpec &m, const juno_kvpool *pool, int layer,
                     const RowSet &rows, int n_splits, int len_bound, cudaStream_t st) {
    const int n = rows.n, dt = net->dt, H = m.heads, rp = m.rp(), dp = m.dp(), vp = m.vp();
    unsigned *err = c->gemv_scratch.qerr;
    const float *gate = net->u + m.gate_col();
    GemmArgs g;
    g.M = n;
    if (dt == DT_BF16 && rows.one_seq && n > kAbsorbRows && flash_fits(m)) {
        JUNO_TRY(ensure_device(&net->ctx_lat, &net->ctx_lat_bytes, (size_t)len_bound * rp * 2));
        JUNO_TRY(ensure_device(&net->ctx_kv, &net->ctx_kv_bytes, (size_t)len_bound * H * (dp + vp) * 2));
        JUNO_TRY(launch_latent_gather(c, pool, layer, rows.slots, len_bound, net->ctx_lat, st));
        g.a = net->ctx_lat;
        g.lda = rp;
        g.w = L.ukv.w;
        g.ldw = rp;
        g.M = len_bound;
        g.N = H * (dp + vp);
        g.K = rp;
        g.out = net->ctx_kv;
        g.ldo = H * (dp + vp);
        JUNO_TRY(launch_gemm_rows(c, dt, g, err, st));
        FlashArgs f{n, len_bound - n, H, dp, vp, m.scale, net->q, net->ctx_kv, H * (dp + vp), gate, net->ldu, net->att};
        return launch_flash_prefill(c, f, st);
    }
    JUNO_REQUIRE(n <= net->lat_cap, "a pass of %d rows exceeds the latent buffers (%d)", n, net->lat_cap);
    g.a = net->q;
    g.lda = H * dp;
    g.w = L.ukt.w;
    g.ldw = dp;
    g.N = rp;
    g.K = dp;
    g.out = net->qlat;
    g.ldo = H * rp;
    g.groups = H;
    g.a_step = dp;
    g.w_step = rp;
    g.o_step = rp;
    JUNO_TRY(launch_gemm_rows(c, dt, g, err, st));
    const uint8_t *w_uv = static_cast<const uint8_t *>(L.ukv.w) + (size_t)H * dp * rp * dt_bytes(dt);
    if (dt == DT_BF16 && rp <= kLatentSplitMaxRank) {
        const size_t ml = (size_t)n * H * n_splits * rp;
        JUNO_REQUIRE(ml + (size_t)n * H * n_splits * 2 <= net->part_floats, "%d context splits of %d rows exceed the buffer", n_splits, n);
        LatentSplitArgs sp{pool, layer, rows, H, rp, n_splits, m.scale, net->qlat, net->part_o, net->part_o + ml};
        JUNO_TRY(launch_latent_attn_split(c, sp, st));
        const bool fold = n <= kMergeRows;  // the value projection inside the merge reads W_uv once per row
        LatentMergeArgs mg{n, H, rp, vp, n_splits, net->part_o, net->part_o + ml, fold ? w_uv : nullptr, gate, net->ldu, fold ? net->att : net->olat};
        JUNO_TRY(launch_latent_merge(c, mg, st));
        if (fold) return JUNO_OK;
    } else {
        LatentAttnArgs at{pool, layer, rows, H, rp, m.scale, net->qlat, net->olat};
        JUNO_TRY(launch_latent_attn_simt(c, dt, at, st));
    }
    g.a = net->olat;
    g.lda = H * rp;
    g.w = w_uv;
    g.ldw = rp;
    g.N = vp;
    g.K = rp;
    g.out = net->att;
    g.ldo = H * vp;
    g.epi = GE_GROUP_GATE;
    g.aux = gate;
    g.ldaux = net->ldu;
    g.a_step = rp;
    g.w_step = vp;
    g.o_step = vp;
    return launch_gemm_rows(c, dt, g, err, st);
}

// ───────────────────────────── a pass over many rows ──────────────────────────────────────
int stack_enqueue_layers(juno_ctx *c, StackNet *net, const juno_kvpool *pool, const RowSet &rows, int n_splits, int len_bound, cudaStream_t st) {
    const StackSpec &s = net->spec;
    net->last_x = 0;
    const int n = rows.n, wp = s.wp(), dt = net->dt, n_layers = (int)s.layers.size();
    unsigned *err = c->gemv_scratch.qerr;
    JUNO_REQUIRE(n >= 1 && n <= net->cap, "a pass of %d rows exceeds the buffers (%d)", n, net->cap);
    auto product = [&](const void *a, int lda, const StackMat &w, void *out, int ldo, int epi, const float *bias = nullptr, const void *aux = nullptr) {
        GemmArgs g;
        g.a = a;
        g.lda = lda;
        g.w = w.w;
        g.ldw = w.cols;
        g.M = n;
        g.N = w.rows;
        g.K = w.cols;
        g.out = out;
        g.ldo = ldo;
        g.epi = epi;
        g.bias = bias;
        g.aux = aux;
        g.ldaux = wp;
        return launch_gemm_rows(c, dt, g, err, st);
    };
    // x += norm(z) of the sublayer that ended, and the next sublayer's normed input
    auto residual = [&](const void *z, float g_z, bool more, float g_next) {
        ResidNormArgs a;
        a.x = net->x;
        a.ldx = wp;
        a.width = s.width;
        a.n = n;
        a.z = z;
        a.ldz = wp;
        a.g_z = g_z;
        a.g_next = g_next;
        a.eps = s.eps;
        a.h = more ? net->h : nullptr;
        a.ldh = wp;
        a.row_scale = net->row_scale;
        return launch_resid_norm(c, dt, a, st);
    };
    JUNO_TRY(launch_embed_norm(c, dt, net->embed.w, net->embed.cols, s.width, s.vocab, net->embed_norm, s.eps, rows, net->x, wp, st));
    JUNO_TRY(residual(nullptr, 0.f, true, net->layers[s.weights(0)].norm1));
    for (int l = 0; l < n_layers; l++) {
        const StackLayerWeights &L = net->layers[s.weights(l)];
        const LatentMixerSpec &m = s.layers[l].mix;
        const bool last = l + 1 == n_layers;
        const float next_norm1 = last ? 0.f : net->layers[s.weights(l + 1)].norm1;
        // mixer
        JUNO_TRY(product(net->h, wp, L.rg1, net->gate, wp, GE_SIGMOID, L.rg1_b));
        ConvArgs cv{net->x, wp, s.width, net->row_scale, L.conv, s.taps, pool, l, net->hc, wp};
        JUNO_TRY(launch_conv(c, dt, cv, rows, st));
        JUNO_TRY(product(net->hc, wp, L.down, net->u, net->ldu, GE_F32));
        LatentNormArgs ln{net->u, net->ldu, m.q_rank, m.kv_col(), m.kv_rank, L.dq_norm, L.dkv_norm, s.eps, net->cq, m.qp(), pool, l};
        JUNO_TRY(launch_latent_norm(c, dt, ln, rows, st));
        JUNO_TRY(product(net->cq, m.qp(), L.uq, net->q, m.heads * m.dp(), GE_OP));
        JUNO_TRY(attention(c, net, L, m, pool, l, rows, n_splits, len_bound, st));
        JUNO_TRY(product(net->att, m.heads * m.vp(), L.o, net->z, wp, GE_MUL, nullptr, net->gate));
        const bool mlp = s.layers[l].ff > 0;
        JUNO_TRY(residual(net->z, L.norm1b, mlp || !last, mlp ? L.norm2 : next_norm1));
        if (!mlp) continue;
        // feed-forward
        JUNO_TRY(product(net->h, wp, L.rg2, net->gate, wp, GE_SIGMOID, L.rg2_b));
        JUNO_TRY(product(net->h, wp, L.up, net->act, L.mdown.cols, GE_RELU2));
        JUNO_TRY(product(net->act, L.mdown.cols, L.mdown, net->z, wp, GE_MUL, nullptr, net->gate));
        JUNO_TRY(residual(net->z, L.norm2b, !last, next_norm1));
    }
    return JUNO_OK;
}

int stack_enqueue_logits(juno_ctx *c, StackNet *net, const int32_t *row_idx, int n, float *logits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    JUNO_REQUIRE(n >= 1 && n <= net->logit_cap, "logits of %d rows exceed the buffer (%d)", n, net->logit_cap);
    JUNO_TRY(launch_gather_norm(c, net->dt, net->x, s.wp(), s.width, row_idx, n, net->final_norm, s.eps, net->fin, s.wp(), st));
    GemmArgs g;
    g.a = net->fin;
    g.lda = s.wp();
    g.w = net->head.w;
    g.ldw = net->head.cols;
    g.M = n;
    g.N = s.vocab;
    g.K = net->head.cols;
    g.w_rows = net->head.rows;
    g.out = logits;
    g.ldo = s.vocab;
    g.epi = GE_F32;
    return launch_gemm_rows(c, net->dt, g, c->gemv_scratch.qerr, st);
}

}  // namespace juno
