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
constexpr int kGroupedFewRows = 16;  // rows of a portion up to which the decode attention is faster than a prompt's
static bool flash_fits(int dp, int vp) { return dp <= kFlashMaxDim && vp <= kFlashMaxDim; }

// ───────────────────────────── buffers ────────────────────────────────────────────────────
// (cos, sin) tables, one per distinct rotation.
static int rotation_tables(juno_ctx *c, StackNet *net, int max_ctx) {
    const StackSpec &s = net->spec;
    net->rot.assign(s.layers.size(), nullptr);
    for (size_t l = 0; l < s.layers.size(); l++) {
        const GroupedMixerSpec &m = s.layers[l].grouped;
        if (s.layers[l].mixer != MIX_GROUPED || m.rot_dims == 0) continue;
        for (size_t k = 0; k < l && !net->rot[l]; k++)
            if (net->rot[k] && s.layers[k].grouped.rot_dims == m.rot_dims && s.layers[k].grouped.rot_base == m.rot_base) net->rot[l] = net->rot[k];
        if (net->rot[l]) continue;
        float2 *t = nullptr;
        JUNO_TRY(net_alloc(net, (void **)&t, (size_t)max_ctx * (m.rot_dims / 2) * sizeof(float2)));
        JUNO_TRY(launch_rotation_table(c, max_ctx, m.rot_dims, m.rot_base, t, c->stream));
        net->rot[l] = t;
    }
    return JUNO_OK;
}

int stack_alloc(juno_ctx *c, StackNet *net, int max_batch, int max_rows, int logit_rows, int max_ctx) {
    const StackSpec &s = net->spec;
    const size_t es = dt_bytes(net->dt);
    const int cap = net->cap = std::max(max_batch, max_rows);
    net->logit_cap = logit_rows;
    // absorbed queries are kept for few rows only, unless some layer has to take the general kernel
    net->lat_cap = net->dt == DT_BF16 ? std::min(cap, std::max(max_batch, kAbsorbRows)) : cap;
    for (const StackLayerSpec &L : s.layers)
        if (L.mixer == MIX_LATENT && (!flash_fits(L.mix.dp(), L.mix.vp()) || L.mix.rp() > kLatentSplitMaxRank)) net->lat_cap = cap;
    const int wp = s.wp(), streams = std::max(1, s.streams), few = std::min(cap, kGvMaxSeqs);
    const size_t gated = s.streams ? 0 : 1;  // buffers of the gated, convolved residual
    int ff = 16;
    bool grouped = false;
    for (const StackLayerSpec &L : s.layers) {
        ff = std::max(ff, pad16(L.ff));
        if (L.mixer == MIX_GROUPED) {
            const GroupedMixerSpec &m = L.grouped;
            grouped = true;
            net->ldu = std::max(net->ldu, m.qkv_rows());
            net->ldq = std::max(net->ldq, m.heads * m.dp());
            net->ldatt = std::max(net->ldatt, m.heads * m.vp());
            if (net->dt == DT_BF16 && std::max(m.dp(), m.vp()) <= kGroupedMaxDim) net->part_floats = std::max(net->part_floats, grouped_part_floats(c, m.vp()));
            continue;
        }
        const LatentMixerSpec &m = L.mix;
        net->ldu = std::max(net->ldu, m.down_rows());
        net->ldcq = std::max(net->ldcq, m.qp());
        net->ldq = std::max(net->ldq, m.heads * m.dp());
        net->ldlat = std::max(net->ldlat, m.heads * m.rp());
        net->ldatt = std::max(net->ldatt, m.heads * m.vp());
        if (net->dt == DT_BF16)
            for (int n = 1; n <= net->lat_cap; n++) net->part_floats = std::max(net->part_floats, latent_part_floats(c, n, m.heads, m.rp()));
    }
    for (const StackLayerSpec &L : s.layers)
        JUNO_REQUIRE((L.mixer == MIX_GROUPED) == (s.streams > 0), "latent attention belongs to the gated residual, grouped attention to residual streams");
    net->ldact = ff;
    net->weight_bytes = (double)net->head.rows * net->head.cols * es;
    for (size_t l = 0; l < s.layers.size(); l++) {
        const StackLayerWeights &L = net->layers[(size_t)s.weights((int)l)];
        for (const StackMat *m : {&L.down, &L.uq, &L.ukt, &L.o, &L.rg1, &L.rg2, &L.up, &L.mdown, &L.qkv, &L.gu}) net->weight_bytes += (double)m->rows * m->cols * es;
        if (s.layers[l].mixer == MIX_LATENT) net->weight_bytes += (double)s.layers[l].mix.heads * s.layers[l].mix.vp() * s.layers[l].mix.rp() * es;  // W_uv
    }
    JUNO_TRY(rotation_tables(c, net, max_ctx));
    const struct { void **p; size_t bytes; } bufs[] = {
        {(void **)&net->x, (size_t)cap * streams * wp * 4},
        {(void **)&net->u, (size_t)cap * net->ldu * 4},
        {(void **)&net->row_scale, gated * cap * 4},
        {&net->h, (size_t)cap * wp * es},
        {&net->hc, gated * cap * wp * es},
        {&net->gate, gated * cap * wp * es},
        {&net->z, (size_t)cap * wp * es},
        {&net->cq, (size_t)cap * net->ldcq * es},
        {&net->q, (size_t)cap * net->ldq * es},
        {&net->qlat, (size_t)net->lat_cap * net->ldlat * es},
        {&net->olat, (size_t)net->lat_cap * net->ldlat * es},
        {&net->att, (size_t)cap * net->ldatt * es},
        {&net->act, (size_t)cap * net->ldact * es},
        {&net->fin, (size_t)std::max(logit_rows, 1) * wp * es},
        {(void **)&net->row_idx, (size_t)cap * 4},
        {(void **)&net->x2, (size_t)few * streams * wp * 4},
        {(void **)&net->dec_gate, gated * few * wp * 4},
        {(void **)&net->dec_z, (size_t)few * wp * 4},
        {(void **)&net->part_o, net->part_floats * 4},
        {(void **)&net->counters, grouped ? grouped_counters(c) * 4 : 0},
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
    if (net->hidden) cudaFree(net->hidden);
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
    net->last_x = stack_fused_ok(c, net, rows) ? stack_decode_hand_overs(net, n) & 1 : 0;
}

int stack_residual(juno_ctx *c, StackNet *net, int n, const float **out, cudaStream_t st) {
    *out = net->last_x ? net->x2 : net->x;
    if (net->spec.streams == 0) return JUNO_OK;
    const int wp = net->spec.wp();
    JUNO_TRY(ensure_device((void **)&net->hidden, &net->hidden_bytes, (size_t)n * wp * 4));
    JUNO_TRY(launch_stream_gather(c, net->dt, *out, net->spec.streams, wp, net->spec.width, nullptr, n, nullptr, 0.f, net->hidden, wp, st));
    *out = net->hidden;
    return JUNO_OK;
}

// One split count for all layers of a step (it is part of the captured step's key): the largest any layer's shape asks for
// that every layer's buffers and kernels take.
int stack_pick_splits(const juno_ctx *c, const StackNet *net, int n, int len_bound) {
    if (net->dt != DT_BF16) return 1;
    int best = 1, most = 1 << 30;
    for (const StackLayerSpec &L : net->spec.layers) {
        if (L.mixer == MIX_GROUPED) {
            const GroupedMixerSpec &m = L.grouped;
            best = std::max(best, grouped_pick_splits(c, n, m.heads, m.kv_heads, std::max(m.dp(), m.vp()), m.span.longest(len_bound)));
            continue;
        }
        if (L.mix.rp() > kLatentSplitMaxRank) continue;
        best = std::max(best, latent_pick_splits(c, n, L.mix.heads, L.mix.rp(), len_bound));
        most = std::min<long long>(most, (long long)(net->part_floats / ((size_t)n * L.mix.heads * (L.mix.rp() + 2))));
    }
    return std::max(1, std::min(best, most));
}

// ───────────────────────────── attention of one layer ─────────────────────────────────────
GroupedAttnArgs grouped_attn_args(const StackNet *net, const StackLayerWeights &L, const juno_kvpool *pool, int layer, const RowSet &rows) {
    const GroupedMixerSpec &m = net->spec.layers[(size_t)layer].grouped;
    GroupedAttnArgs a;
    a.pool = pool;
    a.layer = layer;
    a.rows = rows;
    a.heads = m.heads;
    a.kv_heads = m.kv_heads;
    a.dim = m.dim;
    a.dp = m.dp();
    a.vp = m.vp();
    a.scale = m.scale;
    a.span = m.span;
    a.slopes = L.slopes;
    a.sinks = L.sinks;
    a.u = net->u;
    a.ldu = m.qkv_rows();
    a.q_norm = L.q_norm;
    a.k_norm = L.k_norm;
    a.eps = net->spec.eps;
    a.rot = net->rot[(size_t)layer];
    a.rot_dims = m.rot_dims;
    a.temp_coef = m.temp_coef;
    a.temp_every = m.temp_every;
    a.q = net->q;
    a.out = net->att;
    return a;
}
int grouped_layer_splits(const juno_ctx *c, const GroupedMixerSpec &m, int n, int n_splits) {
    return std::min(n_splits, grouped_pick_splits(c, n, m.heads, m.kv_heads, std::max(m.dp(), m.vp()), m.span.longest(1 << 30)));
}

// u -> att over the layer's pages, this pass's positions appended.
static int grouped_attention(juno_ctx *c, StackNet *net, const StackLayerWeights &L, const juno_kvpool *pool, int layer, const RowSet &rows, int n_splits, int len_bound,
                             cudaStream_t st) {
    const GroupedMixerSpec &m = net->spec.layers[(size_t)layer].grouped;
    const GroupedAttnArgs a = grouped_attn_args(net, L, pool, layer, rows);
    const int d = std::max(a.dp, a.vp);
    JUNO_TRY(launch_grouped_prep(c, net->dt, a, st));
    if (net->dt == DT_F32 || d > kGroupedMaxDim) return launch_grouped_simt(c, net->dt, a, st);
    if (!rows.one_seq || rows.n <= kGroupedFewRows)
        return launch_grouped_split(c, a, grouped_layer_splits(c, m, rows.n, n_splits), false, net->part_o, net->part_floats, net->counters, st);
    FlashArgs f;
    f.n = rows.n;
    f.pos0 = len_bound - rows.n;
    f.heads = a.heads;
    f.dim = a.dp;
    f.vdim = a.vp;
    f.scale = a.scale;
    f.q = a.q;
    f.out = a.out;
    f.kv_heads = a.kv_heads;
    f.pool = pool;
    f.layer = layer;
    f.slot = rows.slots;
    f.span = a.span;
    f.slopes = a.slopes;
    f.sinks = a.sinks;
    return launch_flash_prefill(c, f, st);
}

// q -> att, the head gates applied.  Few rows: the queries are taken into the latent space (q_lat[h] = W_uk[h]^T q[h]) and
// attend the latent pages themselves.  Many rows of one sequence: keys and values are expanded once for the pass.
static int latent_attention(juno_ctx *c, StackNet *net, const StackLayerWeights &L, const LatentMixerSpec &m, const juno_kvpool *pool, int layer,
                     const RowSet &rows, int n_splits, int len_bound, cudaStream_t st) {
    const int n = rows.n, dt = net->dt, H = m.heads, rp = m.rp(), dp = m.dp(), vp = m.vp();
    unsigned *err = c->gemv_scratch.qerr;
    const float *gate = net->u + m.gate_col();
    GemmArgs g;
    g.M = n;
    if (dt == DT_BF16 && rows.one_seq && n > kAbsorbRows && flash_fits(dp, vp)) {
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
    // the residual takes the result z of the sublayer that ended, and gives the next one its normed input
    struct Sublayer {
        const StackLayerWeights *w = nullptr;
        bool ff = false;
    };
    auto hand_over = [&](Sublayer done, Sublayer next) {
        const bool more = next.w != nullptr;
        if (s.streams) {
            StreamStepArgs a;
            a.x = net->x;
            a.streams = s.streams;
            a.ldx = wp;
            a.width = s.width;
            a.n = n;
            a.eps = s.eps;
            if (done.w) {
                const HyperConnection &hc = done.ff ? done.w->hc2 : done.w->hc1;
                a.z = net->z;
                a.ldz = wp;
                a.mix = hc.mix;
                a.out = hc.out;
            }
            if (more) {
                a.in = (next.ff ? next.w->hc2 : next.w->hc1).in;
                a.w = next.ff ? next.w->norm2_w : next.w->norm1_w;
                a.h = net->h;
                a.ldh = wp;
            }
            return launch_stream_step(c, dt, a, st);
        }
        ResidNormArgs a;
        a.x = net->x;
        a.ldx = wp;
        a.width = s.width;
        a.n = n;
        a.z = done.w ? net->z : nullptr;
        a.ldz = wp;
        a.g_z = done.w ? (done.ff ? done.w->norm2b : done.w->norm1b) : 0.f;
        a.g_next = more ? (next.ff ? next.w->norm2 : next.w->norm1) : 0.f;
        a.eps = s.eps;
        a.h = more ? net->h : nullptr;
        a.ldh = wp;
        a.row_scale = net->row_scale;
        return launch_resid_norm(c, dt, a, st);
    };
    // the result of a sublayer; the gated residual multiplies it by its gate
    auto result = [&](const void *a, const StackMat &w) {
        return s.streams ? product(a, w.cols, w, net->z, wp, GE_OP) : product(a, w.cols, w, net->z, wp, GE_MUL, nullptr, net->gate);
    };
    auto weights = [&](int l) { return &net->layers[(size_t)s.weights(l)]; };
    if (s.streams)
        JUNO_TRY(launch_stream_embed(c, dt, net->embed.w, net->embed.cols, s.width, s.vocab, s.streams, rows, net->x, wp, st));
    else
        JUNO_TRY(launch_embed_norm(c, dt, net->embed.w, net->embed.cols, s.width, s.vocab, net->embed_norm, s.eps, rows, net->x, wp, st));
    JUNO_TRY(hand_over({}, {weights(0), false}));
    for (int l = 0; l < n_layers; l++) {
        const StackLayerWeights &L = *weights(l);
        const StackLayerSpec &spec = s.layers[(size_t)l];
        const Sublayer next = {l + 1 < n_layers ? weights(l + 1) : nullptr, false};
        if (!s.streams) JUNO_TRY(product(net->h, wp, L.rg1, net->gate, wp, GE_SIGMOID, L.rg1_b));
        if (spec.mixer == MIX_GROUPED) {
            JUNO_TRY(product(net->h, wp, L.qkv, net->u, L.qkv.rows, GE_F32, L.qkv_b));
            JUNO_TRY(grouped_attention(c, net, L, pool, l, rows, n_splits, len_bound, st));
        } else {
            const LatentMixerSpec &m = spec.mix;
            ConvArgs cv{net->x, wp, s.width, net->row_scale, L.conv, s.taps, pool, l, net->hc, wp};
            JUNO_TRY(launch_conv(c, dt, cv, rows, st));
            JUNO_TRY(product(net->hc, wp, L.down, net->u, net->ldu, GE_F32));
            LatentNormArgs ln{net->u, net->ldu, m.q_rank, m.kv_col(), m.kv_rank, L.dq_norm, L.dkv_norm, s.eps, net->cq, m.qp(), pool, l};
            JUNO_TRY(launch_latent_norm(c, dt, ln, rows, st));
            JUNO_TRY(product(net->cq, m.qp(), L.uq, net->q, m.heads * m.dp(), GE_OP));
            JUNO_TRY(latent_attention(c, net, L, m, pool, l, rows, n_splits, len_bound, st));
        }
        JUNO_TRY(result(net->att, L.o));
        if (spec.ff == 0) {
            JUNO_TRY(hand_over({&L, false}, next));
            continue;
        }
        JUNO_TRY(hand_over({&L, false}, {&L, true}));
        if (!s.streams) JUNO_TRY(product(net->h, wp, L.rg2, net->gate, wp, GE_SIGMOID, L.rg2_b));
        if (spec.ff_kind == FF_GEGLU)
            JUNO_TRY(product(net->h, wp, L.gu, net->act, L.mdown.cols, GE_GEGLU));
        else
            JUNO_TRY(product(net->h, wp, L.up, net->act, L.mdown.cols, GE_RELU2));
        JUNO_TRY(result(net->act, L.mdown));
        JUNO_TRY(hand_over({&L, true}, next));
    }
    return JUNO_OK;
}

int stack_enqueue_logits(juno_ctx *c, StackNet *net, const int32_t *row_idx, int n, float *logits, cudaStream_t st) {
    const StackSpec &s = net->spec;
    JUNO_REQUIRE(n >= 1 && n <= net->logit_cap, "logits of %d rows exceed the buffer (%d)", n, net->logit_cap);
    if (s.streams)
        JUNO_TRY(launch_stream_gather(c, net->dt, net->x, s.streams, s.wp(), s.width, row_idx, n, net->final_w, s.eps, net->fin, s.wp(), st));
    else
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
