// The Desilorn design: a decoder-only stack of two kinds of grouped-head attention (a sliding window with a distance bias, a
// query temperature and learned sinks; chunks with normed and rotated queries and keys and a fixed sink) and gated GELU
// feed-forwards, on residual streams joined by hyper-connections, with a span of layers that runs several times in a row.
// This file knows the keys of its config.json and the names of its tensors; the mechanisms are the generic ones of stack.cuh.
#include "stack_loader.cuh"

#include <algorithm>
#include <cmath>

namespace juno {

static int mixer_spec(const Json *m, const std::string &type, const std::string &where, GroupedMixerSpec *s) {
    constexpr int kMax = 1 << 20;
    const char *w = where.c_str();
    if (type != "attention" && type != "attention_2") {
        set_error("config: %s: mixer '%s' is not part of this design", w, type.c_str());
        return JUNO_ERR_UNSUPPORTED;
    }
    JUNO_TRY(cfg_int(m, "heads", w, 1, 65535, &s->heads));
    JUNO_TRY(cfg_int(m, "kv_heads", w, 1, 65535, &s->kv_heads));
    JUNO_REQUIRE(s->heads % s->kv_heads == 0, "config: %s: %d heads cannot share %d key/value heads", w, s->heads, s->kv_heads);
    JUNO_TRY(cfg_int(m, "dim", w, 1, 8192, &s->dim));
    JUNO_TRY(cfg_int(m, "vdim", w, 1, kGroupedMaxVdim, &s->vdim));
    JUNO_TRY(cfg_float(m, "scale", w, &s->scale));
    const Json *mask = m->find("mask");
    if (type == "attention") {
        JUNO_TRY(cfg_int(mask, "size", (where + ".mask").c_str(), 1, 1 << 30, &s->span.window));
        s->distance_bias = true;
        s->sink = SINK_LEARNED;
        const Json *temp = m->find("q_temp");
        if (temp && !temp->is_null()) {
            JUNO_TRY(cfg_float(temp, "coef", (where + ".q_temp").c_str(), &s->temp_coef));
            JUNO_TRY(cfg_int(temp, "every", (where + ".q_temp").c_str(), 1, 1 << 30, &s->temp_every));
        }
        return JUNO_OK;
    }
    JUNO_TRY(cfg_int(mask, "size", (where + ".mask").c_str(), 1, 1 << 30, &s->span.chunk));
    s->qk_norm = true;
    s->sink = SINK_ZERO;
    const Json *rot = m->find("rot"), *base = rot ? rot->find("base") : nullptr;
    JUNO_TRY(cfg_int(rot, "dims", (where + ".rot").c_str(), 0, kMax, &s->rot_dims));
    JUNO_REQUIRE(s->rot_dims % 2 == 0 && s->rot_dims <= s->dim, "config: %s.rot.dims must be even and at most %d", w, s->dim);
    JUNO_REQUIRE(base && base->kind == Json::NUMBER && base->num > 0, "config: %s.rot.base must be a positive number", w);
    s->rot_base = base->num;
    return JUNO_OK;
}

int desilorn_spec(const Json &cfg, StackSpec *spec) {
    JUNO_TRY(cfg_int(&cfg, "width", "model", 1, 49152, &spec->width));
    JUNO_TRY(cfg_int(&cfg, "vocab", "model", 1, 1 << 24, &spec->vocab));
    JUNO_TRY(cfg_int(&cfg, "streams", "model", 1, kMaxStreams, &spec->streams));
    JUNO_TRY(cfg_float(cfg.find("norm"), "eps", "norm", &spec->eps));
    const Json *layers = cfg.find("layers");
    JUNO_REQUIRE(layers && layers->kind == Json::ARRAY && !layers->arr.empty(), "config: layers must be a non-empty list");
    const int n = (int)layers->arr.size();
    std::vector<StackLayerSpec> one;
    for (int i = 0; i < n; i++) {
        const Json &e = layers->arr[(size_t)i];
        const std::string w = "layers[" + std::to_string(i) + "]";
        StackLayerSpec L;
        std::string type, kind;
        JUNO_TRY(cfg_string(&e, "type", w.c_str(), &type));
        const Json *m = e.find("mixer");
        JUNO_REQUIRE(m && m->kind == Json::OBJECT, "config: %s.mixer is missing", w.c_str());
        L.mixer = MIX_GROUPED;
        L.source = i;
        JUNO_TRY(mixer_spec(m, type, w + ".mixer", &L.grouped));
        const Json *mlp = e.find("mlp");
        if (mlp && !mlp->is_null()) {
            JUNO_TRY(cfg_string(mlp, "kind", (w + ".mlp").c_str(), &kind));
            if (kind != "dense") {
                set_error("config: %s: feed-forward '%s' is not part of this design", w.c_str(), kind.c_str());
                return JUNO_ERR_UNSUPPORTED;
            }
            JUNO_TRY(cfg_int(mlp, "ff", (w + ".mlp").c_str(), 1, 1 << 20, &L.ff));
            L.ff_kind = FF_GEGLU;
        }
        one.push_back(L);
    }
    // the order of the runs: the looped span several times, each pass with a cache of its own and the first pass's weights
    int start = 0, stop = 0, times = 1;
    const Json *loop = cfg.find("loop");
    if (loop && !loop->is_null()) {
        JUNO_TRY(cfg_int(loop, "start", "loop", 0, n, &start));
        JUNO_TRY(cfg_int(loop, "stop", "loop", start, n, &stop));
        JUNO_TRY(cfg_int(loop, "times", "loop", 1, 4096, &times));
    }
    for (int i = 0; i < start; i++) spec->layers.push_back(one[(size_t)i]);
    for (int t = 0; t < times; t++)
        for (int i = start; i < stop; i++) {
            StackLayerSpec L = one[(size_t)i];
            if (t > 0) L.weights_of = i;  // before the span and in its first pass, runs and layers have the same numbers
            spec->layers.push_back(L);
        }
    for (int i = stop; i < n; i++) spec->layers.push_back(one[(size_t)i]);
    return JUNO_OK;
}

namespace {
struct Loader : StackLoader {
    int mixer(const std::string &p, const GroupedMixerSpec &s, StackLayerWeights *L) {
        const int W = net->spec.width, wp = net->spec.wp(), H = s.heads, G = s.kv_heads;
        const struct { const char *name; int heads, size, padded; } part[3] = {{"q", H, s.dim, s.dp()}, {"k", G, s.dim, s.dp()}, {"v", G, s.vdim, s.vp()}};
        HostMat qkv(net->dt, s.qkv_rows(), wp);
        std::vector<float> bias((size_t)s.qkv_rows(), 0.f);
        int row = 0;
        for (const auto &e : part) {
            const StTensor *w, *b;
            JUNO_TRY(get(p + e.name, {(int64_t)e.heads * e.size, W}, &w));
            JUNO_TRY(get(p + e.name + ".b", {(int64_t)e.heads * e.size}, &b));
            put_heads(&qkv, *w, e.heads, e.size, e.padded, W, row);
            for (int h = 0; h < e.heads; h++, row += e.padded)
                for (int i = 0; i < e.size; i++) bias[(size_t)(row + i)] = st_value(f, *b, (int64_t)h * e.size + i);
        }
        JUNO_TRY(stack_upload(c, net, qkv, &L->qkv));
        JUNO_TRY(stack_upload_f32(c, net, bias, &L->qkv_b));
        const StTensor *o;
        JUNO_TRY(get(p + "o", {W, (int64_t)H * s.vdim}, &o));
        HostMat mo(net->dt, wp, H * s.vp());
        put_head_columns(&mo, *o, H, s.vdim, s.vp(), W);
        JUNO_TRY(stack_upload(c, net, mo, &L->o));
        if (s.qk_norm) {
            JUNO_TRY(vector(p + "q.norm", s.dim, s.dp(), &L->q_norm));
            JUNO_TRY(vector(p + "k.norm", s.dim, s.dp(), &L->k_norm));
        }
        if (s.sink == SINK_LEARNED) JUNO_TRY(vector(p + "sink", H, H, &L->sinks));
        if (s.sink == SINK_ZERO) JUNO_TRY(stack_upload_f32(c, net, std::vector<float>((size_t)H, 0.f), &L->sinks));
        if (s.distance_bias) {
            std::vector<float> slopes;
            for (int h = 0; h < H; h++) slopes.push_back((float)std::exp2(-8.0 * (h + 1) / H));
            JUNO_TRY(stack_upload_f32(c, net, slopes, &L->slopes));
        }
        return JUNO_OK;
    }
    int hyper_connection(const std::string &p, HyperConnection *hc) {
        const int S = net->spec.streams;
        JUNO_TRY(vector(p + "in", S, S, &hc->in));
        JUNO_TRY(vector(p + "out", S, S, &hc->out));
        const StTensor *m;
        JUNO_TRY(get(p + "mix", {S, S}, &m));
        std::vector<float> v;
        for (int i = 0; i < S * S; i++) v.push_back(st_value(f, *m, i));
        return stack_upload_f32(c, net, v, &hc->mix);
    }
    int layer(const StackLayerSpec &s, StackLayerWeights *L) {
        const int W = net->spec.width, wp = net->spec.wp();
        const std::string p = "l" + std::to_string(s.source) + ".";
        JUNO_TRY(vector(p + "norm1", W, wp, &L->norm1_w, 1.f));
        JUNO_TRY(hyper_connection(p + "hc1.", &L->hc1));
        JUNO_TRY(mixer(p + "mix.", s.grouped, L));
        if (s.ff == 0) return JUNO_OK;
        JUNO_TRY(vector(p + "norm2", W, wp, &L->norm2_w, 1.f));
        JUNO_TRY(hyper_connection(p + "hc2.", &L->hc2));
        const StTensor *gate, *up;
        JUNO_TRY(get(p + "mlp.gate", {s.ff, W}, &gate));
        JUNO_TRY(get(p + "mlp.up", {s.ff, W}, &up));
        HostMat gu(net->dt, 2 * pad16(s.ff), wp);
        for (int i = 0; i < s.ff; i += 8) {
            gu.put(f, *gate, i, 0, std::min(8, s.ff - i), W, 2 * i, 0);
            gu.put(f, *up, i, 0, std::min(8, s.ff - i), W, 2 * i + 8, 0);
        }
        JUNO_TRY(stack_upload(c, net, gu, &L->gu));
        return matrix(p + "mlp.down", W, s.ff, &L->mdown);
    }
    int all() {
        const StackSpec &spec = net->spec;
        JUNO_TRY(matrix("embed", spec.vocab, spec.width, &net->embed));
        net->head = net->embed;
        JUNO_TRY(vector("final.norm", spec.width, spec.wp(), &net->final_w, 1.f));
        JUNO_TRY(stack_upload_f32(c, net, std::vector<float>((size_t)kMaxStreams, 1.f), &net->ones));
        net->layers.resize(spec.layers.size());
        for (size_t i = 0; i < spec.layers.size(); i++)
            if (spec.layers[i].weights_of < 0) JUNO_TRY(layer(spec.layers[i], &net->layers[i]));
        return JUNO_OK;
    }
};
}  // namespace

int desilorn_load(juno_ctx *c, const juno_safetensors *f, const StackSpec &spec, int dt, StackNet **out) {
    StackNet *net = new StackNet();
    net->spec = spec;
    net->dt = dt;
    Loader l{{c, f, net}};
    const int rc = l.all();
    if (rc != JUNO_OK) {
        stack_free(net);
        return rc;
    }
    *out = net;
    return JUNO_OK;
}

}  // namespace juno
