// The Vosotar design: a decoder-only stack of latent attention without positions and squared-ReLU feed-forwards, scalar RMS
// norms before and after every sublayer, a short causal convolution on the mixer's input, and an element-wise sigmoid gate on
// every sublayer's result.  This file knows the keys of its config.json and the names of its tensors; the mechanisms
// themselves are the generic ones of stack.cuh.
#include "stack_loader.cuh"

namespace juno {

int vosotar_spec(const Json &cfg, StackSpec *spec) {
    constexpr int kMax = 1 << 20;
    JUNO_TRY(cfg_int(&cfg, "width", "model", 1, 49152, &spec->width));
    JUNO_TRY(cfg_int(&cfg, "vocab", "model", 1, 1 << 24, &spec->vocab));
    JUNO_TRY(cfg_float(cfg.find("norm"), "eps", "norm", &spec->eps));
    JUNO_TRY(cfg_int(cfg.find("canon"), "taps", "canon", 1, 64, &spec->taps));
    const Json *layers = cfg.find("layers");
    JUNO_REQUIRE(layers && layers->kind == Json::ARRAY && !layers->arr.empty(), "config: layers must be a non-empty list");
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const Json &e = layers->arr[i];
        const std::string w = "layers[" + std::to_string(i) + "]";
        StackLayerSpec L;
        L.source = (int)i;
        std::string type, kind;
        JUNO_TRY(cfg_string(&e, "type", w.c_str(), &type));
        if (type != "latent_attention") {
            set_error("config: %s: mixer '%s' is not part of this design", w.c_str(), type.c_str());
            return JUNO_ERR_UNSUPPORTED;
        }
        const Json *m = e.find("mixer");
        const std::string wm = w + ".mixer";
        JUNO_TRY(cfg_int(m, "heads", wm.c_str(), 1, 65535, &L.mix.heads));
        JUNO_TRY(cfg_int(m, "dim", wm.c_str(), 1, kMax, &L.mix.dim));
        JUNO_TRY(cfg_int(m, "vdim", wm.c_str(), 1, kMax, &L.mix.vdim));
        JUNO_TRY(cfg_int(m, "q_rank", wm.c_str(), 1, kMax, &L.mix.q_rank));
        JUNO_TRY(cfg_int(m, "kv_rank", wm.c_str(), 1, 2048, &L.mix.kv_rank));
        JUNO_TRY(cfg_float(m, "scale", wm.c_str(), &L.mix.scale));
        JUNO_REQUIRE(L.mix.scale > 0.f, "config: %s.scale must be positive", wm.c_str());
        const Json *mlp = e.find("mlp");
        if (mlp && !mlp->is_null()) {
            JUNO_TRY(cfg_string(mlp, "kind", (w + ".mlp").c_str(), &kind));
            if (kind != "dense") {
                set_error("config: %s: feed-forward '%s' is not part of this design", w.c_str(), kind.c_str());
                return JUNO_ERR_UNSUPPORTED;
            }
            JUNO_TRY(cfg_int(mlp, "ff", (w + ".mlp").c_str(), 1, kMax, &L.ff));
        }
        const Json *src = e.find("weights_of");
        if (src && !src->is_null()) {
            int64_t j = 0;
            JUNO_REQUIRE(src->to_int(0, (int64_t)layers->arr.size() - 1, &j), "config: %s.weights_of must name a layer", w.c_str());
            L.weights_of = (int)j;
        }
        spec->layers.push_back(L);
    }
    for (size_t i = 0; i < spec->layers.size(); i++) {
        size_t j = i, hops = 0;
        while (spec->layers[j].weights_of >= 0 && hops++ < spec->layers.size()) j = (size_t)spec->layers[j].weights_of;
        const StackLayerSpec &L = spec->layers[i], &o = spec->layers[j];
        JUNO_REQUIRE(o.weights_of < 0, "config: layers[%zu].weights_of never reaches a layer with weights", i);
        JUNO_REQUIRE(o.ff == L.ff && o.mix.heads == L.mix.heads && o.mix.dim == L.mix.dim && o.mix.vdim == L.mix.vdim &&
                         o.mix.q_rank == L.mix.q_rank && o.mix.kv_rank == L.mix.kv_rank,
                     "config: layers[%zu] has other sizes than the layer whose weights it uses", i);
    }
    return JUNO_OK;
}

namespace {
struct Loader : StackLoader {
    int mixer(const std::string &p, const LatentMixerSpec &s, StackLayerWeights *L) {
        const int W = net->spec.width, wp = net->spec.wp(), dt = net->dt, H = s.heads;
        const StTensor *dq, *dkv, *g, *uq, *uk, *uv, *o;
        JUNO_TRY(get(p + "dq", {s.q_rank, W}, &dq));
        JUNO_TRY(get(p + "dkv", {s.kv_rank, W}, &dkv));
        JUNO_TRY(get(p + "g", {H, W}, &g));
        HostMat down(dt, s.down_rows(), wp);
        down.put(f, *dq, 0, 0, s.q_rank, W, 0, 0);
        down.put(f, *dkv, 0, 0, s.kv_rank, W, s.kv_col(), 0);
        down.put(f, *g, 0, 0, H, W, s.gate_col(), 0);
        JUNO_TRY(stack_upload(c, net, down, &L->down));
        JUNO_TRY(vector(p + "dq.norm", s.q_rank, s.qp(), &L->dq_norm));
        JUNO_TRY(vector(p + "dkv.norm", s.kv_rank, s.rp(), &L->dkv_norm));
        JUNO_TRY(get(p + "uq", {(int64_t)H * s.dim, s.q_rank}, &uq));
        JUNO_TRY(get(p + "uk", {(int64_t)H * s.dim, s.kv_rank}, &uk));
        JUNO_TRY(get(p + "uv", {(int64_t)H * s.vdim, s.kv_rank}, &uv));
        JUNO_TRY(get(p + "o", {W, (int64_t)H * s.vdim}, &o));
        HostMat muq(dt, H * s.dp(), s.qp()), mukv(dt, H * (s.dp() + s.vp()), s.rp()), mukt(dt, H * s.rp(), s.dp()), mo(dt, wp, H * s.vp());
        put_heads(&muq, *uq, H, s.dim, s.dp(), s.q_rank, 0);
        put_heads(&mukv, *uk, H, s.dim, s.dp(), s.kv_rank, 0);
        put_heads(&mukv, *uv, H, s.vdim, s.vp(), s.kv_rank, H * s.dp());
        put_head_columns(&mo, *o, H, s.vdim, s.vp(), W);
        for (int h = 0; h < H; h++) mukt.put_transposed(f, *uk, (int64_t)h * s.dim, 0, s.dim, s.kv_rank, h * s.rp(), 0);
        JUNO_TRY(stack_upload(c, net, muq, &L->uq));
        JUNO_TRY(stack_upload(c, net, mukv, &L->ukv));
        JUNO_TRY(stack_upload(c, net, mukt, &L->ukt));
        return stack_upload(c, net, mo, &L->o);
    }
    int layer(int i) {
        const StackSpec &spec = net->spec;
        const StackLayerSpec &s = spec.layers[(size_t)i];
        StackLayerWeights *L = &net->layers[(size_t)i];
        const std::string p = "l" + std::to_string(i) + ".";
        const int W = spec.width;
        JUNO_TRY(number(p + "norm1", &L->norm1));
        JUNO_TRY(number(p + "norm1b", &L->norm1b));
        JUNO_TRY(mixer(p + "mix.", s.mix, L));
        const StTensor *cw;
        JUNO_TRY(get(p + "canon1", {W, spec.taps}, &cw));
        HostMat conv(net->dt, spec.taps, spec.wp());
        conv.put_transposed(f, *cw, 0, 0, W, spec.taps, 0, 0);
        StackMat cm;
        JUNO_TRY(stack_upload(c, net, conv, &cm));
        L->conv = cm.w;
        JUNO_TRY(matrix(p + "rg1", W, W, &L->rg1));
        JUNO_TRY(vector(p + "rg1.b", W, spec.wp(), &L->rg1_b));
        if (s.ff == 0) return JUNO_OK;
        JUNO_TRY(number(p + "norm2", &L->norm2));
        JUNO_TRY(number(p + "norm2b", &L->norm2b));
        JUNO_TRY(matrix(p + "mlp.up", s.ff, W, &L->up));
        JUNO_TRY(matrix(p + "mlp.down", W, s.ff, &L->mdown));
        JUNO_TRY(matrix(p + "rg2", W, W, &L->rg2));
        return vector(p + "rg2.b", W, spec.wp(), &L->rg2_b);
    }
    int all() {
        const StackSpec &spec = net->spec;
        JUNO_TRY(matrix("embed", spec.vocab, spec.width, &net->embed));
        JUNO_TRY(number("embed.norm", &net->embed_norm));
        JUNO_TRY(number("final.norm", &net->final_norm));
        JUNO_TRY(matrix("head", spec.vocab, spec.width, &net->head));
        net->layers.resize(spec.layers.size());
        for (size_t i = 0; i < spec.layers.size(); i++)
            if (spec.layers[i].weights_of < 0) JUNO_TRY(layer((int)i));
        return JUNO_OK;
    }
};
}  // namespace

int vosotar_load(juno_ctx *c, const juno_safetensors *f, const StackSpec &spec, int dt, StackNet **out) {
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
