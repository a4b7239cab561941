// Model registry: which files open as which model.  A folder holds config.json (its "architecture" names the design) and
// model.safetensors; a single file is a GGUF file of the quantised LLaMA family.  Every entry ends in the same juno_model, so
// sequences, steps, prefill and the greedy loop are the same calls for all of them.
#include <sys/stat.h>

#include <cstring>

#include "json.hpp"
#include "model.cuh"
#include "stack.cuh"

namespace juno {

struct Design {
    const char *architecture;
    int (*spec)(const Json &cfg, StackSpec *out);
    int (*load)(juno_ctx *c, const juno_safetensors *f, const StackSpec &spec, int dt, StackNet **out);
};
static const Design kDesigns[] = {
    {"Vosotar", vosotar_spec, vosotar_load},
    {"Desilorn", desilorn_spec, desilorn_load},
};

static int open_folder(juno_ctx *c, const std::string &dir, const juno_open_opts &o, juno_model **out) {
    std::string text;
    JUNO_TRY(read_text_file(dir + "/config.json", &text));
    Json cfg;
    JUNO_REQUIRE(JsonParser(text.data(), text.size()).parse(&cfg) && cfg.kind == Json::OBJECT, "%s/config.json is not a JSON object", dir.c_str());
    const Json *a = cfg.find("architecture");
    JUNO_REQUIRE(a && a->kind == Json::STRING, "%s/config.json names no architecture", dir.c_str());
    const Design *d = nullptr;
    for (const Design &e : kDesigns)
        if (a->str == e.architecture) d = &e;
    if (!d) {
        set_error("architecture '%s' is not in the model registry", a->str.c_str());
        return JUNO_ERR_UNSUPPORTED;
    }
    StackSpec spec;
    JUNO_TRY(d->spec(cfg, &spec));
    juno_safetensors *f = nullptr;
    JUNO_TRY(juno_safetensors_open((dir + "/model.safetensors").c_str(), &f));
    StackNet *net = nullptr;
    const int rc = d->load(c, f, spec, o.dtype == JUNO_DTYPE_F32 ? DT_F32 : DT_BF16, &net);
    juno_safetensors_close(f);
    JUNO_TRY(rc);
    return model_from_stack(c, net, d->architecture, o, out);
}

static int open_gguf(juno_ctx *c, const char *path, const juno_open_opts &o, juno_model **out) {
    juno_gguf *g = nullptr;
    JUNO_TRY(juno_gguf_open(path, &g));
    juno_model_cfg cfg;
    memset(&cfg, 0, sizeof(cfg));
    cfg.struct_size = (int32_t)sizeof(cfg);
    cfg.max_batch = o.max_batch;
    cfg.max_seqs = o.max_seqs;
    cfg.max_ctx = o.max_ctx;
    cfg.kv_dtype = o.dtype == JUNO_DTYPE_F32 ? 1 : 0;
    cfg.tp_world = 1;
    juno_model *m = nullptr;
    int rc = juno_gguf_model_cfg(g, &cfg);
    if (rc == JUNO_OK) rc = juno_model_create(c, &cfg, &m);
    if (rc == JUNO_OK) rc = juno_model_load_gguf(m, g);
    if (rc == JUNO_OK) rc = juno_model_finalize(m);
    if (rc != JUNO_OK && m) juno_model_free(m);
    juno_gguf_close(g);
    if (rc == JUNO_OK) *out = m;
    return rc;
}

}  // namespace juno

using namespace juno;

extern "C" int juno_model_open(juno_ctx *c, const char *path, const juno_open_opts *opts, juno_model **out) {
    JUNO_TRY(ctx_check(c));
    JUNO_REQUIRE(path && opts && out, "null argument");
    JUNO_REQUIRE(opts->struct_size == (int32_t)sizeof(juno_open_opts), "juno_open_opts.struct_size is %d, expected %d", opts->struct_size,
                 (int)sizeof(juno_open_opts));
    JUNO_REQUIRE(opts->dtype == JUNO_DTYPE_DEFAULT || opts->dtype == JUNO_DTYPE_F32, "dtype %d", opts->dtype);
    JUNO_REQUIRE(opts->max_batch >= 1 && opts->max_batch <= 1024 && opts->max_seqs >= 1 && opts->max_ctx >= 1 && opts->max_rows >= 0 && opts->max_rows <= 32768,
                 "max_batch/max_seqs/max_ctx/max_rows out of range");
    struct stat sb;
    JUNO_REQUIRE(stat(path, &sb) == 0, "cannot open %s: %s", path, strerror(errno));
    std::lock_guard<std::recursive_mutex> lk(c->mu);
    DeviceGuard g(c->device);
    return S_ISDIR(sb.st_mode) ? open_folder(c, path, *opts, out) : open_gguf(c, path, *opts, out);
}
