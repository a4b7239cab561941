// See stack_loader.cuh.
#include "stack_loader.cuh"

namespace juno {

int cfg_int(const Json *o, const char *key, const char *where, int lo, int hi, int *out) {
    const Json *v = o ? o->find(key) : nullptr;
    int64_t t = 0;
    JUNO_REQUIRE(v && v->to_int(lo, hi, &t), "config: %s.%s must be a whole number in [%d, %d]", where, key, lo, hi);
    *out = (int)t;
    return JUNO_OK;
}
int cfg_float(const Json *o, const char *key, const char *where, float *out) {
    const Json *v = o ? o->find(key) : nullptr;
    JUNO_REQUIRE(v && v->kind == Json::NUMBER, "config: %s.%s must be a number", where, key);
    *out = (float)v->num;
    return JUNO_OK;
}
int cfg_string(const Json *o, const char *key, const char *where, std::string *out) {
    const Json *v = o ? o->find(key) : nullptr;
    JUNO_REQUIRE(v && v->kind == Json::STRING, "config: %s.%s is missing", where, key);
    *out = v->str;
    return JUNO_OK;
}

int StackLoader::get(const std::string &name, std::vector<int64_t> shape, const StTensor **out) {
    const StTensor *t = f->find(name);
    JUNO_REQUIRE(t, "tensor %s is missing", name.c_str());
    JUNO_REQUIRE(t->dtype == ST_BF16 || t->dtype == ST_F32, "tensor %s: weights must be BF16 or F32", name.c_str());
    const bool ok = shape.empty() ? t->nelems == 1 : t->shape == shape;
    if (!ok) {
        std::string have, want;
        for (int64_t d : t->shape) have += (have.empty() ? "" : "x") + std::to_string(d);
        for (int64_t d : shape) want += (want.empty() ? "" : "x") + std::to_string(d);
        set_error("tensor %s has shape [%s], expected [%s]", name.c_str(), have.c_str(), want.c_str());
        return JUNO_ERR_INVALID_ARG;
    }
    *out = t;
    return JUNO_OK;
}
int StackLoader::number(const std::string &name, float *out) {
    const StTensor *t;
    JUNO_TRY(get(name, {}, &t));
    *out = st_value(f, *t, 0);
    return JUNO_OK;
}
int StackLoader::vector(const std::string &name, int n, int padded, float **out, float offset) {
    const StTensor *t;
    JUNO_TRY(get(name, {n}, &t));
    std::vector<float> v((size_t)padded, 0.f);
    for (int i = 0; i < n; i++) v[(size_t)i] = offset + st_value(f, *t, i);
    return stack_upload_f32(c, net, v, out);
}
int StackLoader::matrix(const std::string &name, int rows, int cols, StackMat *out) {
    const StTensor *t;
    JUNO_TRY(get(name, {rows, cols}, &t));
    HostMat m(net->dt, pad16(rows), pad16(cols));
    m.put(f, *t, 0, 0, rows, cols, 0, 0);
    return stack_upload(c, net, m, out);
}
void StackLoader::put_heads(HostMat *m, const StTensor &t, int heads, int size, int padded, int cols, int row0) {
    for (int h = 0; h < heads; h++) m->put(f, t, (int64_t)h * size, 0, size, cols, row0 + h * padded, 0);
}
void StackLoader::put_head_columns(HostMat *m, const StTensor &t, int heads, int size, int padded, int rows) {
    for (int h = 0; h < heads; h++) m->put(f, t, 0, (int64_t)h * size, rows, size, 0, h * padded);
}

}  // namespace juno
