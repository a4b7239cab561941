// What the configuration readers and tensor loaders of layer-stack designs share.
#pragma once
#include "json.hpp"
#include "stack.cuh"

namespace juno {

// A member of a JSON object as a number within bounds, or an error that names its place.
int cfg_int(const Json *o, const char *key, const char *where, int lo, int hi, int *out);
int cfg_float(const Json *o, const char *key, const char *where, float *out);
// The "type" of a layer / the "kind" of a feed-forward.
int cfg_string(const Json *o, const char *key, const char *where, std::string *out);

struct StackLoader {
    juno_ctx *c;
    const juno_safetensors *f;
    StackNet *net;

    // The tensor of that name with exactly that shape (a single number: one element, any rank).
    int get(const std::string &name, std::vector<int64_t> shape, const StTensor **out);
    int number(const std::string &name, float *out);
    // `offset` is added to every element (norm weights stored as their distance from one)
    int vector(const std::string &name, int n, int padded, float **out, float offset = 0.f);
    int matrix(const std::string &name, int rows, int cols, StackMat *out);
    // rows of heads, each padded on its own: head h of `t` at row row0 + h * padded of `m`
    void put_heads(HostMat *m, const StTensor &t, int heads, int size, int padded, int cols, int row0);
    // columns of heads, each padded on its own
    void put_head_columns(HostMat *m, const StTensor &t, int heads, int size, int padded, int rows);
};

}  // namespace juno
