// safetensors container on the host: an 8-byte little-endian header length, a JSON object name -> {dtype, shape,
// data_offsets}, then the data.  Like the GGUF reader this is host code over a read-only mapping and trusts nothing: every
// length, shape and offset is checked against the file before a tensor is handed out.
#include "safetensors.cuh"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <algorithm>
#include <cerrno>
#include <climits>
#include <cstring>

#include "json.hpp"

namespace juno {

static int st_check(juno_safetensors *s) {
    if (!s) {
        set_error("safetensors handle is null");
        return JUNO_ERR_INVALID_ARG;
    }
    if (s->magic != kMagicSafetensors) {
        set_error("safetensors file is closed");
        return JUNO_ERR_CLOSED;
    }
    return JUNO_OK;
}

static void st_release(juno_safetensors *s) {
    if (s->base) munmap(const_cast<uint8_t *>(s->base), (size_t)s->size);
    if (s->fd >= 0) close(s->fd);
    s->base = nullptr;
    s->fd = -1;
}

static int st_dtype(const std::string &d, int *elem) {
    if (d == "BF16") return *elem = 2, ST_BF16;
    if (d == "F16") return *elem = 2, ST_F16;
    if (d == "F32") return *elem = 4, ST_F32;
    if (d == "I32") return *elem = 4, ST_I32;
    *elem = d == "F64" || d == "I64" || d == "U64" ? 8 : d == "I16" || d == "U16" ? 2 : d == "U32" ? 4 : 1;
    return ST_OTHER;
}

int read_text_file(const std::string &path, std::string *out) {
    FILE *f = fopen(path.c_str(), "rb");
    JUNO_REQUIRE(f, "cannot open %s: %s", path.c_str(), strerror(errno));
    out->clear();
    char buf[65536];
    size_t n;
    while ((n = fread(buf, 1, sizeof(buf), f)) > 0) out->append(buf, n);
    const bool bad = ferror(f) != 0;
    fclose(f);
    JUNO_REQUIRE(!bad, "cannot read %s", path.c_str());
    return JUNO_OK;
}

}  // namespace juno

using namespace juno;

extern "C" {

int juno_safetensors_open(const char *path, juno_safetensors **out) {
    JUNO_REQUIRE(path && out, "path or out is null");
    juno_safetensors *s = new juno_safetensors();
    auto fail = [&](int rc) {
        st_release(s);
        delete s;
        return rc;
    };
    s->fd = open(path, O_RDONLY | O_CLOEXEC);
    if (s->fd < 0) {
        set_error("cannot open %s: %s", path, strerror(errno));
        return fail(JUNO_ERR_INVALID_ARG);
    }
    struct stat sb;
    if (fstat(s->fd, &sb) != 0 || sb.st_size < 8) {
        set_error("%s is too short for a safetensors file", path);
        return fail(JUNO_ERR_INVALID_ARG);
    }
    s->size = sb.st_size;
    void *m = mmap(nullptr, (size_t)s->size, PROT_READ, MAP_PRIVATE, s->fd, 0);
    if (m == MAP_FAILED) {
        set_error("cannot map %s: %s", path, strerror(errno));
        return fail(JUNO_ERR_INVALID_ARG);
    }
    s->base = static_cast<const uint8_t *>(m);
    uint64_t hlen = 0;
    memcpy(&hlen, s->base, 8);
    Json h;
    if (hlen > (uint64_t)(s->size - 8) || !JsonParser(reinterpret_cast<const char *>(s->base + 8), (size_t)hlen).parse(&h) ||
        h.kind != Json::OBJECT) {
        set_error("%s: the safetensors header is damaged", path);
        return fail(JUNO_ERR_INVALID_ARG);
    }
    const int64_t data0 = 8 + (int64_t)hlen, data_len = s->size - data0;
    for (const auto &kv : h.obj) {
        if (kv.first == "__metadata__") continue;
        StTensor t;
        t.name = kv.first;
        const Json *dt = kv.second.find("dtype"), *sh = kv.second.find("shape"), *of = kv.second.find("data_offsets");
        bool ok = dt && dt->kind == Json::STRING && sh && sh->kind == Json::ARRAY && of && of->kind == Json::ARRAY && of->arr.size() == 2;
        int elem = 1;
        if (ok) t.dtype = st_dtype(dt->str, &elem);
        if (ok)
            for (const Json &d : sh->arr) {
                int64_t v = 0;
                if (!d.to_int(0, 1ll << 48, &v) || (v && t.nelems > (1ll << 48) / v)) {
                    ok = false;
                    break;
                }
                t.shape.push_back(v);
                t.nelems *= v;
            }
        int64_t a = 0, b = 0;
        ok = ok && of->arr[0].to_int(0, data_len, &a) && of->arr[1].to_int(a, data_len, &b);
        if (ok && t.dtype != ST_OTHER) ok = b - a == t.nelems * elem;
        if (!ok) {
            set_error("%s: the header entry of tensor %s is damaged or runs past the end of the file", path, t.name.c_str());
            return fail(JUNO_ERR_INVALID_ARG);
        }
        t.offset = data0 + a;
        t.nbytes = b - a;
        s->tensors.push_back(std::move(t));
    }
    std::sort(s->tensors.begin(), s->tensors.end(), [](const StTensor &x, const StTensor &y) { return x.offset < y.offset || (x.offset == y.offset && x.name < y.name); });
    for (size_t i = 0; i < s->tensors.size(); i++) s->by_name[s->tensors[i].name] = i;
    *out = s;
    return JUNO_OK;
}

int juno_safetensors_close(juno_safetensors *s) {
    JUNO_TRY(st_check(s));
    st_release(s);
    s->magic = 0;
    delete s;
    return JUNO_OK;
}

int juno_safetensors_count(juno_safetensors *s, int64_t *n_tensors) {
    JUNO_TRY(st_check(s));
    JUNO_REQUIRE(n_tensors, "out is null");
    *n_tensors = (int64_t)s->tensors.size();
    return JUNO_OK;
}

int juno_safetensors_name(juno_safetensors *s, int64_t index, char *buf, int32_t buf_len) {
    JUNO_TRY(st_check(s));
    JUNO_REQUIRE(buf && buf_len > 0, "buf is null or empty");
    JUNO_REQUIRE(index >= 0 && index < (int64_t)s->tensors.size(), "tensor index %lld out of range", (long long)index);
    const std::string &n = s->tensors[(size_t)index].name;
    JUNO_REQUIRE((size_t)buf_len > n.size(), "buffer of %d bytes is too small for a %zu-byte tensor name", buf_len, n.size());
    memcpy(buf, n.c_str(), n.size() + 1);
    return JUNO_OK;
}

int juno_safetensors_tensor(juno_safetensors *s, const char *name, int32_t *dtype, int32_t *n_dims, int64_t *dims8, const void **data,
                            int64_t *n_bytes) {
    JUNO_TRY(st_check(s));
    JUNO_REQUIRE(name, "name is null");
    const StTensor *t = s->find(name);
    JUNO_REQUIRE(t, "Tensor not found: %s  (available: %zu tensors)", name, s->tensors.size());
    JUNO_REQUIRE(t->shape.size() <= 8, "tensor %s has %zu dimensions", name, t->shape.size());
    if (dtype) *dtype = t->dtype;
    if (n_dims) *n_dims = (int32_t)t->shape.size();
    if (dims8)
        for (size_t d = 0; d < 8; d++) dims8[d] = d < t->shape.size() ? t->shape[d] : 1;
    if (data) *data = s->base + t->offset;
    if (n_bytes) *n_bytes = t->nbytes;
    return JUNO_OK;
}

}  // extern "C"
