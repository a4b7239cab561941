// Model folders (config.json + model.safetensors) on the host: a mapped reader for the safetensors container.
#pragma once
#include <map>
#include <string>
#include <vector>

#include "common.cuh"

namespace juno {

constexpr uint32_t kMagicSafetensors = 0x4A535446;  // "JSTF"

enum StDtype { ST_BF16 = 0, ST_F16 = 1, ST_F32 = 2, ST_I32 = 3, ST_OTHER = -1 };

struct StTensor {
    std::string name;
    int dtype = ST_OTHER;
    std::vector<int64_t> shape;  // outermost first, as the header writes it; empty = a single number
    int64_t nelems = 1, offset = 0, nbytes = 0;  // offset from the start of the file
};

}  // namespace juno

struct juno_safetensors {
    uint32_t magic = juno::kMagicSafetensors;
    int fd = -1;
    const uint8_t *base = nullptr;
    int64_t size = 0;
    std::vector<juno::StTensor> tensors;  // in order of their data
    std::map<std::string, size_t> by_name;

    const juno::StTensor *find(const std::string &name) const {
        auto it = by_name.find(name);
        return it == by_name.end() ? nullptr : &tensors[it->second];
    }
};

namespace juno {
// Whole text file; JUNO_ERR_INVALID_ARG when it cannot be read.
int read_text_file(const std::string &path, std::string *out);
}  // namespace juno
