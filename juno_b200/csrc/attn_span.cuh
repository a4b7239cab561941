// Which earlier positions a position attends: all of them, the last `window` (itself included), or those of its own chunk of
// `chunk` positions (counted from position 0 of the sequence).  The first position seen never decreases with the position.
#pragma once

namespace juno {

struct KeySpan {
    int window = 0, chunk = 0;  // 0: no limit of that kind
#if defined(__CUDACC__)
    __host__ __device__ __forceinline__
#endif
    int first(int pos) const {
        int lo = 0;
        if (window > 0 && pos >= window) lo = pos - window + 1;
        if (chunk > 0) {
            const int c = pos - pos % chunk;
            if (c > lo) lo = c;
        }
        return lo;
    }
    // most positions that any position below `len` sees
    int longest(int len) const {
        if (window > 0 && window < len) len = window;
        if (chunk > 0 && chunk < len) len = chunk;
        return len;
    }
};

}  // namespace juno
