// Minimal JSON reader (host): model configurations and safetensors headers.  Objects keep their members in a map, numbers
// are doubles (exact for integers below 2^53), nesting is limited, and damaged text is an error, never an assumption.
#pragma once
#include <cmath>
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <map>
#include <string>
#include <vector>

namespace juno {

struct Json {
    enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::map<std::string, Json> obj;

    const Json *find(const char *key) const {
        if (kind != OBJECT) return nullptr;
        auto it = obj.find(key);
        return it == obj.end() ? nullptr : &it->second;
    }
    bool is_null() const { return kind == NUL; }
    // A whole number within [lo, hi]; false otherwise.
    bool to_int(int64_t lo, int64_t hi, int64_t *out) const {
        if (kind != NUMBER || num != std::floor(num) || num < (double)lo || num > (double)hi) return false;
        *out = (int64_t)num;
        return true;
    }
};

class JsonParser {
  public:
    JsonParser(const char *text, size_t n) : p_(text), end_(text + n) {}
    bool parse(Json *out) {
        if (!value(out, 0)) return false;
        space();
        return p_ == end_;
    }

  private:
    const char *p_, *end_;
    void space() {
        while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) p_++;
    }
    bool word(const char *w) {
        const size_t n = strlen(w);
        if ((size_t)(end_ - p_) < n || memcmp(p_, w, n) != 0) return false;
        p_ += n;
        return true;
    }
    static void utf8(std::string &s, uint32_t c) {
        if (c < 0x80) {
            s += (char)c;
        } else if (c < 0x800) {
            s += (char)(0xC0 | (c >> 6));
            s += (char)(0x80 | (c & 63));
        } else if (c < 0x10000) {
            s += (char)(0xE0 | (c >> 12));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        } else {
            s += (char)(0xF0 | (c >> 18));
            s += (char)(0x80 | ((c >> 12) & 63));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        }
    }
    bool hex4(uint32_t *v) {
        if (end_ - p_ < 4) return false;
        *v = 0;
        for (int i = 0; i < 4; i++, p_++) {
            const char c = *p_;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return false;
            *v = *v * 16 + (uint32_t)d;
        }
        return true;
    }
    bool string(std::string *out) {
        if (p_ >= end_ || *p_ != '"') return false;
        p_++;
        out->clear();
        while (p_ < end_ && *p_ != '"') {
            if (*p_ != '\\') {
                *out += *p_++;
                continue;
            }
            if (++p_ >= end_) return false;
            const char c = *p_++;
            switch (c) {
            case '"': case '\\': case '/': *out += c; break;
            case 'b': *out += '\b'; break;
            case 'f': *out += '\f'; break;
            case 'n': *out += '\n'; break;
            case 'r': *out += '\r'; break;
            case 't': *out += '\t'; break;
            case 'u': {
                uint32_t v, lo;
                if (!hex4(&v)) return false;
                if (v >= 0xD800 && v < 0xDC00) {  // surrogate pair
                    if (!word("\\u") || !hex4(&lo) || lo < 0xDC00 || lo > 0xDFFF) return false;
                    v = 0x10000 + ((v - 0xD800) << 10) + (lo - 0xDC00);
                }
                utf8(*out, v);
                break;
            }
            default: return false;
            }
        }
        if (p_ >= end_) return false;
        p_++;
        return true;
    }
    bool number(double *out) {
        const char *s = p_;
        if (p_ < end_ && *p_ == '-') p_++;
        while (p_ < end_ && ((*p_ >= '0' && *p_ <= '9') || *p_ == '.' || *p_ == 'e' || *p_ == 'E' || *p_ == '+' || *p_ == '-')) p_++;
        const std::string t(s, p_);
        char *stop = nullptr;
        *out = strtod(t.c_str(), &stop);
        return !t.empty() && stop == t.c_str() + t.size() && std::isfinite(*out);
    }
    bool value(Json *out, int depth) {
        if (depth > 64) return false;
        space();
        if (p_ >= end_) return false;
        if (*p_ == '{') {
            p_++;
            out->kind = Json::OBJECT;
            space();
            if (p_ < end_ && *p_ == '}') return p_++, true;
            for (;;) {
                std::string key;
                space();
                if (!string(&key)) return false;
                space();
                if (p_ >= end_ || *p_++ != ':') return false;
                Json v;
                if (!value(&v, depth + 1)) return false;
                out->obj[key] = std::move(v);
                space();
                if (p_ >= end_) return false;
                if (*p_ == ',') {
                    p_++;
                    continue;
                }
                return *p_++ == '}';
            }
        }
        if (*p_ == '[') {
            p_++;
            out->kind = Json::ARRAY;
            space();
            if (p_ < end_ && *p_ == ']') return p_++, true;
            for (;;) {
                Json v;
                if (!value(&v, depth + 1)) return false;
                out->arr.push_back(std::move(v));
                space();
                if (p_ >= end_) return false;
                if (*p_ == ',') {
                    p_++;
                    continue;
                }
                return *p_++ == ']';
            }
        }
        if (*p_ == '"') {
            out->kind = Json::STRING;
            return string(&out->str);
        }
        if (word("true")) return out->kind = Json::BOOL, out->b = true, true;
        if (word("false")) return out->kind = Json::BOOL, out->b = false, true;
        if (word("null")) return out->kind = Json::NUL, true;
        out->kind = Json::NUMBER;
        return number(&out->num);
    }
};

}  // namespace juno
