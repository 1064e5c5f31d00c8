// safetensors files: an 8-byte little-endian header length, that many bytes of JSON
// (name -> {"dtype", "shape", "data_offsets"}, and an optional "__metadata__" object of strings),
// then the tensors' bytes.  The loader reads one tensor at a time and uploads it as dense bf16 or
// f32 rows; the header is checked against the file first.
#include <cerrno>
#include <cstdlib>
#include <cstring>
#include <fstream>
#include <memory>

#include "tlc_internal.h"

extern "C" int32_t tlc_model_create(tlc_ctx *, tlc_model **);
extern "C" int32_t tlc_model_add(tlc_model *, const char *, tlc_qtensor *);
extern "C" int32_t tlc_model_destroy(tlc_model *);

namespace {

struct Entry {
    std::string name, dtype;
    std::vector<int64_t> shape;
    uint64_t begin = 0, end = 0;
    bool has_offsets = false, has_shape = false;
};

// The part of JSON a header uses: objects, arrays, strings with escapes, integers; anything else
// is skipped as a balanced value.
struct Json {
    const char *p, *end;
    bool ok = true;
    int depth = 0;  // of skip()

    void space() {
        while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
    }
    bool eat(char c) {
        space();
        if (p < end && *p == c) {
            p++;
            return true;
        }
        return false;
    }
    void need(char c) {
        if (!eat(c)) ok = false;
    }
    static void put_utf8(std::string &s, uint32_t c) {
        if (c < 0x80) {
            s += (char)c;
        } else if (c < 0x800) {
            s += (char)(0xC0 | (c >> 6));
            s += (char)(0x80 | (c & 0x3F));
        } else if (c < 0x10000) {
            s += (char)(0xE0 | (c >> 12));
            s += (char)(0x80 | ((c >> 6) & 0x3F));
            s += (char)(0x80 | (c & 0x3F));
        } else {
            s += (char)(0xF0 | (c >> 18));
            s += (char)(0x80 | ((c >> 12) & 0x3F));
            s += (char)(0x80 | ((c >> 6) & 0x3F));
            s += (char)(0x80 | (c & 0x3F));
        }
    }
    bool hex4(uint32_t &v) {
        v = 0;
        for (int i = 0; i < 4; i++, p++) {
            if (p >= end) return false;
            const char c = *p;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return false;
            v = 16 * v + (uint32_t)d;
        }
        return true;
    }
    std::string string() {
        std::string s;
        space();
        if (p >= end || *p != '"') {
            ok = false;
            return s;
        }
        for (p++; p < end && *p != '"'; p++) {
            if (*p != '\\') {
                s += *p;
                continue;
            }
            if (++p >= end) break;
            switch (*p) {
                case 'n': s += '\n'; break;
                case 't': s += '\t'; break;
                case 'r': s += '\r'; break;
                case 'b': s += '\b'; break;
                case 'f': s += '\f'; break;
                case 'u': {
                    p++;
                    uint32_t c = 0, lo = 0;
                    if (!hex4(c)) {
                        ok = false;
                        return s;
                    }
                    if (c >= 0xD800 && c < 0xDC00) {  // the first half of a pair
                        if (end - p < 6 || p[0] != '\\' || p[1] != 'u') {
                            ok = false;
                            return s;
                        }
                        p += 2;
                        if (!hex4(lo) || lo < 0xDC00 || lo > 0xDFFF) {
                            ok = false;
                            return s;
                        }
                        c = 0x10000 + ((c - 0xD800) << 10) + (lo - 0xDC00);
                    }
                    put_utf8(s, c);
                    p--;  // the loop steps past the last digit
                    break;
                }
                default: s += *p;
            }
        }
        if (p >= end)
            ok = false;
        else
            p++;
        return s;
    }
    uint64_t integer() {
        space();
        uint64_t v = 0;
        if (p >= end || *p < '0' || *p > '9') ok = false;
        for (; ok && p < end && *p >= '0' && *p <= '9'; p++) {
            if (v > (UINT64_MAX - 9) / 10) {
                ok = false;
                break;
            }
            v = 10 * v + (uint64_t)(*p - '0');
        }
        return v;
    }
    void skip() {
        space();
        if (p >= end || ++depth > 64) {
            ok = false;
            return;
        }
        if (*p == '"') {
            string();
        } else if (*p == '{' || *p == '[') {
            const char close = *p == '{' ? '}' : ']';
            const bool object = *p == '{';
            p++;
            if (!eat(close)) {
                do {
                    if (object) {
                        string();
                        need(':');
                    }
                    if (ok) skip();
                } while (ok && eat(','));
                if (ok) need(close);
            }
        } else {
            while (p < end && *p != ',' && *p != '}' && *p != ']') p++;
        }
        depth--;
    }
    template <typename F>
    void array(F each) {
        need('[');
        if (ok && eat(']')) return;
        do each();
        while (ok && eat(','));
        if (ok) need(']');
    }
    template <typename F>
    void object(F each) {  // each(key) consumes the value
        need('{');
        if (ok && eat('}')) return;
        do {
            const std::string key = string();
            if (ok) need(':');
            if (ok) each(key);
        } while (ok && eat(','));
        if (ok) need('}');
    }
};

int32_t parse_header(const char *path, const std::string &text, uint64_t data_bytes, std::vector<Entry> &out) {
    Json j{text.data(), text.data() + text.size()};
    j.object([&](const std::string &name) {
        if (name == "__metadata__") {
            j.skip();
            return;
        }
        Entry e;
        e.name = name;
        j.object([&](const std::string &key) {
            if (key == "dtype") {
                e.dtype = j.string();
            } else if (key == "shape") {
                e.has_shape = true;
                j.array([&] { e.shape.push_back((int64_t)j.integer()); });
            } else if (key == "data_offsets") {
                uint64_t v[2] = {0, 0};
                int n = 0;
                j.array([&] {
                    const uint64_t x = j.integer();
                    if (n < 2) v[n] = x;
                    n++;
                });
                e.begin = v[0];
                e.end = v[1];
                e.has_offsets = n == 2;
            } else {
                j.skip();
            }
        });
        out.push_back(std::move(e));
    });
    TLC_REQUIRE(j.ok, TLC_ERR_LOAD, "'%s': the safetensors header is not valid JSON", path);
    for (const Entry &e : out) {
        TLC_REQUIRE(e.has_offsets && e.has_shape, TLC_ERR_LOAD, "'%s': tensor '%s' has no shape or no offsets", path, e.name.c_str());
        TLC_REQUIRE(e.begin <= e.end && e.end <= data_bytes, TLC_ERR_LOAD, "'%s': tensor '%s' lies outside the file", path,
                    e.name.c_str());
        const uint64_t elem = e.dtype == "F32" ? 4 : e.dtype == "BF16" || e.dtype == "F16" ? 2 : 0;
        TLC_REQUIRE(elem, TLC_ERR_LOAD, "'%s': tensor '%s' has dtype %s (supported: F32, F16, BF16)", path, e.name.c_str(),
                    e.dtype.c_str());
        uint64_t n = 1;
        for (int64_t s : e.shape) {
            TLC_REQUIRE(s > 0 && n <= data_bytes / (uint64_t)s, TLC_ERR_LOAD, "'%s': tensor '%s' has a bad shape", path, e.name.c_str());
            n *= (uint64_t)s;
        }
        TLC_REQUIRE(n * elem == e.end - e.begin, TLC_ERR_LOAD, "'%s': tensor '%s' has %llu bytes, its shape needs %llu", path,
                    e.name.c_str(), (unsigned long long)(e.end - e.begin), (unsigned long long)(n * elem));
    }
    return TLC_OK;
}

}  // namespace

extern "C" int32_t tlc_model_load_safetensors(tlc_ctx *ctx, const char *path, int32_t store_type, tlc_model **out) {
    if (int32_t rc = tlc_enter(ctx)) return rc;
    TLC_REQUIRE(path && out, TLC_ERR_INVALID_OPERATION, "load_safetensors: null pointer");
    *out = nullptr;
    std::ifstream f(path, std::ios::binary | std::ios::ate);
    TLC_REQUIRE(f.good(), TLC_ERR_LOAD, "Failed to open safetensors file '%s': %s", path, strerror(errno));
    const uint64_t size = (uint64_t)f.tellg();
    uint8_t len8[8];
    f.seekg(0);
    f.read(reinterpret_cast<char *>(len8), 8);
    uint64_t len = 0;
    for (int i = 0; i < 8; i++) len |= (uint64_t)len8[i] << (8 * i);
    TLC_REQUIRE((bool)f && size >= 8 && len <= size - 8, TLC_ERR_LOAD, "'%s' is not a safetensors file", path);
    std::string text(len, '\0');
    f.read(&text[0], (std::streamsize)len);
    TLC_REQUIRE((bool)f, TLC_ERR_LOAD, "'%s': short read on the header", path);
    std::vector<Entry> entries;
    if (int32_t rc = parse_header(path, text, size - 8 - len, entries)) return rc;

    tlc_model *raw = nullptr;
    if (int32_t rc = tlc_model_create(ctx, &raw)) return rc;
    std::unique_ptr<tlc_model, int32_t (*)(tlc_model *)> model(raw, tlc_model_destroy);
    std::vector<char> host;
    for (const Entry &e : entries) {
        host.resize(e.end - e.begin);
        f.seekg((std::streamoff)(8 + len + e.begin));
        f.read(host.data(), (std::streamsize)host.size());
        TLC_REQUIRE((bool)f, TLC_ERR_LOAD, "'%s': short read on tensor '%s'", path, e.name.c_str());
        int64_t rows = 1;
        for (size_t i = 0; i + 1 < e.shape.size(); i++) rows *= e.shape[i];
        const int64_t cols = e.shape.empty() ? 1 : e.shape.back();
        const int32_t src = e.dtype == "F32" ? TLC_TYPE_F32 : e.dtype == "F16" ? TLC_TYPE_F16 : TLC_TYPE_BF16;
        tlc_qtensor *qt = nullptr;
        if (int32_t rc = tlc_qtensor_create_dense(ctx, src, store_type, rows, cols, host.data(), host.size(), &qt)) return rc;
        if (int32_t rc = tlc_model_add(model.get(), e.name.c_str(), qt)) {
            tlc_qtensor_destroy(qt);
            return rc;
        }
    }
    *out = model.release();
    return TLC_OK;
}
