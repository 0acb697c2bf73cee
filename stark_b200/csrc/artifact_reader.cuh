// Host-side reading of a model directory: a small JSON reader, the bounded safetensors header reader (header <= 100 MB,
// crates/stark-engine/src/parameters/safetensors_metadata.rs:117-132) and tensor look-up by name, type and shape.
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <map>
#include <set>
#include <string>
#include <vector>

#include "common.cuh"

namespace sb {

// ---------------------------------------------------------------------------------------- a small JSON reader
struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0.0;
    bool integral = false;
    std::string str;
    std::vector<Json> items;
    std::vector<std::pair<std::string, Json>> fields;

    const Json *get(const char *name) const {
        if (kind != Object) return nullptr;
        for (auto &f : fields)
            if (f.first == name) return &f.second;
        return nullptr;
    }
    bool is_null() const { return kind == Null; }
};

struct JsonParser {
    const char *p, *end;
    int depth = 0;
    bool fail = false;

    void skip() {
        while (p < end && (*p == ' ' || *p == '\n' || *p == '\r' || *p == '\t')) ++p;
    }
    bool literal(const char *word) {
        const size_t n = strlen(word);
        if ((size_t)(end - p) < n || memcmp(p, word, n) != 0) return false;
        p += n;
        return true;
    }
    bool string(std::string &out) {
        if (p >= end || *p != '"') return false;
        ++p;
        while (p < end && *p != '"') {
            if (*p == '\\') {
                if (++p >= end) return false;
                switch (*p) {
                    case '"': out += '"'; break;
                    case '\\': out += '\\'; break;
                    case '/': out += '/'; break;
                    case 'b': out += '\b'; break;
                    case 'f': out += '\f'; break;
                    case 'n': out += '\n'; break;
                    case 'r': out += '\r'; break;
                    case 't': out += '\t'; break;
                    case 'u': {
                        if (end - p < 5) return false;
                        unsigned code = 0;
                        for (int i = 1; i <= 4; ++i) {
                            const char c = p[i];
                            code <<= 4;
                            if (c >= '0' && c <= '9') code |= (unsigned)(c - '0');
                            else if (c >= 'a' && c <= 'f') code |= (unsigned)(c - 'a' + 10);
                            else if (c >= 'A' && c <= 'F') code |= (unsigned)(c - 'A' + 10);
                            else return false;
                        }
                        p += 4;
                        // names and enumerators of this format are ASCII; other code points are kept as UTF-8
                        if (code < 0x80) out += (char)code;
                        else if (code < 0x800) {
                            out += (char)(0xC0 | (code >> 6));
                            out += (char)(0x80 | (code & 0x3F));
                        } else {
                            out += (char)(0xE0 | (code >> 12));
                            out += (char)(0x80 | ((code >> 6) & 0x3F));
                            out += (char)(0x80 | (code & 0x3F));
                        }
                        break;
                    }
                    default: return false;
                }
                ++p;
            } else {
                out += *p++;
            }
        }
        if (p >= end) return false;
        ++p;
        return true;
    }
    Json value() {
        Json v;
        skip();
        if (p >= end || ++depth > 64) {
            fail = true;
            return v;
        }
        const char c = *p;
        if (c == '{') {
            v.kind = Json::Object;
            ++p;
            skip();
            if (p < end && *p == '}') {
                ++p;
            } else {
                for (;;) {
                    skip();
                    std::string key;
                    if (!string(key)) { fail = true; break; }
                    skip();
                    if (p >= end || *p != ':') { fail = true; break; }
                    ++p;
                    Json item = value();
                    if (fail) break;
                    for (auto &f : v.fields)
                        if (f.first == key) fail = true;  // a duplicate key is a malformed file
                    v.fields.emplace_back(std::move(key), std::move(item));
                    skip();
                    if (p < end && *p == ',') { ++p; continue; }
                    if (p < end && *p == '}') { ++p; break; }
                    fail = true;
                    break;
                }
            }
        } else if (c == '[') {
            v.kind = Json::Array;
            ++p;
            skip();
            if (p < end && *p == ']') {
                ++p;
            } else {
                for (;;) {
                    v.items.push_back(value());
                    if (fail) break;
                    skip();
                    if (p < end && *p == ',') { ++p; continue; }
                    if (p < end && *p == ']') { ++p; break; }
                    fail = true;
                    break;
                }
            }
        } else if (c == '"') {
            v.kind = Json::String;
            if (!string(v.str)) fail = true;
        } else if (c == 't') {
            v.kind = Json::Bool;
            v.b = true;
            if (!literal("true")) fail = true;
        } else if (c == 'f') {
            v.kind = Json::Bool;
            if (!literal("false")) fail = true;
        } else if (c == 'n') {
            if (!literal("null")) fail = true;
        } else {
            v.kind = Json::Number;
            const char *start = p;
            if (p < end && *p == '-') ++p;
            bool digits = false, frac = false;
            while (p < end && ((*p >= '0' && *p <= '9') || *p == '.' || *p == 'e' || *p == 'E' || *p == '+' || *p == '-')) {
                if (*p >= '0' && *p <= '9') digits = true;
                else frac = true;
                ++p;
            }
            if (!digits) {
                fail = true;
            } else {
                const std::string text(start, p);
                char *stop = nullptr;
                v.num = strtod(text.c_str(), &stop);
                v.integral = !frac;
                if (!stop || *stop) fail = true;
            }
        }
        --depth;
        return v;
    }
};

inline bool parse_json(const char *data, size_t size, Json &out) {
    JsonParser parser{data, data + size};
    out = parser.value();
    parser.skip();
    return !parser.fail && parser.p == parser.end;
}

inline bool read_file(const std::string &path, std::string &out, size_t limit) {
    FILE *f = fopen(path.c_str(), "rb");
    if (!f) return false;
    char buf[1 << 16];
    size_t n;
    while ((n = fread(buf, 1, sizeof buf, f)) > 0) {
        out.append(buf, n);
        if (out.size() > limit) break;
    }
    const bool ok = !ferror(f) && out.size() <= limit;
    fclose(f);
    return ok;
}

struct Mapping {
    const uint8_t *data = nullptr;
    size_t size = 0;
    ~Mapping() {
        if (data) munmap(const_cast<uint8_t *>(data), size);
    }
    bool open_file(const std::string &path) {
        const int fd = ::open(path.c_str(), O_RDONLY | O_CLOEXEC);
        if (fd < 0) return false;
        struct stat st;
        if (fstat(fd, &st) != 0 || st.st_size <= 0) {
            ::close(fd);
            return false;
        }
        void *p = mmap(nullptr, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
        ::close(fd);
        if (p == MAP_FAILED) return false;
        data = static_cast<const uint8_t *>(p);
        size = (size_t)st.st_size;
        return true;
    }
};

// ---------------------------------------------------------------------------------------- config checks
inline bool is_str(const Json *v, const char *s) { return v && v->kind == Json::String && v->str == s; }
inline bool is_none(const Json *v) { return !v || v->is_null(); }
inline bool is_false(const Json *v) { return v && v->kind == Json::Bool && !v->b; }
inline bool is_true(const Json *v) { return v && v->kind == Json::Bool && v->b; }
inline bool as_u32(const Json *v, uint32_t &out) {
    if (!v || v->kind != Json::Number || !v->integral || v->num < 0 || v->num > 4294967295.0) return false;
    out = (uint32_t)v->num;
    return true;
}

struct Tensor {
    std::string dtype;
    std::vector<uint64_t> shape;
    uint64_t lo = 0, hi = 0;
};

// model.safetensors, mapped; `used` collects the names that were asked for (every tensor must be consumed).
struct TensorFile {
    Mapping file;
    const uint8_t *payload = nullptr;
    size_t payload_size = 0;
    std::map<std::string, Tensor> tensors;
    std::map<std::string, std::string> metadata;
    std::set<std::string> used;
};

inline stark_b200_status read_safetensors(const std::string &path, TensorFile &a) {
    if (!a.file.open_file(path)) return STARK_B200_IO_FAILURE;
    if (a.file.size < 8) return STARK_B200_INVALID_ARGUMENT;
    uint64_t n = 0;
    memcpy(&n, a.file.data, 8);
    if (n > 100ull * 1024 * 1024 || 8 + n > a.file.size) return STARK_B200_INVALID_ARGUMENT;  // safetensors_metadata.rs:117-132
    Json header;
    if (!parse_json(reinterpret_cast<const char *>(a.file.data + 8), (size_t)n, header) || header.kind != Json::Object)
        return STARK_B200_INVALID_ARGUMENT;
    a.payload = a.file.data + 8 + n;
    a.payload_size = a.file.size - 8 - (size_t)n;
    for (auto &f : header.fields) {
        if (f.first == "__metadata__") {
            if (f.second.kind == Json::Object)
                for (auto &mf : f.second.fields)
                    if (mf.second.kind == Json::String) a.metadata[mf.first] = mf.second.str;
            continue;
        }
        Tensor t;
        const Json *dtype = f.second.get("dtype"), *shape = f.second.get("shape"), *offs = f.second.get("data_offsets");
        if (!dtype || dtype->kind != Json::String || !shape || shape->kind != Json::Array || !offs ||
            offs->kind != Json::Array || offs->items.size() != 2)
            return STARK_B200_INVALID_ARGUMENT;
        t.dtype = dtype->str;
        for (auto &d : shape->items) {
            if (d.kind != Json::Number || !d.integral || d.num < 0) return STARK_B200_INVALID_ARGUMENT;
            t.shape.push_back((uint64_t)d.num);
        }
        if (offs->items[0].kind != Json::Number || offs->items[1].kind != Json::Number || offs->items[0].num < 0 ||
            offs->items[1].num < offs->items[0].num)
            return STARK_B200_INVALID_ARGUMENT;
        t.lo = (uint64_t)offs->items[0].num;
        t.hi = (uint64_t)offs->items[1].num;
        a.tensors[f.first] = std::move(t);
    }
    return STARK_B200_OK;
}

// The bytes of tensor `name`, which must have exactly this dtype and shape and consistent offsets.
inline const uint8_t *tensor_bytes(TensorFile &a, const std::string &name, const char *dtype, std::vector<uint64_t> shape,
                            uint32_t element_bytes) {
    auto it = a.tensors.find(name);
    if (it == a.tensors.end() || it->second.dtype != dtype || it->second.shape != shape) return nullptr;
    uint64_t bytes = element_bytes;
    for (uint64_t d : shape) bytes *= d;
    if (it->second.hi - it->second.lo != bytes || it->second.hi > a.payload_size) return nullptr;
    a.used.insert(name);
    return a.payload + it->second.lo;
}

// The layered family's half of stark_b200_load (load_layered.cu): `root` is its config.json.
bool layered_claims(const Json &root);
stark_b200_status load_layered(const std::string &dir, const Json &root, uint64_t context_tokens, stark_b200_model **out_model);

}  // namespace sb
