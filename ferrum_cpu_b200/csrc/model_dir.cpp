// Reader of model folders: a small JSON parser and the safetensors container (an 8-byte little-endian length, that many
// bytes of JSON mapping names to type, shape and offsets, then the data).
#include "model_dir.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>

#include "fc_common.cuh"

namespace fc {

const Json* Json::find(const char* key) const {
    for (auto& m : members)
        if (m.first == key) return &m.second;
    return nullptr;
}

namespace {
struct Parser {
    const char *p, *end;
    std::string err;
    int depth = 0;
    void skip() { while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) ++p; }
    bool bad(const char* what) { if (err.empty()) err = what; return false; }
    bool word(const char* w) {
        const size_t n = std::strlen(w);
        if ((size_t)(end - p) < n || std::memcmp(p, w, n)) return bad("unexpected word");
        p += n;
        return true;
    }
    bool string(std::string* out) {
        if (p >= end || *p != '"') return bad("a string was expected");
        ++p;
        while (p < end && *p != '"') {
            if (*p == '\\') {
                if (++p >= end) break;
                switch (*p) {
                    case 'n': out->push_back('\n'); break;
                    case 't': out->push_back('\t'); break;
                    case 'r': out->push_back('\r'); break;
                    case 'b': out->push_back('\b'); break;
                    case 'f': out->push_back('\f'); break;
                    case 'u': {
                        if (end - p < 5) return bad("truncated escape");
                        char hex[5] = {p[1], p[2], p[3], p[4], 0};
                        const unsigned c = (unsigned)std::strtoul(hex, nullptr, 16);
                        if (c < 0x80) out->push_back((char)c);
                        else if (c < 0x800) { out->push_back((char)(0xC0 | c >> 6)); out->push_back((char)(0x80 | (c & 63))); }
                        else { out->push_back((char)(0xE0 | c >> 12)); out->push_back((char)(0x80 | (c >> 6 & 63))); out->push_back((char)(0x80 | (c & 63))); }
                        p += 4;
                        break;
                    }
                    default: out->push_back(*p);
                }
                ++p;
            } else {
                out->push_back(*p++);
            }
        }
        if (p >= end) return bad("unterminated string");
        ++p;
        return true;
    }
    bool value(Json* out) {
        if (++depth > 64) return bad("nesting too deep");
        skip();
        if (p >= end) return bad("unexpected end");
        bool ok = true;
        if (*p == '{') {
            out->kind = Json::Object;
            ++p; skip();
            if (p < end && *p == '}') ++p;
            else for (;;) {
                skip();
                std::string key;
                Json v;
                if (!string(&key)) return false;
                skip();
                if (p >= end || *p != ':') return bad("':' was expected");
                ++p;
                if (!value(&v)) return false;
                out->members.emplace_back(std::move(key), std::move(v));
                skip();
                if (p < end && *p == ',') { ++p; continue; }
                if (p < end && *p == '}') { ++p; break; }
                return bad("',' or '}' was expected");
            }
        } else if (*p == '[') {
            out->kind = Json::Array;
            ++p; skip();
            if (p < end && *p == ']') ++p;
            else for (;;) {
                Json v;
                if (!value(&v)) return false;
                out->items.push_back(std::move(v));
                skip();
                if (p < end && *p == ',') { ++p; continue; }
                if (p < end && *p == ']') { ++p; break; }
                return bad("',' or ']' was expected");
            }
        } else if (*p == '"') {
            out->kind = Json::String;
            ok = string(&out->str);
        } else if (*p == 't') {
            out->kind = Json::Bool; out->b = true;
            ok = word("true");
        } else if (*p == 'f') {
            out->kind = Json::Bool;
            ok = word("false");
        } else if (*p == 'n') {
            ok = word("null");
        } else {
            out->kind = Json::Number;
            const char* s = p;
            while (p < end && (std::strchr("+-.eE", *p) || (*p >= '0' && *p <= '9'))) ++p;
            const std::string text(s, p);
            char* stop = nullptr;
            out->num = std::strtod(text.c_str(), &stop);
            if (text.empty() || *stop) ok = bad("a value was expected");
        }
        --depth;
        return ok;
    }
};

size_t type_bytes(const std::string& t) {
    if (t == "F64" || t == "I64" || t == "U64") return 8;
    if (t == "F32" || t == "I32" || t == "U32") return 4;
    if (t == "BF16" || t == "F16" || t == "I16" || t == "U16") return 2;
    if (t == "I8" || t == "U8" || t == "BOOL" || t == "F8_E4M3" || t == "F8_E5M2") return 1;
    return 0;
}
}  // namespace

bool json_parse(const char* text, size_t n, Json* out, std::string* error) {
    Parser ps{text, text + n, {}};
    bool ok = ps.value(out);
    ps.skip();
    if (ok && ps.p != ps.end) ok = ps.bad("text after the value");
    if (!ok && error) *error = ps.err;
    return ok;
}

ModelDir::~ModelDir() {
    if (map_) munmap(map_, map_bytes_);
}

const TensorView* ModelDir::tensor(const std::string& name) const {
    auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
}

int ModelDir::open_config(const char* dir) {
    const std::string path = std::string(dir) + "/config.json";
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) return fail(FC_E_FORMAT, "cannot open %s", path.c_str());
    std::string text;
    char buf[65536];
    size_t n;
    while ((n = std::fread(buf, 1, sizeof buf, f)) > 0) text.append(buf, n);
    std::fclose(f);
    std::string err;
    if (!json_parse(text.data(), text.size(), &config, &err)) return fail(FC_E_FORMAT, "%s: %s", path.c_str(), err.c_str());
    if (config.kind != Json::Object) return fail(FC_E_FORMAT, "%s is not an object", path.c_str());
    return FC_OK;
}

int ModelDir::open(const char* dir) {
    FC_TRY(open_config(dir));
    const std::string path = std::string(dir) + "/model.safetensors";
    const int fd = ::open(path.c_str(), O_RDONLY | O_CLOEXEC);
    if (fd < 0) return fail(FC_E_FORMAT, "cannot open %s", path.c_str());
    struct stat sb;
    if (fstat(fd, &sb) != 0 || sb.st_size < 8) { ::close(fd); return fail(FC_E_FORMAT, "%s is too short", path.c_str()); }
    map_bytes_ = (size_t)sb.st_size;
    void* m = mmap(nullptr, map_bytes_, PROT_READ, MAP_PRIVATE, fd, 0);
    ::close(fd);
    if (m == MAP_FAILED) return fail(FC_E_FORMAT, "cannot map %s", path.c_str());
    map_ = m;
    const uint8_t* base = (const uint8_t*)m;
    uint64_t head = 0;
    for (int i = 7; i >= 0; --i) head = head << 8 | base[i];
    if (head > map_bytes_ - 8) return fail(FC_E_FORMAT, "%s: the directory runs past the end of the file", path.c_str());
    Json dirj;
    std::string err;
    if (!json_parse((const char*)base + 8, (size_t)head, &dirj, &err)) return fail(FC_E_FORMAT, "%s: %s", path.c_str(), err.c_str());
    const uint8_t* data = base + 8 + head;
    const size_t data_bytes = map_bytes_ - 8 - (size_t)head;
    for (auto& e : dirj.members) {
        if (e.first == "__metadata__") continue;
        const Json *dt = e.second.find("dtype"), *sh = e.second.find("shape"), *off = e.second.find("data_offsets");
        if (!dt || dt->kind != Json::String || !sh || sh->kind != Json::Array || !off || off->items.size() != 2)
            return fail(FC_E_FORMAT, "%s: tensor %s has no dtype, shape or offsets", path.c_str(), e.first.c_str());
        TensorView v;
        v.dtype = dt->str;
        double count = 1.0;
        for (auto& d : sh->items) {
            if (d.kind != Json::Number || d.num < 0 || d.num != std::floor(d.num) || d.num > 1e12)
                return fail(FC_E_FORMAT, "%s: tensor %s has a bad shape", path.c_str(), e.first.c_str());
            v.shape.push_back((int64_t)d.num);
            count *= d.num;
        }
        const double a = off->items[0].num, b = off->items[1].num;
        if (!(a >= 0 && b >= a && b <= (double)data_bytes)) return fail(FC_E_FORMAT, "%s: tensor %s lies outside the file", path.c_str(), e.first.c_str());
        v.data = data + (size_t)a;
        v.nbytes = (size_t)(b - a);
        const size_t tb = type_bytes(v.dtype);
        if (!tb || count * (double)tb != (double)v.nbytes)
            return fail(FC_E_FORMAT, "%s: tensor %s: %zu bytes do not fit its shape and type %s", path.c_str(), e.first.c_str(), v.nbytes, v.dtype.c_str());
        tensors_[e.first] = std::move(v);
    }
    return FC_OK;
}

}  // namespace fc

// The registry's probe: which architecture a model folder holds.
extern "C" int fc_model_dir_architecture(const char* dir, char* out, int cap) {
    using namespace fc;
    if (!dir || !out || cap <= 0) return fail(FC_E_ARG, "fc_model_dir_architecture: null argument");
    ModelDir md;
    FC_TRY(md.open_config(dir));
    const Json* a = md.config.find("architecture");
    if (!a || a->kind != Json::String) return fail(FC_E_FORMAT, "%s/config.json names no architecture", dir);
    if ((int)a->str.size() >= cap) return fail(FC_E_SHAPE, "the architecture's name does not fit %d bytes", cap);
    std::memcpy(out, a->str.c_str(), a->str.size() + 1);
    return FC_OK;
}
