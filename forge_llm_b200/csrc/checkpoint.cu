// JSON and safetensors readers (host code): an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
// data_offsets), then the data.  Every offset is checked against the file before it is used.
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cmath>
#include <cstdlib>
#include <cstring>

#include "checkpoint.cuh"

namespace forge {

namespace {

struct Parser {
    const char* p;
    const char* end;
    int depth = 0;
    void ws() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p; }
    bool lit(const char* s) {
        const size_t n = strlen(s);
        if (size_t(end - p) < n || memcmp(p, s, n)) return false;
        p += n;
        return true;
    }
    bool hex4(unsigned& v) {
        v = 0;
        for (int i = 0; i < 4; ++i, ++p) {
            if (p >= end) return false;
            const char c = *p;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return false;
            v = v * 16 + unsigned(d);
        }
        return true;
    }
    static void utf8(std::string& s, unsigned c) {
        if (c < 0x80) s += char(c);
        else if (c < 0x800) { s += char(0xC0 | c >> 6); s += char(0x80 | (c & 63)); }
        else if (c < 0x10000) { s += char(0xE0 | c >> 12); s += char(0x80 | (c >> 6 & 63)); s += char(0x80 | (c & 63)); }
        else { s += char(0xF0 | c >> 18); s += char(0x80 | (c >> 12 & 63)); s += char(0x80 | (c >> 6 & 63)); s += char(0x80 | (c & 63)); }
    }
    bool string(std::string& out) {
        if (p >= end || *p != '"') return false;
        ++p;
        while (p < end && *p != '"') {
            if (*p != '\\') { out += *p++; continue; }
            if (++p >= end) return false;
            const char c = *p++;
            switch (c) {
                case '"': case '\\': case '/': out += c; break;
                case 'b': out += '\b'; break;
                case 'f': out += '\f'; break;
                case 'n': out += '\n'; break;
                case 'r': out += '\r'; break;
                case 't': out += '\t'; break;
                case 'u': {
                    unsigned v, w;
                    if (!hex4(v)) return false;
                    if (v >= 0xD800 && v < 0xDC00) {
                        if (!lit("\\u") || !hex4(w) || w < 0xDC00 || w > 0xDFFF) return false;
                        v = 0x10000 + ((v - 0xD800) << 10) + (w - 0xDC00);
                    }
                    utf8(out, v);
                    break;
                }
                default: return false;
            }
        }
        if (p >= end) return false;
        ++p;
        return true;
    }
    bool value(Json& v) {
        if (++depth > 64) return false;
        ws();
        if (p >= end) return false;
        bool ok = true;
        if (*p == '{') {
            v.kind = Json::Object;
            ++p; ws();
            if (p < end && *p == '}') ++p;
            else for (;;) {
                ws();
                std::pair<std::string, Json> f;
                if (!string(f.first)) return false;
                ws();
                if (p >= end || *p++ != ':') return false;
                if (!value(f.second)) return false;
                v.fields.push_back(std::move(f));
                ws();
                if (p >= end) return false;
                const char c = *p++;
                if (c == '}') break;
                if (c != ',') return false;
            }
        } else if (*p == '[') {
            v.kind = Json::Array;
            ++p; ws();
            if (p < end && *p == ']') ++p;
            else for (;;) {
                v.items.emplace_back();
                if (!value(v.items.back())) return false;
                ws();
                if (p >= end) return false;
                const char c = *p++;
                if (c == ']') break;
                if (c != ',') return false;
            }
        } else if (*p == '"') { v.kind = Json::String; ok = string(v.str); }
        else if (lit("true")) { v.kind = Json::Bool; v.flag = true; }
        else if (lit("false")) v.kind = Json::Bool;
        else if (lit("null")) v.kind = Json::Null;
        else {
            const char* b = p;
            while (p < end && (strchr("+-.eE", *p) || (*p >= '0' && *p <= '9'))) ++p;
            const std::string t(b, p);
            char* e = nullptr;
            v.kind = Json::Number;
            v.num = strtod(t.c_str(), &e);
            ok = !t.empty() && e == t.c_str() + t.size();
        }
        --depth;
        return ok;
    }
};

size_t dtype_bytes(const std::string& t) {
    if (t == "F64" || t == "I64" || t == "U64") return 8;
    if (t == "F32" || t == "I32" || t == "U32") return 4;
    if (t == "BF16" || t == "F16" || t == "I16" || t == "U16") return 2;
    if (t == "I8" || t == "U8" || t == "BOOL") return 1;
    return 0;
}

}  // namespace

int32_t json_parse(const char* text, size_t len, Json* out) {
    Parser ps{text, text + len};
    *out = Json();
    bool ok = ps.value(*out);
    ps.ws();
    if (!ok || ps.p != ps.end) { set_error("malformed JSON near byte %zu", size_t(ps.p - text)); return FORGE_ERR_SHAPE; }
    return FORGE_OK;
}

float TensorView::at(size_t i) const {
    if (dtype == "BF16") { uint16_t h; memcpy(&h, data + 2 * i, 2); const uint32_t u = uint32_t(h) << 16; float f; memcpy(&f, &u, 4); return f; }
    if (dtype == "F16") { __half h; memcpy(&h, data + 2 * i, 2); return __half2float(h); }
    float f;
    memcpy(&f, data + 4 * i, 4);
    return f;
}

Checkpoint::~Checkpoint() { if (map_) munmap(map_, map_len_); }

int32_t Checkpoint::open(const char* dir) {
    const std::string cfg_path = std::string(dir) + "/config.json", st_path = std::string(dir) + "/model.safetensors";
    std::string text;
    {
        FILE* f = fopen(cfg_path.c_str(), "rb");
        if (!f) { set_error("cannot open %s", cfg_path.c_str()); return FORGE_ERR_INVALID_ARG; }
        char buf[4096];
        for (size_t n; (n = fread(buf, 1, sizeof buf, f)) > 0;) text.append(buf, n);
        fclose(f);
    }
    FORGE_TRY(json_parse(text.data(), text.size(), &config_));
    if (config_.kind != Json::Object) { set_error("config.json is not an object"); return FORGE_ERR_SHAPE; }
    const int fd = ::open(st_path.c_str(), O_RDONLY);
    if (fd < 0) { set_error("cannot open %s", st_path.c_str()); return FORGE_ERR_INVALID_ARG; }
    struct stat sb;
    if (fstat(fd, &sb) != 0 || sb.st_size < 8) { ::close(fd); set_error("%s is truncated", st_path.c_str()); return FORGE_ERR_SHAPE; }
    map_len_ = size_t(sb.st_size);
    map_ = mmap(nullptr, map_len_, PROT_READ, MAP_PRIVATE, fd, 0);
    ::close(fd);
    if (map_ == MAP_FAILED) { map_ = nullptr; set_error("cannot map %s", st_path.c_str()); return FORGE_ERR_INVALID_ARG; }
    const uint8_t* base = static_cast<const uint8_t*>(map_);
    uint64_t hl;
    memcpy(&hl, base, 8);
    if (hl > map_len_ - 8) { set_error("%s: the header is longer than the file", st_path.c_str()); return FORGE_ERR_SHAPE; }
    Json head;
    FORGE_TRY(json_parse(reinterpret_cast<const char*>(base + 8), size_t(hl), &head));
    const size_t data_len = map_len_ - 8 - size_t(hl);
    for (const auto& f : head.fields) {
        if (f.first == "__metadata__") continue;
        const Json *dt = f.second.get("dtype"), *sh = f.second.get("shape"), *off = f.second.get("data_offsets");
        if (!dt || dt->kind != Json::String || !sh || sh->kind != Json::Array || !off || off->items.size() != 2) { set_error("tensor %s: bad header entry", f.first.c_str()); return FORGE_ERR_SHAPE; }
        TensorView t;
        t.dtype = dt->str;
        double n = 1;
        for (const Json& s : sh->items) {
            if (s.kind != Json::Number || !(s.num >= 0) || s.num != std::floor(s.num)) { set_error("tensor %s: bad shape", f.first.c_str()); return FORGE_ERR_SHAPE; }
            t.shape.push_back(int64_t(s.num)); n *= s.num;
        }
        const double a = off->items[0].num, b = off->items[1].num;
        if (!(a >= 0) || !(b >= a) || b > double(data_len) || dtype_bytes(t.dtype) == 0 || n * dtype_bytes(t.dtype) != b - a) { set_error("tensor %s: its data does not fit the file", f.first.c_str()); return FORGE_ERR_SHAPE; }
        t.data = base + 8 + hl + size_t(a);
        t.bytes = size_t(b - a);
        tensors_[f.first] = t;
    }
    return FORGE_OK;
}

const TensorView* Checkpoint::tensor(const std::string& name, const std::vector<int64_t>& shape) const {
    auto it = tensors_.find(name);
    if (it == tensors_.end()) { set_error("tensor %s is missing", name.c_str()); return nullptr; }
    const TensorView& t = it->second;
    if (t.shape != shape) {
        std::string want, got;
        for (int64_t s : shape) want += " " + std::to_string(s);
        for (int64_t s : t.shape) got += " " + std::to_string(s);
        set_error("tensor %s has shape [%s ], the configuration needs [%s ]", name.c_str(), got.c_str(), want.c_str());
        return nullptr;
    }
    if (t.dtype != "BF16" && t.dtype != "F16" && t.dtype != "F32") { set_error("tensor %s: type %s unsupported", name.c_str(), t.dtype.c_str()); return nullptr; }
    return &t;
}

int64_t Checkpoint::parameters() const {
    int64_t n = 0;
    for (const auto& t : tensors_) n += t.second.count();
    return n;
}

}  // namespace forge
