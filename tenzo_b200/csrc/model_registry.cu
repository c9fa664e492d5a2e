// Model registry, JSON reader and safetensors reader (host code).
#include "model_registry.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstdio>
#include <cstdlib>
#include <cstring>

#include "engine_core.h"

namespace tz {

// ---- JSON -----------------------------------------------------------------------------------------------------------------
namespace {

class Parser {
public:
    explicit Parser(const std::string& t) : s(t) {}
    Json document() {
        Json v = value(0);
        space();
        if (p != s.size()) fail("text after the document");
        return v;
    }

private:
    const std::string& s;
    size_t p = 0;

    [[noreturn]] void fail(const char* what) { throw std::invalid_argument(std::string("JSON, byte ") + std::to_string(p) + ": " + what); }
    void space() { while (p < s.size() && (s[p] == ' ' || s[p] == '\t' || s[p] == '\n' || s[p] == '\r')) ++p; }
    bool eat(char c) {
        space();
        if (p < s.size() && s[p] == c) { ++p; return true; }
        return false;
    }
    void literal(const char* w) {
        const size_t n = std::strlen(w);
        if (s.compare(p, n, w) != 0) fail("unknown literal");
        p += n;
    }
    static void utf8(std::string& out, unsigned c) {
        if (c < 0x80) out += (char)c;
        else if (c < 0x800) { out += (char)(0xC0 | (c >> 6)); out += (char)(0x80 | (c & 63)); }
        else if (c < 0x10000) { out += (char)(0xE0 | (c >> 12)); out += (char)(0x80 | ((c >> 6) & 63)); out += (char)(0x80 | (c & 63)); }
        else { out += (char)(0xF0 | (c >> 18)); out += (char)(0x80 | ((c >> 12) & 63)); out += (char)(0x80 | ((c >> 6) & 63)); out += (char)(0x80 | (c & 63)); }
    }
    unsigned hex4() {
        if (p + 4 > s.size()) fail("short \\u escape");
        unsigned v = 0;
        for (int i = 0; i < 4; ++i) {
            const char c = s[p++];
            v = v * 16 + (c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : (fail("bad \\u escape"), 0));
        }
        return v;
    }
    std::string text() {
        if (!eat('"')) fail("a string was expected");
        std::string out;
        for (;;) {
            if (p >= s.size()) fail("unterminated string");
            const char c = s[p++];
            if (c == '"') return out;
            if (c != '\\') { out += c; continue; }
            if (p >= s.size()) fail("unterminated escape");
            const char e = s[p++];
            switch (e) {
                case 'n': out += '\n'; break;
                case 't': out += '\t'; break;
                case 'r': out += '\r'; break;
                case 'b': out += '\b'; break;
                case 'f': out += '\f'; break;
                case '"': case '\\': case '/': out += e; break;
                case 'u': {
                    unsigned v = hex4();
                    if (v >= 0xD800 && v < 0xDC00 && s.compare(p, 2, "\\u") == 0) { p += 2; v = 0x10000 + ((v - 0xD800) << 10) + (hex4() - 0xDC00); }
                    utf8(out, v);
                    break;
                }
                default: fail("unknown escape");
            }
        }
    }
    Json value(int depth) {
        if (depth > 64) fail("nesting too deep");
        space();
        if (p >= s.size()) fail("unexpected end");
        Json v;
        const char c = s[p];
        if (c == '{') {
            ++p;
            v.kind = Json::Object;
            if (eat('}')) return v;
            do {
                space();
                std::string k = text();
                if (!eat(':')) fail("':' was expected");
                v.fields[k] = value(depth + 1);
            } while (eat(','));
            if (!eat('}')) fail("'}' was expected");
        } else if (c == '[') {
            ++p;
            v.kind = Json::Array;
            if (eat(']')) return v;
            do v.items.push_back(value(depth + 1)); while (eat(','));
            if (!eat(']')) fail("']' was expected");
        } else if (c == '"') {
            v.kind = Json::String;
            v.str = text();
        } else if (c == 't') { literal("true"); v.kind = Json::Bool; v.b = true; }
        else if (c == 'f') { literal("false"); v.kind = Json::Bool; }
        else if (c == 'n') { literal("null"); }
        else {
            const char* b = s.c_str() + p;
            char* e = nullptr;
            if (!((c >= '0' && c <= '9') || c == '-')) fail("unexpected character");
            v.num = std::strtod(b, &e);
            if (e == b) fail("bad number");
            p += (size_t)(e - b);
            v.kind = Json::Number;
        }
        return v;
    }
};

std::vector<ModelFamily>& registry() {
    static std::vector<ModelFamily> r;
    return r;
}

}  // namespace

Json parse_json(const std::string& text) { return Parser(text).document(); }

// ---- registry -------------------------------------------------------------------------------------------------------------
ModelRegistration::ModelRegistration(const ModelFamily& f) { registry().push_back(f); }
const std::vector<ModelFamily>& model_families() { return registry(); }

std::string read_text_file(const std::string& path) {
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) throw IoError("cannot open " + path);
    std::string text;
    char buf[1 << 16];
    size_t n;
    while ((n = std::fread(buf, 1, sizeof buf, f)) > 0) text.append(buf, n);
    std::fclose(f);
    return text;
}

EngineCore* open_model(const OpenOptions& o) {
    const std::string path = o.dir + "/config.json";
    Json cfg;
    try {
        cfg = parse_json(read_text_file(path));
        const std::string& arch = cfg.at("architecture").string();
        for (const ModelFamily& f : registry())
            if (arch == f.architecture) return f.open(cfg, o);
        throw ParseError("no model of this library has architecture '" + arch + "'");
    } catch (const std::invalid_argument& e) {
        throw ParseError(path + ": " + e.what());
    }
}

// ---- safetensors ----------------------------------------------------------------------------------------------------------
SafeTensors::SafeTensors(const std::string& path) {
    const int fd = ::open(path.c_str(), O_RDONLY);
    if (fd < 0) throw IoError("cannot open " + path);
    struct stat st;
    if (fstat(fd, &st) != 0 || st.st_size < 8) { ::close(fd); throw IoError(path + " is too short"); }
    size = (size_t)st.st_size;
    base = mmap(nullptr, size, PROT_READ, MAP_PRIVATE, fd, 0);
    ::close(fd);
    if (base == MAP_FAILED) { base = nullptr; throw IoError("cannot map " + path); }
    try {
        const unsigned char* b = static_cast<const unsigned char*>(base);
        unsigned long long n = 0;
        for (int i = 7; i >= 0; --i) n = n << 8 | b[i];
        if (n > size - 8) throw ParseError(path + ": header runs past the end of the file");
        const size_t data0 = 8 + (size_t)n;
        const Json head = parse_json(std::string(reinterpret_cast<const char*>(b) + 8, (size_t)n));
        for (const auto& kv : head.fields) {
            if (kv.first == "__metadata__") continue;
            TensorView t;
            t.dtype = kv.second.at("dtype").string();
            for (const Json& d : kv.second.at("shape").array()) t.shape.push_back((long long)d.number());
            const auto& off = kv.second.at("data_offsets").array();
            if (off.size() != 2) throw ParseError(path + ": bad data_offsets of " + kv.first);
            const double lo = off[0].number(), hi = off[1].number();
            if (lo < 0 || hi < lo || hi > (double)(size - data0)) throw ParseError(path + ": " + kv.first + " lies outside the file");
            t.data = b + data0 + (size_t)lo;
            t.bytes = (size_t)hi - (size_t)lo;
            const size_t es = t.dtype == "BF16" || t.dtype == "F16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : 0;
            if (es && t.bytes != es * (size_t)t.count()) throw ParseError(path + ": size of " + kv.first + " does not fit its shape");
            tensors[kv.first] = t;
        }
    } catch (const std::invalid_argument& e) {
        munmap(base, size);
        throw ParseError(path + ": " + e.what());
    } catch (...) {
        munmap(base, size);
        throw;
    }
}

SafeTensors::~SafeTensors() { if (base) munmap(base, size); }

const TensorView& SafeTensors::at(const std::string& name) const {
    auto it = tensors.find(name);
    if (it == tensors.end()) throw ParseError("tensor '" + name + "' is missing");
    return it->second;
}

const TensorView& SafeTensors::bf16(const std::string& name, const std::vector<long long>& shape) const {
    const TensorView& t = at(name);
    bool ok = t.shape.size() == shape.size();
    for (size_t i = 0; ok && i < shape.size(); ++i) ok = shape[i] < 0 || t.shape[i] == shape[i];
    if (!ok) {
        std::string m = "tensor '" + name + "' has shape [";
        for (size_t i = 0; i < t.shape.size(); ++i) m += (i ? ", " : "") + std::to_string(t.shape[i]);
        m += "], expected [";
        for (size_t i = 0; i < shape.size(); ++i) m += (i ? ", " : "") + (shape[i] < 0 ? std::string("?") : std::to_string(shape[i]));
        throw ParseError(m + "]");
    }
    if (t.dtype != "BF16") throw ParseError("tensor '" + name + "' is " + t.dtype + ", expected BF16");
    return t;
}

std::vector<float> SafeTensors::floats(const std::string& name, const std::vector<long long>& shape) const {
    const TensorView& t = bf16(name, shape);
    std::vector<float> out((size_t)t.count());
    for (size_t i = 0; i < out.size(); ++i) {
        const uint32_t bits = (uint32_t)(t.data[2 * i] | t.data[2 * i + 1] << 8) << 16;
        std::memcpy(&out[i], &bits, 4);
    }
    return out;
}

}  // namespace tz
