// Readers of a model folder: a small JSON parser (config.json, the safetensors header) and the safetensors container
// (an 8-byte little-endian header length, that many bytes of JSON name -> dtype, shape, data_offsets, then the data).
// Both throw std::runtime_error with a message that names what is wrong.
#pragma once
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <fstream>
#include <map>
#include <stdexcept>
#include <string>
#include <vector>

namespace wick {

class JsonValue {
  public:
    enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT };
    Kind kind = NUL;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<JsonValue> items;
    std::map<std::string, JsonValue> members;

    bool is_null() const { return kind == NUL; }
    bool is_string() const { return kind == STRING; }
    bool is_object() const { return kind == OBJECT; }
    bool is_array() const { return kind == ARRAY; }
    bool is_number() const { return kind == NUMBER; }
    const JsonValue* find(const std::string& key) const {
        auto it = members.find(key);
        return it == members.end() ? nullptr : &it->second;
    }
    const JsonValue& at(const std::string& key) const {
        const JsonValue* v = find(key);
        if (!v) throw std::runtime_error("missing key: " + key);
        return *v;
    }
    // a positive integer that fits an int
    int count(const std::string& key) const {
        const JsonValue& v = at(key);
        if (v.kind != NUMBER || v.num < 1 || v.num > 1e9 || v.num != (double)(int64_t)v.num)
            throw std::runtime_error("key " + key + ": expected a positive integer");
        return (int)v.num;
    }
    int count_or(const std::string& key, int fallback) const {
        const JsonValue* v = find(key);
        if (!v || v->is_null()) return fallback;
        if (v->kind != NUMBER || v->num < 0 || v->num > 1e9 || v->num != (double)(int64_t)v->num)
            throw std::runtime_error("key " + key + ": expected an integer");
        return (int)v->num;
    }
    double number(const std::string& key) const {
        const JsonValue& v = at(key);
        if (v.kind != NUMBER) throw std::runtime_error("key " + key + ": expected a number");
        return v.num;
    }
    double number_or(const std::string& key, double fallback) const {
        const JsonValue* v = find(key);
        return !v || v->is_null() ? fallback : number(key);
    }

    static JsonValue parse(const char* p, size_t n) {
        Parser ps{p, p + n};
        JsonValue v = ps.value(0);
        ps.space();
        if (ps.p != ps.end) throw std::runtime_error("JSON: text after the value");
        return v;
    }
    static JsonValue parse_file(const std::string& path) {
        std::ifstream f(path, std::ios::binary);
        if (!f) throw std::runtime_error("cannot open " + path);
        std::string s((std::istreambuf_iterator<char>(f)), std::istreambuf_iterator<char>());
        try {
            return parse(s.data(), s.size());
        } catch (const std::exception& e) {
            throw std::runtime_error(path + ": " + e.what());
        }
    }

  private:
    struct Parser {
        const char *p, *end;
        [[noreturn]] void bad(const char* what) { throw std::runtime_error(std::string("JSON: ") + what); }
        void space() {
            while (p != end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
        }
        bool take(const char* word) {
            const size_t n = strlen(word);
            if ((size_t)(end - p) < n || memcmp(p, word, n)) return false;
            p += n;
            return true;
        }
        void utf8(std::string& s, unsigned c) {
            if (c < 0x80) s += (char)c;
            else if (c < 0x800) { s += (char)(0xC0 | c >> 6); s += (char)(0x80 | (c & 63)); }
            else if (c < 0x10000) { s += (char)(0xE0 | c >> 12); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
            else { s += (char)(0xF0 | c >> 18); s += (char)(0x80 | (c >> 12 & 63)); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
        }
        unsigned hex4() {
            if (end - p < 4) bad("short \\u escape");
            unsigned v = 0;
            for (int i = 0; i < 4; i++, p++) {
                const char c = *p;
                v = v * 16 + (c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : (bad("bad \\u escape"), 0));
            }
            return v;
        }
        std::string string() {
            std::string s;
            p++;  // opening quote
            while (true) {
                if (p == end) bad("unterminated string");
                char c = *p++;
                if (c == '"') return s;
                if (c != '\\') { s += c; continue; }
                if (p == end) bad("unterminated string");
                c = *p++;
                switch (c) {
                    case 'n': s += '\n'; break;
                    case 't': s += '\t'; break;
                    case 'r': s += '\r'; break;
                    case 'b': s += '\b'; break;
                    case 'f': s += '\f'; break;
                    case 'u': {
                        unsigned u = hex4();
                        if (u >= 0xD800 && u < 0xDC00 && take("\\u")) u = 0x10000 + ((u - 0xD800) << 10) + (hex4() - 0xDC00);
                        utf8(s, u);
                        break;
                    }
                    default: s += c;
                }
            }
        }
        JsonValue value(int depth) {
            if (depth > 64) bad("nested too deeply");
            space();
            if (p == end) bad("empty text");
            JsonValue v;
            if (*p == '{') {
                v.kind = OBJECT;
                p++;
                space();
                if (p != end && *p == '}') { p++; return v; }
                while (true) {
                    space();
                    if (p == end || *p != '"') bad("expected a key");
                    std::string k = string();
                    space();
                    if (p == end || *p != ':') bad("expected ':'");
                    p++;
                    v.members[k] = value(depth + 1);
                    space();
                    if (p != end && *p == ',') { p++; continue; }
                    if (p != end && *p == '}') { p++; return v; }
                    bad("expected ',' or '}'");
                }
            }
            if (*p == '[') {
                v.kind = ARRAY;
                p++;
                space();
                if (p != end && *p == ']') { p++; return v; }
                while (true) {
                    v.items.push_back(value(depth + 1));
                    space();
                    if (p != end && *p == ',') { p++; continue; }
                    if (p != end && *p == ']') { p++; return v; }
                    bad("expected ',' or ']'");
                }
            }
            if (*p == '"') { v.kind = STRING; v.str = string(); return v; }
            if (take("true")) { v.kind = BOOL; v.b = true; return v; }
            if (take("false")) { v.kind = BOOL; return v; }
            if (take("null")) return v;
            std::string t;
            while (p != end && (strchr("+-.eE", *p) ? *p != 0 : (*p >= '0' && *p <= '9'))) t += *p++;
            char* e = nullptr;
            v.num = strtod(t.c_str(), &e);
            if (t.empty() || *e) bad("unexpected character");
            v.kind = NUMBER;
            return v;
        }
    };
};

struct SafeTensor {
    std::string dtype;
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;
    size_t bytes = 0;
    size_t elems() const {
        size_t n = 1;
        for (int64_t d : shape) n *= (size_t)d;
        return n;
    }
};

class SafeTensors {
  public:
    explicit SafeTensors(const std::string& path) {
        std::ifstream f(path, std::ios::binary | std::ios::ate);
        if (!f) throw std::runtime_error("cannot open " + path);
        const size_t len = (size_t)f.tellg();
        f.seekg(0);
        buf_.resize(len);
        if (len && !f.read((char*)buf_.data(), (std::streamsize)len)) throw std::runtime_error("cannot read " + path);
        uint64_t hl = 0;
        if (len < 8) throw std::runtime_error(path + ": too short for a safetensors file");
        memcpy(&hl, buf_.data(), 8);
        if (hl > len - 8) throw std::runtime_error(path + ": header beyond the end of the file");
        const JsonValue head = JsonValue::parse((const char*)buf_.data() + 8, (size_t)hl);
        if (!head.is_object()) throw std::runtime_error(path + ": header is not a JSON object");
        const size_t base = 8 + (size_t)hl, room = len - base;
        for (const auto& kv : head.members) {
            if (kv.first == "__metadata__") continue;
            SafeTensor t;
            t.dtype = kv.second.at("dtype").str;
            double total = 1.0;
            for (const JsonValue& d : kv.second.at("shape").items) {
                if (!d.is_number() || d.num < 0 || d.num > 1e12) throw std::runtime_error("tensor " + kv.first + ": implausible shape");
                t.shape.push_back((int64_t)d.num);
                total *= d.num;
            }
            if (total > 1e13) throw std::runtime_error("tensor " + kv.first + ": implausible shape");
            const JsonValue& off = kv.second.at("data_offsets");
            if (off.items.size() != 2 || !off.items[0].is_number() || !off.items[1].is_number() || off.items[0].num < 0 ||
                off.items[1].num < off.items[0].num || off.items[1].num > (double)room)
                throw std::runtime_error("tensor " + kv.first + ": data beyond the end of the file");
            const size_t a = (size_t)off.items[0].num, e = (size_t)off.items[1].num;
            const size_t es = t.dtype == "BF16" || t.dtype == "F16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : t.dtype == "I64" || t.dtype == "F64" ? 8 : 1;
            if (t.elems() * es != e - a) throw std::runtime_error("tensor " + kv.first + ": byte count does not fit its shape");
            t.data = buf_.data() + base + a;
            t.bytes = e - a;
            map_[kv.first] = t;
        }
    }
    const SafeTensor* find(const std::string& name) const {
        auto it = map_.find(name);
        return it == map_.end() ? nullptr : &it->second;
    }
    // The tensor of this name and shape, or an exception that says what is wrong.
    const SafeTensor& get(const std::string& name, const std::vector<int64_t>& shape, const char* dtype = "BF16") const {
        const SafeTensor* t = find(name);
        if (!t) throw std::runtime_error("tensor not found: " + name);
        if (t->dtype != dtype) throw std::runtime_error("tensor " + name + ": dtype " + t->dtype + ", expected " + dtype);
        if (t->shape != shape) {
            std::string a, b;
            for (int64_t d : t->shape) a += " " + std::to_string(d);
            for (int64_t d : shape) b += " " + std::to_string(d);
            throw std::runtime_error("tensor " + name + ": shape [" + a + " ], expected [" + b + " ]");
        }
        return *t;
    }

  private:
    std::vector<uint8_t> buf_;
    std::map<std::string, SafeTensor> map_;
};

}  // namespace wick
