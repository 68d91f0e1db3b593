// A small JSON reader for model configuration files (config.json, the header of a safetensors file).
// Numbers are kept as doubles; objects keep their keys in file order. Depth and size are bounded by the caller's text.
#pragma once
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace sp {

struct Json {
    enum Type { NUL, BOOL, NUM, STR, ARR, OBJ };
    Type type = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::vector<std::pair<std::string, Json>> obj;

    bool is_null() const { return type == NUL; }
    const Json* get(const char* key) const {
        if (type != OBJ) return nullptr;
        for (const auto& kv : obj)
            if (kv.first == key) return kv.second.type == NUL ? nullptr : &kv.second;  // null reads as absent
        return nullptr;
    }

    // false on malformed input
    static bool parse(const char* text, size_t n, Json* out) {
        Parser p{text, text + n};
        if (!p.value(*out, 0)) return false;
        p.skip();
        return p.s == p.end;
    }

  private:
    struct Parser {
        const char *s, *end;
        void skip() { while (s < end && (*s == ' ' || *s == '\n' || *s == '\t' || *s == '\r')) ++s; }
        bool lit(const char* w) {
            const size_t k = std::strlen(w);
            if ((size_t)(end - s) < k || std::memcmp(s, w, k) != 0) return false;
            s += k;
            return true;
        }
        static void utf8(unsigned c, std::string& o) {
            if (c < 0x80) o += (char)c;
            else if (c < 0x800) { o += (char)(0xC0 | c >> 6); o += (char)(0x80 | (c & 63)); }
            else { o += (char)(0xE0 | c >> 12); o += (char)(0x80 | (c >> 6 & 63)); o += (char)(0x80 | (c & 63)); }
        }
        bool string(std::string& o) {
            if (s >= end || *s != '"') return false;
            for (++s; s < end && *s != '"'; ++s) {
                if (*s != '\\') { o += *s; continue; }
                if (++s >= end) return false;
                switch (*s) {
                    case 'n': o += '\n'; break;
                    case 't': o += '\t'; break;
                    case 'r': o += '\r'; break;
                    case 'b': o += '\b'; break;
                    case 'f': o += '\f'; break;
                    case 'u': {
                        if (end - s < 5) return false;
                        const std::string hex(s + 1, s + 5);
                        char* stop = nullptr;
                        const long c = std::strtol(hex.c_str(), &stop, 16);
                        if (stop != hex.c_str() + 4) return false;
                        utf8((unsigned)c, o);
                        s += 4;
                        break;
                    }
                    default: o += *s;  // quote, backslash, slash
                }
            }
            if (s >= end) return false;
            ++s;
            return true;
        }
        bool value(Json& v, int depth) {
            if (depth > 64) return false;
            skip();
            if (s >= end) return false;
            if (*s == '{') {
                v.type = OBJ;
                ++s;
                skip();
                if (s < end && *s == '}') { ++s; return true; }
                for (;;) {
                    skip();
                    std::pair<std::string, Json> kv;
                    if (!string(kv.first)) return false;
                    skip();
                    if (s >= end || *s++ != ':') return false;
                    if (!value(kv.second, depth + 1)) return false;
                    v.obj.push_back(std::move(kv));
                    skip();
                    if (s >= end) return false;
                    if (*s == ',') { ++s; continue; }
                    if (*s == '}') { ++s; return true; }
                    return false;
                }
            }
            if (*s == '[') {
                v.type = ARR;
                ++s;
                skip();
                if (s < end && *s == ']') { ++s; return true; }
                for (;;) {
                    v.arr.emplace_back();
                    if (!value(v.arr.back(), depth + 1)) return false;
                    skip();
                    if (s >= end) return false;
                    if (*s == ',') { ++s; continue; }
                    if (*s == ']') { ++s; return true; }
                    return false;
                }
            }
            if (*s == '"') { v.type = STR; return string(v.str); }
            if (lit("null")) { v.type = NUL; return true; }
            if (lit("true")) { v.type = BOOL; v.b = true; return true; }
            if (lit("false")) { v.type = BOOL; return true; }
            // the text need not be NUL-terminated: copy the number out
            const char* e = s;
            while (e < end && (std::strchr("+-.eE", *e) ? *e != 0 : (*e >= '0' && *e <= '9'))) ++e;
            if (e == s) return false;
            const std::string t(s, e);
            char* stop = nullptr;
            v.num = std::strtod(t.c_str(), &stop);
            if (stop != t.c_str() + t.size()) return false;
            v.type = NUM;
            s = e;
            return true;
        }
    };
};

}  // namespace sp
