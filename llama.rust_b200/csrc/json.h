// A small JSON reader for model configurations and safetensors headers (host only, no dependency).
#pragma once
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace b200 {

class Json {
public:
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ };
    Kind kind = NUL;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<Json> items;
    std::vector<std::pair<std::string, Json>> members;

    // false: not JSON (or nested deeper than 64)
    static bool parse(const char *p, size_t n, Json *out) {
        Reader r{p, p + n, 0};
        if (!r.value(out)) return false;
        r.space();
        return r.p == r.end;
    }
    const Json *find(const char *key) const {
        for (const auto &m : members)
            if (m.first == key) return &m.second;
        return nullptr;
    }
    bool is_null() const { return kind == NUL; }

private:
    struct Reader {
        const char *p, *end;
        int depth;
        void space() {
            while (p < end && (*p == ' ' || *p == '\n' || *p == '\r' || *p == '\t')) p++;
        }
        bool word(const char *w) {
            const size_t n = strlen(w);
            if ((size_t)(end - p) < n || memcmp(p, w, n) != 0) return false;
            p += n;
            return true;
        }
        bool hex4(unsigned *v) {
            if (end - p < 4) return false;
            *v = 0;
            for (int i = 0; i < 4; i++, p++) {
                const char c = *p;
                const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
                if (d < 0) return false;
                *v = *v * 16 + (unsigned)d;
            }
            return true;
        }
        static void utf8(unsigned v, std::string *s) {
            if (v < 0x80) { *s += (char)v; return; }
            if (v < 0x800) { *s += (char)(0xc0 | v >> 6); *s += (char)(0x80 | (v & 63)); return; }
            if (v < 0x10000) { *s += (char)(0xe0 | v >> 12); *s += (char)(0x80 | (v >> 6 & 63)); *s += (char)(0x80 | (v & 63)); return; }
            *s += (char)(0xf0 | v >> 18); *s += (char)(0x80 | (v >> 12 & 63)); *s += (char)(0x80 | (v >> 6 & 63)); *s += (char)(0x80 | (v & 63));
        }
        bool string(std::string *s) {
            if (p >= end || *p != '"') return false;
            for (p++; p < end && *p != '"';) {
                if (*p != '\\') { *s += *p++; continue; }
                if (++p >= end) return false;
                const char c = *p++;
                switch (c) {
                    case '"': case '\\': case '/': *s += c; break;
                    case 'b': *s += '\b'; break;
                    case 'f': *s += '\f'; break;
                    case 'n': *s += '\n'; break;
                    case 'r': *s += '\r'; break;
                    case 't': *s += '\t'; break;
                    case 'u': {
                        unsigned v = 0, w = 0;
                        if (!hex4(&v)) return false;
                        if (v >= 0xd800 && v < 0xdc00 && word("\\u")) {
                            if (!hex4(&w)) return false;
                            v = 0x10000 + ((v - 0xd800) << 10) + (w - 0xdc00);
                        }
                        utf8(v, s);
                        break;
                    }
                    default: return false;
                }
            }
            if (p >= end) return false;
            p++;
            return true;
        }
        bool value(Json *v) {
            if (++depth > 64) return false;
            space();
            if (p >= end) return false;
            bool ok = true;
            if (*p == '{') {
                v->kind = OBJ;
                p++;
                space();
                if (p < end && *p == '}') { p++; depth--; return true; }
                for (;;) {
                    std::pair<std::string, Json> m;
                    space();
                    if (!string(&m.first)) return false;
                    space();
                    if (p >= end || *p++ != ':' || !value(&m.second)) return false;
                    v->members.push_back(std::move(m));
                    space();
                    if (p >= end) return false;
                    if (*p == ',') { p++; continue; }
                    ok = *p++ == '}';
                    break;
                }
            } else if (*p == '[') {
                v->kind = ARR;
                p++;
                space();
                if (p < end && *p == ']') { p++; depth--; return true; }
                for (;;) {
                    v->items.emplace_back();
                    if (!value(&v->items.back())) return false;
                    space();
                    if (p >= end) return false;
                    if (*p == ',') { p++; continue; }
                    ok = *p++ == ']';
                    break;
                }
            } else if (*p == '"') {
                v->kind = STR;
                ok = string(&v->str);
            } else if (word("true")) {
                v->kind = BOOL;
                v->b = true;
            } else if (word("false")) {
                v->kind = BOOL;
            } else if (word("null")) {
                v->kind = NUL;
            } else {
                const char *q = p;
                while (q < end && (strchr("+-.eE", *q) || (*q >= '0' && *q <= '9'))) q++;
                const std::string s(p, q);
                char *stop = nullptr;
                v->kind = NUM;
                v->num = strtod(s.c_str(), &stop);
                ok = !s.empty() && stop == s.c_str() + s.size();
                p = q;
            }
            depth--;
            return ok;
        }
    };
};

}  // namespace b200
