// Minimal JSON reader (host only): model configurations and safetensors headers.
#pragma once
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace b200p {

struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object };
    Kind kind = Null;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<Json> items;                                  // Array
    std::vector<std::pair<std::string, Json>> fields;         // Object, in file order

    // The member `key` of an object; null (as a pointer) when it is absent or JSON null.
    const Json* get(const char* key) const {
        if (kind != Object) return nullptr;
        for (const auto& f : fields)
            if (f.first == key) return f.second.kind == Null ? nullptr : &f.second;
        return nullptr;
    }
    bool is_int() const { return kind == Number && num == double((long long)(num)); }

    // false on malformed text (then *out is unspecified)
    static bool parse(const char* text, size_t n, Json* out) {
        Reader r{text, text + n, 0};
        r.skip();
        if (!r.value(out)) return false;
        r.skip();
        return r.p == r.end;
    }

private:
    struct Reader {
        const char *p, *end;
        int depth;
        void skip() { while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) ++p; }
        bool word(const char* w) {
            const char* q = p;
            for (; *w; ++w, ++q) if (q >= end || *q != *w) return false;
            p = q;
            return true;
        }
        static void utf8(unsigned c, std::string* s) {
            if (c < 0x80) s->push_back(char(c));
            else if (c < 0x800) { s->push_back(char(0xC0 | (c >> 6))); s->push_back(char(0x80 | (c & 63))); }
            else { s->push_back(char(0xE0 | (c >> 12))); s->push_back(char(0x80 | ((c >> 6) & 63))); s->push_back(char(0x80 | (c & 63))); }
        }
        bool string(std::string* s) {
            if (p >= end || *p != '"') return false;
            for (++p; p < end && *p != '"'; ++p) {
                if (*p != '\\') { s->push_back(*p); continue; }
                if (++p >= end) return false;
                switch (*p) {
                    case 'n': s->push_back('\n'); break;
                    case 't': s->push_back('\t'); break;
                    case 'r': s->push_back('\r'); break;
                    case 'b': s->push_back('\b'); break;
                    case 'f': s->push_back('\f'); break;
                    case 'u': {
                        if (end - p < 5) return false;
                        utf8(unsigned(std::strtoul(std::string(p + 1, p + 5).c_str(), nullptr, 16)), s);
                        p += 4;
                        break;
                    }
                    default: s->push_back(*p);                 // \" \\ \/
                }
            }
            if (p >= end) return false;
            ++p;
            return true;
        }
        bool value(Json* v) {
            if (p >= end || depth > 64) return false;
            if (*p == '"') { v->kind = String; return string(&v->str); }
            if (*p == '{' || *p == '[') {
                const bool obj = *p == '{';
                const char close = obj ? '}' : ']';
                v->kind = obj ? Object : Array;
                ++p; ++depth; skip();
                if (p < end && *p == close) { ++p; --depth; return true; }
                for (;;) {
                    std::string key;
                    skip();
                    if (obj) {
                        if (!string(&key)) return false;
                        skip();
                        if (p >= end || *p != ':') return false;
                        ++p; skip();
                    }
                    Json item;
                    if (!value(&item)) return false;
                    if (obj) v->fields.emplace_back(std::move(key), std::move(item)); else v->items.push_back(std::move(item));
                    skip();
                    if (p >= end) return false;
                    if (*p == ',') { ++p; continue; }
                    if (*p != close) return false;
                    ++p; --depth;
                    return true;
                }
            }
            if (word("true")) { v->kind = Bool; v->b = true; return true; }
            if (word("false")) { v->kind = Bool; return true; }
            if (word("null")) return true;
            const char* q = p;                                 // a number: copied out, strtod needs a terminated string
            while (q < end && ((*q >= '0' && *q <= '9') || *q == '+' || *q == '-' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
            if (q == p) return false;
            const std::string t(p, q);
            char* e = nullptr;
            v->kind = Number; v->num = std::strtod(t.c_str(), &e);
            p = q;
            return *e == '\0';
        }
    };
};

} // namespace b200p
