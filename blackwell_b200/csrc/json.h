// A small JSON reader for model configurations, safetensors headers and JSON-lines requests (host only).
#pragma once
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include <string>
#include <utility>
#include <vector>

namespace bw {

struct Json {
    enum Type { kNull, kBool, kNumber, kString, kArray, kObject };
    Type type = kNull;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::vector<std::pair<std::string, Json>> obj;

    const Json* get(const char* key) const {
        for (const auto& kv : obj)
            if (kv.first == key) return &kv.second;
        return nullptr;
    }
    bool is_null() const { return type == kNull; }
    bool is_int() const { return type == kNumber && num == floor(num) && fabs(num) < 9e15; }

    // Parses one document; on failure returns false and says where in `err`.
    static bool parse(const char* text, size_t n, Json* out, std::string* err) {
        Parser p{text, text + n, text, 0};
        if (p.value(out) && (p.space(), p.p == p.end)) return true;
        if (err) *err = "malformed JSON at byte " + std::to_string(p.p - p.begin);
        return false;
    }

private:
    struct Parser {
        const char *p, *end, *begin;
        int depth;
        void space() { while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) ++p; }
        bool word(const char* w) {
            const size_t n = strlen(w);
            if ((size_t)(end - p) < n || memcmp(p, w, n) != 0) return false;
            p += n;
            return true;
        }
        static void utf8(std::string& s, unsigned c) {
            if (c < 0x80) s += (char)c;
            else if (c < 0x800) { s += (char)(0xC0 | c >> 6); s += (char)(0x80 | (c & 0x3F)); }
            else if (c < 0x10000) { s += (char)(0xE0 | c >> 12); s += (char)(0x80 | (c >> 6 & 0x3F)); s += (char)(0x80 | (c & 0x3F)); }
            else { s += (char)(0xF0 | c >> 18); s += (char)(0x80 | (c >> 12 & 0x3F)); s += (char)(0x80 | (c >> 6 & 0x3F)); s += (char)(0x80 | (c & 0x3F)); }
        }
        bool hex4(unsigned* v) {
            if (end - p < 4) return false;
            *v = 0;
            for (int i = 0; i < 4; ++i, ++p) {
                const char c = *p;
                const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
                if (d < 0) return false;
                *v = *v * 16 + d;
            }
            return true;
        }
        bool string(std::string* s) {
            if (p >= end || *p != '"') return false;
            for (++p; p < end && *p != '"'; ++p) {
                if (*p != '\\') { *s += *p; continue; }
                if (++p >= end) return false;
                switch (*p) {
                    case 'n': *s += '\n'; break;
                    case 't': *s += '\t'; break;
                    case 'r': *s += '\r'; break;
                    case 'b': *s += '\b'; break;
                    case 'f': *s += '\f'; break;
                    case 'u': {
                        ++p;
                        unsigned c, lo;
                        if (!hex4(&c)) return false;
                        if (c >= 0xD800 && c < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {
                            p += 2;
                            if (!hex4(&lo)) return false;
                            c = 0x10000 + ((c - 0xD800) << 10) + (lo - 0xDC00);
                        }
                        utf8(*s, c);
                        --p;
                        break;
                    }
                    default: *s += *p;
                }
            }
            if (p >= end) return false;
            ++p;
            return true;
        }
        bool value(Json* v) {
            space();
            if (p >= end || depth > 64) return false;
            if (*p == '{') {
                v->type = kObject;
                ++p; ++depth;
                space();
                if (p < end && *p == '}') { ++p; --depth; return true; }
                for (;;) {
                    std::pair<std::string, Json> kv;
                    space();
                    if (!string(&kv.first)) return false;
                    space();
                    if (p >= end || *p++ != ':') return false;
                    if (!value(&kv.second)) return false;
                    v->obj.push_back(std::move(kv));
                    space();
                    if (p >= end) return false;
                    const char c = *p++;
                    if (c == '}') { --depth; return true; }
                    if (c != ',') { --p; return false; }
                }
            }
            if (*p == '[') {
                v->type = kArray;
                ++p; ++depth;
                space();
                if (p < end && *p == ']') { ++p; --depth; return true; }
                for (;;) {
                    v->arr.emplace_back();
                    if (!value(&v->arr.back())) return false;
                    space();
                    if (p >= end) return false;
                    const char c = *p++;
                    if (c == ']') { --depth; return true; }
                    if (c != ',') { --p; return false; }
                }
            }
            if (*p == '"') { v->type = kString; return string(&v->str); }
            if (word("true")) { v->type = kBool; v->b = true; return true; }
            if (word("false")) { v->type = kBool; return true; }
            if (word("null")) return true;
            if (!(*p == '-' || (*p >= '0' && *p <= '9'))) return false;
            const char* q = p;
            while (q < end && (strchr("+-.eE", *q) || (*q >= '0' && *q <= '9'))) ++q;
            const std::string digits(p, q);
            char* stop = nullptr;
            v->type = kNumber;
            v->num = strtod(digits.c_str(), &stop);
            if (stop != digits.c_str() + digits.size()) return false;
            p = q;
            return true;
        }
    };
};

}  // namespace bw
