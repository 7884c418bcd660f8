// A small JSON reader for model directories (config.json, the header of a safetensors file): the whole text becomes a
// tree of values.  Host only.
#pragma once
#include <stdlib.h>
#include <string.h>

#include <string>
#include <utility>
#include <vector>

namespace cq {

struct Json {
    enum Kind { Null, Bool, Num, Str, Arr, Obj } kind = Null;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::vector<std::pair<std::string, Json>> obj;

    // Member of an object; null when this is no object or has no such member.
    const Json* get(const char* key) const {
        if (kind != Obj) return nullptr;
        for (const auto& kv : obj) if (kv.first == key) return &kv.second;
        return nullptr;
    }
    bool is_null() const { return kind == Null; }
};

class JsonReader {
public:
    // False when the text is not one JSON value (and nothing but white space after it).
    static bool parse(const char* text, size_t n, Json* out) {
        JsonReader r(text, text + n);
        if (!r.value(out, 0)) return false;
        r.space();
        return r.p_ == r.end_;
    }

private:
    JsonReader(const char* p, const char* end) : p_(p), end_(end) {}
    void space() { while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_; }
    bool take(char c) { space(); if (p_ < end_ && *p_ == c) { ++p_; return true; } return false; }
    bool word(const char* w) { const size_t n = strlen(w); if ((size_t)(end_ - p_) < n || memcmp(p_, w, n)) return false; p_ += n; return true; }
    bool value(Json* v, int depth) {
        if (depth > 64) return false;
        space();
        if (p_ >= end_) return false;
        switch (*p_) {
            case '{': {
                ++p_; v->kind = Json::Obj;
                if (take('}')) return true;
                do {
                    std::string k;
                    space();
                    if (!string(&k) || !take(':')) return false;
                    v->obj.emplace_back(std::move(k), Json());
                    if (!value(&v->obj.back().second, depth + 1)) return false;
                } while (take(','));
                return take('}');
            }
            case '[': {
                ++p_; v->kind = Json::Arr;
                if (take(']')) return true;
                do { v->arr.emplace_back(); if (!value(&v->arr.back(), depth + 1)) return false; } while (take(','));
                return take(']');
            }
            case '"': v->kind = Json::Str; return string(&v->str);
            case 't': v->kind = Json::Bool; v->b = true; return word("true");
            case 'f': v->kind = Json::Bool; v->b = false; return word("false");
            case 'n': v->kind = Json::Null; return word("null");
            default: return number(v);
        }
    }
    bool number(Json* v) {
        const char* s = p_;
        while (p_ < end_ && (strchr("+-.eE", *p_) || (*p_ >= '0' && *p_ <= '9'))) ++p_;
        if (p_ == s) return false;
        const std::string t(s, p_);
        char* stop = nullptr;
        v->kind = Json::Num; v->num = strtod(t.c_str(), &stop);
        return stop == t.c_str() + t.size();
    }
    static void utf8(std::string* o, unsigned c) {
        if (c < 0x80) *o += (char)c;
        else if (c < 0x800) { *o += (char)(0xc0 | c >> 6); *o += (char)(0x80 | (c & 63)); }
        else if (c < 0x10000) { *o += (char)(0xe0 | c >> 12); *o += (char)(0x80 | (c >> 6 & 63)); *o += (char)(0x80 | (c & 63)); }
        else { *o += (char)(0xf0 | c >> 18); *o += (char)(0x80 | (c >> 12 & 63)); *o += (char)(0x80 | (c >> 6 & 63)); *o += (char)(0x80 | (c & 63)); }
    }
    bool hex4(unsigned* c) {
        if (end_ - p_ < 4) return false;
        *c = 0;
        for (int i = 0; i < 4; ++i, ++p_) {
            const char h = *p_;
            const int d = h >= '0' && h <= '9' ? h - '0' : h >= 'a' && h <= 'f' ? h - 'a' + 10 : h >= 'A' && h <= 'F' ? h - 'A' + 10 : -1;
            if (d < 0) return false;
            *c = *c * 16 + (unsigned)d;
        }
        return true;
    }
    bool string(std::string* o) {
        if (p_ >= end_ || *p_ != '"') return false;
        ++p_;
        while (p_ < end_ && *p_ != '"') {
            if (*p_ != '\\') { *o += *p_++; continue; }
            if (++p_ >= end_) return false;
            switch (*p_++) {
                case '"': *o += '"'; break;
                case '\\': *o += '\\'; break;
                case '/': *o += '/'; break;
                case 'b': *o += '\b'; break;
                case 'f': *o += '\f'; break;
                case 'n': *o += '\n'; break;
                case 'r': *o += '\r'; break;
                case 't': *o += '\t'; break;
                case 'u': {
                    unsigned c, d;
                    if (!hex4(&c)) return false;
                    if (c >= 0xd800 && c < 0xdc00 && end_ - p_ >= 6 && p_[0] == '\\' && p_[1] == 'u') { p_ += 2; if (!hex4(&d)) return false; c = 0x10000 + ((c - 0xd800) << 10) + (d - 0xdc00); }
                    utf8(o, c);
                    break;
                }
                default: return false;
            }
        }
        return take_quote();
    }
    bool take_quote() { if (p_ < end_ && *p_ == '"') { ++p_; return true; } return false; }
    const char *p_, *end_;
};

}  // namespace cq
