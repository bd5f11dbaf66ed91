// Small JSON reader for model configurations and safetensors headers: one recursive-descent pass into a value tree.
// Host code only.
#pragma once

#include <cctype>
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace qbjson {

struct Value {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0.0;
    std::string s;
    std::vector<Value> items;                                // array elements
    std::vector<std::pair<std::string, Value>> members;      // object members in file order

    const Value *get(const char *key) const {
        if (kind == Object)
            for (const auto &m : members) if (m.first == key) return &m.second;
        return nullptr;
    }
    bool is_null() const { return kind == Null; }
};

class Parser {
public:
    Parser(const char *p, size_t n) : p_(p), end_(p + n) {}
    // False on malformed input or anything but blanks after the value.
    bool parse(Value &out) {
        if (!value(out, 0)) return false;
        blanks();
        return p_ == end_;
    }

private:
    const char *p_, *end_;
    static constexpr int MAX_DEPTH = 64;

    void blanks() { while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_; }
    bool lit(const char *w) {
        const size_t n = strlen(w);
        if ((size_t)(end_ - p_) < n || strncmp(p_, w, n) != 0) return false;
        p_ += n;
        return true;
    }
    static void put_utf8(std::string &s, uint32_t c) {
        if (c < 0x80) s += (char)c;
        else if (c < 0x800) { s += (char)(0xC0 | c >> 6); s += (char)(0x80 | (c & 63)); }
        else if (c < 0x10000) { s += (char)(0xE0 | c >> 12); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
        else { s += (char)(0xF0 | c >> 18); s += (char)(0x80 | (c >> 12 & 63)); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
    }
    bool hex4(uint32_t &v) {
        if (end_ - p_ < 4) return false;
        v = 0;
        for (int i = 0; i < 4; ++i, ++p_) {
            if (!isxdigit((unsigned char)*p_)) return false;
            v = v * 16 + (uint32_t)(*p_ <= '9' ? *p_ - '0' : (*p_ | 32) - 'a' + 10);
        }
        return true;
    }
    bool string(std::string &s) {
        if (p_ >= end_ || *p_ != '"') return false;
        ++p_;
        while (p_ < end_ && *p_ != '"') {
            if (*p_ != '\\') { s += *p_++; continue; }
            if (++p_ >= end_) return false;
            const char e = *p_++;
            switch (e) {
                case 'n': s += '\n'; break;
                case 't': s += '\t'; break;
                case 'r': s += '\r'; break;
                case 'b': s += '\b'; break;
                case 'f': s += '\f'; break;
                case '"': case '\\': case '/': s += e; break;
                case 'u': {
                    uint32_t c, d;
                    if (!hex4(c)) return false;
                    if (c >= 0xD800 && c < 0xDC00) {
                        if (!lit("\\u") || !hex4(d) || d < 0xDC00 || d > 0xDFFF) return false;
                        c = 0x10000 + ((c - 0xD800) << 10) + (d - 0xDC00);
                    }
                    put_utf8(s, c);
                    break;
                }
                default: return false;
            }
        }
        if (p_ >= end_) return false;
        ++p_;
        return true;
    }
    bool number(double &v) {
        const char *q = p_;
        while (q < end_ && (isdigit((unsigned char)*q) || *q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
        if (q == p_) return false;
        const std::string t(p_, q);
        char *stop = nullptr;
        v = strtod(t.c_str(), &stop);
        if (!stop || *stop) return false;
        p_ = q;
        return true;
    }
    bool value(Value &v, int depth) {
        if (depth > MAX_DEPTH) return false;
        blanks();
        if (p_ >= end_) return false;
        switch (*p_) {
            case '{':
                v.kind = Value::Object;
                ++p_;
                blanks();
                if (p_ < end_ && *p_ == '}') { ++p_; return true; }
                for (;;) {
                    std::pair<std::string, Value> m;
                    blanks();
                    if (!string(m.first)) return false;
                    blanks();
                    if (p_ >= end_ || *p_++ != ':') return false;
                    if (!value(m.second, depth + 1)) return false;
                    v.members.push_back(std::move(m));
                    blanks();
                    if (p_ >= end_) return false;
                    if (*p_ == ',') { ++p_; continue; }
                    return *p_++ == '}';
                }
            case '[':
                v.kind = Value::Array;
                ++p_;
                blanks();
                if (p_ < end_ && *p_ == ']') { ++p_; return true; }
                for (;;) {
                    v.items.emplace_back();
                    if (!value(v.items.back(), depth + 1)) return false;
                    blanks();
                    if (p_ >= end_) return false;
                    if (*p_ == ',') { ++p_; continue; }
                    return *p_++ == ']';
                }
            case '"': v.kind = Value::String; return string(v.s);
            case 't': v.kind = Value::Bool; v.b = true; return lit("true");
            case 'f': v.kind = Value::Bool; return lit("false");
            case 'n': v.kind = Value::Null; return lit("null");
            default: v.kind = Value::Number; return number(v.num);
        }
    }
};

}  // namespace qbjson
