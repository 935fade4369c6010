// A small JSON reader (host only): enough for model configuration files and safetensors headers.
#pragma once
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace l2b {

struct JsonValue {
    enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<JsonValue> items;                            // ARRAY
    std::vector<std::pair<std::string, JsonValue>> members;  // OBJECT, in file order
    const JsonValue* find(const char* key) const {           // null when absent or when this is not an object
        if (kind == OBJECT)
            for (const auto& m : members)
                if (m.first == key) return &m.second;
        return nullptr;
    }
    bool is_null() const { return kind == NUL; }
};

class JsonParser {
public:
    // Parses the whole of [text, text + n); false on anything malformed.
    static bool parse(const char* text, size_t n, JsonValue& out) {
        JsonParser p(text, n);
        if (!p.value(out, 0)) return false;
        p.space();
        return p.i_ == n;
    }

private:
    JsonParser(const char* t, size_t n) : t_(t), n_(n) {}
    void space() {
        while (i_ < n_ && (t_[i_] == ' ' || t_[i_] == '\n' || t_[i_] == '\t' || t_[i_] == '\r')) ++i_;
    }
    bool word(const char* w) {
        const size_t k = strlen(w);
        if (n_ - i_ < k || memcmp(t_ + i_, w, k) != 0) return false;
        i_ += k;
        return true;
    }
    bool string(std::string& s) {
        if (i_ >= n_ || t_[i_] != '"') return false;
        ++i_;
        while (i_ < n_ && t_[i_] != '"') {
            char c = t_[i_++];
            if (c != '\\') {
                s.push_back(c);
                continue;
            }
            if (i_ >= n_) return false;
            c = t_[i_++];
            switch (c) {
                case 'n': s.push_back('\n'); break;
                case 't': s.push_back('\t'); break;
                case 'r': s.push_back('\r'); break;
                case 'b': s.push_back('\b'); break;
                case 'f': s.push_back('\f'); break;
                case 'u': {  // a code unit below 0x800 as UTF-8; others (not found in keys or names) as three bytes
                    if (n_ - i_ < 4) return false;
                    const unsigned u = (unsigned)strtoul(std::string(t_ + i_, 4).c_str(), nullptr, 16);
                    i_ += 4;
                    if (u < 0x80) s.push_back((char)u);
                    else if (u < 0x800) { s.push_back((char)(0xC0 | (u >> 6))); s.push_back((char)(0x80 | (u & 63))); }
                    else { s.push_back((char)(0xE0 | (u >> 12))); s.push_back((char)(0x80 | ((u >> 6) & 63))); s.push_back((char)(0x80 | (u & 63))); }
                    break;
                }
                default: s.push_back(c);
            }
        }
        if (i_ >= n_) return false;
        ++i_;
        return true;
    }
    bool value(JsonValue& v, int depth) {
        if (depth > 64) return false;
        space();
        if (i_ >= n_) return false;
        const char c = t_[i_];
        if (c == '{') {
            v.kind = JsonValue::OBJECT;
            ++i_;
            space();
            if (i_ < n_ && t_[i_] == '}') return ++i_, true;
            for (;;) {
                space();
                v.members.emplace_back();
                if (!string(v.members.back().first)) return false;
                space();
                if (i_ >= n_ || t_[i_++] != ':') return false;
                if (!value(v.members.back().second, depth + 1)) return false;
                space();
                if (i_ >= n_) return false;
                if (t_[i_] == '}') return ++i_, true;
                if (t_[i_++] != ',') return false;
            }
        }
        if (c == '[') {
            v.kind = JsonValue::ARRAY;
            ++i_;
            space();
            if (i_ < n_ && t_[i_] == ']') return ++i_, true;
            for (;;) {
                v.items.emplace_back();
                if (!value(v.items.back(), depth + 1)) return false;
                space();
                if (i_ >= n_) return false;
                if (t_[i_] == ']') return ++i_, true;
                if (t_[i_++] != ',') return false;
            }
        }
        if (c == '"') {
            v.kind = JsonValue::STRING;
            return string(v.str);
        }
        if (c == 't') { v.kind = JsonValue::BOOL; v.b = true; return word("true"); }
        if (c == 'f') { v.kind = JsonValue::BOOL; v.b = false; return word("false"); }
        if (c == 'n') { v.kind = JsonValue::NUL; return word("null"); }
        size_t e = i_;
        while (e < n_ && strchr("+-.0123456789eE", t_[e])) ++e;
        if (e == i_) return false;
        const std::string s(t_ + i_, e - i_);
        char* end = nullptr;
        v.kind = JsonValue::NUMBER;
        v.num = strtod(s.c_str(), &end);
        i_ = e;
        return end && *end == 0;
    }
    const char* t_;
    size_t n_, i_ = 0;
};

}  // namespace l2b
