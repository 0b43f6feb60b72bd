// A small JSON reader (host code): the token-level pieces the safetensors header is parsed with, and a
// document tree for configuration files.
#pragma once
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

struct JsonValue {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<JsonValue> items;                           // Array
    std::vector<std::pair<std::string, JsonValue>> members; // Object, in file order
    const JsonValue *get(const char *key) const { // null when absent (or not an object)
        for (const auto &m : members)
            if (m.first == key) return &m.second;
        return nullptr;
    }
};

struct Json {
    const char *p, *e;
    bool ok = true;
    void ws() {
        while (p < e && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p;
    }
    bool eat(char c) {
        ws();
        if (p < e && *p == c) { ++p; return true; }
        return false;
    }
    bool str(std::string &out) {
        ws();
        if (p >= e || *p != '"') return ok = false;
        ++p;
        out.clear();
        while (p < e && *p != '"') {
            if (*p == '\\') {
                if (++p >= e) return ok = false;
                switch (*p) {
                    case 'n': out += '\n'; break;
                    case 't': out += '\t'; break;
                    case 'r': out += '\r'; break;
                    case 'b': out += '\b'; break;
                    case 'f': out += '\f'; break;
                    case 'u': { // basic multilingual plane -> UTF-8
                        if (e - p < 5) return ok = false;
                        unsigned v = 0;
                        for (int i = 1; i <= 4; ++i) {
                            const char h = p[i];
                            v <<= 4;
                            if (h >= '0' && h <= '9') v |= h - '0';
                            else if (h >= 'a' && h <= 'f') v |= h - 'a' + 10;
                            else if (h >= 'A' && h <= 'F') v |= h - 'A' + 10;
                            else return ok = false;
                        }
                        p += 4;
                        if (v < 0x80) out += (char)v;
                        else if (v < 0x800) { out += (char)(0xC0 | (v >> 6)); out += (char)(0x80 | (v & 0x3F)); }
                        else { out += (char)(0xE0 | (v >> 12)); out += (char)(0x80 | ((v >> 6) & 0x3F)); out += (char)(0x80 | (v & 0x3F)); }
                        break;
                    }
                    default: out += *p; // \" \\ \/
                }
                ++p;
            } else {
                out += *p++;
            }
        }
        if (p >= e) return ok = false;
        ++p;
        return true;
    }
    bool uint(size_t &v) {
        ws();
        if (p >= e || *p < '0' || *p > '9') return ok = false;
        v = 0;
        while (p < e && *p >= '0' && *p <= '9') v = v * 10 + (size_t)(*p++ - '0');
        return true;
    }
    bool skip() { // any value
        ws();
        if (p >= e) return ok = false;
        if (*p == '"') { std::string s; return str(s); }
        if (*p == '{' || *p == '[') {
            const char close = *p == '{' ? '}' : ']';
            const bool obj = *p == '{';
            ++p;
            if (eat(close)) return true;
            do {
                if (obj) { std::string k; if (!str(k) || !eat(':')) return ok = false; }
                if (!skip()) return false;
            } while (eat(','));
            return eat(close) ? true : (ok = false);
        }
        while (p < e && *p != ',' && *p != '}' && *p != ']') ++p; // number / true / false / null
        return true;
    }
    bool number(double &v) {
        ws();
        const char *s = p;
        while (p < e && ((*p >= '0' && *p <= '9') || *p == '-' || *p == '+' || *p == '.' || *p == 'e' || *p == 'E')) ++p;
        if (s == p) return ok = false;
        const std::string t(s, p);
        char *end = nullptr;
        v = strtod(t.c_str(), &end);
        return end && !*end ? true : (ok = false);
    }
    bool word(const char *w) {
        const char *q = p;
        while (*w && q < e && *q == *w) { ++q; ++w; }
        if (*w) return false;
        p = q;
        return true;
    }
    bool value(JsonValue &v, int depth = 0) {
        ws();
        if (p >= e || depth > 64) return ok = false;
        if (*p == '"') { v.kind = JsonValue::String; return str(v.str); }
        if (eat('{')) {
            v.kind = JsonValue::Object;
            if (eat('}')) return true;
            do {
                v.members.emplace_back();
                if (!str(v.members.back().first) || !eat(':') || !value(v.members.back().second, depth + 1)) return ok = false;
            } while (eat(','));
            return eat('}') ? true : (ok = false);
        }
        if (eat('[')) {
            v.kind = JsonValue::Array;
            if (eat(']')) return true;
            do {
                v.items.emplace_back();
                if (!value(v.items.back(), depth + 1)) return ok = false;
            } while (eat(','));
            return eat(']') ? true : (ok = false);
        }
        if (word("true")) { v.kind = JsonValue::Bool; v.b = true; return true; }
        if (word("false")) { v.kind = JsonValue::Bool; return true; }
        if (word("null")) return true;
        v.kind = JsonValue::Number;
        return number(v.num);
    }
};
