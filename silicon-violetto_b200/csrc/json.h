// A small JSON reader: enough for a model folder's config.json and a safetensors header.
#pragma once
#include <cmath>
#include <cstdlib>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "common.h"

namespace vlt {

struct Json {
    enum class Kind { Null, Bool, Number, String, Array, Object } kind = Kind::Null;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> items;
    std::map<std::string, Json> fields;

    bool is_null() const { return kind == Kind::Null; }
    // A field that is absent, or null, is null.
    const Json& operator[](const std::string& key) const {
        static const Json none;
        auto it = fields.find(key);
        return it == fields.end() ? none : it->second;
    }
    const Json& at(const std::string& key) const {
        auto it = fields.find(key);
        if (it == fields.end()) throw Error("config: no field `" + key + "`");
        return it->second;
    }
    double number(const std::string& what) const {
        if (kind != Kind::Number) throw Error("config: `" + what + "` is not a number");
        return num;
    }
    uint32_t count(const std::string& what) const {  // a whole number that fits a size
        const double v = number(what);
        if (!(v >= 0 && v <= 4294967295.0) || v != std::floor(v)) throw Error("config: `" + what + "` is not a size");
        return uint32_t(v);
    }
    bool flag(const std::string& what) const {  // (absent or null: no)
        if (kind != Kind::Bool && kind != Kind::Null) throw Error("config: `" + what + "` is neither true nor false");
        return kind == Kind::Bool && b;
    }
    const std::string& text(const std::string& what) const {
        if (kind != Kind::String) throw Error("config: `" + what + "` is not a string");
        return str;
    }

    static Json parse(const char* s, size_t n, const std::string& where) {
        Parser p{s, s + n, where, 0};
        Json v = p.value();
        p.space();
        if (p.at != p.end) p.fail("text after the value");
        return v;
    }

  private:
    struct Parser {
        const char *at, *end;
        const std::string& where;
        int depth;
        [[noreturn]] void fail(const char* what) const { throw Error(where + ": not valid JSON (" + what + ")"); }
        void space() { while (at != end && (*at == ' ' || *at == '\n' || *at == '\t' || *at == '\r')) at++; }
        char peek() {
            space();
            if (at == end) fail("it ends early");
            return *at;
        }
        void expect(char c) {
            if (peek() != c) fail("a character is missing");
            at++;
        }
        bool word(const char* w) {
            const size_t n = std::strlen(w);
            if (size_t(end - at) < n || std::memcmp(at, w, n) != 0) return false;
            at += n;
            return true;
        }
        std::string string() {
            expect('"');
            std::string out;
            for (;;) {
                if (at == end) fail("an open string");
                char c = *at++;
                if (c == '"') return out;
                if (c != '\\') { out += c; continue; }
                if (at == end) fail("an open string");
                c = *at++;
                switch (c) {
                case 'n': out += '\n'; break;
                case 't': out += '\t'; break;
                case 'r': out += '\r'; break;
                case 'b': out += '\b'; break;
                case 'f': out += '\f'; break;
                case 'u': {
                    if (end - at < 4) fail("a short escape");
                    const uint32_t u = uint32_t(std::strtoul(std::string(at, 4).c_str(), nullptr, 16));
                    at += 4;
                    if (u < 0x80) out += char(u);
                    else if (u < 0x800) { out += char(0xC0 | u >> 6); out += char(0x80 | (u & 63)); }
                    else { out += char(0xE0 | u >> 12); out += char(0x80 | (u >> 6 & 63)); out += char(0x80 | (u & 63)); }
                    break;
                }
                default: out += c;
                }
            }
        }
        Json value() {
            if (++depth > 64) fail("too deep");
            Json v;
            const char c = peek();
            if (c == '{') {
                v.kind = Kind::Object;
                at++;
                if (peek() == '}') at++;
                else
                    for (;;) {
                        std::string key = string();
                        expect(':');
                        v.fields[key] = value();
                        if (peek() == ',') { at++; peek(); continue; }
                        expect('}');
                        break;
                    }
            } else if (c == '[') {
                v.kind = Kind::Array;
                at++;
                if (peek() == ']') at++;
                else
                    for (;;) {
                        v.items.push_back(value());
                        if (peek() == ',') { at++; continue; }
                        expect(']');
                        break;
                    }
            } else if (c == '"') {
                v.kind = Kind::String;
                v.str = string();
            } else if (word("true")) {
                v.kind = Kind::Bool;
                v.b = true;
            } else if (word("false")) {
                v.kind = Kind::Bool;
            } else if (word("null")) {
            } else {
                const char* s = at;
                while (at != end && (std::strchr("+-.eE", *at) || (*at >= '0' && *at <= '9'))) at++;
                const std::string t(s, at);
                char* stop = nullptr;
                v.kind = Kind::Number;
                v.num = std::strtod(t.c_str(), &stop);
                if (t.empty() || *stop) fail("a bad number");
            }
            depth--;
            return v;
        }
    };
};

}  // namespace vlt
