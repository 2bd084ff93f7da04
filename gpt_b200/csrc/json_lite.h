// A small JSON reader for configuration files and safetensors headers (host only, no dependencies).
// Numbers are kept as double (exact for the integers that occur).  Errors throw std::runtime_error with the byte position.
#pragma once

#include <cctype>
#include <cstdlib>
#include <map>
#include <memory>
#include <stdexcept>
#include <string>
#include <vector>

namespace gptb200 {

struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool boolean = false;
    double number = 0.0;
    std::string string;
    std::vector<Json> items;
    std::map<std::string, Json> fields;

    bool is_null() const { return kind == Null; }
    bool has(const std::string &key) const { return kind == Object && fields.count(key) && !fields.at(key).is_null(); }
    const Json &at(const std::string &key) const
    {
        if (kind != Object || !fields.count(key)) throw std::runtime_error("missing key '" + key + "'");
        return fields.at(key);
    }
    double num(const std::string &key) const
    {
        const Json &v = at(key);
        if (v.kind != Number) throw std::runtime_error("'" + key + "' is not a number");
        return v.number;
    }
    // a positive integer that fits an int
    int size(const std::string &key) const
    {
        const double v = num(key);
        if (!(v >= 1.0 && v <= 2147483647.0) || v != static_cast<double>(static_cast<long long>(v))) throw std::runtime_error("'" + key + "' is not a positive integer");
        return static_cast<int>(v);
    }
    bool flag(const std::string &key) const
    {
        const Json &v = at(key);
        if (v.kind != Bool) throw std::runtime_error("'" + key + "' is not true or false");
        return v.boolean;
    }
    const std::string &str(const std::string &key) const
    {
        const Json &v = at(key);
        if (v.kind != String) throw std::runtime_error("'" + key + "' is not a string");
        return v.string;
    }

    static Json parse(const std::string &text)
    {
        Parser p{text, 0, 0};
        Json v = p.value();
        p.space();
        if (p.at != text.size()) p.fail("trailing characters");
        return v;
    }

private:
    struct Parser {
        const std::string &s;
        size_t at;
        int depth;
        [[noreturn]] void fail(const char *what) const { throw std::runtime_error(std::string("JSON: ") + what + " at byte " + std::to_string(at)); }
        void space()
        {
            while (at < s.size() && (s[at] == ' ' || s[at] == '\n' || s[at] == '\t' || s[at] == '\r')) ++at;
        }
        char peek()
        {
            space();
            if (at >= s.size()) fail("unexpected end");
            return s[at];
        }
        void expect(char c)
        {
            if (peek() != c) fail("unexpected character");
            ++at;
        }
        bool word(const char *w)
        {
            const size_t n = std::string(w).size();
            if (s.compare(at, n, w) != 0) return false;
            at += n;
            return true;
        }
        std::string text()
        {
            expect('"');
            std::string out;
            while (true) {
                if (at >= s.size()) fail("unterminated string");
                const char c = s[at++];
                if (c == '"') return out;
                if (c != '\\') {
                    out += c;
                    continue;
                }
                if (at >= s.size()) fail("unterminated string");
                const char e = s[at++];
                switch (e) {
                    case 'n': out += '\n'; break;
                    case 't': out += '\t'; break;
                    case 'r': out += '\r'; break;
                    case 'b': out += '\b'; break;
                    case 'f': out += '\f'; break;
                    case 'u': {
                        if (at + 4 > s.size()) fail("bad escape");
                        const unsigned u = static_cast<unsigned>(strtoul(s.substr(at, 4).c_str(), nullptr, 16));
                        at += 4;
                        if (u < 0x80) {
                            out += static_cast<char>(u);
                        } else if (u < 0x800) {
                            out += static_cast<char>(0xC0 | (u >> 6));
                            out += static_cast<char>(0x80 | (u & 0x3F));
                        } else {
                            out += static_cast<char>(0xE0 | (u >> 12));
                            out += static_cast<char>(0x80 | ((u >> 6) & 0x3F));
                            out += static_cast<char>(0x80 | (u & 0x3F));
                        }
                        break;
                    }
                    default: out += e;   // quote, backslash, slash
                }
            }
        }
        Json value()
        {
            if (++depth > 64) fail("nested too deeply");
            Json v;
            const char c = peek();
            if (c == '{') {
                v.kind = Object;
                ++at;
                if (peek() == '}') {
                    ++at;
                } else {
                    while (true) {
                        space();
                        const std::string key = text();
                        expect(':');
                        v.fields[key] = value();
                        if (peek() == ',') { ++at; continue; }
                        expect('}');
                        break;
                    }
                }
            } else if (c == '[') {
                v.kind = Array;
                ++at;
                if (peek() == ']') {
                    ++at;
                } else {
                    while (true) {
                        v.items.push_back(value());
                        if (peek() == ',') { ++at; continue; }
                        expect(']');
                        break;
                    }
                }
            } else if (c == '"') {
                v.kind = String;
                v.string = text();
            } else if (word("true")) {
                v.kind = Bool;
                v.boolean = true;
            } else if (word("false")) {
                v.kind = Bool;
            } else if (word("null")) {
                v.kind = Null;
            } else {
                char *end = nullptr;
                v.kind = Number;
                v.number = strtod(s.c_str() + at, &end);
                if (end == s.c_str() + at) fail("unexpected character");
                at = static_cast<size_t>(end - s.c_str());
            }
            --depth;
            return v;
        }
    };
};

}  // namespace gptb200
