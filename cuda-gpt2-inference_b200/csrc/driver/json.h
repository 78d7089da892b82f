// A small JSON reader: config.json and the header of a safetensors file.
#pragma once
#include <cstdlib>
#include <map>
#include <stdexcept>
#include <string>
#include <vector>

namespace b200 {

struct Json {
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::map<std::string, Json> obj;

    bool is_null() const { return kind == NUL; }
    bool has(const std::string& k) const { return kind == OBJ && obj.count(k) > 0; }
    // member k; throws std::runtime_error with the path if it is not there
    const Json& at(const std::string& k) const {
        auto it = obj.find(k);
        if (kind != OBJ || it == obj.end()) throw std::runtime_error("missing key '" + k + "'");
        return it->second;
    }
    double number(const std::string& k) const {
        const Json& j = at(k);
        if (j.kind != NUM) throw std::runtime_error("'" + k + "' is not a number");
        return j.num;
    }
    int integer(const std::string& k) const {
        const double d = number(k);
        const int i = (int)d;
        if ((double)i != d) throw std::runtime_error("'" + k + "' is not an integer");
        return i;
    }
    const std::string& string(const std::string& k) const {
        const Json& j = at(k);
        if (j.kind != STR) throw std::runtime_error("'" + k + "' is not a string");
        return j.str;
    }

    static Json parse(const char* p, const char* end) {
        Parser ps{p, end, 0};
        Json j = ps.value();
        ps.space();
        if (ps.p != ps.end) throw std::runtime_error("JSON: text behind the value");
        return j;
    }

   private:
    struct Parser {
        const char *p, *end;
        int depth;
        [[noreturn]] void fail(const char* what) { throw std::runtime_error(std::string("JSON: ") + what); }
        void space() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p; }
        char peek() { space(); if (p >= end) fail("unexpected end"); return *p; }
        void expect(char c) { if (peek() != c) fail("unexpected character"); ++p; }
        bool word(const char* w) {
            const char* q = p;
            while (*w) { if (q >= end || *q != *w) return false; ++q; ++w; }
            p = q;
            return true;
        }
        void utf8(unsigned u, std::string& s) {
            if (u < 0x80) s += (char)u;
            else if (u < 0x800) { s += (char)(0xC0 | u >> 6); s += (char)(0x80 | (u & 63)); }
            else if (u < 0x10000) { s += (char)(0xE0 | u >> 12); s += (char)(0x80 | (u >> 6 & 63)); s += (char)(0x80 | (u & 63)); }
            else { s += (char)(0xF0 | u >> 18); s += (char)(0x80 | (u >> 12 & 63)); s += (char)(0x80 | (u >> 6 & 63)); s += (char)(0x80 | (u & 63)); }
        }
        unsigned hex4() {
            if (end - p < 4) fail("bad escape");
            unsigned u = 0;
            for (int i = 0; i < 4; ++i, ++p) {
                const char c = *p;
                u = u * 16 + (c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : (fail("bad escape"), 0));
            }
            return u;
        }
        std::string text() {
            expect('"');
            std::string s;
            while (true) {
                if (p >= end) fail("unterminated string");
                char c = *p++;
                if (c == '"') return s;
                if (c != '\\') { s += c; continue; }
                if (p >= end) fail("unterminated string");
                c = *p++;
                switch (c) {
                    case 'n': s += '\n'; break;
                    case 't': s += '\t'; break;
                    case 'r': s += '\r'; break;
                    case 'b': s += '\b'; break;
                    case 'f': s += '\f'; break;
                    case 'u': {
                        unsigned u = hex4();
                        if (u >= 0xD800 && u < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {
                            p += 2;
                            u = 0x10000 + ((u - 0xD800) << 10) + (hex4() - 0xDC00);
                        }
                        utf8(u, s);
                        break;
                    }
                    default: s += c;
                }
            }
        }
        Json value() {
            if (++depth > 100) fail("nested too deeply");
            Json j;
            const char c = peek();
            if (c == '{') {
                j.kind = OBJ;
                ++p;
                if (peek() == '}') ++p;
                else
                    while (true) {
                        peek();
                        std::string k = text();
                        expect(':');
                        j.obj[k] = value();
                        if (peek() == ',') { ++p; continue; }
                        expect('}');
                        break;
                    }
            } else if (c == '[') {
                j.kind = ARR;
                ++p;
                if (peek() == ']') ++p;
                else
                    while (true) {
                        j.arr.push_back(value());
                        if (peek() == ',') { ++p; continue; }
                        expect(']');
                        break;
                    }
            } else if (c == '"') {
                j.kind = STR;
                j.str = text();
            } else if (word("true")) { j.kind = BOOL; j.b = true; }
            else if (word("false")) j.kind = BOOL;
            else if (word("null")) j.kind = NUL;
            else {
                std::string t;
                while (p < end && (std::string("+-.eE").find(*p) != std::string::npos || (*p >= '0' && *p <= '9'))) t += *p++;
                char* stop = nullptr;
                j.kind = NUM;
                j.num = strtod(t.c_str(), &stop);
                if (t.empty() || *stop) fail("bad number");
            }
            --depth;
            return j;
        }
    };
};

}  // namespace b200
