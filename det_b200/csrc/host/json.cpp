#include "json.hpp"
#include <cmath>
#include <cstdlib>
#include <stdexcept>

namespace det {

namespace {
struct Parser {
    const char* p;
    const char* begin;
    const char* end;
    int depth = 0;

    [[noreturn]] void fail(const char* what) const {
        throw std::runtime_error(std::string("JSON: ") + what + " at offset " + std::to_string(p - begin));
    }
    void space() {
        while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
    }
    bool eat(char c) {
        space();
        if (p < end && *p == c) {
            p++;
            return true;
        }
        return false;
    }
    void word(const char* w) {
        for (; *w; w++, p++)
            if (p >= end || *p != *w) fail("bad literal");
    }
    unsigned hex4() {
        unsigned v = 0;
        for (int i = 0; i < 4; i++, p++) {
            if (p >= end) fail("bad escape");
            const char c = *p;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) fail("bad escape");
            v = v * 16 + (unsigned)d;
        }
        return v;
    }
    static void utf8(std::string& s, unsigned c) {
        if (c < 0x80) s += (char)c;
        else if (c < 0x800) {
            s += (char)(0xC0 | (c >> 6));
            s += (char)(0x80 | (c & 63));
        } else if (c < 0x10000) {
            s += (char)(0xE0 | (c >> 12));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        } else {
            s += (char)(0xF0 | (c >> 18));
            s += (char)(0x80 | ((c >> 12) & 63));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        }
    }
    std::string text() {
        std::string s;
        if (p >= end || *p != '"') fail("expected a string");
        for (p++;; p++) {
            if (p >= end) fail("unterminated string");
            if (*p == '"') break;
            if (*p != '\\') {
                s += *p;
                continue;
            }
            if (++p >= end) fail("bad escape");
            switch (*p) {
                case 'b': s += '\b'; break;
                case 'f': s += '\f'; break;
                case 'n': s += '\n'; break;
                case 'r': s += '\r'; break;
                case 't': s += '\t'; break;
                case 'u': {
                    p++;
                    unsigned c = hex4();
                    if (c >= 0xD800 && c < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {
                        p += 2;
                        c = 0x10000 + ((c - 0xD800) << 10) + (hex4() - 0xDC00);
                    }
                    utf8(s, c);
                    p--;
                    break;
                }
                default: s += *p;   // quote, backslash, slash
            }
        }
        p++;
        return s;
    }
    Json value() {
        if (++depth > 64) fail("nested too deeply");
        space();
        if (p >= end) fail("unexpected end");
        Json j;
        switch (*p) {
            case '{':
                j.kind = Json::Object;
                p++;
                if (eat('}')) break;
                do {
                    space();
                    std::string key = text();
                    if (!eat(':')) fail("expected ':'");
                    j.members.emplace_back(std::move(key), value());
                } while (eat(','));
                if (!eat('}')) fail("expected '}'");
                break;
            case '[':
                j.kind = Json::Array;
                p++;
                if (eat(']')) break;
                do j.items.push_back(value());
                while (eat(','));
                if (!eat(']')) fail("expected ']'");
                break;
            case '"':
                j.kind = Json::String;
                j.str = text();
                break;
            case 't': word("true"); j.kind = Json::Bool; j.b = true; break;
            case 'f': word("false"); j.kind = Json::Bool; break;
            case 'n': word("null"); break;
            default: {
                const char* q = p;
                while (q < end && (std::string("+-.eE").find(*q) != std::string::npos || (*q >= '0' && *q <= '9'))) q++;
                const std::string n(p, q);
                char* stop = nullptr;
                j.kind = Json::Number;
                j.num = std::strtod(n.c_str(), &stop);
                if (n.empty() || *stop) fail("bad number");
                p = q;
            }
        }
        depth--;
        return j;
    }
};
}  // namespace

Json Json::parse(const char* text, size_t len) {
    Parser ps{text, text, text + len};
    Json j = ps.value();
    ps.space();
    if (ps.p != ps.end) ps.fail("trailing characters");
    return j;
}
const Json* Json::find(const std::string& key) const {
    for (const auto& m : members)
        if (m.first == key) return &m.second;
    return nullptr;
}
const Json& Json::at(const std::string& key) const {
    const Json* j = find(key);
    if (!j) throw std::runtime_error("'" + key + "' is missing");
    return *j;
}
double Json::number(const std::string& key) const {
    const Json& j = at(key);
    if (j.kind != Number) throw std::runtime_error("'" + key + "' is not a number");
    return j.num;
}
size_t Json::size(const std::string& key) const {
    const double v = number(key);
    if (v < 0 || v != std::floor(v) || v > 1e15) throw std::runtime_error("'" + key + "' is not a size");
    return (size_t)v;
}
const std::string& Json::string(const std::string& key) const {
    const Json& j = at(key);
    if (j.kind != String) throw std::runtime_error("'" + key + "' is not a string");
    return j.str;
}

}  // namespace det
