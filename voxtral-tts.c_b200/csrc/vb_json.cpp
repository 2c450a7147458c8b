/* vb_json.cpp - recursive-descent JSON reader (vb_json.h). */
#include "vb_json.h"

#include <stdint.h>
#include <stdlib.h>
#include <string.h>

namespace vb {

const Json *Json::get(const char *key) const {
    if (kind != OBJECT) return nullptr;
    for (const auto &m : members)
        if (m.first == key) return m.second.kind == NIL ? nullptr : &m.second;
    return nullptr;
}

namespace {

constexpr int kMaxDepth = 64;

struct Reader {
    const char *p, *end;
    const char *error = nullptr;

    bool fail(const char *what) {
        if (!error) error = what;
        return false;
    }
    void space() {
        while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
    }
    bool word(const char *w) {
        const size_t n = strlen(w);
        if ((size_t)(end - p) < n || memcmp(p, w, n) != 0) return fail("unknown word");
        p += n;
        return true;
    }
    bool hex4(uint32_t *v) {
        if (end - p < 4) return fail("short \\u escape");
        *v = 0;
        for (int i = 0; i < 4; i++, p++) {
            const char c = *p;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return fail("bad \\u escape");
            *v = *v * 16 + (uint32_t)d;
        }
        return true;
    }
    static void utf8(std::string *s, uint32_t c) {
        if (c < 0x80) *s += (char)c;
        else if (c < 0x800) { *s += (char)(0xC0 | (c >> 6)); *s += (char)(0x80 | (c & 63)); }
        else if (c < 0x10000) { *s += (char)(0xE0 | (c >> 12)); *s += (char)(0x80 | ((c >> 6) & 63)); *s += (char)(0x80 | (c & 63)); }
        else { *s += (char)(0xF0 | (c >> 18)); *s += (char)(0x80 | ((c >> 12) & 63)); *s += (char)(0x80 | ((c >> 6) & 63)); *s += (char)(0x80 | (c & 63)); }
    }
    bool string(std::string *out) {
        p++;                                             /* opening quote */
        while (true) {
            if (p >= end) return fail("unterminated string");
            const char c = *p++;
            if (c == '"') return true;
            if (c != '\\') { *out += c; continue; }
            if (p >= end) return fail("unterminated string");
            const char e = *p++;
            uint32_t u = 0;
            switch (e) {
            case 'n': *out += '\n'; break;
            case 't': *out += '\t'; break;
            case 'r': *out += '\r'; break;
            case 'b': *out += '\b'; break;
            case 'f': *out += '\f'; break;
            case '"': case '\\': case '/': *out += e; break;
            case 'u':
                if (!hex4(&u)) return false;
                if (u >= 0xD800 && u < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {
                    uint32_t lo = 0;
                    p += 2;
                    if (!hex4(&lo)) return false;
                    u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
                }
                utf8(out, u);
                break;
            default: return fail("unknown escape");
            }
        }
    }
    bool value(Json *v, int depth) {
        if (depth > kMaxDepth) return fail("nested too deeply");
        space();
        if (p >= end) return fail("value missing");
        switch (*p) {
        case '{': {
            v->kind = Json::OBJECT;
            p++;
            space();
            if (p < end && *p == '}') { p++; return true; }
            while (true) {
                space();
                if (p >= end || *p != '"') return fail("member name expected");
                std::string name;
                if (!string(&name)) return false;
                space();
                if (p >= end || *p != ':') return fail("':' expected");
                p++;
                v->members.emplace_back(std::move(name), Json());
                if (!value(&v->members.back().second, depth + 1)) return false;
                space();
                if (p < end && *p == ',') { p++; continue; }
                if (p < end && *p == '}') { p++; return true; }
                return fail("',' or '}' expected");
            }
        }
        case '[': {
            v->kind = Json::ARRAY;
            p++;
            space();
            if (p < end && *p == ']') { p++; return true; }
            while (true) {
                v->items.emplace_back();
                if (!value(&v->items.back(), depth + 1)) return false;
                space();
                if (p < end && *p == ',') { p++; continue; }
                if (p < end && *p == ']') { p++; return true; }
                return fail("',' or ']' expected");
            }
        }
        case '"': v->kind = Json::STRING; return string(&v->text);
        case 't': v->kind = Json::BOOL; v->truth = true; return word("true");
        case 'f': v->kind = Json::BOOL; return word("false");
        case 'n': v->kind = Json::NIL; return word("null");
        default: {
            char buf[64];
            size_t n = 0;
            while (p < end && n + 1 < sizeof(buf) && (strchr("+-.eE", *p) || (*p >= '0' && *p <= '9'))) buf[n++] = *p++;
            buf[n] = 0;
            char *stop = nullptr;
            v->kind = Json::NUMBER;
            v->number = strtod(buf, &stop);
            if (n == 0 || stop != buf + n) return fail("number expected");
            return true;
        }
        }
    }
};

} // namespace

bool json_parse(const char *text, size_t n, Json *out, std::string *err) {
    Reader r{text, text + n};
    *out = Json();
    bool ok = r.value(out, 0);
    if (ok) {
        r.space();
        if (r.p != r.end && *r.p != 0) ok = r.fail("text after the value");
    }
    if (!ok && err) *err = std::string(r.error ? r.error : "malformed") + " at byte " + std::to_string(r.p - text);
    return ok;
}

} // namespace vb
