#include "json.h"

#include <cmath>
#include <cstdlib>
#include <cstring>

using namespace std;

struct json_parser {
    const char* at;
    const char* end;
    string error;
    static constexpr int kMaxDepth = 64;

    bool fail(const char* what) {
        if (error.empty()) error = what;
        return false;
    }
    void space() { while (at < end && (*at == ' ' || *at == '\t' || *at == '\n' || *at == '\r')) ++at; }
    bool literal(const char* s) {
        const size_t n = strlen(s);
        if (size_t(end - at) < n || memcmp(at, s, n) != 0) return fail("bad literal");
        at += n;
        return true;
    }
    static void utf8(string* out, u32 c) {
        if (c < 0x80) { *out += char(c); return; }
        if (c < 0x800) { *out += char(0xc0 | c >> 6); *out += char(0x80 | (c & 63)); return; }
        if (c < 0x10000) { *out += char(0xe0 | c >> 12); *out += char(0x80 | (c >> 6 & 63)); *out += char(0x80 | (c & 63)); return; }
        *out += char(0xf0 | c >> 18); *out += char(0x80 | (c >> 12 & 63)); *out += char(0x80 | (c >> 6 & 63)); *out += char(0x80 | (c & 63));
    }
    bool hex4(u32* out) {
        if (end - at < 4) return fail("bad escape");
        u32 v = 0;
        for (int i = 0; i < 4; ++i) {
            const char c = *at++;
            v = v * 16 + (c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : 99);
            if (v > 0xffff) return fail("bad escape");
        }
        *out = v;
        return true;
    }
    bool text(string* out) {
        ++at;                                              // opening quote
        while (at < end && *at != '"') {
            if (*at != '\\') { *out += *at++; continue; }
            if (++at == end) break;
            const char c = *at++;
            switch (c) {
                case 'n': *out += '\n'; break;
                case 't': *out += '\t'; break;
                case 'r': *out += '\r'; break;
                case 'b': *out += '\b'; break;
                case 'f': *out += '\f'; break;
                case '"': case '\\': case '/': *out += c; break;
                case 'u': {
                    u32 v = 0, w = 0;
                    if (!hex4(&v)) return false;
                    if (v >= 0xd800 && v < 0xdc00 && end - at >= 6 && at[0] == '\\' && at[1] == 'u') {
                        at += 2;
                        if (!hex4(&w)) return false;
                        v = 0x10000 + ((v - 0xd800) << 10) + ((w - 0xdc00) & 0x3ff);
                    }
                    utf8(out, v);
                    break;
                }
                default: return fail("bad escape");
            }
        }
        if (at == end) return fail("unterminated string");
        ++at;
        return true;
    }
    bool value(json_value* out, int depth) {
        if (depth > kMaxDepth) return fail("nested too deeply");
        space();
        if (at == end) return fail("unexpected end");
        switch (*at) {
            case '{': {
                out->type_ = json_value::kind::object;
                ++at;
                space();
                if (at < end && *at == '}') { ++at; return true; }
                for (;;) {
                    space();
                    if (at == end || *at != '"') return fail("expected a key");
                    string key;
                    if (!text(&key)) return false;
                    space();
                    if (at == end || *at != ':') return fail("expected ':'");
                    ++at;
                    out->members_.emplace_back(std::move(key), json_value());
                    if (!value(&out->members_.back().second, depth + 1)) return false;
                    space();
                    if (at < end && *at == ',') { ++at; continue; }
                    if (at < end && *at == '}') { ++at; return true; }
                    return fail("expected ',' or '}'");
                }
            }
            case '[': {
                out->type_ = json_value::kind::array;
                ++at;
                space();
                if (at < end && *at == ']') { ++at; return true; }
                for (;;) {
                    out->items_.emplace_back();
                    if (!value(&out->items_.back(), depth + 1)) return false;
                    space();
                    if (at < end && *at == ',') { ++at; continue; }
                    if (at < end && *at == ']') { ++at; return true; }
                    return fail("expected ',' or ']'");
                }
            }
            case '"': out->type_ = json_value::kind::text; return text(&out->text_);
            case 't': out->type_ = json_value::kind::boolean; out->number_ = 1; return literal("true");
            case 'f': out->type_ = json_value::kind::boolean; return literal("false");
            case 'n': return literal("null");
            default: {
                const char* p = at;
                while (p < end && (strchr("+-.eE", *p) != nullptr || (*p >= '0' && *p <= '9')) && *p != 0) ++p;
                const string digits(at, p);
                char* stop = nullptr;
                out->number_ = strtod(digits.c_str(), &stop);
                if (digits.empty() || *stop != 0) return fail("bad number");
                out->type_ = json_value::kind::number;
                at = p;
                return true;
            }
        }
    }
};

bool json_value::parse(const char* text, size_t size, json_value* out, string* error) {
    json_parser p{text, text + size, {}};
    *out = json_value();
    bool ok = p.value(out, 0);
    if (ok) {
        p.space();
        if (p.at != p.end) ok = p.fail("text after the value");
    }
    if (!ok && error) *error = p.error + " at byte " + to_string(p.at - text);
    return ok;
}

const json_value* json_value::find(const string& key) const {
    for (const auto& m : members_)
        if (m.first == key) return &m.second;
    return nullptr;
}

bool json_value::as_u64(u64* out) const {
    if (type_ != kind::number || number_ < 0 || number_ > 9007199254740992.0 || number_ != floor(number_)) return false;
    *out = u64(number_);
    return true;
}

bool json_value::as_u32(u32* out) const {
    u64 v;
    if (!as_u64(&v) || v > 0xffffffffull) return false;
    *out = u32(v);
    return true;
}

bool json_value::as_float(float* out) const {
    if (type_ != kind::number || !isfinite(number_)) return false;
    *out = float(number_);
    return true;
}
