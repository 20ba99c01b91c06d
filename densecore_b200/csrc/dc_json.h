// A small JSON reader for config.json and safetensors headers (host code, header only).
#pragma once
#include <stdint.h>
#include <stdlib.h>
#include <string.h>

#include <map>
#include <string>
#include <utility>
#include <vector>

struct dc_json {
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<dc_json> arr;
    std::vector<std::pair<std::string, dc_json>> obj;   // in file order

    const dc_json* get(const char* key) const {
        for (auto& kv : obj)
            if (kv.first == key) return &kv.second;
        return nullptr;
    }
    bool is_null() const { return kind == NUL; }
};

// Recursive-descent parser; nesting is limited so that a malformed file cannot exhaust the stack.
class dc_json_parser {
public:
    dc_json_parser(const char* s, size_t n) : p_(s), end_(s + n) {}
    bool parse(dc_json* out, std::string* err) {
        const bool ok = value(out, 0) && (ws(), p_ == end_);
        if (!ok && err) *err = err_.empty() ? "trailing characters" : err_;
        return ok;
    }

private:
    const char *p_, *end_;
    std::string err_;

    bool fail(const char* m) {
        if (err_.empty()) err_ = m;
        return false;
    }
    void ws() {
        while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_;
    }
    bool lit(const char* w) {
        const size_t n = strlen(w);
        if ((size_t)(end_ - p_) < n || strncmp(p_, w, n) != 0) return fail("unknown literal");
        p_ += n;
        return true;
    }
    static void utf8(std::string* s, uint32_t c) {
        if (c < 0x80) {
            s->push_back((char)c);
        } else if (c < 0x800) {
            s->push_back((char)(0xC0 | (c >> 6)));
            s->push_back((char)(0x80 | (c & 63)));
        } else {
            s->push_back((char)(0xE0 | (c >> 12)));
            s->push_back((char)(0x80 | ((c >> 6) & 63)));
            s->push_back((char)(0x80 | (c & 63)));
        }
    }
    bool string(std::string* out) {
        if (p_ >= end_ || *p_ != '"') return fail("string expected");
        ++p_;
        out->clear();
        while (p_ < end_ && *p_ != '"') {
            if (*p_ != '\\') {
                out->push_back(*p_++);
                continue;
            }
            if (++p_ >= end_) break;
            const char c = *p_++;
            switch (c) {
            case 'n': out->push_back('\n'); break;
            case 't': out->push_back('\t'); break;
            case 'r': out->push_back('\r'); break;
            case 'b': out->push_back('\b'); break;
            case 'f': out->push_back('\f'); break;
            case 'u': {
                if (end_ - p_ < 4) return fail("short \\u escape");
                char hex[5] = {p_[0], p_[1], p_[2], p_[3], 0};
                utf8(out, (uint32_t)strtoul(hex, nullptr, 16));
                p_ += 4;
                break;
            }
            default: out->push_back(c);
            }
        }
        if (p_ >= end_) return fail("unterminated string");
        ++p_;
        return true;
    }
    bool value(dc_json* v, int depth) {
        if (depth > 64) return fail("nested too deeply");
        ws();
        if (p_ >= end_) return fail("unexpected end");
        *v = dc_json();
        const char c = *p_;
        if (c == '{') {
            v->kind = dc_json::OBJ;
            ++p_;
            ws();
            if (p_ < end_ && *p_ == '}') return ++p_, true;
            for (;;) {
                ws();
                std::string k;
                if (!string(&k)) return false;
                ws();
                if (p_ >= end_ || *p_ != ':') return fail("':' expected");
                ++p_;
                v->obj.emplace_back(std::move(k), dc_json());
                if (!value(&v->obj.back().second, depth + 1)) return false;
                ws();
                if (p_ < end_ && *p_ == ',') {
                    ++p_;
                    continue;
                }
                if (p_ < end_ && *p_ == '}') return ++p_, true;
                return fail("',' or '}' expected");
            }
        }
        if (c == '[') {
            v->kind = dc_json::ARR;
            ++p_;
            ws();
            if (p_ < end_ && *p_ == ']') return ++p_, true;
            for (;;) {
                v->arr.emplace_back();
                if (!value(&v->arr.back(), depth + 1)) return false;
                ws();
                if (p_ < end_ && *p_ == ',') {
                    ++p_;
                    continue;
                }
                if (p_ < end_ && *p_ == ']') return ++p_, true;
                return fail("',' or ']' expected");
            }
        }
        if (c == '"') {
            v->kind = dc_json::STR;
            return string(&v->str);
        }
        if (c == 't') {
            v->kind = dc_json::BOOL;
            v->b = true;
            return lit("true");
        }
        if (c == 'f') {
            v->kind = dc_json::BOOL;
            return lit("false");
        }
        if (c == 'n') return lit("null");
        char buf[64];
        size_t n = 0;
        while (p_ < end_ && n < sizeof(buf) - 1 && (strchr("+-.eE", *p_) || (*p_ >= '0' && *p_ <= '9'))) buf[n++] = *p_++;
        buf[n] = 0;
        char* e = nullptr;
        v->kind = dc_json::NUM;
        v->num = strtod(buf, &e);
        return n > 0 && e == buf + n ? true : fail("number expected");
    }
};
