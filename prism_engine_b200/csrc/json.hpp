// Minimal JSON reader for the headers of weight containers (.cimage, .safetensors).
#pragma once

#include <cstdint>
#include <string>

namespace prism {

// Pull parser over one document: enough for the headers serde_json and safetensors write.
struct Json {
    const char *p, *end;
    bool ok = true;
    void ws() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) p++; }
    bool eat(char c) { ws(); if (p < end && *p == c) { p++; return true; } return false; }
    std::string str() {
        std::string s;
        ws();
        if (p >= end || *p != '"') { ok = false; return s; }
        p++;
        while (p < end && *p != '"') {
            if (*p == '\\' && p + 1 < end) {
                p++;
                switch (*p) {
                case 'n': s += '\n'; break;
                case 't': s += '\t'; break;
                case 'r': s += '\r'; break;
                case 'b': s += '\b'; break;
                case 'f': s += '\f'; break;
                case 'u': {  // keep BMP code points below 0x80 exact, others as '?': keys are ASCII
                    unsigned v = 0;
                    for (int i = 0; i < 4 && p + 1 < end; i++) {
                        p++;
                        char ch = *p;
                        v = v * 16 + (ch >= '0' && ch <= '9' ? ch - '0' : (ch | 32) >= 'a' && (ch | 32) <= 'f' ? (ch | 32) - 'a' + 10 : 0);
                    }
                    s += v < 0x80 ? (char)v : '?';
                    break;
                }
                default: s += *p;
                }
                p++;
            } else {
                s += *p++;
            }
        }
        if (p >= end) { ok = false; return s; }
        p++;
        return s;
    }
    uint64_t num() {
        ws();
        uint64_t v = 0;
        bool any = false;
        while (p < end && *p >= '0' && *p <= '9') { v = v * 10 + (uint64_t)(*p - '0'); p++; any = true; }
        if (!any) ok = false;
        // tolerate a fractional/exponent tail (not produced for integer fields)
        while (p < end && (*p == '.' || *p == 'e' || *p == 'E' || *p == '+' || *p == '-' || (*p >= '0' && *p <= '9'))) p++;
        return v;
    }
    void skip() {  // any value
        ws();
        if (p >= end) { ok = false; return; }
        if (*p == '"') { str(); return; }
        if (*p == '{' || *p == '[') {
            char open = *p, close = open == '{' ? '}' : ']';
            p++;
            ws();
            if (p < end && *p == close) { p++; return; }
            while (ok && p < end) {
                if (open == '{') { str(); if (!eat(':')) { ok = false; return; } }
                skip();
                if (eat(',')) continue;
                if (eat(close)) return;
                ok = false;
                return;
            }
            ok = false;
            return;
        }
        while (p < end && *p != ',' && *p != '}' && *p != ']') p++;  // number / true / false / null
    }
};

}  // namespace prism
