// A small JSON reader, shared by the tokenizer and by the reader of model folders (config.json, safetensors headers).  The text
// must be NUL-terminated behind `end` (a std::string's data), since numbers are read with strtod.
#pragma once
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace tlb {

struct JVal {
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<JVal> arr;
    std::vector<std::pair<std::string, JVal>> obj;
    const JVal *get(const char *key) const
    {
        for (auto &kv : obj)
            if (kv.first == key) return &kv.second;
        return nullptr;
    }
    bool is(Kind k) const { return kind == k; }
};

inline void put_utf8(std::string &s, uint32_t cp)
{
    if (cp < 0x80) s += (char)cp;
    else if (cp < 0x800) { s += (char)(0xC0 | (cp >> 6)); s += (char)(0x80 | (cp & 0x3F)); }
    else if (cp < 0x10000) { s += (char)(0xE0 | (cp >> 12)); s += (char)(0x80 | ((cp >> 6) & 0x3F)); s += (char)(0x80 | (cp & 0x3F)); }
    else { s += (char)(0xF0 | (cp >> 18)); s += (char)(0x80 | ((cp >> 12) & 0x3F)); s += (char)(0x80 | ((cp >> 6) & 0x3F)); s += (char)(0x80 | (cp & 0x3F)); }
}

struct JReader {
    const char *p, *end;
    bool ok = true;
    int depth = 0;
    void ws() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\r' || *p == '\t')) p++; }
    bool lit(const char *s) { size_t n = strlen(s); if ((size_t)(end - p) >= n && !memcmp(p, s, n)) { p += n; return true; } return false; }
    int hex4()
    {
        if (end - p < 4) return -1;
        int v = 0;
        for (int i = 0; i < 4; i++) {
            char c = p[i];
            int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return -1;
            v = v * 16 + d;
        }
        p += 4;
        return v;
    }
    bool string(std::string &out)
    {
        if (p >= end || *p != '"') return false;
        p++;
        while (p < end && *p != '"') {
            if (*p == '\\') {
                if (++p >= end) return false;
                char c = *p++;
                switch (c) {
                    case 'n': out += '\n'; break; case 't': out += '\t'; break; case 'r': out += '\r'; break;
                    case 'b': out += '\b'; break; case 'f': out += '\f'; break;
                    case 'u': {
                        int hi = hex4();
                        if (hi < 0) return false;
                        uint32_t cp = (uint32_t)hi;
                        if (hi >= 0xD800 && hi < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {   // surrogate pair
                            p += 2;
                            int lo = hex4();
                            if (lo < 0xDC00 || lo > 0xDFFF) return false;
                            cp = 0x10000 + (((uint32_t)hi - 0xD800) << 10) + ((uint32_t)lo - 0xDC00);
                        }
                        put_utf8(out, cp);
                        break;
                    }
                    default: out += c;   // \" \\ \/
                }
            } else out += *p++;
        }
        if (p >= end) return false;
        p++;
        return true;
    }
    bool value(JVal &v)
    {
        if (++depth > 64) return false;
        ws();
        bool r = false;
        if (p >= end) r = false;
        else if (*p == '{') {
            p++;
            v.kind = JVal::OBJ;
            ws();
            if (p < end && *p == '}') { p++; r = true; }
            else for (;;) {
                ws();
                std::string k;
                if (!string(k)) break;
                ws();
                if (p >= end || *p++ != ':') break;
                v.obj.emplace_back(std::move(k), JVal());
                if (!value(v.obj.back().second)) break;
                ws();
                if (p < end && *p == ',') { p++; continue; }
                if (p < end && *p == '}') { p++; r = true; }
                break;
            }
        } else if (*p == '[') {
            p++;
            v.kind = JVal::ARR;
            ws();
            if (p < end && *p == ']') { p++; r = true; }
            else for (;;) {
                v.arr.emplace_back();
                if (!value(v.arr.back())) break;
                ws();
                if (p < end && *p == ',') { p++; continue; }
                if (p < end && *p == ']') { p++; r = true; }
                break;
            }
        } else if (*p == '"') { v.kind = JVal::STR; r = string(v.str); }
        else if (lit("true")) { v.kind = JVal::BOOL; v.b = true; r = true; }
        else if (lit("false")) { v.kind = JVal::BOOL; v.b = false; r = true; }
        else if (lit("null")) { v.kind = JVal::NUL; r = true; }
        else {
            char *e = nullptr;
            v.num = strtod(p, &e);
            if (e && e > p && e <= end) { v.kind = JVal::NUM; p = e; r = true; }
        }
        depth--;
        return r;
    }
};

}  // namespace tlb
