// Host-side file helpers: a small JSON reader and a read-only file mapping.
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>
#include <cstdlib>
#include <cstring>
#include <map>
#include <string>
#include <vector>
#include "lc_common.cuh"

namespace lc {

// ---- a small JSON reader: enough for manifests and configs (objects, arrays, strings, numbers, true/false/null) ----------------
struct JValue {
    enum Kind { NUL, NUM, STR, BOOL, ARR, OBJ } kind = NUL;
    double num = 0;
    std::string str;
    std::vector<JValue> arr;
    std::map<std::string, JValue> obj;
    const JValue* get(const char* k) const {
        auto it = obj.find(k);
        return it == obj.end() ? nullptr : &it->second;
    }
};
struct JReader {
    const char* p;
    const char* e;
    bool ok = true;
    void ws() { while (p < e && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) p++; }
    bool eat(char c) { ws(); if (p < e && *p == c) { p++; return true; } return false; }
    std::string str() {
        std::string s;
        if (!eat('"')) { ok = false; return s; }
        while (p < e && *p != '"') {
            if (*p == '\\' && p + 1 < e) {
                p++;
                switch (*p) {
                    case 'n': s += '\n'; break;
                    case 't': s += '\t'; break;
                    case 'u': if (p + 4 < e) p += 4; s += '?'; break;  // names and paths in a manifest are ASCII
                    default: s += *p;
                }
                p++;
            } else {
                s += *p++;
            }
        }
        if (p >= e) ok = false; else p++;
        return s;
    }
    JValue value(int depth = 0) {
        JValue v;
        ws();
        if (p >= e || depth > 16) { ok = false; return v; }
        if (*p == '{') {
            p++;
            v.kind = JValue::OBJ;
            if (eat('}')) return v;
            do {
                std::string k = str();
                if (!ok || !eat(':')) { ok = false; return v; }
                v.obj[k] = value(depth + 1);
            } while (ok && eat(','));
            if (!eat('}')) ok = false;
        } else if (*p == '[') {
            p++;
            v.kind = JValue::ARR;
            if (eat(']')) return v;
            do v.arr.push_back(value(depth + 1)); while (ok && eat(','));
            if (!eat(']')) ok = false;
        } else if (*p == '"') {
            v.kind = JValue::STR;
            v.str = str();
        } else if (!strncmp(p, "true", 4) && e - p >= 4) { v.kind = JValue::BOOL; v.num = 1; p += 4; }
        else if (!strncmp(p, "false", 5) && e - p >= 5) { v.kind = JValue::BOOL; p += 5; }
        else if (!strncmp(p, "null", 4) && e - p >= 4) { p += 4; }
        else {
            char* end = nullptr;
            v.kind = JValue::NUM;
            v.num = strtod(p, &end);
            if (end == p || end > e) ok = false; else p = end;
        }
        return v;
    }
};

struct Mapping {
    int fd = -1;
    void* base = MAP_FAILED;
    size_t size = 0;
    int32_t open_file(const std::string& path) {
        fd = open(path.c_str(), O_RDONLY);
        LC_CHECK(fd >= 0, LC_ERR_INVALID, "cannot open %s", path.c_str());
        struct stat st;
        LC_CHECK(fstat(fd, &st) == 0 && st.st_size > 0, LC_ERR_INVALID, "%s: empty or unreadable", path.c_str());
        size = (size_t)st.st_size;
        base = mmap(nullptr, size, PROT_READ, MAP_PRIVATE, fd, 0);
        LC_CHECK(base != MAP_FAILED, LC_ERR_INVALID, "cannot map %s", path.c_str());
        return LC_OK;
    }
    ~Mapping() {
        if (base != MAP_FAILED) munmap(base, size);
        if (fd >= 0) close(fd);
    }
};

}  // namespace lc
