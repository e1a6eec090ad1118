// A small JSON reader for model configurations and safetensors headers (host only).
#pragma once
#include <cmath>
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace tmb {

struct Json {
    enum Kind { kNull, kBool, kNumber, kString, kArray, kObject } kind = kNull;
    bool                                      boolean = false;
    double                                    number  = 0;
    std::string                               text;
    std::vector<Json>                         items;
    std::vector<std::pair<std::string, Json>> fields;

    const Json* find(const char* key) const
    {
        if (kind != kObject) return nullptr;
        for (const auto& f : fields) {
            if (f.first == key) return &f.second;
        }
        return nullptr;
    }
    bool is_null() const { return kind == kNull; }

    static bool parse(const std::string& s, Json* out)
    {
        size_t i = 0;
        if (!value(s, i, out, 0)) return false;
        space(s, i);
        return i == s.size();
    }

private:
    static void space(const std::string& s, size_t& i)
    {
        while (i < s.size() && (s[i] == ' ' || s[i] == '\t' || s[i] == '\n' || s[i] == '\r')) ++i;
    }
    static bool word(const std::string& s, size_t& i, const char* w)
    {
        const std::string t(w);
        if (s.compare(i, t.size(), t) != 0) return false;
        i += t.size();
        return true;
    }
    static void utf8(unsigned c, std::string* out)
    {
        if (c < 0x80) {
            *out += (char)c;
        }
        else if (c < 0x800) {
            *out += (char)(0xc0 | (c >> 6));
            *out += (char)(0x80 | (c & 0x3f));
        }
        else {
            *out += (char)(0xe0 | (c >> 12));
            *out += (char)(0x80 | ((c >> 6) & 0x3f));
            *out += (char)(0x80 | (c & 0x3f));
        }
    }
    static bool string(const std::string& s, size_t& i, std::string* out)
    {
        if (i >= s.size() || s[i] != '"') return false;
        for (++i; i < s.size(); ++i) {
            if (s[i] == '"') {
                ++i;
                return true;
            }
            if (s[i] != '\\') {
                *out += s[i];
                continue;
            }
            if (++i >= s.size()) return false;
            switch (s[i]) {
                case 'n': *out += '\n'; break;
                case 't': *out += '\t'; break;
                case 'r': *out += '\r'; break;
                case 'b': *out += '\b'; break;
                case 'f': *out += '\f'; break;
                case 'u': {
                    if (i + 4 >= s.size()) return false;
                    utf8((unsigned)std::strtoul(s.substr(i + 1, 4).c_str(), nullptr, 16), out);
                    i += 4;
                    break;
                }
                default: *out += s[i];
            }
        }
        return false;
    }
    static bool value(const std::string& s, size_t& i, Json* out, int depth)
    {
        if (depth > 64) return false;
        space(s, i);
        if (i >= s.size()) return false;
        if (s[i] == '{' || s[i] == '[') {
            const bool object = s[i] == '{';
            const char close  = object ? '}' : ']';
            out->kind         = object ? kObject : kArray;
            ++i;
            space(s, i);
            if (i < s.size() && s[i] == close) return ++i, true;
            for (;;) {
                Json        v;
                std::string key;
                if (object) {
                    space(s, i);
                    if (!string(s, i, &key)) return false;
                    space(s, i);
                    if (i >= s.size() || s[i++] != ':') return false;
                }
                if (!value(s, i, &v, depth + 1)) return false;
                if (object) {
                    out->fields.emplace_back(std::move(key), std::move(v));
                }
                else {
                    out->items.push_back(std::move(v));
                }
                space(s, i);
                if (i >= s.size()) return false;
                const char c = s[i++];
                if (c == close) return true;
                if (c != ',') return false;
            }
        }
        if (s[i] == '"') {
            out->kind = kString;
            return string(s, i, &out->text);
        }
        if (word(s, i, "null")) return true;
        if (word(s, i, "true")) return out->kind = kBool, out->boolean = true, true;
        if (word(s, i, "false")) return out->kind = kBool, true;
        char*        end   = nullptr;
        const char*  begin = s.c_str() + i;
        const double x     = std::strtod(begin, &end);
        if (end == begin) return false;
        out->kind   = kNumber;
        out->number = x;
        i += (size_t)(end - begin);
        return true;
    }
};

}  // namespace tmb
