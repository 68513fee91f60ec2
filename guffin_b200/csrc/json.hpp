// A small JSON reader for configuration files and safetensors headers: whole documents, numbers as doubles,
// no writer.  Malformed text makes parse() return false with the offset in `error_at`.
#pragma once

#include <cstddef>
#include <cstdint>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace gf {

struct Json {
    enum Kind { kNull, kBool, kNumber, kString, kArray, kObject } kind = kNull;
    bool truth = false;
    double number = 0.0;
    std::string text;
    std::vector<Json> items;                                  // arrays
    std::vector<std::pair<std::string, Json>> members;        // objects, in file order

    const Json* find(const char* key) const {
        for (const auto& m : members)
            if (m.first == key) return &m.second;
        return nullptr;
    }
    bool is_null() const { return kind == kNull; }

    static bool parse(const char* data, size_t size, Json& out, size_t* error_at = nullptr) {
        Reader r{data, size, 0};
        const bool ok = r.value(out, 0) && (r.space(), r.at == r.size);
        if (error_at) *error_at = r.at;
        return ok;
    }

private:
    struct Reader {
        const char* data;
        size_t size, at;
        void space() { while (at < size && (data[at] == ' ' || data[at] == '\n' || data[at] == '\t' || data[at] == '\r')) ++at; }
        bool take(char c) { space(); if (at < size && data[at] == c) { ++at; return true; } return false; }
        bool word(const char* w) {
            const size_t n = std::strlen(w);
            if (size - at < n || std::memcmp(data + at, w, n) != 0) return false;
            at += n;
            return true;
        }
        static void utf8(std::string& out, uint32_t c) {
            if (c < 0x80u) out += (char)c;
            else if (c < 0x800u) { out += (char)(0xC0u | (c >> 6)); out += (char)(0x80u | (c & 0x3Fu)); }
            else if (c < 0x10000u) { out += (char)(0xE0u | (c >> 12)); out += (char)(0x80u | ((c >> 6) & 0x3Fu)); out += (char)(0x80u | (c & 0x3Fu)); }
            else {
                out += (char)(0xF0u | (c >> 18)); out += (char)(0x80u | ((c >> 12) & 0x3Fu));
                out += (char)(0x80u | ((c >> 6) & 0x3Fu)); out += (char)(0x80u | (c & 0x3Fu));
            }
        }
        bool hex4(uint32_t& out) {
            if (size - at < 4u) return false;
            out = 0;
            for (int i = 0; i < 4; ++i) {
                const char c = data[at++];
                const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
                if (d < 0) return false;
                out = out * 16u + (uint32_t)d;
            }
            return true;
        }
        bool string(std::string& out) {
            if (!take('"')) return false;
            out.clear();
            while (at < size) {
                const char c = data[at++];
                if (c == '"') return true;
                if (c != '\\') { out += c; continue; }
                if (at >= size) return false;
                switch (const char e = data[at++]) {
                    case 'b': out += '\b'; break;
                    case 'f': out += '\f'; break;
                    case 'n': out += '\n'; break;
                    case 'r': out += '\r'; break;
                    case 't': out += '\t'; break;
                    case '"': case '\\': case '/': out += e; break;
                    case 'u': {
                        uint32_t code = 0, low = 0;
                        if (!hex4(code)) return false;
                        if (code >= 0xD800u && code < 0xDC00u && word("\\u")) {
                            if (!hex4(low)) return false;
                            code = 0x10000u + ((code - 0xD800u) << 10) + (low - 0xDC00u);
                        }
                        utf8(out, code);
                        break;
                    }
                    default: return false;
                }
            }
            return false;
        }
        bool value(Json& out, int depth) {
            if (depth > 64) return false;
            space();
            if (at >= size) return false;
            const char c = data[at];
            if (c == '{') {
                ++at;
                out.kind = kObject;
                if (take('}')) return true;
                do {
                    std::pair<std::string, Json> m;
                    space();
                    if (!string(m.first) || !take(':') || !value(m.second, depth + 1)) return false;
                    out.members.push_back(std::move(m));
                } while (take(','));
                return take('}');
            }
            if (c == '[') {
                ++at;
                out.kind = kArray;
                if (take(']')) return true;
                do {
                    out.items.emplace_back();
                    if (!value(out.items.back(), depth + 1)) return false;
                } while (take(','));
                return take(']');
            }
            if (c == '"') { out.kind = kString; return string(out.text); }
            if (word("true")) { out.kind = kBool; out.truth = true; return true; }
            if (word("false")) { out.kind = kBool; return true; }
            if (word("null")) return true;
            size_t end = at;
            while (end < size && (std::strchr("+-.eE", data[end]) || (data[end] >= '0' && data[end] <= '9'))) ++end;
            if (end == at) return false;
            const std::string digits(data + at, end - at);
            char* stop = nullptr;
            out.kind = kNumber;
            out.number = std::strtod(digits.c_str(), &stop);
            if (stop != digits.c_str() + digits.size()) return false;
            at = end;
            return true;
        }
    };
};

}  // namespace gf
