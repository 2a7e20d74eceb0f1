// A small JSON reader (RFC 8259) for model folders: config.json and the header of a safetensors file. Values keep their text form until
// they are asked for, so an integer beyond 2^53 (a byte offset) loses nothing.
#pragma once
#include <cmath>
#include <cstdint>
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace qtb {

struct JsonValue {
    enum Kind { kNull, kBool, kNumber, kString, kArray, kObject } kind = kNull;
    bool b = false;
    std::string s;                                          // strings, and the text of numbers
    std::vector<JsonValue> items;                           // arrays
    std::vector<std::pair<std::string, JsonValue>> fields;  // objects, in file order
    const JsonValue* get(const char* key) const {
        for (const auto& f : fields)
            if (f.first == key) return &f.second;
        return nullptr;
    }
    bool is(Kind k) const { return kind == k; }
    double number() const { return std::strtod(s.c_str(), nullptr); }
    // The value as a non-negative integer; false when it is not one (a fraction, a sign, another kind).
    bool as_u64(uint64_t* out) const {
        if (kind != kNumber) return false;
        if (s.find_first_not_of("0123456789") == std::string::npos) {
            *out = std::strtoull(s.c_str(), nullptr, 10);
            return true;
        }
        const double v = number();  // 1e3, 64.0
        if (!(v >= 0.0) || v > 9007199254740992.0 || v != std::floor(v)) return false;
        *out = static_cast<uint64_t>(v);
        return true;
    }
};

class JsonReader {
  public:
    JsonReader(const char* p, size_t n) : p_(p), end_(p + n) {}
    // Parses the whole text into *out; on failure returns false and says why and where.
    bool parse(JsonValue* out, std::string* why) {
        const char* begin = p_;
        if (value(out, 0)) {
            space();
            if (p_ == end_) return true;
            error_ = "text after the end of the value";
        }
        *why = error_ + " at byte " + std::to_string(p_ - begin);
        return false;
    }

  private:
    const char *p_, *end_;
    std::string error_;
    bool bad(const char* what) {
        if (error_.empty()) error_ = what;
        return false;
    }
    void space() {
        while (p_ != end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_;
    }
    bool word(const char* w) {
        const char* q = p_;
        for (; *w; ++w, ++q)
            if (q == end_ || *q != *w) return bad("unknown word");
        p_ = q;
        return true;
    }
    static void utf8(uint32_t c, std::string* out) {
        if (c < 0x80) {
            out->push_back(static_cast<char>(c));
        } else if (c < 0x800) {
            out->push_back(static_cast<char>(0xC0 | (c >> 6))), out->push_back(static_cast<char>(0x80 | (c & 63)));
        } else if (c < 0x10000) {
            out->push_back(static_cast<char>(0xE0 | (c >> 12))), out->push_back(static_cast<char>(0x80 | ((c >> 6) & 63))), out->push_back(static_cast<char>(0x80 | (c & 63)));
        } else {
            out->push_back(static_cast<char>(0xF0 | (c >> 18))), out->push_back(static_cast<char>(0x80 | ((c >> 12) & 63)));
            out->push_back(static_cast<char>(0x80 | ((c >> 6) & 63))), out->push_back(static_cast<char>(0x80 | (c & 63)));
        }
    }
    bool hex4(uint32_t* out) {
        uint32_t v = 0;
        for (int i = 0; i < 4; ++i, ++p_) {
            if (p_ == end_) return bad("unfinished escape");
            const char c = *p_;
            v = v * 16 + (c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : 99);
            if (v > 0xFFFF) return bad("bad escape");
        }
        *out = v;
        return true;
    }
    bool string(std::string* out) {
        ++p_;  // the opening quote
        while (p_ != end_ && *p_ != '"') {
            if (*p_ != '\\') {
                out->push_back(*p_++);
                continue;
            }
            if (++p_ == end_) break;
            const char c = *p_++;
            switch (c) {
                case '"': case '\\': case '/': out->push_back(c); break;
                case 'b': out->push_back('\b'); break;
                case 'f': out->push_back('\f'); break;
                case 'n': out->push_back('\n'); break;
                case 'r': out->push_back('\r'); break;
                case 't': out->push_back('\t'); break;
                case 'u': {
                    uint32_t u = 0, lo = 0;
                    if (!hex4(&u)) return false;
                    if (u >= 0xD800 && u < 0xDC00 && end_ - p_ >= 6 && p_[0] == '\\' && p_[1] == 'u') {
                        p_ += 2;
                        if (!hex4(&lo)) return false;
                        u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
                    }
                    utf8(u, out);
                    break;
                }
                default: return bad("unknown escape");
            }
        }
        if (p_ == end_) return bad("unfinished string");
        ++p_;
        return true;
    }
    bool value(JsonValue* out, int depth) {
        if (depth > 64) return bad("nested too deeply");
        space();
        if (p_ == end_) return bad("unexpected end");
        switch (*p_) {
            case '{':
                out->kind = JsonValue::kObject;
                for (++p_, space(); p_ != end_ && *p_ != '}';) {
                    if (*p_ != '"') return bad("a key must be a string");
                    out->fields.emplace_back();
                    auto& f = out->fields.back();
                    if (!string(&f.first)) return false;
                    space();
                    if (p_ == end_ || *p_ != ':') return bad("':' expected");
                    ++p_;
                    if (!value(&f.second, depth + 1)) return false;
                    space();
                    if (p_ != end_ && *p_ == ',') {
                        ++p_, space();
                        if (p_ != end_ && *p_ == '}') return bad("a key must follow ','");
                    } else if (p_ == end_ || *p_ != '}') {
                        return bad("',' or '}' expected");
                    }
                }
                if (p_ == end_) return bad("unfinished object");
                ++p_;
                return true;
            case '[':
                out->kind = JsonValue::kArray;
                for (++p_, space(); p_ != end_ && *p_ != ']';) {
                    out->items.emplace_back();
                    if (!value(&out->items.back(), depth + 1)) return false;
                    space();
                    if (p_ != end_ && *p_ == ',') {
                        ++p_, space();
                        if (p_ != end_ && *p_ == ']') return bad("a value must follow ','");
                    } else if (p_ == end_ || *p_ != ']') {
                        return bad("',' or ']' expected");
                    }
                }
                if (p_ == end_) return bad("unfinished array");
                ++p_;
                return true;
            case '"': out->kind = JsonValue::kString; return string(&out->s);
            case 't': out->kind = JsonValue::kBool, out->b = true; return word("true");
            case 'f': out->kind = JsonValue::kBool, out->b = false; return word("false");
            case 'n': out->kind = JsonValue::kNull; return word("null");
            default: {
                const char* q = p_;
                while (q != end_ && ((*q >= '0' && *q <= '9') || *q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
                if (q == p_) return bad("a value expected");
                out->kind = JsonValue::kNumber;
                out->s.assign(p_, q);
                char* stop = nullptr;
                std::strtod(out->s.c_str(), &stop);
                if (*stop != 0) return bad("malformed number");
                p_ = q;
                return true;
            }
        }
    }
};

}  // namespace qtb
