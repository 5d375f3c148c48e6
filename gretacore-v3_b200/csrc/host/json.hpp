// A small JSON reader (objects, arrays, strings, numbers, literals) for config.json files, safetensors headers and the
// step lines of a trace.
#pragma once
#include <cmath>
#include <cstdint>
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace gcore::host {

class Json {
public:
  enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT };
  Kind kind = NUL;
  bool boolean = false;
  double number = 0.0;
  std::string string;
  std::vector<Json> items;                            // ARRAY
  std::vector<std::pair<std::string, Json>> members;  // OBJECT, in file order

  bool is_null() const { return kind == NUL; }
  // Member of an object; nullptr when absent, null or not an object.
  const Json *get(const char *key) const {
    for (const auto &m : members)
      if (m.first == key) return m.second.is_null() ? nullptr : &m.second;
    return nullptr;
  }
  // A non-negative whole number (up to 2^32 - 1).
  bool as_u32(uint32_t *out) const {
    if (kind != NUMBER || number < 0 || number > 4294967295.0 || number != std::floor(number)) return false;
    *out = (uint32_t)number;
    return true;
  }
  bool as_float(float *out) const {
    if (kind != NUMBER) return false;
    *out = (float)number;
    return true;
  }

  static bool parse(const char *text, size_t n, Json *out, std::string *err) {
    Reader r{text, text + n};
    if (!r.value(out, 0) || (r.space(), r.p != r.end)) {
      if (err) *err = "JSON: malformed at byte " + std::to_string(r.p - text);
      return false;
    }
    return true;
  }
  static bool parse(const std::string &text, Json *out, std::string *err) { return parse(text.data(), text.size(), out, err); }

private:
  struct Reader {
    const char *p, *end;
    void space() {
      while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p;
    }
    bool literal(const char *s) {
      const char *q = p;
      for (; *s; ++s, ++q)
        if (q >= end || *q != *s) return false;
      p = q;
      return true;
    }
    static void utf8(std::string *s, uint32_t c) {
      if (c < 0x80) {
        *s += (char)c;
      } else if (c < 0x800) {
        *s += (char)(0xC0 | (c >> 6));
        *s += (char)(0x80 | (c & 63));
      } else if (c < 0x10000) {
        *s += (char)(0xE0 | (c >> 12));
        *s += (char)(0x80 | ((c >> 6) & 63));
        *s += (char)(0x80 | (c & 63));
      } else {
        *s += (char)(0xF0 | (c >> 18));
        *s += (char)(0x80 | ((c >> 12) & 63));
        *s += (char)(0x80 | ((c >> 6) & 63));
        *s += (char)(0x80 | (c & 63));
      }
    }
    bool hex4(uint32_t *c) {
      if (end - p < 4) return false;
      *c = 0;
      for (int i = 0; i < 4; ++i, ++p) {
        const char h = *p;
        const int d = h >= '0' && h <= '9' ? h - '0' : h >= 'a' && h <= 'f' ? h - 'a' + 10 : h >= 'A' && h <= 'F' ? h - 'A' + 10 : -1;
        if (d < 0) return false;
        *c = *c * 16 + (uint32_t)d;
      }
      return true;
    }
    bool str(std::string *s) {
      if (p >= end || *p != '"') return false;
      ++p;
      s->clear();
      while (p < end && *p != '"') {
        if (*p != '\\') {
          *s += *p++;
          continue;
        }
        if (++p >= end) return false;
        const char e = *p++;
        switch (e) {
          case 'n': *s += '\n'; break;
          case 't': *s += '\t'; break;
          case 'r': *s += '\r'; break;
          case 'b': *s += '\b'; break;
          case 'f': *s += '\f'; break;
          case '"': case '\\': case '/': *s += e; break;
          case 'u': {
            uint32_t c, d;
            if (!hex4(&c)) return false;
            if (c >= 0xD800 && c < 0xDC00) {
              if (end - p < 2 || p[0] != '\\' || p[1] != 'u') return false;
              p += 2;
              if (!hex4(&d) || d < 0xDC00 || d > 0xDFFF) return false;
              c = 0x10000 + ((c - 0xD800) << 10) + (d - 0xDC00);
            }
            utf8(s, c);
            break;
          }
          default: return false;
        }
      }
      if (p >= end) return false;
      ++p;
      return true;
    }
    bool value(Json *v, int depth) {
      if (depth > 64) return false;
      space();
      if (p >= end) return false;
      if (*p == '{') {
        v->kind = OBJECT;
        ++p;
        space();
        if (p < end && *p == '}') return ++p, true;
        for (;;) {
          std::pair<std::string, Json> m;
          space();
          if (!str(&m.first)) return false;
          space();
          if (p >= end || *p++ != ':' || !value(&m.second, depth + 1)) return false;
          v->members.push_back(std::move(m));
          space();
          if (p >= end) return false;
          if (*p == '}') return ++p, true;
          if (*p++ != ',') return false;
        }
      }
      if (*p == '[') {
        v->kind = ARRAY;
        ++p;
        space();
        if (p < end && *p == ']') return ++p, true;
        for (;;) {
          v->items.emplace_back();
          if (!value(&v->items.back(), depth + 1)) return false;
          space();
          if (p >= end) return false;
          if (*p == ']') return ++p, true;
          if (*p++ != ',') return false;
        }
      }
      if (*p == '"') {
        v->kind = STRING;
        return str(&v->string);
      }
      if (literal("null")) return v->kind = NUL, true;
      if (literal("true")) return v->kind = BOOL, v->boolean = true, true;
      if (literal("false")) return v->kind = BOOL, true;
      const char *q = p;
      while (q < end && ((*q >= '0' && *q <= '9') || *q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
      if (q == p) return false;
      const std::string num(p, q);
      char *stop = nullptr;
      v->kind = NUMBER;
      v->number = std::strtod(num.c_str(), &stop);
      if (*stop) return false;
      p = q;
      return true;
    }
  };
};

}  // namespace gcore::host
