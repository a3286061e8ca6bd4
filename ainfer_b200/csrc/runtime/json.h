// Small JSON reader for model configurations: a value tree, no external code.
#pragma once
#include <cstdlib>
#include <map>
#include <string>
#include <vector>

namespace ainfer {

struct Json {
  enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
  bool b = false;
  double n = 0;
  std::string s;
  std::vector<Json> a;
  std::map<std::string, Json> o;

  bool is_null() const { return kind == NUL; }
  bool has(const char *k) const { return kind == OBJ && o.count(k) != 0; }
  const Json &at(const char *k) const {
    static const Json none;
    auto it = o.find(k);
    return it == o.end() ? none : it->second;
  }
  double num(double d) const { return kind == NUM ? n : d; }
  int integer(int d) const { return kind == NUM ? (int)n : d; }
  const std::string &str() const { return s; }

  // Returns false (with err set) unless the whole text is one JSON value.
  static bool parse(const std::string &text, Json &out, std::string &err) {
    Reader r{text.data(), text.data() + text.size(), 0};
    if (!r.value(out)) { err = "not valid JSON"; return false; }
    r.ws();
    if (r.p != r.end) { err = "not valid JSON: text after the value"; return false; }
    return true;
  }

 private:
  struct Reader {
    const char *p, *end;
    int depth;
    void ws() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p; }
    bool lit(char c) { ws(); if (p < end && *p == c) { ++p; return true; } return false; }
    bool word(const char *w) {
      const char *q = p;
      for (; *w; ++w, ++q)
        if (q >= end || *q != *w) return false;
      p = q;
      return true;
    }
    bool string(std::string &out) {
      if (!lit('"')) return false;
      out.clear();
      while (p < end && *p != '"') {
        if (*p == '\\') {
          if (++p >= end) return false;
          switch (*p) {
            case 'n': out += '\n'; break;
            case 't': out += '\t'; break;
            case 'r': out += '\r'; break;
            case 'b': out += '\b'; break;
            case 'f': out += '\f'; break;
            case 'u':   // configuration text is ASCII
              if (end - p < 5) return false;
              out += '?';
              p += 4;
              break;
            default: out += *p;
          }
          ++p;
        } else {
          out += *p++;
        }
      }
      return lit('"');
    }
    bool value(Json &v) {
      ws();
      if (p >= end || ++depth > 64) return false;
      bool ok = true;
      if (*p == '"') { v.kind = STR; ok = string(v.s); }
      else if (*p == '{') {
        v.kind = OBJ;
        ++p;
        if (!lit('}')) {
          do {
            std::string k;
            if (!string(k) || !lit(':') || !value(v.o[k])) return false;
          } while (lit(','));
          ok = lit('}');
        }
      } else if (*p == '[') {
        v.kind = ARR;
        ++p;
        if (!lit(']')) {
          do {
            v.a.emplace_back();
            if (!value(v.a.back())) return false;
          } while (lit(','));
          ok = lit(']');
        }
      } else if (word("true")) { v.kind = BOOL; v.b = true; }
      else if (word("false")) { v.kind = BOOL; }
      else if (word("null")) { v.kind = NUL; }
      else {
        const char *q = p;
        while (q < end && (*q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E' || (*q >= '0' && *q <= '9'))) ++q;
        const std::string t(p, q);
        char *stop = nullptr;
        v.n = std::strtod(t.c_str(), &stop);
        v.kind = NUM;
        ok = !t.empty() && *stop == 0;
        p = q;
      }
      --depth;
      return ok;
    }
  };
};

}  // namespace ainfer
