// Minimal JSON reader for the model folder's config.json and the header of a
// safetensors file. Host code only; numbers are kept as double (integers up to
// 2^53 are exact, more than any offset a header carries).
#pragma once

#include <cctype>
#include <cstdint>
#include <cstdlib>
#include <stdexcept>
#include <string>
#include <utility>
#include <vector>

namespace lb {

class Json {
 public:
  enum Kind { Null, Bool, Number, String, Array, Object };
  Kind kind = Null;
  bool boolean = false;
  double number = 0.0;
  std::string text;
  std::vector<Json> items;                              // Array
  std::vector<std::pair<std::string, Json>> members;    // Object, in file order

  static Json parse(const std::string &s) {
    Parser p{s.c_str(), s.c_str() + s.size()};
    Json j = p.value(0);
    p.space();
    if (p.at != p.end) p.fail("trailing characters");
    return j;
  }

  const Json *find(const std::string &key) const {
    if (kind != Object) return nullptr;
    for (const auto &m : members)
      if (m.first == key) return &m.second;
    return nullptr;
  }
  // A member that is absent or null counts as missing.
  bool has(const std::string &key) const {
    const Json *j = find(key);
    return j != nullptr && j->kind != Null;
  }
  const Json &at(const std::string &key) const {
    const Json *j = find(key);
    if (j == nullptr || j->kind == Null) throw std::runtime_error("missing key \"" + key + "\"");
    return *j;
  }
  double as_number() const {
    if (kind != Number) throw std::runtime_error("expected a number");
    return number;
  }
  long long as_int() const {
    const double v = as_number();
    const long long i = (long long)v;
    if ((double)i != v) throw std::runtime_error("expected an integer");
    return i;
  }
  const std::string &as_string() const {
    if (kind != String) throw std::runtime_error("expected a string");
    return text;
  }
  const std::vector<Json> &as_array() const {
    if (kind != Array) throw std::runtime_error("expected an array");
    return items;
  }

 private:
  struct Parser {
    const char *at, *end;
    [[noreturn]] void fail(const char *what) const { throw std::runtime_error(std::string("JSON: ") + what); }
    void space() {
      while (at != end && (*at == ' ' || *at == '\t' || *at == '\n' || *at == '\r')) ++at;
    }
    char peek() {
      space();
      if (at == end) fail("unexpected end");
      return *at;
    }
    void expect(char c) {
      if (peek() != c) fail("unexpected character");
      ++at;
    }
    bool word(const char *w) {
      const char *p = at;
      for (; *w; ++w, ++p)
        if (p == end || *p != *w) return false;
      at = p;
      return true;
    }
    unsigned hex4() {
      unsigned v = 0;
      for (int i = 0; i < 4; ++i) {
        if (at == end || !std::isxdigit((unsigned char)*at)) fail("bad \\u escape");
        const char c = *at++;
        v = v * 16 + (unsigned)(c <= '9' ? c - '0' : (c | 32) - 'a' + 10);
      }
      return v;
    }
    std::string string() {
      expect('"');
      std::string out;
      while (true) {
        if (at == end) fail("unterminated string");
        const char c = *at++;
        if (c == '"') return out;
        if (c != '\\') {
          out += c;
          continue;
        }
        if (at == end) fail("unterminated string");
        const char e = *at++;
        switch (e) {
          case 'n': out += '\n'; break;
          case 't': out += '\t'; break;
          case 'r': out += '\r'; break;
          case 'b': out += '\b'; break;
          case 'f': out += '\f'; break;
          case 'u': {
            const unsigned v = hex4();  // UTF-8, surrogate halves kept apart
            if (v < 0x80) out += (char)v;
            else if (v < 0x800) { out += (char)(0xC0 | v >> 6); out += (char)(0x80 | (v & 63)); }
            else { out += (char)(0xE0 | v >> 12); out += (char)(0x80 | (v >> 6 & 63)); out += (char)(0x80 | (v & 63)); }
            break;
          }
          default: out += e;
        }
      }
    }
    Json value(int depth) {
      if (depth > 64) fail("nested too deeply");
      Json j;
      const char c = peek();
      if (c == '{') {
        j.kind = Object;
        ++at;
        if (peek() == '}') { ++at; return j; }
        while (true) {
          peek();
          std::string key = string();
          expect(':');
          j.members.emplace_back(std::move(key), value(depth + 1));
          if (peek() == ',') { ++at; continue; }
          expect('}');
          return j;
        }
      }
      if (c == '[') {
        j.kind = Array;
        ++at;
        if (peek() == ']') { ++at; return j; }
        while (true) {
          j.items.push_back(value(depth + 1));
          if (peek() == ',') { ++at; continue; }
          expect(']');
          return j;
        }
      }
      if (c == '"') {
        j.kind = String;
        j.text = string();
        return j;
      }
      if (word("true")) { j.kind = Bool; j.boolean = true; return j; }
      if (word("false")) { j.kind = Bool; return j; }
      if (word("null")) return j;
      const char *start = at;
      while (at != end && (std::isalnum((unsigned char)*at) || *at == '+' || *at == '-' || *at == '.')) ++at;
      const std::string lit(start, at);
      char *stop = nullptr;
      j.kind = Number;
      j.number = std::strtod(lit.c_str(), &stop);
      if (lit.empty() || stop != lit.c_str() + lit.size()) fail("bad number");
      return j;
    }
  };
};

}  // namespace lb
