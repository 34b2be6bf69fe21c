// A small JSON reader (internal): model configurations and safetensors headers. Input is untrusted: depth and sizes are
// bounded, every access is checked, errors are a flag and a message, never an exception or a crash.
#pragma once
#include <math.h>
#include <stdint.h>
#include <stdlib.h>
#include <string.h>

#include <string>
#include <utility>
#include <vector>

namespace nfai {

struct Json {
  enum Kind { Null, Bool, Number, String, Array, Object };
  Kind kind = Null;
  bool b = false;
  double num = 0;
  std::string str;
  std::vector<Json> items;                             // Array
  std::vector<std::pair<std::string, Json>> members;   // Object, in file order

  const Json* get(const char* key) const {
    if (kind != Object) return nullptr;
    for (const auto& m : members)
      if (m.first == key) return &m.second;
    return nullptr;
  }
  bool is_null() const { return kind == Null; }
};

class JsonReader {
 public:
  JsonReader(const char* text, size_t len) : p_(text), end_(text + len) {}
  bool parse(Json* out, std::string* err) {
    bool ok = value(out, 0);
    if (ok) {
      space();
      if (p_ != end_) ok = bad("text after the document");
    }
    if (!ok && err) *err = err_;
    return ok;
  }

 private:
  const char* p_;
  const char* end_;
  std::string err_;

  bool bad(const char* what) {
    if (err_.empty()) err_ = std::string("malformed JSON: ") + what;
    return false;
  }
  void space() {
    while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_;
  }
  bool literal(const char* word) {
    const size_t n = strlen(word);
    if ((size_t)(end_ - p_) < n || memcmp(p_, word, n) != 0) return bad("unknown word");
    p_ += n;
    return true;
  }
  static void put_utf8(std::string* s, uint32_t c) {
    if (c < 0x80) s->push_back((char)c);
    else if (c < 0x800) { s->push_back((char)(0xC0 | (c >> 6))); s->push_back((char)(0x80 | (c & 63))); }
    else if (c < 0x10000) { s->push_back((char)(0xE0 | (c >> 12))); s->push_back((char)(0x80 | ((c >> 6) & 63))); s->push_back((char)(0x80 | (c & 63))); }
    else { s->push_back((char)(0xF0 | (c >> 18))); s->push_back((char)(0x80 | ((c >> 12) & 63))); s->push_back((char)(0x80 | ((c >> 6) & 63))); s->push_back((char)(0x80 | (c & 63))); }
  }
  bool hex4(uint32_t* out) {
    if (end_ - p_ < 4) return bad("short escape");
    uint32_t v = 0;
    for (int i = 0; i < 4; ++i, ++p_) {
      const char c = *p_;
      v <<= 4;
      if (c >= '0' && c <= '9') v |= (uint32_t)(c - '0');
      else if (c >= 'a' && c <= 'f') v |= (uint32_t)(c - 'a' + 10);
      else if (c >= 'A' && c <= 'F') v |= (uint32_t)(c - 'A' + 10);
      else return bad("bad escape");
    }
    *out = v;
    return true;
  }
  bool string(std::string* out) {
    if (p_ >= end_ || *p_ != '"') return bad("a string was expected");
    ++p_;
    while (p_ < end_ && *p_ != '"') {
      if (*p_ != '\\') { out->push_back(*p_++); continue; }
      if (++p_ >= end_) return bad("unterminated string");
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
          if (u >= 0xD800 && u < 0xDC00 && end_ - p_ >= 2 && p_[0] == '\\' && p_[1] == 'u') {
            p_ += 2;
            if (!hex4(&lo)) return false;
            if (lo < 0xDC00 || lo > 0xDFFF) return bad("bad surrogate pair");
            u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
          }
          put_utf8(out, u);
          break;
        }
        default: return bad("bad escape");
      }
    }
    if (p_ >= end_) return bad("unterminated string");
    ++p_;
    return true;
  }
  bool value(Json* out, int depth) {
    if (depth > 32) return bad("nested too deeply");
    space();
    if (p_ >= end_) return bad("unexpected end");
    switch (*p_) {
      case '{': {
        ++p_;
        out->kind = Json::Object;
        space();
        if (p_ < end_ && *p_ == '}') { ++p_; return true; }
        for (;;) {
          space();
          out->members.emplace_back();
          if (!string(&out->members.back().first)) return false;
          space();
          if (p_ >= end_ || *p_++ != ':') return bad("':' expected");
          if (!value(&out->members.back().second, depth + 1)) return false;
          space();
          if (p_ >= end_) return bad("unterminated object");
          const char c = *p_++;
          if (c == '}') return true;
          if (c != ',') return bad("',' expected");
        }
      }
      case '[': {
        ++p_;
        out->kind = Json::Array;
        space();
        if (p_ < end_ && *p_ == ']') { ++p_; return true; }
        for (;;) {
          out->items.emplace_back();
          if (!value(&out->items.back(), depth + 1)) return false;
          space();
          if (p_ >= end_) return bad("unterminated array");
          const char c = *p_++;
          if (c == ']') return true;
          if (c != ',') return bad("',' expected");
        }
      }
      case '"': out->kind = Json::String; return string(&out->str);
      case 't': out->kind = Json::Bool; out->b = true; return literal("true");
      case 'f': out->kind = Json::Bool; return literal("false");
      case 'n': return literal("null");
      default: {
        const char* a = p_;
        while (p_ < end_ && ((*p_ >= '0' && *p_ <= '9') || *p_ == '-' || *p_ == '+' || *p_ == '.' || *p_ == 'e' || *p_ == 'E')) ++p_;
        if (a == p_ || p_ - a > 64) return bad("a value was expected");
        const std::string t(a, (size_t)(p_ - a));
        char* e = nullptr;
        out->kind = Json::Number;
        out->num = strtod(t.c_str(), &e);
        if (!e || *e || !isfinite(out->num)) return bad("bad number");
        return true;
      }
    }
  }
};

}  // namespace nfai
