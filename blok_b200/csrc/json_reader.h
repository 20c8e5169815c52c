// A small JSON reader for model configurations and safetensors headers: objects keep their order, numbers are doubles.
#pragma once
#include <cctype>
#include <cstdint>
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace blok {

struct Json {
  enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
  bool flag = false;
  double number = 0;
  std::string text;
  std::vector<Json> items;                          // Array
  std::vector<std::pair<std::string, Json>> fields;  // Object

  const Json *find(const char *name) const {
    for (const auto &f : fields)
      if (f.first == name) return &f.second;
    return nullptr;
  }
  bool is_null() const { return kind == Null; }
};

class JsonParser {
 public:
  JsonParser(const char *begin, const char *end) : p_(begin), end_(end) {}
  // False (and a message in error()) when the text is not one JSON value.
  bool parse(Json *out) {
    if (!value(out, 0)) return false;
    space();
    return p_ == end_ || fail("text after the value");
  }
  const std::string &error() const { return error_; }

 private:
  static constexpr int kMaxDepth = 64;
  const char *p_, *end_;
  std::string error_;

  bool fail(const char *what) {
    if (error_.empty()) error_ = what;
    return false;
  }
  void space() {
    while (p_ < end_ && (*p_ == ' ' || *p_ == '\t' || *p_ == '\n' || *p_ == '\r')) ++p_;
  }
  bool word(const char *w) {
    const char *q = p_;
    for (; *w; ++w, ++q)
      if (q == end_ || *q != *w) return fail("unknown word");
    p_ = q;
    return true;
  }
  static void utf8(std::string *s, unsigned c) {
    if (c < 0x80) s->push_back((char)c);
    else if (c < 0x800) s->push_back((char)(0xC0 | c >> 6)), s->push_back((char)(0x80 | (c & 63)));
    else if (c < 0x10000) s->push_back((char)(0xE0 | c >> 12)), s->push_back((char)(0x80 | (c >> 6 & 63))), s->push_back((char)(0x80 | (c & 63)));
    else
      s->push_back((char)(0xF0 | c >> 18)), s->push_back((char)(0x80 | (c >> 12 & 63))), s->push_back((char)(0x80 | (c >> 6 & 63))),
          s->push_back((char)(0x80 | (c & 63)));
  }
  bool hex4(unsigned *out) {
    unsigned v = 0;
    for (int i = 0; i < 4; ++i, ++p_) {
      if (p_ == end_ || !isxdigit((unsigned char)*p_)) return fail("bad \\u escape");
      const char c = *p_;
      v = v * 16 + (unsigned)(c <= '9' ? c - '0' : (c | 32) - 'a' + 10);
    }
    *out = v;
    return true;
  }
  bool string(std::string *s) {
    ++p_;  // the opening quote
    while (p_ < end_ && *p_ != '"') {
      if (*p_ != '\\') {
        s->push_back(*p_++);
        continue;
      }
      if (++p_ == end_) break;
      const char c = *p_++;
      switch (c) {
        case 'n': s->push_back('\n'); break;
        case 't': s->push_back('\t'); break;
        case 'r': s->push_back('\r'); break;
        case 'b': s->push_back('\b'); break;
        case 'f': s->push_back('\f'); break;
        case '"': case '\\': case '/': s->push_back(c); break;
        case 'u': {
          unsigned v = 0, lo = 0;
          if (!hex4(&v)) return false;
          if (v >= 0xD800 && v < 0xDC00 && end_ - p_ >= 6 && p_[0] == '\\' && p_[1] == 'u') {
            p_ += 2;
            if (!hex4(&lo)) return false;
            v = 0x10000 + ((v - 0xD800) << 10) + (lo - 0xDC00);
          }
          utf8(s, v);
          break;
        }
        default: return fail("bad escape");
      }
    }
    if (p_ == end_) return fail("unterminated string");
    ++p_;
    return true;
  }
  bool value(Json *out, int depth) {
    space();
    if (p_ == end_) return fail("unexpected end");
    if (depth > kMaxDepth) return fail("nested too deeply");
    switch (*p_) {
      case '{': {
        out->kind = Json::Object;
        ++p_;
        space();
        if (p_ < end_ && *p_ == '}') return ++p_, true;
        for (;;) {
          space();
          if (p_ == end_ || *p_ != '"') return fail("expected a field name");
          out->fields.emplace_back();
          if (!string(&out->fields.back().first)) return false;
          space();
          if (p_ == end_ || *p_ != ':') return fail("expected ':'");
          ++p_;
          if (!value(&out->fields.back().second, depth + 1)) return false;
          space();
          if (p_ < end_ && *p_ == ',') {
            ++p_;
            continue;
          }
          if (p_ < end_ && *p_ == '}') return ++p_, true;
          return fail("expected ',' or '}'");
        }
      }
      case '[': {
        out->kind = Json::Array;
        ++p_;
        space();
        if (p_ < end_ && *p_ == ']') return ++p_, true;
        for (;;) {
          out->items.emplace_back();
          if (!value(&out->items.back(), depth + 1)) return false;
          space();
          if (p_ < end_ && *p_ == ',') {
            ++p_;
            continue;
          }
          if (p_ < end_ && *p_ == ']') return ++p_, true;
          return fail("expected ',' or ']'");
        }
      }
      case '"': out->kind = Json::String; return string(&out->text);
      case 't': out->kind = Json::Bool; out->flag = true; return word("true");
      case 'f': out->kind = Json::Bool; out->flag = false; return word("false");
      case 'n': out->kind = Json::Null; return word("null");
      default: {
        const char *q = p_;
        while (q < end_ && (isdigit((unsigned char)*q) || *q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
        const std::string n(p_, q);
        char *stop = nullptr;
        out->kind = Json::Number;
        out->number = strtod(n.c_str(), &stop);
        if (n.empty() || *stop) return fail("bad number");
        p_ = q;
        return true;
      }
    }
  }
};

}  // namespace blok
