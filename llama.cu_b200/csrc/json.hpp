// Small JSON reader for model configuration files and safetensors headers (host only).
#pragma once
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace lcu {

struct json_value {
  enum kind_t { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
  bool boolean = false;
  double number = 0;
  std::string text;
  std::vector<json_value> items;                            // ARRAY
  std::vector<std::pair<std::string, json_value>> members;  // OBJECT, in file order

  bool is(kind_t k) const { return kind == k; }
  const json_value* find(const char* key) const {
    for (auto& m : members)
      if (m.first == key) return &m.second;
    return nullptr;
  }
  // member that is present and not null
  const json_value* get(const char* key) const {
    const json_value* v = find(key);
    return v && v->kind != NUL ? v : nullptr;
  }
};

class json_reader {
 public:
  json_reader(const char* begin, const char* end) : p_(begin), end_(end) {}
  // false (with the offset of the fault in fault_at) on malformed text
  bool parse(json_value& out) {
    if (!value(out, 0)) return false;
    blanks();
    return p_ == end_;
  }
  const char* fault_at() const { return p_; }

 private:
  static constexpr int MAX_DEPTH = 64;
  const char *p_, *end_;

  void blanks() {
    while (p_ < end_ && (*p_ == ' ' || *p_ == '\n' || *p_ == '\t' || *p_ == '\r')) ++p_;
  }
  bool take(char c) {
    blanks();
    if (p_ >= end_ || *p_ != c) return false;
    ++p_;
    return true;
  }
  bool word(const char* w) {
    const char* q = p_;
    for (; *w; ++w, ++q)
      if (q >= end_ || *q != *w) return false;
    p_ = q;
    return true;
  }
  bool string(std::string& s) {
    if (!take('"')) return false;
    s.clear();
    while (p_ < end_ && *p_ != '"') {
      char c = *p_++;
      if (c == '\\') {
        if (p_ >= end_) return false;
        c = *p_++;
        switch (c) {
          case 'n': s.push_back('\n'); break;
          case 't': s.push_back('\t'); break;
          case 'r': s.push_back('\r'); break;
          case 'b': s.push_back('\b'); break;
          case 'f': s.push_back('\f'); break;
          case 'u': {  // code points of the basic plane, as UTF-8
            if (end_ - p_ < 4) return false;
            const std::string hex(p_, 4);
            char* stop = nullptr;
            const unsigned long u = std::strtoul(hex.c_str(), &stop, 16);
            if (*stop) return false;
            p_ += 4;
            if (u < 0x80) {
              s.push_back((char)u);
            } else if (u < 0x800) {
              s.push_back((char)(0xc0 | (u >> 6)));
              s.push_back((char)(0x80 | (u & 0x3f)));
            } else {
              s.push_back((char)(0xe0 | (u >> 12)));
              s.push_back((char)(0x80 | ((u >> 6) & 0x3f)));
              s.push_back((char)(0x80 | (u & 0x3f)));
            }
            break;
          }
          default: s.push_back(c);
        }
      } else {
        s.push_back(c);
      }
    }
    return take('"');
  }
  bool value(json_value& v, int depth) {
    if (depth > MAX_DEPTH) return false;
    blanks();
    if (p_ >= end_) return false;
    switch (*p_) {
      case '{': {
        ++p_;
        v.kind = json_value::OBJECT;
        if (take('}')) return true;
        do {
          v.members.emplace_back();
          blanks();
          if (!string(v.members.back().first) || !take(':') || !value(v.members.back().second, depth + 1)) return false;
        } while (take(','));
        return take('}');
      }
      case '[': {
        ++p_;
        v.kind = json_value::ARRAY;
        if (take(']')) return true;
        do {
          v.items.emplace_back();
          if (!value(v.items.back(), depth + 1)) return false;
        } while (take(','));
        return take(']');
      }
      case '"': v.kind = json_value::STRING; return string(v.text);
      case 't': v.kind = json_value::BOOL; v.boolean = true; return word("true");
      case 'f': v.kind = json_value::BOOL; return word("false");
      case 'n': v.kind = json_value::NUL; return word("null");
      default: {
        const char* q = p_;
        while (q < end_ && ((*q >= '0' && *q <= '9') || *q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E')) ++q;
        if (q == p_) return false;
        const std::string num(p_, q);
        char* stop = nullptr;
        v.kind = json_value::NUMBER;
        v.number = std::strtod(num.c_str(), &stop);
        if (*stop) return false;
        p_ = q;
        return true;
      }
    }
  }
};

}  // namespace lcu
