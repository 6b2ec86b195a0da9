// A small JSON reader (objects, arrays, strings, numbers, literals): Safetensors headers, model
// configuration files, request lines of the command-line driver.  Header-only, host-only.
#pragma once

#include <cstddef>
#include <cstdlib>
#include <cstring>
#include <string>
#include <utility>
#include <vector>

namespace evob {

struct Json {
  enum Kind { kNull, kBool, kNumber, kString, kArray, kObject } kind = kNull;
  bool boolean = false;
  double number = 0;
  std::string text;
  std::vector<Json> items;
  std::vector<std::pair<std::string, Json>> members;  // insertion order
  const Json *get(const std::string &key) const {
    for (const auto &m : members)
      if (m.first == key) return &m.second;
    return nullptr;
  }
};

class JsonParser {
 public:
  JsonParser(const char *begin, const char *end) : p_(begin), end_(end) {}
  bool parse(Json *out) {
    skip();
    if (!value(out, 0)) return false;
    skip();
    return p_ == end_;
  }

 private:
  const char *p_, *end_;
  void skip() {
    while (p_ < end_ && (*p_ == ' ' || *p_ == '\n' || *p_ == '\t' || *p_ == '\r')) ++p_;
  }
  bool literal(const char *word) {
    const std::size_t n = std::strlen(word);
    if (static_cast<std::size_t>(end_ - p_) < n || std::memcmp(p_, word, n) != 0) return false;
    p_ += n;
    return true;
  }
  bool string(std::string *out) {
    if (p_ >= end_ || *p_ != '"') return false;
    ++p_;
    out->clear();
    while (p_ < end_ && *p_ != '"') {
      if (*p_ == '\\') {
        if (++p_ >= end_) return false;
        switch (*p_) {
          case '"': out->push_back('"'); break;
          case '\\': out->push_back('\\'); break;
          case '/': out->push_back('/'); break;
          case 'b': out->push_back('\b'); break;
          case 'f': out->push_back('\f'); break;
          case 'n': out->push_back('\n'); break;
          case 'r': out->push_back('\r'); break;
          case 't': out->push_back('\t'); break;
          case 'u': {
            if (end_ - p_ < 5) return false;
            unsigned code = 0;
            for (int i = 1; i <= 4; ++i) {
              const char c = p_[i];
              code <<= 4;
              if (c >= '0' && c <= '9') code |= c - '0';
              else if (c >= 'a' && c <= 'f') code |= c - 'a' + 10;
              else if (c >= 'A' && c <= 'F') code |= c - 'A' + 10;
              else return false;
            }
            p_ += 4;
            if (code < 0x80) out->push_back(static_cast<char>(code));
            else if (code < 0x800) {
              out->push_back(static_cast<char>(0xc0 | (code >> 6)));
              out->push_back(static_cast<char>(0x80 | (code & 0x3f)));
            } else {
              out->push_back(static_cast<char>(0xe0 | (code >> 12)));
              out->push_back(static_cast<char>(0x80 | ((code >> 6) & 0x3f)));
              out->push_back(static_cast<char>(0x80 | (code & 0x3f)));
            }
            break;
          }
          default: return false;
        }
        ++p_;
      } else {
        out->push_back(*p_++);
      }
    }
    if (p_ >= end_) return false;
    ++p_;
    return true;
  }
  bool value(Json *out, const int depth) {
    if (depth > 16 || p_ >= end_) return false;
    if (*p_ == '{') {
      out->kind = Json::kObject;
      ++p_;
      skip();
      if (p_ < end_ && *p_ == '}') { ++p_; return true; }
      for (;;) {
        std::string key;
        skip();
        if (!string(&key)) return false;
        skip();
        if (p_ >= end_ || *p_ != ':') return false;
        ++p_;
        skip();
        Json member;
        if (!value(&member, depth + 1)) return false;
        out->members.emplace_back(std::move(key), std::move(member));
        skip();
        if (p_ < end_ && *p_ == ',') { ++p_; continue; }
        if (p_ < end_ && *p_ == '}') { ++p_; return true; }
        return false;
      }
    }
    if (*p_ == '[') {
      out->kind = Json::kArray;
      ++p_;
      skip();
      if (p_ < end_ && *p_ == ']') { ++p_; return true; }
      for (;;) {
        Json item;
        skip();
        if (!value(&item, depth + 1)) return false;
        out->items.push_back(std::move(item));
        skip();
        if (p_ < end_ && *p_ == ',') { ++p_; continue; }
        if (p_ < end_ && *p_ == ']') { ++p_; return true; }
        return false;
      }
    }
    if (*p_ == '"') {
      out->kind = Json::kString;
      return string(&out->text);
    }
    if (literal("true")) { out->kind = Json::kBool; out->boolean = true; return true; }
    if (literal("false")) { out->kind = Json::kBool; return true; }
    if (literal("null")) { out->kind = Json::kNull; return true; }
    const char *start = p_;
    while (p_ < end_ && (std::strchr("+-0123456789.eE", *p_) != nullptr)) ++p_;
    if (p_ == start) return false;
    out->kind = Json::kNumber;
    out->number = std::strtod(std::string(start, p_).c_str(), nullptr);
    return true;
  }
};

}  // namespace evob
