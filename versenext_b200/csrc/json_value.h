// A small JSON reader for model configurations (objects, arrays, numbers, strings, booleans, null).
#pragma once
#include <stdlib.h>
#include <string>
#include <utility>
#include <vector>

struct JsonValue {
  enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
  double num = 0;
  std::string str;
  std::vector<JsonValue> arr;
  std::vector<std::pair<std::string, JsonValue>> obj;

  const JsonValue* find(const char* key) const {
    for (auto& kv : obj)
      if (kv.first == key) return &kv.second;
    return nullptr;
  }
  // number (or boolean) under `key`; `dflt` when it is absent or null
  double number(const char* key, double dflt) const {
    const JsonValue* v = find(key);
    return v && (v->kind == NUM || v->kind == BOOL) ? v->num : dflt;
  }
  std::string text(const char* key) const {
    const JsonValue* v = find(key);
    return v && v->kind == STR ? v->str : std::string();
  }
};

class JsonReader {
 public:
  // false on malformed input
  static bool parse(const std::string& s, JsonValue* out) {
    JsonReader r(s);
    if (!r.value(out, 0)) return false;
    r.space();
    return r.i_ == s.size();
  }

 private:
  explicit JsonReader(const std::string& s) : s_(s) {}
  void space() { while (i_ < s_.size() && (s_[i_] == ' ' || s_[i_] == '\n' || s_[i_] == '\t' || s_[i_] == '\r')) ++i_; }
  bool eat(char c) { space(); if (i_ < s_.size() && s_[i_] == c) { ++i_; return true; } return false; }
  bool word(const char* w) { const size_t n = std::string(w).size(); if (s_.compare(i_, n, w)) return false; i_ += n; return true; }
  bool string(std::string* out) {
    if (!eat('"')) return false;
    while (i_ < s_.size() && s_[i_] != '"') {
      if (s_[i_] == '\\') { if (++i_ >= s_.size()) return false; }      // escapes: the character itself (names are plain)
      out->push_back(s_[i_++]);
    }
    return i_ < s_.size() && s_[i_++] == '"';
  }
  bool value(JsonValue* v, int depth) {
    if (depth > 32) return false;
    space();
    if (i_ >= s_.size()) return false;
    const char c = s_[i_];
    if (c == '{') {
      ++i_;
      v->kind = JsonValue::OBJ;
      if (eat('}')) return true;
      do {
        std::pair<std::string, JsonValue> kv;
        space();
        if (!string(&kv.first) || !eat(':') || !value(&kv.second, depth + 1)) return false;
        v->obj.push_back(std::move(kv));
      } while (eat(','));
      return eat('}');
    }
    if (c == '[') {
      ++i_;
      v->kind = JsonValue::ARR;
      if (eat(']')) return true;
      do {
        v->arr.emplace_back();
        if (!value(&v->arr.back(), depth + 1)) return false;
      } while (eat(','));
      return eat(']');
    }
    if (c == '"') { v->kind = JsonValue::STR; return string(&v->str); }
    if (word("null")) return true;
    if (word("true")) { v->kind = JsonValue::BOOL; v->num = 1; return true; }
    if (word("false")) { v->kind = JsonValue::BOOL; return true; }
    char* end = nullptr;
    v->kind = JsonValue::NUM;
    v->num = strtod(s_.c_str() + i_, &end);
    const size_t n = end - (s_.c_str() + i_);
    i_ += n;
    return n > 0;
  }
  const std::string& s_;
  size_t i_ = 0;
};
