// Small JSON reader for model folders (config.json, the header of a safetensors file): a value tree, no writer.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace b200 {

struct Json {
  enum Kind { Null, Bool, Number, String, Array, Object };
  Kind kind = Null;
  bool b = false;
  double num = 0;
  std::string str;
  std::vector<Json> items;
  std::map<std::string, Json> fields;

  bool is_null() const { return kind == Null; }
  // Field of an object, or nullptr when it is absent or null.
  const Json* find(const std::string& key) const {
    if (kind != Object) return nullptr;
    auto it = fields.find(key);
    return it == fields.end() || it->second.is_null() ? nullptr : &it->second;
  }
  // Required fields; a missing one or one of another kind throws std::runtime_error naming the key.
  const Json& at(const std::string& key) const;
  double number(const std::string& key) const;
  int integer(const std::string& key) const;
  const std::string& text(const std::string& key) const;
};

// Throws std::runtime_error on malformed input.
Json json_parse(const char* text, size_t n);

}  // namespace b200
