#include "safetensors.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cctype>
#include <cmath>
#include <cstdlib>
#include <cstring>
#include <stdexcept>

#include "json.h"

namespace b200 {

// ---- JSON --------------------------------------------------------------------------------------------------------
const Json& Json::at(const std::string& key) const {
  const Json* j = find(key);
  if (!j) throw std::runtime_error("missing field '" + key + "'");
  return *j;
}
double Json::number(const std::string& key) const {
  const Json& j = at(key);
  if (j.kind != Number) throw std::runtime_error("field '" + key + "' is not a number");
  return j.num;
}
int Json::integer(const std::string& key) const {
  const double v = number(key);
  if (v != std::floor(v) || std::fabs(v) > 2147483647.0) throw std::runtime_error("field '" + key + "' is not an integer");
  return (int)v;
}
const std::string& Json::text(const std::string& key) const {
  const Json& j = at(key);
  if (j.kind != String) throw std::runtime_error("field '" + key + "' is not a string");
  return j.str;
}

namespace {
struct Parser {
  const char* p;
  const char* end;
  int depth = 0;

  [[noreturn]] void bad(const char* what) { throw std::runtime_error(std::string("malformed JSON: ") + what); }
  void space() { while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) ++p; }
  bool eat(char c) {
    space();
    if (p < end && *p == c) { ++p; return true; }
    return false;
  }
  void word(const char* w) {
    const size_t n = std::strlen(w);
    if ((size_t)(end - p) < n || std::memcmp(p, w, n)) bad("unknown word");
    p += n;
  }
  unsigned hex4() {
    if (end - p < 4) bad("short escape");
    unsigned v = 0;
    for (int i = 0; i < 4; ++i, ++p) {
      if (!std::isxdigit((unsigned char)*p)) bad("bad escape");
      v = v * 16 + (unsigned)(*p <= '9' ? *p - '0' : (*p | 32) - 'a' + 10);
    }
    return v;
  }
  void utf8(std::string& s, unsigned c) {
    if (c < 0x80) s += (char)c;
    else if (c < 0x800) { s += (char)(0xC0 | c >> 6); s += (char)(0x80 | (c & 63)); }
    else if (c < 0x10000) { s += (char)(0xE0 | c >> 12); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
    else { s += (char)(0xF0 | c >> 18); s += (char)(0x80 | (c >> 12 & 63)); s += (char)(0x80 | (c >> 6 & 63)); s += (char)(0x80 | (c & 63)); }
  }
  std::string string() {
    if (!eat('"')) bad("string expected");
    std::string s;
    while (p < end && *p != '"') {
      if (*p != '\\') { s += *p++; continue; }
      if (++p >= end) bad("short escape");
      const char c = *p++;
      switch (c) {
        case 'n': s += '\n'; break;
        case 't': s += '\t'; break;
        case 'r': s += '\r'; break;
        case 'b': s += '\b'; break;
        case 'f': s += '\f'; break;
        case 'u': {
          unsigned v = hex4();
          if (v >= 0xD800 && v < 0xDC00 && end - p >= 6 && p[0] == '\\' && p[1] == 'u') {
            p += 2;
            v = 0x10000 + ((v - 0xD800) << 10) + (hex4() - 0xDC00);
          }
          utf8(s, v);
          break;
        }
        default: s += c;
      }
    }
    if (p >= end) bad("unterminated string");
    ++p;
    return s;
  }
  Json value() {
    if (++depth > 64) bad("nested too deeply");
    space();
    if (p >= end) bad("unexpected end");
    Json j;
    if (*p == '{') {
      ++p;
      j.kind = Json::Object;
      if (!eat('}')) {
        do {
          space();
          std::string k = string();
          if (!eat(':')) bad("':' expected");
          j.fields[k] = value();
        } while (eat(','));
        if (!eat('}')) bad("'}' expected");
      }
    } else if (*p == '[') {
      ++p;
      j.kind = Json::Array;
      if (!eat(']')) {
        do j.items.push_back(value()); while (eat(','));
        if (!eat(']')) bad("']' expected");
      }
    } else if (*p == '"') {
      j.kind = Json::String;
      j.str = string();
    } else if (*p == 't') {
      word("true"); j.kind = Json::Bool; j.b = true;
    } else if (*p == 'f') {
      word("false"); j.kind = Json::Bool;
    } else if (*p == 'n') {
      word("null");
    } else {
      std::string n;
      while (p < end && (std::isalnum((unsigned char)*p) || *p == '-' || *p == '+' || *p == '.')) n += *p++;
      char* stop = nullptr;
      j.kind = Json::Number;
      j.num = std::strtod(n.c_str(), &stop);
      if (n.empty() || *stop) bad("number expected");
    }
    --depth;
    return j;
  }
};
}  // namespace

Json json_parse(const char* text, size_t n) {
  Parser ps{text, text + n};
  Json j = ps.value();
  ps.space();
  if (ps.p != ps.end) ps.bad("text after the value");
  return j;
}

// ---- safetensors -------------------------------------------------------------------------------------------------
StFile::~StFile() {
  if (map_base) munmap(const_cast<uint8_t*>(map_base), map_size);
  if (fd >= 0) close(fd);
}

void safetensors_open(const std::string& path, StFile& out) {
  out.fd = open(path.c_str(), O_RDONLY | O_CLOEXEC);
  if (out.fd < 0) throw std::runtime_error("cannot open " + path);
  struct stat st;
  if (fstat(out.fd, &st) || st.st_size < 10) throw std::runtime_error(path + " is not a safetensors file");
  out.map_size = (size_t)st.st_size;
  void* m = mmap(nullptr, out.map_size, PROT_READ, MAP_PRIVATE, out.fd, 0);
  if (m == MAP_FAILED) throw std::runtime_error("cannot map " + path);
  out.map_base = static_cast<const uint8_t*>(m);
  uint64_t hlen = 0;
  std::memcpy(&hlen, out.map_base, 8);
  if (hlen > out.map_size - 8) throw std::runtime_error(path + ": header longer than the file");
  const uint8_t* data = out.map_base + 8 + hlen;
  const size_t data_bytes = out.map_size - 8 - (size_t)hlen;
  const Json head = json_parse(reinterpret_cast<const char*>(out.map_base) + 8, (size_t)hlen);
  if (head.kind != Json::Object) throw std::runtime_error(path + ": header is not an object");
  for (const auto& kv : head.fields) {
    if (kv.first == "__metadata__") continue;
    StTensor t;
    t.dtype = kv.second.text("dtype");
    const size_t esz = t.dtype == "BF16" || t.dtype == "F16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : t.dtype == "I64" || t.dtype == "F64" ? 8 : 1;
    for (const Json& d : kv.second.at("shape").items) {
      if (d.kind != Json::Number || d.num < 0) throw std::runtime_error(path + ": bad shape of " + kv.first);
      t.shape.push_back((int64_t)d.num);
    }
    const Json& off = kv.second.at("data_offsets");
    if (off.items.size() != 2) throw std::runtime_error(path + ": bad offsets of " + kv.first);
    const double lo = off.items[0].num, hi = off.items[1].num;
    if (lo < 0 || hi < lo || hi > (double)data_bytes || (double)t.elems() * esz != hi - lo)
      throw std::runtime_error(path + ": data of " + kv.first + " does not match its shape");
    t.data = data + (size_t)lo;
    t.bytes = (size_t)(hi - lo);
    out.tensors.emplace(kv.first, std::move(t));
  }
}

}  // namespace b200
