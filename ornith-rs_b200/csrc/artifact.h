// Artifact files shared by the loaders of all architectures: a small JSON reader and memory-mapped
// safetensors shards (src/safetensors.rs:189-308 of the reference: 8-byte little-endian header
// length, JSON header, raw tensor bytes).
#pragma once

#include <fcntl.h>
#include <stdint.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cctype>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <map>
#include <string>
#include <utility>
#include <vector>

namespace orna {

// ---------------------------------------------------------------- tiny JSON
struct JVal {
  enum Type { Null, Bool, Num, Str, Arr, Obj } type = Null;
  bool b = false;
  double num = 0;
  std::string str;
  std::vector<JVal> arr;
  std::vector<std::pair<std::string, JVal>> obj;
  const JVal* get(const std::string& k) const {
    if (type != Obj) return nullptr;
    for (auto& kv : obj)
      if (kv.first == k) return &kv.second;
    return nullptr;
  }
};

struct JParser {
  const char* p;
  const char* end;
  bool ok = true;
  void ws() { while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p; }
  bool lit(const char* s) {
    size_t n = strlen(s);
    if ((size_t)(end - p) >= n && memcmp(p, s, n) == 0) { p += n; return true; }
    return false;
  }
  std::string string() {
    std::string out;
    if (p >= end || *p != '"') { ok = false; return out; }
    ++p;
    while (p < end && *p != '"') {
      if (*p == '\\' && p + 1 < end) {
        ++p;
        switch (*p) {
          case 'n': out += '\n'; break;
          case 't': out += '\t'; break;
          case 'r': out += '\r'; break;
          case 'b': out += '\b'; break;
          case 'f': out += '\f'; break;
          case 'u': {  // keep the escape verbatim; tensor names are ASCII
            out += "\\u";
            break;
          }
          default: out += *p; break;
        }
        ++p;
      } else {
        out += *p++;
      }
    }
    if (p >= end) { ok = false; return out; }
    ++p;
    return out;
  }
  JVal value() {
    JVal v;
    ws();
    if (p >= end) { ok = false; return v; }
    if (*p == '{') {
      v.type = JVal::Obj;
      ++p; ws();
      if (p < end && *p == '}') { ++p; return v; }
      while (ok) {
        ws();
        std::string k = string();
        ws();
        if (p >= end || *p != ':') { ok = false; break; }
        ++p;
        JVal c = value();
        v.obj.emplace_back(std::move(k), std::move(c));
        ws();
        if (p < end && *p == ',') { ++p; continue; }
        if (p < end && *p == '}') { ++p; break; }
        ok = false;
      }
    } else if (*p == '[') {
      v.type = JVal::Arr;
      ++p; ws();
      if (p < end && *p == ']') { ++p; return v; }
      while (ok) {
        v.arr.push_back(value());
        ws();
        if (p < end && *p == ',') { ++p; continue; }
        if (p < end && *p == ']') { ++p; break; }
        ok = false;
      }
    } else if (*p == '"') {
      v.type = JVal::Str;
      v.str = string();
    } else if (lit("true")) { v.type = JVal::Bool; v.b = true; }
    else if (lit("false")) { v.type = JVal::Bool; v.b = false; }
    else if (lit("null")) { v.type = JVal::Null; }
    else {
      // the header of a memory-mapped file is not NUL-terminated: parse from a bounded copy
      char tmp[64];
      size_t n = 0;
      while (p + n < end && n + 1 < sizeof tmp && (isdigit((unsigned char)p[n]) || strchr("+-.eE", p[n]) != nullptr)) {
        tmp[n] = p[n];
        ++n;
      }
      tmp[n] = 0;
      char* e = nullptr;
      v.type = JVal::Num;
      v.num = strtod(tmp, &e);
      if (e == tmp) ok = false;
      p += (e - tmp);
    }
    return v;
  }
};

inline bool parse_json(const char* data, size_t n, JVal* out) {
  JParser ps{data, data + n};
  *out = ps.value();
  return ps.ok;
}

inline bool read_file(const std::string& path, std::string* out) {
  FILE* f = fopen(path.c_str(), "rb");
  if (!f) return false;
  fseek(f, 0, SEEK_END);
  long n = ftell(f);
  fseek(f, 0, SEEK_SET);
  out->resize((size_t)n);
  bool ok = n == 0 || fread(&(*out)[0], 1, (size_t)n, f) == (size_t)n;
  fclose(f);
  return ok;
}

// ---------------------------------------------------------------- safetensors
struct TInfo {
  std::string dtype;
  std::vector<int64_t> shape;
  const uint8_t* data = nullptr;
  size_t nbytes = 0;
};
struct Shard {
  void* map = nullptr;
  size_t size = 0;
};
struct Store {
  Store() = default;
  Store(const Store&) = delete;
  Store& operator=(const Store&) = delete;
  std::vector<Shard> shards;
  std::map<std::string, TInfo> tensors;
  ~Store() {
    for (auto& s : shards)
      if (s.map) munmap(s.map, s.size);
  }
};

inline bool open_shard(const std::string& path, Store* st, std::string* err) {
  int fd = open(path.c_str(), O_RDONLY);
  if (fd < 0) { *err = "cannot open " + path; return false; }
  struct stat sb;
  if (fstat(fd, &sb) != 0 || sb.st_size < 8) { close(fd); *err = "short file " + path; return false; }
  void* mp = mmap(nullptr, (size_t)sb.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
  close(fd);
  if (mp == MAP_FAILED) { *err = "mmap failed for " + path; return false; }
  st->shards.push_back(Shard{mp, (size_t)sb.st_size});
  const uint8_t* base = (const uint8_t*)mp;
  uint64_t hlen = 0;
  memcpy(&hlen, base, 8);
  if (hlen > (uint64_t)sb.st_size - 8) { *err = "bad header length in " + path; return false; }
  JVal hdr;
  if (!parse_json((const char*)base + 8, (size_t)hlen, &hdr) || hdr.type != JVal::Obj) {
    *err = "bad safetensors header in " + path;
    return false;
  }
  const uint8_t* data = base + 8 + hlen;
  const size_t data_size = (size_t)sb.st_size - 8 - (size_t)hlen;
  for (auto& kv : hdr.obj) {
    if (kv.first == "__metadata__") continue;
    const JVal* dt = kv.second.get("dtype");
    const JVal* sh = kv.second.get("shape");
    const JVal* off = kv.second.get("data_offsets");
    if (!dt || !sh || !off || off->arr.size() != 2) { *err = "bad tensor entry " + kv.first; return false; }
    TInfo ti;
    ti.dtype = dt->str;
    bool shape_ok = true;
    for (auto& d : sh->arr) {
      if (d.type != JVal::Num || d.num < 0 || d.num > 2147483647.0 || d.num != (double)(int64_t)d.num) shape_ok = false;
      ti.shape.push_back((int64_t)d.num);
    }
    if (!shape_ok) { *err = "bad shape for " + kv.first; return false; }
    size_t a = (size_t)off->arr[0].num, b = (size_t)off->arr[1].num;
    if (a > b || b > data_size) { *err = "tensor out of bounds: " + kv.first; return false; }
    ti.data = data + a;
    ti.nbytes = b - a;
    st->tensors[kv.first] = ti;
  }
  return true;
}

// every shard of an artifact: those model.safetensors.index.json lists, else model.safetensors
// (src/safetensors.rs:296-308)
inline bool open_shards(const std::string& dir, Store* st, std::string* err) {
  std::vector<std::string> files;
  std::string idx;
  if (read_file(dir + "/model.safetensors.index.json", &idx)) {
    JVal ij;
    if (!parse_json(idx.data(), idx.size(), &ij)) { *err = "model.safetensors.index.json: parse error"; return false; }
    const JVal* wm = ij.get("weight_map");
    if (!wm || wm->type != JVal::Obj) { *err = "index has no weight_map"; return false; }
    for (auto& kv : wm->obj) {
      bool seen = false;
      for (auto& fnm : files) seen = seen || fnm == kv.second.str;
      if (!seen) files.push_back(kv.second.str);
    }
  } else {
    files.push_back("model.safetensors");
  }
  for (auto& fnm : files)
    if (!open_shard(dir + "/" + fnm, st, err)) return false;
  return true;
}

inline bool ends_with(const std::string& s, const std::string& suf) {
  return s.size() >= suf.size() && s.compare(s.size() - suf.size(), suf.size(), suf) == 0;
}

inline int64_t numel(const TInfo& t) {
  int64_t n = 1;
  for (auto d : t.shape) n *= d;
  return n;
}
// bytes the declared dtype and shape ask for must be the bytes the file holds for the tensor
inline bool bytes_match(const TInfo& t, size_t elem) { return !t.shape.empty() && numel(t) > 0 && (size_t)numel(t) * elem == t.nbytes; }

}  // namespace orna
