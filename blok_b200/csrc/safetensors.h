// Reader of a safetensors file: an 8-byte little-endian header length, the header (JSON: name -> dtype, shape,
// data_offsets), then the tensors' bytes.  Every extent is checked against the file's size before anything is read.
#pragma once
#include <fcntl.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cerrno>
#include <cstring>
#include <map>

#include "common.cuh"
#include "json_reader.h"

namespace blok {

struct StoredTensor {
  std::string dtype;
  std::vector<long> shape;
  uint64_t at = 0, bytes = 0;  // place in the file
  long elements() const {
    long n = 1;
    for (long d : shape) n *= d;
    return n;
  }
};

class Safetensors {
 public:
  ~Safetensors() {
    if (fd_ >= 0) close(fd_);
  }
  int open(const std::string &path) {
    path_ = path;
    fd_ = ::open(path.c_str(), O_RDONLY);
    BLOK_REQUIRE(fd_ >= 0, BLOK_ERR_ARG, "cannot open %s: %s", path.c_str(), strerror(errno));
    struct stat st;
    BLOK_REQUIRE(fstat(fd_, &st) == 0 && st.st_size >= 8, BLOK_ERR_ARG, "%s is not a safetensors file", path.c_str());
    const uint64_t size = (uint64_t)st.st_size;
    unsigned char len8[8];
    if (int rc = read_at(0, len8, 8)) return rc;
    uint64_t n = 0;
    for (int i = 7; i >= 0; --i) n = n << 8 | len8[i];
    BLOK_REQUIRE(n <= size - 8 && n <= (1u << 30), BLOK_ERR_ARG, "%s: bad header length", path.c_str());
    std::string head(n, '\0');
    if (int rc = read_at(8, &head[0], n)) return rc;
    Json j;
    JsonParser parser(head.data(), head.data() + head.size());
    BLOK_REQUIRE(parser.parse(&j) && j.kind == Json::Object, BLOK_ERR_ARG, "%s: bad header (%s)", path.c_str(), parser.error().c_str());
    for (const auto &f : j.fields) {
      if (f.first == "__metadata__") continue;
      const Json *dt = f.second.find("dtype"), *sh = f.second.find("shape"), *off = f.second.find("data_offsets");
      BLOK_REQUIRE(dt && sh && off && off->items.size() == 2, BLOK_ERR_ARG, "%s: incomplete entry for %s", path.c_str(), f.first.c_str());
      StoredTensor t;
      t.dtype = dt->text;
      for (const Json &d : sh->items) t.shape.push_back((long)d.number);
      const double lo = off->items[0].number, hi = off->items[1].number;
      BLOK_REQUIRE(lo >= 0 && hi >= lo && hi <= (double)(size - 8 - n), BLOK_ERR_ARG, "%s: %s lies outside the file", path.c_str(),
                   f.first.c_str());
      t.at = 8 + n + (uint64_t)lo;
      t.bytes = (uint64_t)hi - (uint64_t)lo;
      tensors_[f.first] = t;
    }
    return BLOK_OK;
  }
  // The tensor `name`, which must have this dtype ("BF16", "I32") and shape.
  int need(const std::string &name, const char *dtype, const std::vector<long> &shape, const StoredTensor **out) const {
    auto it = tensors_.find(name);
    BLOK_REQUIRE(it != tensors_.end(), BLOK_ERR_ARG, "%s: missing tensor %s", path_.c_str(), name.c_str());
    const StoredTensor &t = it->second;
    const uint64_t esz = t.dtype == "BF16" ? 2 : 4;
    BLOK_REQUIRE(t.dtype == dtype && t.shape == shape && t.bytes == (uint64_t)t.elements() * esz, BLOK_ERR_SHAPE,
                 "%s: tensor %s has another type, shape or size than config.json asks for", path_.c_str(), name.c_str());
    *out = &t;
    return BLOK_OK;
  }
  const StoredTensor *find(const std::string &name) const {
    auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
  }
  int read(const StoredTensor &t, void *dst) const { return read_at(t.at, dst, t.bytes); }
  // `bytes` of the tensor from byte `from` on; the caller has checked its shape
  int read(const StoredTensor &t, void *dst, uint64_t from, uint64_t bytes) const {
    BLOK_REQUIRE(from <= t.bytes && bytes <= t.bytes - from, BLOK_ERR_SHAPE, "%s: a part outside its tensor", path_.c_str());
    return read_at(t.at + from, dst, bytes);
  }

 private:
  int fd_ = -1;
  std::string path_;
  std::map<std::string, StoredTensor> tensors_;

  int read_at(uint64_t at, void *dst, uint64_t n) const {
    char *d = static_cast<char *>(dst);
    while (n) {
      const ssize_t got = pread(fd_, d, n, (off_t)at);
      BLOK_REQUIRE(got > 0, BLOK_ERR_ARG, "%s: short read", path_.c_str());
      d += got;
      at += (uint64_t)got;
      n -= (uint64_t)got;
    }
    return BLOK_OK;
  }
};

}  // namespace blok
