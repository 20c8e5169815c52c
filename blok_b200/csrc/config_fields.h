// Typed access to the fields of a config.json, shared by the families that are opened from one.
#pragma once
#include <cmath>

#include "common.cuh"
#include "json_reader.h"

namespace blok {

// Reads fields of one JSON object; the first field that is missing or of another kind leaves an error.
class Fields {
 public:
  Fields(const Json *object, std::string where) : j_(object), where_(std::move(where)) {
    if (!j_ || j_->kind != Json::Object) fail("is not an object");
  }
  int rc() const { return rc_; }
  double number(const char *name) {
    const Json *v = get(name);
    if (v && v->kind != Json::Number) fail(name, "is not a number");
    return v && v->kind == Json::Number ? v->number : 0;
  }
  int size(const char *name) {
    const double v = number(name);
    if (!rc_ && !(v >= 1 && v <= (1 << 30) && v == std::floor(v))) fail(name, "is not a positive integer");
    return rc_ ? 0 : (int)v;
  }
  bool has(const char *name) const {  // the field is there and not null
    const Json *v = rc_ ? nullptr : j_->find(name);
    return v && !v->is_null();
  }
  std::string text(const char *name) {
    const Json *v = get(name);
    if (v && v->kind != Json::String) fail(name, "is not a string");
    return v ? v->text : std::string();
  }
  std::vector<double> numbers(const char *name) {
    std::vector<double> out;
    const Json *v = get(name);
    if (v && v->kind != Json::Array) fail(name, "is not a list");
    if (v)
      for (const Json &x : v->items) {
        if (x.kind != Json::Number) fail(name, "holds something else than numbers");
        out.push_back(x.number);
      }
    return out;
  }
  // A field that is an object; after an error here its fields report nothing more.
  Fields object(const char *name) {
    const Json *v = get(name);
    if (!rc_) return Fields(v, where_ + "." + name);
    Fields none;
    none.rc_ = rc_;
    return none;
  }
  void fail(const char *name, const char *what) { fail((std::string(name) + " " + what).c_str()); }

 private:
  const Json *j_ = nullptr;
  std::string where_;
  int rc_ = BLOK_OK;

  Fields() = default;
  const Json *get(const char *name) {
    if (rc_) return nullptr;
    const Json *v = j_->find(name);
    if (!v) fail(name, "is missing");
    return v;
  }
  void fail(const char *what) {
    if (!rc_) set_error("config.json: %s: %s", where_.c_str(), what);
    rc_ = BLOK_ERR_ARG;
  }
};

}  // namespace blok
