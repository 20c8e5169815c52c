// blok-trace-run: replays a trace of token ids through a model, step by step, and writes the logits that are asked for.
//
//   blok-trace-run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N
//
// Standard input holds one JSON object a line:
//   {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}
// entries: the next tokens of each sequence and the places among them whose logits are wanted; end: sequences that are
// finished after the step and give back what they hold.  OUT/<step>.f32 receives the wanted rows, in order, as
// little-endian fp32 [wanted, vocab]; "done <step>" is printed after every step.  --max-tokens bounds the tokens that the
// live sequences hold together and sizes the cache.  Nothing is sampled: the sequences go through the same slots, pages,
// prompt chunks and decode steps as generation (blok_model_extend_slot).
#include <cuda_runtime.h>

#include <cstdint>
#include <cstdio>
#include <cstring>
#include <iostream>
#include <map>
#include <string>
#include <vector>

#include "../csrc/json_reader.h"
#include "blok_b200.h"

namespace {

struct Fail {
  std::string message;
};
void require(bool ok, const std::string &message) {
  if (!ok) throw Fail{message};
}
void require_ok(int rc, const char *stage) {
  if (rc != BLOK_OK) throw Fail{std::string(stage) + ": " + blok_last_error()};
}

constexpr int kSlots = 16;  // live sequences

class Replay {
 public:
  Replay(const std::string &dir, int dtype, const std::string &out, long max_tokens) : out_(out) {
    blok_model_options o;
    blok_model_default_options(&o);
    o.dtype = dtype;
    o.max_batch = kSlots;
    o.max_ctx = (int)max_tokens;
    // every live sequence may leave its last page partly empty
    o.kv_pages = (int)((max_tokens + o.kv_page_rows - 1) / o.kv_page_rows) + kSlots;
    require_ok(blok_model_open(dir.c_str(), &o, &model_), "model");
    blok_model_config cfg;
    require_ok(blok_model_get_config(model_, &cfg), "model");
    vocab_ = (size_t)cfg.vocab;
    require(cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking) == cudaSuccess, "cannot create a stream");
    for (int s = kSlots - 1; s >= 0; --s) free_.push_back(s);
  }
  ~Replay() {
    if (stream_) cudaStreamDestroy(stream_);
    if (model_) blok_model_destroy(model_);
  }
  void step(const blok::Json &j) {
    const blok::Json *number = j.find("step"), *entries = j.find("entries"), *end = j.find("end");
    require(number && entries, "a step needs \"step\" and \"entries\"");
    const long n = (long)number->number;
    std::vector<float> rows;
    for (const blok::Json &e : entries->items) {
      const blok::Json *id = e.find("id"), *tokens = e.find("tokens"), *want = e.find("want");
      require(id && tokens && !tokens->items.empty(), "an entry needs \"id\" and \"tokens\"");
      const std::vector<uint32_t> ids = ints<uint32_t>(*tokens);
      const std::vector<int> places = want ? ints<int>(*want) : std::vector<int>();
      const size_t at = rows.size();
      rows.resize(at + places.size() * vocab_);
      require_ok(blok_model_extend_slot(model_, slot_of(id->text), ids.data(), (int)ids.size(), places.data(), (int)places.size(), rows.data() + at,
                                        stream_),
                 "step");
    }
    require_ok(blok_model_check(model_, stream_), "step");
    if (!rows.empty()) {
      const std::string path = out_ + "/" + std::to_string(n) + ".f32";
      FILE *f = std::fopen(path.c_str(), "wb");
      require(f && std::fwrite(rows.data(), 4, rows.size(), f) == rows.size() && std::fclose(f) == 0, "cannot write " + path);
    }
    if (end)
      for (const blok::Json &id : end->items) {
        auto it = live_.find(id.text);
        if (it == live_.end()) continue;
        require_ok(blok_model_slot_release(model_, it->second, stream_), "end");
        free_.push_back(it->second);
        live_.erase(it);
      }
    std::printf("done %ld\n", n);
    std::fflush(stdout);
  }

 private:
  std::string out_;
  blok_model_t *model_ = nullptr;
  cudaStream_t stream_ = nullptr;
  size_t vocab_ = 0;
  std::map<std::string, int> live_;
  std::vector<int> free_;

  template <typename T>
  static std::vector<T> ints(const blok::Json &list) {
    std::vector<T> v;
    for (const blok::Json &x : list.items) {
      require(x.kind == blok::Json::Number && x.number >= 0, "a list holds something else than counts");
      v.push_back((T)x.number);
    }
    return v;
  }
  int slot_of(const std::string &id) {
    auto it = live_.find(id);
    if (it != live_.end()) return it->second;
    require(!free_.empty(), "more than " + std::to_string(kSlots) + " live sequences");
    const int slot = free_.back();
    free_.pop_back();
    live_[id] = slot;
    return slot;
  }
};

int run(int argc, char **argv) {
  std::string model, out;
  int dtype = BLOK_DTYPE_BF16;
  long max_tokens = 4096;
  require(argc % 2 == 1, "usage: blok-trace-run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N");
  for (int i = 1; i + 1 < argc; i += 2) {
    const std::string flag = argv[i], value = argv[i + 1];
    if (flag == "--model") model = value;
    else if (flag == "--out") out = value;
    else if (flag == "--dtype") {
      require(value == "bfloat16" || value == "float32", "unknown dtype: " + value);
      dtype = value == "float32" ? BLOK_DTYPE_F32 : BLOK_DTYPE_BF16;
    } else if (flag == "--max-tokens") {
      max_tokens = std::strtol(value.c_str(), nullptr, 10);
      require(max_tokens >= 1 && max_tokens <= (1 << 28), "bad --max-tokens");
    } else require(false, "unknown flag: " + flag);
  }
  require(!model.empty() && !out.empty(), "--model and --out are needed");
  Replay replay(model, dtype, out, max_tokens);
  std::string line;
  while (std::getline(std::cin, line)) {
    if (line.find_first_not_of(" \t\r") == std::string::npos) continue;
    blok::Json j;
    blok::JsonParser parser(line.data(), line.data() + line.size());
    require(parser.parse(&j), "input: " + parser.error());
    replay.step(j);
  }
  return 0;
}

}  // namespace

int main(int argc, char **argv) {
  try {
    return run(argc, argv);
  } catch (const Fail &f) {
    std::fprintf(stderr, "blok-trace-run: %s\n", f.message.c_str());
    return 1;
  }
}
