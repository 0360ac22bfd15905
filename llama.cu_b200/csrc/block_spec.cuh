// Block models: decoder stacks described by a config.json (sizes, mixers, order of layers) with their weights in a
// safetensors file.  This header is the host-side description every part works from - loader, caches, step programs - and
// the registry that turns a configuration of a named architecture into it.  Nothing here depends on one architecture.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

#include "json.hpp"

namespace lcu {

// A layer's mixer is one or more branches that read the same normalised row; their results are scaled and added.
enum branch_kind {
  BRANCH_WINDOW_ATTN,  // softmax attention: causal sliding window, optionally with one mean key / value per block before it
  BRANCH_RETENTION,    // linear attention with a fixed decay per head, rotary positions, normalised and gated heads
  BRANCH_WKV           // linear attention with a data-dependent decay per channel, token-shifted inputs, bonus for the current token
};

struct branch_spec {
  branch_kind kind = BRANCH_WINDOW_ATTN;
  std::string prefix;       // of its tensors below '<layer>.mix.'
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  float out_scale = 1.0f;   // of the branch's result
  // attention
  float score_scale = 1.0f;
  int window = 0, pool = 0;  // pool 0: no blocks
  // retention
  int rot_dims = 0;          // 0: no rotation
  double rot_base = 0;
  std::vector<float> decay;  // per head
  int out_cols() const { return heads * vdim; }
};

struct layer_spec {
  std::vector<branch_spec> branches;
  int ff = 0;  // 0: no feed-forward
  bool is_wkv() const { return branches.size() == 1 && branches[0].kind == BRANCH_WKV; }
};

struct block_spec {
  std::string architecture;
  int vocab = 0, width = 0, streams = 1;
  float eps = 0.f, embed_scale = 1.f;
  int buckets = 0;  // 0: no bigram embedding
  long long mul_prev = 0, mul_cur = 0;  // modulo buckets
  std::vector<layer_spec> layers;
  std::vector<int> runs;  // layer of every layer run, in order: a looped range appears once per pass
};

struct architecture {
  const char* name;  // config.json "architecture"
  int (*read)(const json_value& config, block_spec& out);
};
const architecture* find_architecture(const std::string& name);
std::string architecture_names();

// parses configuration text and reads it with the architecture it names; checks what the runtime needs of the sizes
int read_block_config(const std::string& text, block_spec& out);

// ---- safetensors
struct tensor_entry {
  std::string dtype;
  std::vector<long long> shape;
  size_t offset = 0, bytes = 0;  // within the file
};
struct tensor_file {
  std::string path;
  size_t file_bytes = 0;
  std::map<std::string, tensor_entry> tensors;
  int open(const std::string& path);  // reads the header
  const tensor_entry* find(const std::string& name) const {
    auto it = tensors.find(name);
    return it == tensors.end() ? nullptr : &it->second;
  }
};
int read_text_file(const std::string& path, std::string& out);

}  // namespace lcu
