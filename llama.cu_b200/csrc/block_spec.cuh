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
  BRANCH_WKV,          // linear attention with a data-dependent decay per channel, token-shifted inputs, bonus for the current token
  BRANCH_LATENT_ATTN   // softmax attention over a sliding window; keys and values of all heads come from one normalised latent
                       // per token (which is what the cache holds), beside one rotated key part shared by all heads
};

struct branch_spec {
  branch_kind kind = BRANCH_WINDOW_ATTN;
  std::string prefix;       // of its tensors below '<layer>.mix.'
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  float out_scale = 1.0f;   // of the branch's result
  // attention
  float score_scale = 1.0f;
  int window = 0, pool = 0;  // pool 0: no blocks
  bool sink = false;         // one more term exp(sink of the head) in every denominator
  bool head_gate = false;    // every head's result times sigmoid of a projection of the row
  // latent attention: per head `dim` unrotated and `rot_dim` rotated query / key dimensions
  int kv_rank = 0, rot_dim = 0;
  int dim_pad() const { return (dim + 7) / 8 * 8; }      // columns of the parts in memory: whole 16-byte vectors
  int rot_pad() const { return (rot_dim + 7) / 8 * 8; }
  int vdim_pad() const { return (vdim + 7) / 8 * 8; }
  int rank_pad() const { return (kv_rank + 7) / 8 * 8; }
  // rotary positions
  int rot_dims = 0;          // 0: no rotation
  double rot_base = 0;
  // retention
  std::vector<float> decay;  // per head
  int out_cols() const { return heads * vdim; }
};

constexpr int MAX_EXPERTS = 1024, MAX_TOP = 32;

struct layer_spec {
  std::vector<branch_spec> branches;
  int ff = 0;  // 0: no feed-forward; of one expert where there are several
  int experts = 0, top = 0;  // experts: 0 = dense, else every token runs `top` of them
  bool is_wkv() const { return branches.size() == 1 && branches[0].kind == BRANCH_WKV; }
};

struct block_spec {
  std::string architecture;
  int vocab = 0, width = 0, streams = 1;
  float eps = 0.f, embed_scale = 1.f;
  int buckets = 0;  // 0: no bigram embedding
  long long mul_prev = 0, mul_cur = 0;  // modulo buckets
  std::vector<layer_spec> layers;
  // residual: plain sum of sublayer results that are normed and scaled channel by channel (norms before and after,
  // factor w) or hyper-connected streams (norm before only, factor 1 + w)
  bool sandwich = false;
  bool loop_input = false;  // a pass over the looped range starts from a linear map of [residual row; embedding row]
  std::vector<int> runs;    // layer of every layer run, in order: a looped range appears once per pass
  std::vector<char> pass_start;  // per run: first of a pass over the looped range
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
