// Block models on the device: weights of a block_spec in one arena, and the loader of a config.json + model.safetensors
// directory.
#pragma once
#include "block_ops.cuh"
#include "block_spec.cuh"
#include "runtime.cuh"

namespace lcu {

// number format of a block model: weights, activations and caches
enum block_dtype : int { BLOCK_BF16 = 0, BLOCK_F32 = 1 };

// Matrices are stored [rows][K] with rows padded to a multiple of 128 and K to a multiple of 256 (zeros), so that every
// size takes the same product kernels; matrices that share an input are stacked.
constexpr int pad_rows(int n) { return (n + 127) / 128 * 128; }
constexpr int pad_stack(int n) { return n > 2048 ? (n + 255) / 256 * 256 : pad_rows(n); }  // long stacks: whole tiles of SM pairs
constexpr int pad_k(int k) { return (k + 255) / 256 * 256; }

struct hyper_weights {
  float *in = nullptr, *out = nullptr, *mix = nullptr;
};
struct branch_weights {
  int q = 0, k = 0, v = 0, g = 0;  // columns of the branch's parts in a row of the stacked projection (latent attention: k is
                                   // the latent, v the shared key part that is rotated)
  int out_col = 0;                 // first column of its output in the mixer's output row
  float* decay = nullptr;          // retention
  float* sink = nullptr;           // attention: per head
  // latent attention: norm of the latent; [keys of all heads; values of all heads] from it, heads padded to 16-byte vectors
  float* latent_norm = nullptr;
  void* up = nullptr;
  int up_rows = 0, up_v = 0, up_k = 0;  // rows, first value row, row length
};
// feed-forward with several experts: expert e's matrices are `gate_up_stride` / `down_stride` elements after expert 0's, in
// gate_up blocks of EXPERT_GATE_BLOCK gate rows alternate with the blocks of the same up rows
constexpr int EXPERT_GATE_BLOCK = 32;
struct expert_weights {
  void *router = nullptr, *gate_up = nullptr, *down = nullptr;
  int router_rows = 0;
  size_t gate_up_stride = 0, down_stride = 0;
};
struct block_layer {
  float *norm1 = nullptr, *norm2 = nullptr;
  float *norm1b = nullptr, *norm2b = nullptr;  // of a sublayer's result, times its channel scale once the weights are in place
  float *scale1 = nullptr, *scale2 = nullptr;
  hyper_weights hc1, hc2;
  std::vector<branch_weights> branches;
  // branches that read the row itself: one stacked projection
  void* proj = nullptr;
  int proj_rows = 0;
  // wkv: r, k, v, g and the first product of the decay, each with its own shifted input
  void* shifted[5] = {};
  int shifted_rows[5] = {};
  float *mu = nullptr, *w2t = nullptr, *w0 = nullptr, *u = nullptr, *head_norm = nullptr;
  int rank = 0;
  // output: columns of all branches side by side
  void* out = nullptr;
  int out_k = 0;
  // feed-forward: [gate; up] and down
  void *gate_up = nullptr, *down = nullptr;
  int ff_pad = 0;
  expert_weights experts;  // (instead of gate_up and down)
};

struct block_model : model_base {
  block_spec spec;
  block_dtype dtype = BLOCK_BF16;
  int device = 0;
  int k_width = 0, n_width = 0, n_vocab_pad = 0;  // padded input / output width, padded vocabulary
  void *embed = nullptr, *bigram = nullptr, *head = nullptr;
  float *final_norm = nullptr, *ones = nullptr;   // ones: [streams], the sum of the streams as an input vector
  float* zeros = nullptr;                         // [streams * streams]
  void* loop_in = nullptr;                        // [n_width][k_loop]
  int k_loop = 0;                                 // padded length of a [residual; embedding] row
  std::vector<block_layer> layers;

  const char* family() const override { return spec.architecture.c_str(); }
  int vocab() const override { return spec.vocab; }
  int width() const override { return spec.width; }
  int n_layers() const override { return (int)spec.layers.size(); }
  size_t elem_bytes() const { return dtype == BLOCK_F32 ? 4 : 2; }

  // allocates everything (zeros) for a description; rank of the wkv decays per layer where it is not in the description
  static int create(std::unique_ptr<block_model>& out, const block_spec& spec, block_dtype dtype, const std::vector<int>& wkv_rank);
  // <dir>/config.json and <dir>/model.safetensors
  static int load(std::unique_ptr<block_model>& out, const std::string& dir, block_dtype dtype);
  int fill_synthetic(uint64_t seed, float scale) override;
  int new_context(std::unique_ptr<context_impl>& out, const context_options& opt) override;

 private:
  struct slot {  // one named tensor and where it goes
    std::string name;
    int rows = 0, cols = 0;   // a vector is one row
    void* dst = nullptr;
    int ld = 0;
    bool f32 = false;         // kept in binary32
    bool transpose = false;
    row_groups groups;        // where rows go
    enum fill_t { MATRIX, ZEROS, ONES, IDENTITY, MEAN, UNIFORM } fill = MATRIX;  // synthetic values
    bool optional = false;    // may be missing: the synthetic values stand
  };
  std::vector<slot> slots() const;
  int set_default(const slot& s);
  int fold_scales();
};

}  // namespace lcu
