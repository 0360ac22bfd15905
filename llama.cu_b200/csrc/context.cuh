// Shared part of every context: the step driver's state (position, streams, staging, captured decode steps) and the
// interface a model family implements - the layer programs of a single-token step and of a multi-row pass.
#pragma once
#include <vector>

#include "gemv.cuh"
#include "runtime.cuh"

namespace lcu {

#define LCU_TRY(expr)      \
  do {                     \
    int _rc = (expr);      \
    if (_rc) return _rc;   \
  } while (0)

constexpr size_t ALIGN = 256;
struct carve {  // offsets of the parts of one allocation
  size_t off = 0;
  size_t take(size_t bytes) {
    size_t o = off;
    off += round_up(bytes, ALIGN);
    return o;
  }
};

struct gpu_state {
  int device = 0;
  cudaStream_t stream = nullptr;
  cudaEvent_t ev = nullptr;
  void* arena = nullptr;
  size_t arena_bytes = 0;
  __half *x = nullptr, *norm = nullptr, *q = nullptr, *kn = nullptr, *vn = nullptr, *att = nullptr;
  __half *h1 = nullptr, *h3 = nullptr, *hs = nullptr;
  __half* scores = nullptr;  // prompt attention on tcgen05: [heads][context_len][round_up(context_len, 128)] scores / probabilities
  __half* deq = nullptr;  // u8 models: the dequantized matrix (or stack of matrices) of the prompt GEMM in flight
  size_t deq_halves = 0;
  // prompt path of u8 models: matrices are expanded to fp16 one job ahead on a side stream, into two alternating buffers
  __half* deq_buf[2] = {nullptr, nullptr};
  cudaStream_t side = nullptr;
  cudaEvent_t deq_done[2] = {nullptr, nullptr}, gemm_done[2] = {nullptr, nullptr};
  long deq_issued = 0, deq_used = 0;  // jobs expanded / consumed so far (job j lives in buffer j % 2)
  float2* rope = nullptr;
  int* state = nullptr;  // [0] position, [1] step counter, [2] last token, [3] error word
};

// What a multi-row pass is asked for beside advancing the caches: binary32 logits of some of its rows (host memory,
// [n_want][n_vocab], rows in the order of `want`), and the next token unless the caller only replays given tokens.
struct pass_request {
  const int* want = nullptr;
  int n_want = 0;
  float* logits_out = nullptr;
  bool token = true;
};

struct context_impl {
  context_options opt;
  int n_vocab = 0, width = 0;
  int start_pos = 0;
  std::vector<gpu_state> gpus;           // in order of first use
  std::vector<void*> kv_arenas;          // one per GPU
  size_t kv_bytes = 0;
  short* ids = nullptr;                  // token ids on the embedding GPU [context_len]
  __half* probs = nullptr;               // on the output GPU
  short* log = nullptr;                  // generated tokens of a chained run [context_len]
  int* h_stage = nullptr;                // pinned: [0] position, [1] zero, [2] token read-back
  short* h_ids = nullptr;                // pinned token staging [context_len]
  cudaEvent_t t0 = nullptr, t1 = nullptr;
  // captured decode steps, one per variant (decode_variant)
  cudaGraphExec_t graph[2] = {nullptr, nullptr};
  bool graph_failed = false;
  bool warmed_variant[2] = {false, false};
  int last_row = 0;                      // row of the activations that holds the last token's residual stream

  virtual ~context_impl() = default;
  gpu_state& first() { return gpus.front(); }
  gpu_state& last() { return gpus.back(); }

  // ---- what a model family implements
  // kernels of one single-token step, in stream order: reads the position from the state words, advances it, leaves the
  // token in state[2] and in ids[0]; capturable
  virtual int enqueue_decode_step(int variant) = 0;
  // m_rows tokens (in `ids`) from start_pos on
  virtual int enqueue_prefill(int m_rows, const pass_request& rq) = 0;
  // which captured step serves a step that sees n_keys positions (0 or 1)
  virtual int decode_variant(int n_keys) const = 0;
  virtual int kernels_per_step() const = 0;
  // single tokens take the multi-row pass (no fused step exists for them)
  virtual bool rows_only() const { return false; }
  // binary32 logits of the last single-token step, to the host
  virtual int read_step_logits(float* out_host) = 0;
  virtual int read_hidden(__half* out_host) = 0;
  virtual int rollover(int keep) = 0;
  virtual int bench_kernel(int which, int reps, float* ms_per_launch, uint64_t* bytes_per_launch) = 0;

  // ---- shared
  int open_streams(int context_len);     // pinned staging and events; gpus must be filled in
  int build_graph(int variant);
  int run_decode_step(int n_keys);
  int stage_inputs(const short* tokens, int n);
};

}  // namespace lcu
