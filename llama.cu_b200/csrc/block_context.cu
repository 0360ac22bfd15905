// Step programs and caches of the block models: what a context of theirs adds to the shared driver (context.cuh).
//
// Every layer run - a looped layer counts once per pass - has caches of its own: window attention a key / value cache and
// the means of its completed blocks, recurrences a binary32 state per head, token-shifted mixers the previous token's row.
// Nothing is cleared between sequences: position 0 ignores what earlier sequences left.
//
// A single token runs as one captured graph: per sublayer one pass over the residual streams (update, input, norm and,
// where the mixer wants it, the token shift), one weight-streaming product, one launch for all heads of all branches, the
// output product.  Several rows run the tensor-core products, the window attention and the scans over all rows at once;
// passes longer than ROWS rows are cut, which changes nothing but the number of launches.
#include <algorithm>
#include <cstring>

#include "block_model.cuh"
#include "block_ops.cuh"
#include "context.cuh"
#include "gemm_tc.cuh"
#include "ops.cuh"
#include "prefill.cuh"

namespace lcu {
namespace {

constexpr int ROWS = 2048;      // rows of one pass
constexpr int LOGIT_ROWS = 128; // rows of logits formed at once

template <typename T>
struct run_cache {  // of one layer run
  window_cache<T> window{};
  float* state = nullptr;
  T* prev = nullptr;
};

template <typename T>
struct block_context : context_impl {
  block_model* m = nullptr;
  int rows_cap = 0;
  std::vector<run_cache<T>> runs;
  std::vector<std::pair<std::pair<int, double>, float2*>> rotations;  // (dims, base) -> table
  // activations [rows_cap]
  float *xs = nullptr, *y = nullptr, *raw = nullptr, *packed = nullptr, *packed_v = nullptr, *low = nullptr, *hidden = nullptr, *logits = nullptr;
  T *h = nullptr, *mix = nullptr, *proj = nullptr, *cat = nullptr, *gu = nullptr, *act = nullptr;
  T* shifted[4] = {};
  int ld_raw = 0, ld_shift = 0;
  int* row_list = nullptr;
  int* h_rows = nullptr;  // pinned
  int launches = 0;       // kernels of the step being put together
  int step_launches = 0;

  ~block_context() override {
    if (h_rows) cudaFreeHost(h_rows);
    for (auto& r : rotations) cudaFree(r.second);
  }

  int create(block_model* model, const context_options& o);
  int enqueue_decode_step(int variant) override;
  int enqueue_prefill(int m_rows, const pass_request& rq) override;
  int decode_variant(int) const override { return 0; }
  int kernels_per_step() const override { return step_launches; }
  int read_step_logits(float* out_host) override {
    LCU_CUDA(cudaMemcpy(out_host, logits, (size_t)n_vocab * 4, cudaMemcpyDeviceToHost));
    return LCU_OK;
  }
  int read_hidden(__half* out_host) override {
    std::vector<float> v(width);
    LCU_CUDA(cudaMemcpy(v.data(), hidden, (size_t)width * 4, cudaMemcpyDeviceToHost));
    for (int i = 0; i < width; ++i) out_host[i] = __float2half(v[i]);
    return LCU_OK;
  }
  int rollover(int) override { LCU_REQUIRE(false, "rollover: a recurrent state cannot drop its oldest tokens (%s)", m->family()); }
  int bench_kernel(int, int, float*, uint64_t*) override { LCU_REQUIRE(false, "bench_kernel: not available for %s models", m->family()); }

  cudaStream_t stream() { return gpus[0].stream; }
  int* err() { return gpus[0].state + 3; }
  float2* rotation(const branch_spec& b) const {
    for (auto& r : rotations)
      if (r.first.first == b.rot_dims && r.first.second == b.rot_base) return r.second;
    return nullptr;
  }
  int product(void* out, bool f32_out, const T* x, int ldx, const void* w, int rows, int N, int K);
  int hyper(const hyper_weights& in, const float* norm_w, const hyper_weights* done, int rows, const block_layer* shift, T* prev);
  attn_rows<T> attention(int run, int b, int ld);
  scan_rows<T> recurrence(int run, int b, int ld);
  int mixer_rows(int run, int rows, int pos0);
  int mixer_one(int run);
  int feed_forward(const block_layer& L, int rows);
  int rows_to_logits(const hyper_weights* done, const int* list, size_t row0, int n);
  int pick_token(bool advance_only, int advance, short* next, short* log_at, int* step, int log_cap, int pdl);
};

template <typename T>
constexpr bool is_f32() { return sizeof(T) == 4; }

// out[rows][N] = x . w^T; f32_out: binary32 results, else T
template <typename T>
int block_context<T>::product(void* out, bool f32_out, const T* x, int ldx, const void* w, int rows, int N, int K) {
  ++launches;
  if (is_f32<T>()) return launch_matmul_f32((float*)out, (const float*)x, ldx, (const float*)w, rows, N, K, stream());
  if (rows == 1) {
    gemv_batch b;
    b.n = 1;
    b.w[0] = w;
    b.x[0] = x;
    b.out[0] = out;
    b.rows[0] = N;
    b.f32[0] = f32_out;
    return launch_gemv_bf16(b, K, err(), stream(), opt.use_pdl);
  }
  return launch_gemm_tc(f32_out ? TC_BF16_F32 : TC_BF16, out, x, ldx, w, rows, N, K, 0.f, err(), stream());
}

// residual pass in front of a sublayer (done: the sublayer whose result is in y, or null)
template <typename T>
int block_context<T>::hyper(const hyper_weights& in, const float* norm_w, const hyper_weights* done, int rows, const block_layer* shift, T* prev) {
  hyper_params<T> p{};
  p.xs = xs;
  p.width = width;
  p.streams = m->spec.streams;
  if (done) {
    p.y = y;
    p.ldy = m->n_width;
    p.up_mix = done->mix;
    p.up_out = done->out;
    p.store = 1;
  }
  p.in = in.in;
  p.norm_w = norm_w;
  p.eps = m->spec.eps;
  p.h = h;
  p.ldh = m->k_width;
  if (shift && rows == 1) {
    p.prev = prev;
    p.mu = shift->mu;
    p.mix = mix;
    p.mix_stride = (size_t)rows_cap * m->k_width;
    p.n_mix = 5;
    p.pos = gpus[0].state;
  }
  ++launches;
  return launch_hyper_rows(p, rows, stream());
}

template <typename T>
attn_rows<T> block_context<T>::attention(int run, int b, int ld) {
  const int l = m->spec.runs[run];
  const branch_spec& bs = m->spec.layers[l].branches[b];
  const branch_weights& bw = m->layers[l].branches[b];
  attn_rows<T> a{};
  a.q = proj + bw.q;
  a.k = proj + bw.k;
  a.v = proj + bw.v;
  a.ld = ld;
  a.cache = runs[run].window;
  a.heads = bs.heads;
  a.kv_heads = bs.kv_heads;
  a.dim = bs.dim;
  a.vdim = bs.vdim;
  a.window = bs.window;
  a.pool = bs.pool;
  a.scale = bs.score_scale;
  a.out_scale = bs.out_scale;
  a.out = cat + bw.out_col;
  a.ldo = m->layers[l].out_k;
  return a;
}

template <typename T>
scan_rows<T> block_context<T>::recurrence(int run, int b, int ld) {
  const int l = m->spec.runs[run];
  const branch_spec& bs = m->spec.layers[l].branches[b];
  const block_layer& L = m->layers[l];
  scan_rows<T> s{};
  s.heads = bs.heads;
  s.dim = bs.dim;
  s.vdim = bs.vdim;
  s.state = runs[run].state;
  if (bs.kind == BRANCH_WKV) {
    s.q = shifted[0];
    s.k = shifted[1];
    s.v = shifted[2];
    s.ldq = s.ldk = s.ldv = L.shifted_rows[0];
    s.u = L.u;
  } else {
    const branch_weights& bw = L.branches[b];
    s.q = proj + bw.q;
    s.k = proj + bw.k;
    s.v = proj + bw.v;
    s.ldq = s.ldk = s.ldv = ld;
    s.rope = rotation(bs);
    s.rot_dims = bs.rot_dims;
    s.kscale = (float)(1.0 / std::sqrt((double)bs.dim));
    s.decay = bw.decay;
  }
  s.out = raw;
  s.ldo = bs.out_cols();
  s.packed = packed;
  s.packed_v = packed_v;
  s.err = gpus[0].state + 3;
  return s;
}

// mixer of several rows: h -> y
template <typename T>
int block_context<T>::mixer_rows(int run, int rows, int pos0) {
  const int l = m->spec.runs[run];
  const layer_spec& ls = m->spec.layers[l];
  const block_layer& L = m->layers[l];
  const int K = m->k_width;
  if (ls.is_wkv()) {
    const size_t stride = (size_t)rows_cap * K;
    const branch_spec& bs = ls.branches[0];
    LCU_TRY(launch_token_shift(h, K, runs[run].prev, L.mu, mix, stride, 5, rows, width, pos0, stream()));
    for (int j = 0; j < 4; ++j) LCU_TRY(product(shifted[j], false, mix + j * stride, K, L.shifted[j], rows, L.shifted_rows[j], K));
    LCU_TRY(product(low, true, mix + 4 * stride, K, L.shifted[4], rows, L.shifted_rows[4], K));
    size_t head_stride, row_stride, offset;
    scan_decay_layout(bs.dim, bs.vdim, rows, &head_stride, &row_stride, &offset);
    LCU_TRY(launch_wkv_decay(packed + offset, head_stride, row_stride, low, L.shifted_rows[4], L.w2t, L.w0, L.rank, bs.heads, bs.dim, rows, stream()));
    LCU_TRY(launch_scan(recurrence(run, 0, 0), true, rows, pos0, stream()));
    LCU_TRY(launch_head_gate(cat, L.out_k, raw, bs.out_cols(), shifted[3], L.shifted_rows[3], L.head_norm, bs.heads, bs.vdim, m->spec.eps, bs.out_scale,
                             rows, stream()));
  } else {
    LCU_TRY(product(proj, false, h, K, L.proj, rows, L.proj_rows, K));
    for (size_t b = 0; b < ls.branches.size(); ++b) {
      const branch_spec& bs = ls.branches[b];
      const branch_weights& bw = L.branches[b];
      if (bs.kind == BRANCH_WINDOW_ATTN) {
        const attn_rows<T> a = attention(run, (int)b, L.proj_rows);
        LCU_TRY(launch_window_append(a, rows, pos0, stream()));
        LCU_TRY(launch_window_attention(a, rows, pos0, stream()));
      } else {
        LCU_TRY(launch_scan(recurrence(run, (int)b, L.proj_rows), false, rows, pos0, stream()));
        LCU_TRY(launch_head_gate(cat + bw.out_col, L.out_k, raw, bs.out_cols(), proj + bw.g, L.proj_rows, (const float*)nullptr, bs.heads, bs.vdim,
                                 m->spec.eps, bs.out_scale, rows, stream()));
      }
    }
  }
  return product(y, true, cat, L.out_k, L.out, rows, m->n_width, L.out_k);
}

// mixer of one token: h (and its shifted copies) -> y
template <typename T>
int block_context<T>::mixer_one(int run) {
  const int l = m->spec.runs[run];
  const layer_spec& ls = m->spec.layers[l];
  const block_layer& L = m->layers[l];
  const int K = m->k_width;
  if (ls.is_wkv()) {
    const size_t stride = (size_t)rows_cap * K;
    if (is_f32<T>()) {
      for (int j = 0; j < 5; ++j) LCU_TRY(product(j < 4 ? (void*)shifted[j] : low, j == 4, mix + j * stride, K, L.shifted[j], 1, L.shifted_rows[j], K));
    } else {
      gemv_batch b;
      b.n = 5;
      for (int j = 0; j < 5; ++j) {
        b.w[j] = L.shifted[j];
        b.x[j] = mix + j * stride;
        b.out[j] = j < 4 ? (void*)shifted[j] : low;
        b.rows[j] = L.shifted_rows[j];
        b.f32[j] = j == 4;
      }
      ++launches;
      LCU_TRY(launch_gemv_bf16(b, K, err(), stream(), opt.use_pdl));
    }
  } else {
    LCU_TRY(product(proj, false, h, K, L.proj, 1, L.proj_rows, K));
  }
  mixer_step<T> st{};
  st.n_branches = (int)ls.branches.size();
  LCU_REQUIRE(st.n_branches <= STEP_MAX_BRANCHES, "mixer with %d branches", st.n_branches);
  for (int i = 0; i < st.n_branches; ++i) {
    const branch_spec& bs = ls.branches[i];
    const branch_weights& bw = L.branches[i];
    step_branch<T>& b = st.b[i];
    b.kind = bs.kind;
    b.first = st.n_clusters;
    st.n_clusters += bs.heads;
    b.eps = m->spec.eps;
    b.out_scale = bs.out_scale;
    b.out = cat + bw.out_col;
    if (bs.kind == BRANCH_WINDOW_ATTN) {
      b.attn = attention(run, i, L.proj_rows);
    } else {
      b.scan = recurrence(run, i, L.proj_rows);
      if (bs.kind == BRANCH_WKV) {
        b.g = shifted[3];
        b.low = low;
        b.w2t = L.w2t;
        b.w0 = L.w0;
        b.rank = L.rank;
        b.norm = L.head_norm;
      } else {
        b.g = proj + bw.g;
      }
    }
  }
  st.pos = gpus[0].state;
  ++launches;
  LCU_TRY(launch_mixer_step(st, opt.context_len, stream()));
  return product(y, true, cat, L.out_k, L.out, 1, m->n_width, L.out_k);
}

template <typename T>
int block_context<T>::feed_forward(const block_layer& L, int rows) {
  const int K = m->k_width, f = L.ff_pad;
  if (!is_f32<T>() && rows == 1) {
    ++launches;
    LCU_TRY(launch_gemv_bf16_gated(act, h, L.gate_up, f, K, err(), stream(), opt.use_pdl));
  } else {
    const int tile = is_f32<T>() ? 0 : gemm_tc_gated_tile(rows, f, K);
    if (tile && gemm_tc_gated_supported(rows, f, K, K, h, L.gate_up, act)) {
      LCU_TRY(launch_gemm_tc_gated(TC_BF16, act, h, K, L.gate_up, rows, f, K, err(), stream(), tile));
    } else {
      LCU_TRY(product(gu, false, h, K, L.gate_up, rows, 2 * f, K));
      ++launches;
      LCU_TRY(launch_gate_rows(act, gu, rows, f, stream()));
    }
  }
  return product(y, true, act, f, L.down, rows, m->n_width, f);
}

// the last residual pass and the output matrix for n rows: list[i], or row0 alone when list is null
template <typename T>
int block_context<T>::rows_to_logits(const hyper_weights* done, const int* list, size_t row0, int n) {
  hyper_params<T> p{};
  p.xs = xs + row0 * m->spec.streams * width;
  p.width = width;
  p.streams = m->spec.streams;
  if (done) {
    p.y = y + row0 * m->n_width;
    p.ldy = m->n_width;
    p.up_mix = done->mix;
    p.up_out = done->out;
  }
  p.in = m->ones;
  p.norm_w = m->final_norm;
  p.eps = m->spec.eps;
  p.rows = list;
  p.h = h;
  p.ldh = m->k_width;
  p.u_out = list ? nullptr : hidden;
  ++launches;
  LCU_TRY(launch_hyper_rows(p, n, stream()));
  return product(logits, true, h, m->k_width, m->head, n, m->n_vocab_pad, m->k_width);
}

template <typename T>
int block_context<T>::pick_token(bool advance_only, int advance, short* next, short* log_at, int* step, int log_cap, int pdl) {
  gpu_state& g = gpus[0];
  if (advance_only) return launch_bump_pos(g.state, advance, g.stream);
  head_params hp{};
  hp.logits_f32 = logits;
  hp.probs = probs;
  hp.n_vocab = n_vocab;
  hp.temperature = opt.temperature;
  hp.token_out = g.state + 2;
  hp.next_ids = next;
  hp.pos = g.state;
  hp.advance = advance;
  hp.log = log_at;
  hp.step = step;
  hp.log_capacity = log_cap;
  ++launches;
  LCU_TRY(launch_logits_head(hp, g.stream, pdl));
  if (opt.sampling) {
    ++launches;
    LCU_TRY(launch_sample(probs, n_vocab, opt.sample_seed, g.state, 0.f, g.state + 2, next, log_at, step, log_cap, g.stream));
  }
  return LCU_OK;
}

template <typename T>
int block_context<T>::enqueue_decode_step(int) {
  gpu_state& g = gpus[0];
  device_guard dg(g.device);
  launches = 0;
  embed_params<T> e{};
  e.xs = xs;
  e.table = (const T*)m->embed;
  e.bigram = (const T*)m->bigram;
  e.ids = ids;
  e.prev_token = g.state + 4;
  e.pos = g.state;
  e.m = 1;
  e.width = width;
  e.streams = m->spec.streams;
  e.buckets = m->spec.buckets;
  e.mul_prev = m->spec.mul_prev;
  e.mul_cur = m->spec.mul_cur;
  e.scale = m->spec.embed_scale;
  ++launches;
  LCU_TRY(launch_block_embed(e, g.stream));
  const hyper_weights* done = nullptr;
  for (size_t run = 0; run < m->spec.runs.size(); ++run) {
    const int l = m->spec.runs[run];
    const block_layer& L = m->layers[l];
    const bool wkv = m->spec.layers[l].is_wkv();
    LCU_TRY(hyper(L.hc1, L.norm1, done, 1, wkv ? &L : nullptr, runs[run].prev));
    LCU_TRY(mixer_one((int)run));
    done = &L.hc1;
    if (m->spec.layers[l].ff > 0) {
      LCU_TRY(hyper(L.hc2, L.norm2, done, 1, nullptr, nullptr));
      LCU_TRY(feed_forward(L, 1));
      done = &L.hc2;
    }
  }
  LCU_TRY(rows_to_logits(done, nullptr, 0, 1));
  LCU_TRY(pick_token(false, 1, ids, log, g.state + 1, opt.context_len, opt.use_pdl));
  step_launches = launches;
  return LCU_OK;
}

template <typename T>
int block_context<T>::enqueue_prefill(int m_rows, const pass_request& rq) {
  gpu_state& g = gpus[0];
  device_guard dg(g.device);
  for (int r0 = 0; r0 < m_rows; r0 += rows_cap) {
    const int rows = std::min(rows_cap, m_rows - r0), pos0 = start_pos + r0;
    embed_params<T> e{};
    e.xs = xs;
    e.table = (const T*)m->embed;
    e.bigram = (const T*)m->bigram;
    e.ids = ids + r0;
    e.prev_token = g.state + 4;
    e.pos_value = pos0;
    e.m = rows;
    e.width = width;
    e.streams = m->spec.streams;
    e.buckets = m->spec.buckets;
    e.mul_prev = m->spec.mul_prev;
    e.mul_cur = m->spec.mul_cur;
    e.scale = m->spec.embed_scale;
    LCU_TRY(launch_block_embed(e, g.stream));
    const hyper_weights* done = nullptr;
    for (size_t run = 0; run < m->spec.runs.size(); ++run) {
      const int l = m->spec.runs[run];
      const block_layer& L = m->layers[l];
      LCU_TRY(hyper(L.hc1, L.norm1, done, rows, nullptr, nullptr));
      LCU_TRY(mixer_rows((int)run, rows, pos0));
      done = &L.hc1;
      if (m->spec.layers[l].ff > 0) {
        LCU_TRY(hyper(L.hc2, L.norm2, done, rows, nullptr, nullptr));
        LCU_TRY(feed_forward(L, rows));
        done = &L.hc2;
      }
    }
    // logits of the wanted rows of this pass, LOGIT_ROWS at a time
    std::vector<int> at;  // index into want
    for (int i = 0; i < rq.n_want; ++i)
      if (rq.want[i] >= r0 && rq.want[i] < r0 + rows) at.push_back(i);
    std::vector<float> slab;
    for (size_t a0 = 0; a0 < at.size(); a0 += LOGIT_ROWS) {
      const int n = (int)std::min<size_t>(LOGIT_ROWS, at.size() - a0);
      for (int i = 0; i < n; ++i) h_rows[i] = rq.want[at[a0 + i]] - r0;
      LCU_CUDA(cudaMemcpyAsync(row_list, h_rows, n * sizeof(int), cudaMemcpyHostToDevice, g.stream));
      LCU_TRY(rows_to_logits(done, row_list, 0, n));
      slab.resize((size_t)n * m->n_vocab_pad);
      LCU_CUDA(cudaMemcpyAsync(slab.data(), logits, slab.size() * 4, cudaMemcpyDeviceToHost, g.stream));
      LCU_CUDA(cudaStreamSynchronize(g.stream));
      for (int i = 0; i < n; ++i)
        memcpy(rq.logits_out + (size_t)at[a0 + i] * n_vocab, slab.data() + (size_t)i * m->n_vocab_pad, (size_t)n_vocab * 4);
    }
    if (r0 + rows == m_rows) {
      if (rq.token) LCU_TRY(rows_to_logits(done, nullptr, rows - 1, 1));
      LCU_TRY(pick_token(!rq.token, m_rows, nullptr, nullptr, nullptr, 0, 0));
    }
  }
  return LCU_OK;
}

template <typename T>
int block_context<T>::create(block_model* model, const context_options& o) {
  m = model;
  opt = o;
  n_vocab = m->spec.vocab;
  width = m->spec.width;
  const size_t ctxl = opt.context_len;
  rows_cap = std::min(opt.context_len, ROWS);
  gpus.resize(1);
  kv_arenas.assign(1, nullptr);
  gpu_state& g = gpus[0];
  g.device = m->device;
  device_guard dg(g.device);
  LCU_CUDA(cudaStreamCreateWithFlags(&g.stream, cudaStreamNonBlocking));
  LCU_CUDA(cudaEventCreateWithFlags(&g.ev, cudaEventDisableTiming));
  // widest rows over the layers
  size_t w_proj = 0, w_cat = 0, w_gu = 0, w_raw = 0, w_shift = 0, w_low = 0, w_packed = 0, w_values = 0;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const block_layer& L = m->layers[i];
    w_proj = std::max(w_proj, (size_t)L.proj_rows);
    w_cat = std::max(w_cat, (size_t)L.out_k);
    w_gu = std::max(w_gu, (size_t)L.ff_pad);
    w_shift = std::max(w_shift, (size_t)L.shifted_rows[0]);
    w_low = std::max(w_low, (size_t)L.shifted_rows[4]);
    for (auto& b : m->spec.layers[i].branches) {
      w_raw = std::max(w_raw, (size_t)b.out_cols());
      if (b.kind == BRANCH_WINDOW_ATTN) continue;
      size_t pk = 0, pv = 0;
      scan_scratch(b.heads, b.dim, b.vdim, b.kind == BRANCH_WKV, rows_cap, &pk, &pv);
      w_packed = std::max(w_packed, pk);
      w_values = std::max(w_values, pv);
    }
  }
  const size_t R = rows_cap, K = m->k_width, es = sizeof(T);
  for (int pass = 0; pass < 2; ++pass) {
    carve cv;
    char* base = (char*)g.arena;
    auto take = [&](auto*& p, size_t bytes) { p = reinterpret_cast<std::remove_reference_t<decltype(p)>>(base + cv.take(bytes)); };
    take(g.state, 64);
    take(ids, ctxl * 2);
    take(log, ctxl * 2);
    take(probs, (size_t)n_vocab * 2);
    take(row_list, LOGIT_ROWS * sizeof(int));
    take(xs, R * m->spec.streams * width * 4);
    take(y, R * m->n_width * 4);
    take(raw, R * w_raw * 4);
    take(packed, w_packed * 4);
    take(packed_v, w_values * 4);
    take(low, R * w_low * 4);
    take(hidden, (size_t)width * 4);
    take(logits, std::min<size_t>(R, LOGIT_ROWS) * m->n_vocab_pad * 4);
    take(h, R * K * es);
    take(mix, (w_shift ? 5 : 0) * R * K * es);
    take(proj, R * w_proj * es);
    take(cat, R * w_cat * es);
    take(gu, 2 * R * w_gu * es);
    take(act, R * w_gu * es);
    for (auto& s : shifted) take(s, R * w_shift * es);
    if (pass == 0) {
      g.arena_bytes = cv.off;
      LCU_CUDA(cudaMalloc(&g.arena, cv.off));
      LCU_CUDA(cudaMemsetAsync(g.arena, 0, cv.off, g.stream));
    }
  }
  // caches of every layer run
  runs.resize(m->spec.runs.size());
  for (int pass = 0; pass < 2; ++pass) {
    carve cv;
    char* base = (char*)kv_arenas[0];
    auto take = [&](auto*& p, size_t bytes) { p = reinterpret_cast<std::remove_reference_t<decltype(p)>>(base + cv.take(bytes)); };
    for (size_t r = 0; r < runs.size(); ++r)
      for (auto& b : m->spec.layers[m->spec.runs[r]].branches) {
        if (b.kind == BRANCH_WINDOW_ATTN) {
          window_cache<T>& w = runs[r].window;
          w.ctx_len = opt.context_len;
          w.n_blocks = b.pool > 0 ? opt.context_len / b.pool : 0;
          w.ldk = (int)round_up(b.dim, 8);
          w.ldv = (int)round_up(b.vdim, 8);
          take(w.k, b.kv_heads * ctxl * w.ldk * es);
          take(w.v, b.kv_heads * ctxl * w.ldv * es);
          take(w.kp, (size_t)b.kv_heads * w.n_blocks * w.ldk * es);
          take(w.vp, (size_t)b.kv_heads * w.n_blocks * w.ldv * es);
        } else {
          take(runs[r].state, (size_t)b.heads * b.dim * b.vdim * 4);
          if (b.kind == BRANCH_WKV) take(runs[r].prev, (size_t)width * es);
        }
      }
    if (pass == 0) {
      kv_bytes = cv.off;
      LCU_CUDA(cudaMalloc(&kv_arenas[0], std::max<size_t>(cv.off, ALIGN)));
      LCU_CUDA(cudaMemsetAsync(kv_arenas[0], 0, std::max<size_t>(cv.off, ALIGN), g.stream));
    }
  }
  for (auto& l : m->spec.layers)
    for (auto& b : l.branches)
      if (b.rot_dims > 0 && !rotation(b)) {
        float2* t = nullptr;
        LCU_CUDA(cudaMalloc(&t, ctxl * (b.rot_dims / 2) * sizeof(float2)));
        rotations.push_back({{b.rot_dims, b.rot_base}, t});
        LCU_TRY(launch_rotation_table(t, opt.context_len, b.rot_dims, b.rot_base, g.stream));
      }
  LCU_CUDA(cudaMallocHost(&h_rows, LOGIT_ROWS * sizeof(int)));
  LCU_CUDA(cudaStreamSynchronize(g.stream));
  return open_streams(opt.context_len);
}

template <typename T>
int make_context(block_model* m, std::unique_ptr<context_impl>& out, const context_options& opt) {
  auto holder = std::make_unique<context>();  // (its destructor releases what was allocated if a step below fails)
  holder->impl = std::make_unique<block_context<T>>();
  LCU_TRY(static_cast<block_context<T>&>(*holder->impl).create(m, opt));
  out = std::move(holder->impl);
  return LCU_OK;
}

}  // namespace

int block_model::new_context(std::unique_ptr<context_impl>& out, const context_options& opt) {
  return dtype == BLOCK_F32 ? make_context<float>(this, out, opt) : make_context<__nv_bfloat16>(this, out, opt);
}

}  // namespace lcu
