// Step programs and caches of the block models: what a context of theirs adds to the shared driver (context.cuh).
//
// Every layer run - a looped layer counts once per pass - has caches of its own: window attention a key / value cache and
// the means of its completed blocks, latent attention the normed latents and the shared key part, recurrences a binary32
// state per head, token-shifted mixers the previous token's row.  Nothing is cleared between sequences: position 0 ignores what earlier sequences left.
//
// A single token runs as one captured graph: per sublayer one pass over the residual streams (update, input, norm and,
// where the mixer wants it, the token shift), one weight-streaming product, one launch for all heads of all branches, the
// output product.  Several rows run the tensor-core products, the window attention and the scans over all rows at once;
// latent attention first forms the keys and values of all positions its rows see, a routed feed-forward lays the rows out
// expert by expert;
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
  latent_cache<T> latent{};
  float* state = nullptr;
  T* prev = nullptr;
};

// a sublayer result in y that the residual has not taken in yet
struct pending_result {
  const hyper_weights* streams = nullptr;            // null: nothing is pending
  const float* post = nullptr;                       // output norm and channel scale
  const int* pieces = nullptr;                       // rows of y that make up a row's result [row][n_pieces]
  int n_pieces = 0;
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
  T *loop_row = nullptr, *staged = nullptr, *kv = nullptr;  // [residual; embedding] rows; latents, keys and values of a pass
  // routed feed-forward: router logits, rows by expert, their weights and places; picks of a single token
  float *z = nullptr, *row_weight = nullptr, *pick_weight = nullptr;
  T* packed_rows = nullptr;
  int *places = nullptr, *route_ints = nullptr, *n_tiles = nullptr, *pick = nullptr, *first_rows = nullptr;
  int4* tiles = nullptr;
  hyper_weights replace;  // the result becomes the residual
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
  int residual(hyper_params<T>& p, const pending_result& done, int n_rows);
  int hyper(const hyper_weights& in, const float* norm_w, const pending_result& done, int rows, const block_layer* shift, T* prev, const layer_spec* routed,
            const block_layer* experts);
  int start_pass(const pending_result& done, int rows);
  int layers(int rows, int pos0, pending_result& done);
  attn_rows<T> attention(int run, int b, int ld);
  scan_rows<T> recurrence(int run, int b, int ld);
  latent_rows<T> latents(int run, int b, int ld);
  int latent_attention_rows(int run, int b, int rows, int pos0);
  int mixer_rows(int run, int rows, int pos0);
  int mixer_one(int run);
  int feed_forward(const block_layer& L, int rows);
  int expert_rows(const layer_spec& ls, const block_layer& L, int rows, pending_result& done);
  int expert_one(const layer_spec& ls, const block_layer& L, pending_result& done);
  int rows_to_logits(const pending_result& done, const int* list, size_t row0, int n);
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

// a residual pass: what every one of them shares
template <typename T>
int block_context<T>::residual(hyper_params<T>& p, const pending_result& done, int n_rows) {
  p.width = width;
  p.streams = m->spec.streams;
  p.norm_base = m->spec.sandwich ? 0.f : 1.f;
  p.eps = m->spec.eps;
  if (done.streams) {
    p.ldy = m->n_width;
    p.up_mix = done.streams->mix;
    p.up_out = done.streams->out;
    p.post_w = done.post;
    p.n_y = done.n_pieces;
  }
  ++launches;
  return launch_hyper_rows(p, n_rows, stream());
}

// residual pass in front of a sublayer (done: the sublayer whose result is in y); a single row of a routed feed-forward also
// picks its experts
template <typename T>
int block_context<T>::hyper(const hyper_weights& in, const float* norm_w, const pending_result& done, int rows, const block_layer* shift, T* prev,
                            const layer_spec* routed, const block_layer* experts) {
  hyper_params<T> p{};
  p.xs = xs;
  if (done.streams) {
    p.y = y;
    p.y_rows = done.pieces;
    p.store = 1;
  }
  p.in = in.in;
  p.norm_w = norm_w;
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
  if (routed && rows == 1 && !is_f32<T>()) {
    p.router = (const T*)experts->experts.router;
    p.ld_router = m->k_width;
    p.experts = routed->experts;
    p.top = routed->top;
    p.pick = pick;
    p.pick_weight = pick_weight;
  }
  return residual(p, done, rows);
}

// a pass over the looped range begins: y = loop_in [residual; embedding], which becomes the residual
template <typename T>
int block_context<T>::start_pass(const pending_result& done, int rows) {
  hyper_params<T> p{};
  p.xs = xs;
  if (done.streams) {
    p.y = y;
    p.y_rows = done.pieces;
  }
  p.in = m->ones;
  p.h = loop_row;  // (the embedding half was written with the rows themselves)
  p.ldh = m->k_loop;
  LCU_TRY(residual(p, done, rows));
  return product(y, true, loop_row, m->k_loop, m->loop_in, rows, m->n_width, m->k_loop);
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
  a.q_head = bs.dim;
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
latent_rows<T> block_context<T>::latents(int run, int b, int ld) {
  const int l = m->spec.runs[run];
  const branch_spec& bs = m->spec.layers[l].branches[b];
  const branch_weights& bw = m->layers[l].branches[b];
  latent_rows<T> p{};
  p.q = proj + bw.q;
  p.c = proj + bw.k;
  p.k = proj + bw.v;
  p.ld = ld;
  p.cache = runs[run].latent;
  p.heads = bs.heads;
  p.dim = bs.dim;
  p.rot_dim = bs.rot_dim;
  p.kv_rank = bs.kv_rank;
  p.vdim = bs.vdim;
  p.window = bs.window;
  p.rope = rotation(bs);
  p.rot_dims = bs.rot_dims;
  p.norm = bw.latent_norm;
  p.eps = m->spec.eps;
  p.staged = staged;
  p.ld_staged = bw.up_k;
  return p;
}

// keys and values of every position the rows see are formed for the pass, so its cost does not depend on how heads share them
template <typename T>
int block_context<T>::latent_attention_rows(int run, int b, int rows, int pos0) {
  const int l = m->spec.runs[run];
  const branch_spec& bs = m->spec.layers[l].branches[b];
  const branch_weights& bw = m->layers[l].branches[b];
  const int ld = m->layers[l].proj_rows, first = window_first(pos0, bs.window), keys = pos0 + rows - first;
  const latent_rows<T> p = latents(run, b, ld);
  LCU_TRY(launch_latent_rows(p, rows, pos0, stream()));
  LCU_TRY(product(kv, false, staged, bw.up_k, bw.up, keys, bw.up_rows, bw.up_k));
  attn_rows<T> a{};
  a.q = p.q;
  a.ld = ld;
  a.q_head = bs.dim_pad() + bs.rot_pad();
  a.cache.k = kv;
  a.cache.v = kv + bw.up_v;
  a.cache.ldk = a.cache.ldv = bw.up_rows;
  a.cache.k_head = bs.dim_pad();
  a.cache.v_head = bs.vdim_pad();
  a.cache.first = first;
  a.key2 = p.cache.rows + p.cache.rot;
  a.ld2 = p.cache.ld;
  a.dim2 = bs.rot_dim;
  a.heads = a.kv_heads = bs.heads;
  a.dim = bs.dim;
  a.vdim = bs.vdim;
  a.window = bs.window;
  a.sink = bs.sink ? bw.sink : nullptr;
  a.gate = bs.head_gate ? proj + bw.g : nullptr;
  a.ldg = ld;
  a.scale = bs.score_scale;
  a.out_scale = bs.out_scale;
  a.out = cat + bw.out_col;
  a.ldo = m->layers[l].out_k;
  return launch_window_attention(a, rows, pos0, stream());
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
      } else if (bs.kind == BRANCH_LATENT_ATTN) {
        LCU_TRY(latent_attention_rows(run, (int)b, rows, pos0));
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
  for (int i = 0; i < (int)ls.branches.size(); ++i) {
    const branch_spec& bs = ls.branches[i];
    const branch_weights& bw = L.branches[i];
    if (bs.kind == BRANCH_LATENT_ATTN) {
      latent_step<T> a{};
      a.rows = latents(run, i, L.proj_rows);
      a.up = (const T*)bw.up;
      a.ld_up = bw.up_k;
      a.up_v = bw.up_v;
      a.scale = bs.score_scale;
      a.out_scale = bs.out_scale;
      a.sink = bs.sink ? bw.sink : nullptr;
      a.gate = bs.head_gate ? proj + bw.g : nullptr;
      a.out = cat + bw.out_col;
      a.pos = gpus[0].state;
      a.err = err();
      ++launches;
      LCU_TRY(launch_latent_step(a, stream()));
      continue;
    }
    LCU_REQUIRE(st.n_branches < STEP_MAX_BRANCHES, "mixer with more than %d branches", STEP_MAX_BRANCHES);
    step_branch<T>& b = st.b[st.n_branches++];
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
  if (st.n_branches > 0) {
    st.pos = gpus[0].state;
    ++launches;
    LCU_TRY(launch_mixer_step(st, opt.context_len, stream()));
  }
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

// routed feed-forward of several rows (and of single ones in binary32): h -> rows of y, in pieces
template <typename T>
int block_context<T>::expert_rows(const layer_spec& ls, const block_layer& L, int rows, pending_result& done) {
  const expert_weights& x = L.experts;
  const int K = m->k_width, f = L.ff_pad, total = rows * ls.top;
  if (is_f32<T>() || rows == 1) {
    LCU_TRY(product(z, true, h, K, x.router, rows, x.router_rows, K));
  } else {  // (one narrow matrix: K split over clusters fills more SMs than a few tiles of SM pairs)
    ++launches;
    LCU_TRY(launch_gemm_tc(TC_BF16_F32, z, h, K, x.router, rows, x.router_rows, K, 0.f, err(), stream(), 0, 0));
  }
  route_rows<T> r{};
  r.z = z;
  r.ldz = x.router_rows;
  r.experts = ls.experts;
  r.top = ls.top;
  r.rows = rows;
  r.h = h;
  r.ldh = r.cols = K;
  r.packed = packed_rows;
  r.weight = row_weight;
  r.at = places;
  r.tiles = tiles;
  r.n_tiles = n_tiles;
  r.tile_rows = is_f32<T>() ? MATMUL_F32_TILE : gemm_tc_group_tile(total, ls.experts);
  r.scratch = route_ints;
  LCU_TRY(launch_route(r, stream()));
  const int most = total / r.tile_rows + std::min(total, ls.experts);
  launches += 4;
  if (is_f32<T>()) {
    LCU_TRY(launch_matmul_f32_grouped((float*)gu, (const float*)packed_rows, K, (const float*)x.gate_up, 2 * f, K, tiles, n_tiles, most, stream()));
    LCU_TRY(launch_gate_rows(act, gu, total, f, stream(), row_weight, EXPERT_GATE_BLOCK));
    LCU_TRY(launch_matmul_f32_grouped(y, (const float*)act, f, (const float*)x.down, m->n_width, f, tiles, n_tiles, most, stream()));
    ++launches;
  } else {
    const gemm_groups g{tiles, n_tiles, most, r.tile_rows, ls.experts, row_weight};
    LCU_TRY(launch_gemm_tc_grouped(TC_BF16, act, packed_rows, K, x.gate_up, total, 2 * f, K, true, g, err(), stream()));
    LCU_TRY(launch_gemm_tc_grouped(TC_BF16_F32, y, act, f, x.down, total, m->n_width, f, false, g, err(), stream()));
  }
  done.pieces = places;
  done.n_pieces = ls.top;
  return LCU_OK;
}

// the same for one token whose experts are picked already: the weights of those experts stream through, one piece each
template <typename T>
int block_context<T>::expert_one(const layer_spec& ls, const block_layer& L, pending_result& done) {
  const expert_weights& x = L.experts;
  const int f = L.ff_pad, batches = (ls.top + GEMV_MAX_BATCH - 1) / GEMV_MAX_BATCH;
  for (int part = 0; part < 2; ++part)  // gate and up, down
    for (int i = 0; i < batches; ++i) {
      const int k0 = i * GEMV_MAX_BATCH;
      gemv_batch b;
      b.n = std::min(GEMV_MAX_BATCH, ls.top - k0);
      b.choice = pick + k0;
      b.choice_bytes = (part ? x.down_stride : x.gate_up_stride) * sizeof(T);
      b.choice_settled = part > 0 || i > 0;  // (all of these launches but the last hold the next one back until the picks stand)
      b.hold = part == 0 || i + 1 < batches;
      for (int k = 0; k < b.n; ++k) {
        b.w[k] = part ? x.down : x.gate_up;
        b.x[k] = part ? act + (size_t)(k0 + k) * f : h;
        b.out[k] = part ? (void*)(y + (size_t)(k0 + k) * m->n_width) : act + (size_t)(k0 + k) * f;
        b.rows[k] = m->n_width;
        b.f32[k] = part;
      }
      ++launches;
      if (part) {
        LCU_TRY(launch_gemv_bf16(b, f, err(), stream(), opt.use_pdl));
      } else {
        b.gate_scale = pick_weight + k0;
        b.gate_shift = 5;
        static_assert(EXPERT_GATE_BLOCK == 1 << 5, "row blocks of the experts' gate and up parts");
        LCU_TRY(launch_gemv_bf16_gated_picked(b, f, m->k_width, err(), stream(), opt.use_pdl));
      }
    }
  done.pieces = first_rows;
  done.n_pieces = ls.top;
  return LCU_OK;
}

// every layer run of a pass (rows == 1 at the position of the state words: the captured step, pos0 < 0)
template <typename T>
int block_context<T>::layers(int rows, int pos0, pending_result& done) {
  const bool step = pos0 < 0, sandwich = m->spec.sandwich;
  for (size_t run = 0; run < m->spec.runs.size(); ++run) {
    const int l = m->spec.runs[run];
    const layer_spec& ls = m->spec.layers[l];
    const block_layer& L = m->layers[l];
    if (m->spec.loop_input && m->spec.pass_start[run]) {
      LCU_TRY(start_pass(done, rows));
      done = pending_result{&replace};
    }
    LCU_TRY(hyper(L.hc1, L.norm1, done, rows, step && ls.is_wkv() ? &L : nullptr, runs[run].prev, nullptr, nullptr));
    LCU_TRY(step ? mixer_one((int)run) : mixer_rows((int)run, rows, pos0));
    done = pending_result{&L.hc1};
    if (sandwich) done.post = L.norm1b;
    if (ls.ff > 0) {
      const bool fused_pick = step && ls.experts > 0 && !is_f32<T>();
      LCU_TRY(hyper(L.hc2, L.norm2, done, rows, nullptr, nullptr, fused_pick ? &ls : nullptr, &L));
      done = pending_result{&L.hc2};
      if (sandwich) done.post = L.norm2b;
      if (fused_pick) LCU_TRY(expert_one(ls, L, done));
      else if (ls.experts > 0) LCU_TRY(expert_rows(ls, L, rows, done));
      else LCU_TRY(feed_forward(L, rows));
    }
  }
  return LCU_OK;
}

// the last residual pass and the output matrix for n rows: list[i], or row0 alone when list is null
template <typename T>
int block_context<T>::rows_to_logits(const pending_result& done, const int* list, size_t row0, int n) {
  hyper_params<T> p{};
  p.xs = xs + row0 * m->spec.streams * width;
  if (done.streams) {
    p.y = y + (done.pieces ? 0 : row0 * m->n_width);
    p.y_rows = done.pieces ? done.pieces + row0 * done.n_pieces : nullptr;
  }
  p.in = m->ones;
  p.norm_w = m->final_norm;
  p.rows = list;
  p.h = h;
  p.ldh = m->k_width;
  p.u_out = list ? nullptr : hidden;
  LCU_TRY(residual(p, done, n));
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
  if (m->spec.loop_input) {
    e.copy = loop_row + width;
    e.ld_copy = m->k_loop;
  }
  ++launches;
  LCU_TRY(launch_block_embed(e, g.stream));
  pending_result done;
  LCU_TRY(layers(1, -1, done));
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
    if (m->spec.loop_input) {
      e.copy = loop_row + width;
      e.ld_copy = m->k_loop;
    }
    LCU_TRY(launch_block_embed(e, g.stream));
    pending_result done;
    LCU_TRY(layers(rows, pos0, done));
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
  size_t w_z = 0, w_tiles = 0, w_route = 0, w_staged = 0, w_kv = 0;
  int top = 1;  // experts a token runs at most
  size_t w_proj = 0, w_cat = 0, w_gu = 0, w_act = 0, w_raw = 0, w_shift = 0, w_low = 0, w_packed = 0, w_values = 0;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const block_layer& L = m->layers[i];
    w_proj = std::max(w_proj, (size_t)L.proj_rows);
    w_cat = std::max(w_cat, (size_t)L.out_k);
    const layer_spec& ls = m->spec.layers[i];
    const size_t per_row = std::max(1, ls.top);
    if (ls.experts == 0 || is_f32<T>()) w_gu = std::max(w_gu, L.ff_pad * per_row);  // (the tensor-core experts gate at once)
    w_act = std::max(w_act, L.ff_pad * per_row);
    if (ls.experts > 0) {
      top = std::max(top, ls.top);
      w_z = std::max(w_z, (size_t)L.experts.router_rows);
      w_route = std::max(w_route, route_scratch(rows_cap, ls.experts, ls.top));
      w_tiles = std::max(w_tiles, (size_t)rows_cap * ls.top / MATMUL_F32_TILE + ls.experts);
    }
    w_shift = std::max(w_shift, (size_t)L.shifted_rows[0]);
    w_low = std::max(w_low, (size_t)L.shifted_rows[4]);
    for (auto& b : m->spec.layers[i].branches) {
      w_raw = std::max(w_raw, (size_t)b.out_cols());
      if (b.kind == BRANCH_LATENT_ATTN) {
        const branch_weights& bw = L.branches[&b - m->spec.layers[i].branches.data()];
        const size_t keys = std::min<size_t>(ctxl, (size_t)b.window - 1 + rows_cap);
        w_staged = std::max(w_staged, keys * bw.up_k);
        w_kv = std::max(w_kv, keys * bw.up_rows);
      }
      if (b.kind == BRANCH_WINDOW_ATTN || b.kind == BRANCH_LATENT_ATTN) continue;
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
    take(y, R * top * m->n_width * 4);
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
    take(act, R * w_act * es);
    take(loop_row, R * m->k_loop * es);
    take(staged, w_staged * es);
    take(kv, w_kv * es);
    take(z, R * w_z * 4);
    take(packed_rows, (w_z ? R * top : 0) * K * es);
    take(row_weight, R * top * 4);
    take(places, R * top * sizeof(int));
    take(route_ints, w_route * sizeof(int));
    take(tiles, w_tiles * sizeof(int4));
    take(n_tiles, sizeof(int));
    take(pick, MAX_TOP * sizeof(int));
    take(pick_weight, MAX_TOP * 4);
    take(first_rows, MAX_TOP * sizeof(int));
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
          w.k_head = ctxl * w.ldk;
          w.v_head = ctxl * w.ldv;
          take(w.k, b.kv_heads * ctxl * w.ldk * es);
          take(w.v, b.kv_heads * ctxl * w.ldv * es);
          take(w.kp, (size_t)b.kv_heads * w.n_blocks * w.ldk * es);
          take(w.vp, (size_t)b.kv_heads * w.n_blocks * w.ldv * es);
        } else if (b.kind == BRANCH_LATENT_ATTN) {
          latent_cache<T>& c = runs[r].latent;
          c.ctx_len = opt.context_len;
          c.rot = b.rank_pad();
          c.ld = c.rot + b.rot_pad();
          take(c.rows, ctxl * c.ld * es);
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
  replace = hyper_weights{m->ones, m->ones, m->zeros};
  int first[MAX_TOP];
  for (int i = 0; i < MAX_TOP; ++i) first[i] = i;
  LCU_CUDA(cudaStreamSynchronize(g.stream));  // (the arena has been cleared)
  LCU_CUDA(cudaMemcpy(first_rows, first, sizeof first, cudaMemcpyHostToDevice));
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
