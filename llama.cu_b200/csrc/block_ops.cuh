// Kernels of the block models beside the matrix products: embedding with bigrams, hyper-connected or normed residual rows with
// the following norm, window-and-blocks attention, latent attention, linear recurrences (retention, wkv), token shift, head
// normalisation and gates, routing of rows to experts.  T is the activation / cache / weight type of the model: __nv_bfloat16 or float.  Norms, residual streams,
// positions, scores, softmax, decays, recurrent state and everything that enters a recurrence beside the projections are
// binary32 in both.
#pragma once
#include <cuda_bf16.h>

#include "block_spec.cuh"
#include "common.cuh"

namespace lcu {

// rows of the residual: xs[row][stream][width] = (table[token] * scale + bigram row), the same in every stream.  The first
// token of a sequence (position 0) takes bigram row `buckets`.  *prev_token is the token before the first row and becomes
// the last row's token.
template <typename T>
struct embed_params {
  float* xs;
  const T *table, *bigram;
  const short* ids;
  int* prev_token;
  const int* pos;  // device position of row 0, or null: pos_value
  int pos_value;
  int m, width, streams, buckets;
  long long mul_prev, mul_cur;
  float scale;
  T* copy;       // optional: the rows once more, ld_copy apart
  int ld_copy;
};
template <typename T>
int launch_block_embed(const embed_params<T>& p, cudaStream_t stream);

// One pass over residual rows between two sublayers:
//   y <- sum_k y[y_rows[row][k]]                     (optional: a result that lies in pieces)
//   y <- y / sqrt(mean(y^2) + eps) * post_w          (optional: a sublayer's output norm, its channel scale included)
//   x_t <- sum_s up_mix[s][t] x_s + up_out[t] y      (the sublayer just computed; skipped when y is null)
//   u = sum_s in[s] x_s;  h = u / sqrt(mean(u^2) + eps) * (norm_base + norm_w)    (the norm of the next one; without norm_w h = u)
// and, for a single row, what follows at once: the inputs mix_i = h + (h_prev - h) * mu_i of a token-shifted mixer, with
// h_prev replaced by h; the experts of a routed feed-forward (as launch_route picks them).
template <typename T>
struct hyper_params {
  float* xs;             // [rows][streams][width]
  int width, streams;
  const float* y;        // [rows][ldy]
  int ldy;
  const float *up_mix, *up_out;
  int store;             // write the new streams back
  const float* in;
  const float* norm_w;
  float norm_base, eps;
  const float* post_w;
  const int* y_rows;     // [rows][n_y]
  int n_y;
  const int* rows;       // row numbers to work on, or null: 0 .. n-1; results are dense
  T* h;                  // [n][ldh]
  int ldh;
  float* u_out;          // optional: u of every row [n][width]
  // token shift of a single row
  T* prev;               // [width]
  const float* mu;       // [n_mix][width]
  T* mix;                // n_mix rows, mix_stride apart
  size_t mix_stride;
  int n_mix;
  const int* pos;
  // experts of a single row
  const T* router;       // [experts][ld_router]
  int ld_router, experts, top;
  int* pick;             // [top]
  float* pick_weight;    // [top]
};
int& hyper_row_one_cta();  // a single row of up to this many columns (all streams: twice as many) is one CTA's, a longer one a cluster's
template <typename T>
int launch_hyper_rows(const hyper_params<T>& p, int n_rows, cudaStream_t stream);

// mix_i[row] = h[row] + (h[row-1] - h[row]) * mu_i; row -1 is `prev` (zeros at position 0), which becomes the last row
template <typename T>
int launch_token_shift(const T* h, int ldh, T* prev, const float* mu, T* mix, size_t mix_stride, int n_mix, int m, int width, int pos0,
                       cudaStream_t stream);

// cos / sin of position * base^(-2 i / dims), angles in binary64: table[pos][dims / 2]
int launch_rotation_table(float2* table, int n_pos, int dims, double base, cudaStream_t stream);

// ---- attention over a sliding window and one mean key / value per block of `pool` tokens that lies wholly before it.
// Caches are [kv_head][position][ld] and [kv_head][block][ld], ld = dim rounded up to 8.  The kernels that only read keys and
// values take any strides: element (head g, position p) starts at g * k_head + (p - first) * ldk.
template <typename T>
struct window_cache {
  T *k, *v, *kp, *vp;
  int ctx_len, n_blocks, ldk, ldv;
  size_t k_head, v_head;
  int first;           // position of row 0
};
template <typename T>
struct attn_rows {
  const T *q, *k, *v;  // new rows; row stride ld
  int ld;
  int q_head;          // elements between the heads of a query row
  window_cache<T> cache;
  int heads, kv_heads, dim, vdim, window, pool;
  // a second part of the keys, shared by all heads: key2 row (p - first2) * ld2; its queries follow the first part's, which
  // are padded to whole 16-byte vectors of zeros
  const T* key2;
  int ld2, dim2, first2;
  const float* sink;   // per head, or null: one more term exp(sink) of the denominator
  const T* gate;       // [rows][ldg], or null: every head's result times sigmoid(gate[head])
  int ldg;
  float scale, out_scale;
  T* out;
  int ldo;
};
// cache rows pos0 .. pos0+m-1, then the blocks they complete, then attention of the rows
template <typename T>
int launch_window_append(const attn_rows<T>& p, int m, int pos0, cudaStream_t stream);
// (bfloat16 rows with heads of up to 128 take the tensor-core kernel of block_attn.cu)
bool window_mma_supported(int dim, int dim2, int vdim);
int launch_window_mma(const attn_rows<__nv_bfloat16>& p, int m, int pos0, cudaStream_t stream);
int& window_mma_mode();  // 1 (default) = where supported, 0 = never
template <typename T>
int launch_window_attention(const attn_rows<T>& p, int m, int pos0, cudaStream_t stream);

// ---- latent attention: keys and values of every head come from one normed latent per token, which is cached beside the key
// part that all heads share: cache row = [latent, padded to 8 | rotated key part, padded to 8].
template <typename T>
struct latent_cache {
  T* rows;             // [ctx_len][ld]
  int ctx_len, ld, rot;  // rot: first column of the rotated part
};
template <typename T>
struct latent_rows {
  T *q;                // projected rows: heads of [dim | rot_dim], each part padded to 8; the rotated part is turned in place
  const T *c, *k;      // latent before its norm, key part before its rotation
  int ld;              // stride of all three
  latent_cache<T> cache;
  int heads, dim, rot_dim, kv_rank, vdim, window;
  const float2* rope;
  int rot_dims;        // of rot_dim, in pairs (2i, 2i + 1)
  const float* norm;
  float eps;
  T* staged;           // [keys][ld_staged]: the latents that the rows see, zero-padded
  int ld_staged;
};
// first position that row `pos0` of a pass sees
__host__ __device__ inline int window_first(int pos0, int window) { return pos0 + 1 > window ? pos0 + 1 - window : 0; }
// norm and rotation of m new rows, into the cache; staged[i] = latent of position window_first(pos0) + i
template <typename T>
int launch_latent_rows(const latent_rows<T>& p, int m, int pos0, cudaStream_t stream);

// One token in one launch, without forming keys or values: a query goes through its head's key matrix once, so that a key is a
// cache row and the result a sum of cache rows, which the head's value matrix turns into the output.
template <typename T>
struct latent_step {
  latent_rows<T> rows;   // of the token; staged is not used
  const T* up;           // [heads * dim_pad | heads * vdim_pad][ld_up]: keys and values of all heads from a latent
  int ld_up, up_v;       // up_v: first value row
  float scale, out_scale;
  const float* sink;     // as attn_rows
  const T* gate;
  T* out;                // [heads * vdim]
  const int* pos;
  int* err;
};
template <typename T>
int launch_latent_step(const latent_step<T>& p, cudaStream_t stream);

// ---- linear recurrences over rows, per head:
//   retention: S <- decay S + k v^T, o = S^T q          (k and q rotated, k times kscale)
//   wkv:       o = (S + diag(u) k v^T)^T q, S <- diag(w) S + k v^T
template <typename T>
struct scan_rows {
  const T *q, *k, *v;     // row stride ld (of the recurrences' projections)
  int ldq, ldk, ldv;
  int heads, dim, vdim;
  float* state;           // [heads][dim][vdim]
  const float2* rope;     // retention: rotation table, or null
  int rot_dims;
  float kscale;
  const float* decay;     // retention: per head
  const float* u;         // wkv: [heads][dim]
  float* out;             // [rows][ldo] binary32
  int ldo;
  float *packed, *packed_v;  // scratch of scan_scratch() floats; wkv: the decays are in `packed` already (scan_decay_layout)
  int* err;
};
void scan_scratch(int heads, int dim, int vdim, bool wkv, size_t rows, size_t* packed_floats, size_t* value_floats);
// where the decay of (head, row, channel) of an m-row pass goes: packed[offset + head * head_stride + row * row_stride + channel]
void scan_decay_layout(int dim, int vdim, int m, size_t* head_stride, size_t* row_stride, size_t* offset);
template <typename T>
int launch_scan(const scan_rows<T>& p, bool wkv, int m, int pos0, cudaStream_t stream);

// decay of channel ch = head * dim + d: w[head * head_stride + row * row_stride + d] = exp(-exp(w0[ch] + sum_r w2t[r][ch] tanh(low[row][r])))
int launch_wkv_decay(float* w, size_t head_stride, size_t row_stride, const float* low, int ld_low, const float* w2t, const float* w0, int rank, int heads,
                     int dim, int m, cudaStream_t stream);

// out[row][head * vdim + j] = o / rms(o of the head) * norm * silu(g) * out_scale
template <typename T>
int launch_head_gate(T* out, int ldo, const float* o, int ld_raw, const T* g, int ldg, const float* norm, int heads, int vdim, float eps,
                     float out_scale, int m, cudaStream_t stream);

// ---- one token through all branches of a mixer in one launch: a cluster of CTAs per head
template <typename T>
struct step_branch {
  int kind;               // branch_kind
  int first;              // first cluster of the launch
  attn_rows<T> attn;      // attention (row pointers: the token's row)
  scan_rows<T> scan;      // recurrences
  const T* g;             // gate projection of the token
  const float* low;       // wkv: input of the decay's second product
  const float *w2t, *w0;
  int rank;
  const float* norm;      // wkv: weight of the normalised heads, or null
  float eps, out_scale;
  T* out;                 // the branch's columns
};
// ---- routed feed-forward: z[row][experts] are the router's logits; every row takes its `top` largest (ties: the lower expert)
// with the weights sigmoid(z).  The rows are then laid out expert by expert:
//   packed[at[row * top + k]] = h[row],  weight[at] its weight,  tiles / n_tiles as gemm_groups (tiles of tile_rows rows)
template <typename T>
struct route_rows {
  const float* z;
  int ldz, experts, top, rows;
  const T* h;
  int ldh, cols;         // columns copied
  T* packed;             // [rows * top][ldh]
  float* weight;         // [rows * top]
  int* at;               // [rows * top]
  int4* tiles;
  int* n_tiles;
  int tile_rows;
  int* scratch;          // route_scratch() ints
};
size_t route_scratch(int rows, int experts, int top);
template <typename T>
int launch_route(const route_rows<T>& p, cudaStream_t stream);

constexpr int STEP_MAX_BRANCHES = 2;
template <typename T>
struct mixer_step {
  step_branch<T> b[STEP_MAX_BRANCHES];
  int n_branches, n_clusters;
  const int* pos;
};
template <typename T>
int launch_mixer_step(const mixer_step<T>& p, int ctx_len, cudaStream_t stream);

// out[row][j] = silu(s a) * (s b), s = row_scale[row] (or 1): a = ab[row][j] and b = ab[row][f + j], or, with `block`, columns
// that alternate in blocks of that many
template <typename T>
int launch_gate_rows(T* out, const T* ab, int m, int f, cudaStream_t stream, const float* row_scale = nullptr, int block = 0);

// ---- weights: bfloat16 (or binary32) source rows into a matrix of the model
enum place_source { PLACE_BF16 = 0, PLACE_F32 = 1 };
// rows in groups: row r of the source goes to row r / group * stride + r % group, `gap` rows later where r % group >= split
struct row_groups {
  int group = 1 << 30, stride = 0, split = 1 << 30, gap = 0;
};
template <typename T>
int launch_place(T* dst, int ld, const void* src, place_source type, int rows, int cols, bool transpose, cudaStream_t stream,
                 const row_groups& groups = row_groups{});

// dst[i] *= src[i]
int launch_scale_vector(float* dst, const float* src, int n, cudaStream_t stream);

// ---- binary32 products: out[m][N] = x[m][ldx] . w[N][K]^T
int launch_matmul_f32(float* out, const float* x, int ldx, const float* w, int m, int N, int K, cudaStream_t stream);
// row groups with a matrix each, as gemm_groups: most_tiles tiles of up to MATMUL_F32_TILE rows
constexpr int MATMUL_F32_TILE = 64;
int launch_matmul_f32_grouped(float* out, const float* x, int ldx, const float* w, int N, int K, const int4* tiles, const int* n_tiles, int most_tiles,
                              cudaStream_t stream);

}  // namespace lcu
