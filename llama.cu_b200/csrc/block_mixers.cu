// Mixers of the block models: attention over a sliding window and pooled blocks, linear recurrences, and the fused
// one-token launch of all branches of a mixer.
#include <algorithm>

#include <math_constants.h>

#include "block_ops.cuh"
#include "elem.cuh"

namespace lcu {
namespace {

constexpr int MX_THREADS = 256;
constexpr int PART_FLOATS = 4096;  // partial sums of the value pass (groups x value columns)

__host__ __device__ __forceinline__ int pow2_at_least(int n) {
  int p = 1;
  while (p < n) p *= 2;
  return p;
}

// what position i sees: blocks 0 .. blocks-1 and tokens lo .. i
__host__ __device__ __forceinline__ void window_of(int i, int window, int pool, int& lo, int& blocks) {
  lo = i + 1 > window ? i + 1 - window : 0;
  const int past = i + 1 - window;  // positions that have left the window
  blocks = pool > 0 && past > 0 ? past / pool : 0;
}

__device__ __forceinline__ float block_max(float v, float* red) {
  v = warp_max(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float m = red[0];
#pragma unroll
  for (int w = 1; w < MX_THREADS / 32; ++w) m = fmaxf(m, red[w]);
  return m;
}
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < MX_THREADS / 32; ++w) s += red[w];
  return s;
}

// ------------------------------------------------------------------ attention of one query row and head
template <typename T>
__host__ __device__ __forceinline__ int query_cols(const attn_rows<T>& p) {
  return (p.dim + 7) / 8 * 8 + (p.key2 ? (p.dim2 + 7) / 8 * 8 : 0);
}
// `rank` of `C` CTAs takes a slice of the visible keys.  The row's own key and value come from `cur_k` / `cur_v` (shared
// memory copies) when given, else from the cache.  Leaves max, sum and the unnormalised value row in res[0], res[1],
// res[2 ..].  Shared memory: q [query_cols], scores [slice], part [PART_FLOATS].
template <typename T>
__device__ void attend_slice(const attn_rows<T>& p, const T* q_row, int head, int pos, int rank, int C, const T* cur_k, const T* cur_v, float* q,
                             float* sc, float* part, float* red, float* res) {
  constexpr int VEC = 16 / sizeof(T);
  const int tid = threadIdx.x;
  const int kvh = head / (p.heads / p.kv_heads);
  const int ldk = p.cache.ldk, ldv = p.cache.ldv;
  const int k_cols = (p.dim + 7) / 8 * 8, v_cols = (p.vdim + 7) / 8 * 8, q_cols = query_cols(p);
  const T* kc = p.cache.k + kvh * p.cache.k_head;
  const T* vc = p.cache.v + kvh * p.cache.v_head;
  const T* kp = p.cache.kp + (size_t)kvh * p.cache.n_blocks * ldk;
  const T* vp = p.cache.vp + (size_t)kvh * p.cache.n_blocks * ldv;
  int lo, blocks;
  window_of(pos, p.window, p.pool, lo, blocks);
  const int total = blocks + pos + 1 - lo;
  const int t0 = (int)((long long)total * rank / C), n = (int)((long long)total * (rank + 1) / C) - t0;
  for (int d = tid; d < q_cols; d += MX_THREADS) q[d] = d < p.dim || p.key2 ? to_f(q_row[head * p.q_head + d]) : 0.f;
  __syncthreads();
  auto key_at = [&](int t) -> const T* {
    if (t < blocks) return kp + (size_t)t * ldk;
    const int j = lo + t - blocks;
    return cur_k && j == pos ? cur_k : kc + (size_t)(j - p.cache.first) * ldk;
  };
  auto value_at = [&](int t) -> const T* {
    if (t < blocks) return vp + (size_t)t * ldv;
    const int j = lo + t - blocks;
    return cur_v && j == pos ? cur_v : vc + (size_t)(j - p.cache.first) * ldv;
  };
  // scores: lpk lanes per key
  {
    const int lpk = min(32, pow2_at_least((k_cols + VEC - 1) / VEC)), groups = MX_THREADS / lpk, grp = tid / lpk, sub = tid % lpk;
    constexpr int U = 4;
    const int rounds = (n + groups * U - 1) / (groups * U);  // (the same for every lane: the shuffles below are warp-wide)
    for (int rd = 0; rd < rounds; ++rd) {
      float s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        s[u] = 0.f;
        const int t = (rd * U + u) * groups + grp;
        if (t < n) {
          const T* k = key_at(t0 + t);
          for (int d = sub * VEC; d < k_cols; d += lpk * VEC) {
            const uint4 raw = *reinterpret_cast<const uint4*>(k + d);
#pragma unroll
            for (int e = 0; e < VEC; ++e) s[u] = fmaf(q[d + e], to_f(reinterpret_cast<const T*>(&raw)[e]), s[u]);
          }
          if (p.key2) {
            const T* k2 = p.key2 + (size_t)(lo + t0 + t - blocks - p.first2) * p.ld2 - k_cols;
            for (int d = k_cols + sub * VEC; d < q_cols; d += lpk * VEC) {
              const uint4 raw = *reinterpret_cast<const uint4*>(k2 + d);
#pragma unroll
              for (int e = 0; e < VEC; ++e) s[u] = fmaf(q[d + e], to_f(reinterpret_cast<const T*>(&raw)[e]), s[u]);
            }
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        for (int o = lpk >> 1; o > 0; o >>= 1) s[u] += __shfl_xor_sync(0xffffffffu, s[u], o);
        const int t = (rd * U + u) * groups + grp;
        if (sub == 0 && t < n) sc[t] = s[u] * p.scale;
      }
    }
  }
  __syncthreads();
  float mx = -CUDART_INF_F;
  for (int t = tid; t < n; t += MX_THREADS) mx = fmaxf(mx, sc[t]);
  mx = block_max(mx, red);
  float sum = 0.f;
  for (int t = tid; t < n; t += MX_THREADS) {
    const float e = expf(sc[t] - mx);
    sc[t] = e;
    sum += e;
  }
  sum = block_sum(sum, red);  // (its barriers also publish the exponentials)
  // values: lpv lanes per row of values, groups of them walk the keys
  const int lpv = min(32, pow2_at_least((v_cols + VEC - 1) / VEC)), groups = MX_THREADS / lpv, grp = tid / lpv, sub = tid % lpv;
  for (int d0 = 0; d0 < v_cols; d0 += lpv * VEC) {
    const int d = d0 + sub * VEC;
    float acc[VEC] = {};
    if (d < v_cols) {
#pragma unroll 4
      for (int t = grp; t < n; t += groups) {
        const uint4 raw = *reinterpret_cast<const uint4*>(value_at(t0 + t) + d);
        const float w = sc[t];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(w, to_f(reinterpret_cast<const T*>(&raw)[e]), acc[e]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < VEC; ++e) part[(grp * lpv + sub) * VEC + e] = acc[e];
    __syncthreads();
    for (int j = tid; j < lpv * VEC && d0 + j < p.vdim; j += MX_THREADS) {
      float v = 0.f;
      for (int g = 0; g < groups; ++g) v += part[g * lpv * VEC + j];
      res[2 + d0 + j] = v;
    }
  }
  if (tid == 0) {
    res[0] = n > 0 ? mx : -CUDART_INF_F;
    res[1] = n > 0 ? sum : 0.f;
  }
  __syncthreads();
}

// rows of a pass, one CTA per (row, head); keys and blocks are in the cache already
template <typename T>
__global__ void __launch_bounds__(MX_THREADS) window_rows_kernel(const attn_rows<T> p, int pos0, int max_keys) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[MX_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.x, r = blockIdx.y;
  float* q = sm;
  float* part = q + query_cols(p);
  float* res = part + PART_FLOATS;
  float* sc = res + 2 + round_up_dev(p.vdim + 2, 4);
  attend_slice(p, p.q + (size_t)r * p.ld, head, pos0 + r, 0, 1, (const T*)nullptr, (const T*)nullptr, q, sc, part, red, res);
  float inv = p.out_scale / res[1];
  if (p.sink) {
    const float top = fmaxf(res[0], p.sink[head]), f = expf(res[0] - top);
    inv = p.out_scale * f / (res[1] * f + expf(p.sink[head] - top));
  }
  if (p.gate) inv *= sigmoid_f(to_f(p.gate[(size_t)r * p.ldg + head]));
  for (int d = threadIdx.x; d < p.vdim; d += MX_THREADS) p.out[(size_t)r * p.ldo + head * p.vdim + d] = from_f<T>(res[2 + d] * inv);
}

// new rows of k and v into the cache
template <typename T>
__global__ void __launch_bounds__(256) window_append_kernel(const attn_rows<T> p, int m, int pos0) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  for (int i = threadIdx.x; i < p.kv_heads * p.dim; i += 256) {
    const int g = i / p.dim, d = i - g * p.dim;
    p.cache.k[((size_t)g * p.cache.ctx_len + pos0 + r) * p.cache.ldk + d] = p.k[(size_t)r * p.ld + i];
  }
  for (int i = threadIdx.x; i < p.kv_heads * p.vdim; i += 256) {
    const int g = i / p.vdim, d = i - g * p.vdim;
    p.cache.v[((size_t)g * p.cache.ctx_len + pos0 + r) * p.cache.ldv + d] = p.v[(size_t)r * p.ld + i];
  }
}

// mean of the cached rows of one block
template <typename T>
__device__ __forceinline__ void pool_block(const T* rows, int ld, int pool, const T* last, T* out, int dim) {
  for (int d = threadIdx.x; d < dim; d += blockDim.x) {
    float s = 0.f;
    for (int j = 0; j < pool; ++j) s += to_f(last && j == pool - 1 ? last[d] : rows[(size_t)j * ld + d]);
    out[d] = from_f<T>(s / (float)pool);
  }
}
template <typename T>
__global__ void __launch_bounds__(128) window_pool_kernel(const attn_rows<T> p, int first_block) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = first_block + blockIdx.x, g = blockIdx.y;
  const size_t row = (size_t)g * p.cache.ctx_len + (size_t)b * p.pool, dst = (size_t)g * p.cache.n_blocks + b;
  pool_block(p.cache.k + row * p.cache.ldk, p.cache.ldk, p.pool, (const T*)nullptr, p.cache.kp + dst * p.cache.ldk, p.dim);
  pool_block(p.cache.v + row * p.cache.ldv, p.cache.ldv, p.pool, (const T*)nullptr, p.cache.vp + dst * p.cache.ldv, p.vdim);
}

// ------------------------------------------------------------------ recurrences over rows
// Two launches.  The first lays a pass's rows out for the second, in binary32: per head and row q, k (rotated and scaled),
// the decays of a wkv layer and its bonus sum_i q_i u_i k_i (the same for every value column) as one run of `stride`
// floats, and the values by blocks of `cols` columns.  The second walks the rows: a CTA owns `cols` value columns of one
// head with their whole state in registers - G lanes share NC columns, each lane holding KC channels of each - and rows
// come in SC_ROWS at a time by bulk copies into a ring of stages.  Lane `sub` of a group holds channels
// (c / 4) * 4 G + 4 sub + c % 4, so that a warp reads row vectors as contiguous 16-byte pieces.  The state is updated once
// per row in row order, so neither the cut of a sequence into passes nor the pass length enters the arithmetic.
constexpr int SC_THREADS = 128;
constexpr int SC_ROWS = 16;
constexpr int SC_MAX_STAGES = 4;
constexpr int SC_NC = 2;

struct scan_shape {
  int kc, G, dimp, cols, blocks, stride;
};
scan_shape scan_shape_of(int dim, int vdim, bool wkv) {
  scan_shape s;
  s.kc = dim <= 128 ? 4 : dim <= 256 ? 8 : 16;
  s.G = std::max(2, pow2_at_least((dim + s.kc - 1) / s.kc));
  s.dimp = s.G * s.kc;
  s.cols = SC_THREADS / s.G * SC_NC;
  s.blocks = (vdim + s.cols - 1) / s.cols;
  s.stride = (wkv ? 3 : 2) * s.dimp + 4;
  return s;
}

constexpr int SP_ROWS = 4;  // rows per warp
template <typename T, bool WKV>
__global__ void __launch_bounds__(256) scan_prepare_kernel(const scan_rows<T> p, const scan_shape z, int m, int pos0) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.rot_dims >> 1;
  const int head = blockIdx.y * 8 + warp, r0 = blockIdx.x * SP_ROWS, nr = min(SP_ROWS, m - r0);
  if (head >= p.heads) return;
  float* out = p.packed + ((size_t)head * m + r0) * z.stride;
  float bonus[SP_ROWS] = {};
  for (int d = lane; d < z.dimp; d += 32) {
    const bool in = d < p.dim, turn = !WKV && d < p.rot_dims, low = d < half;
    const int pd = low ? d + half : d - half;
    const float u = WKV && in ? p.u[head * p.dim + d] : 0.f;
    float q[SP_ROWS], k[SP_ROWS], qo[SP_ROWS], ko[SP_ROWS];
    float2 cs[SP_ROWS];
#pragma unroll
    for (int r = 0; r < SP_ROWS; ++r) {
      const T* qr = p.q + (size_t)(r0 + r) * p.ldq + head * p.dim;
      const T* kr = p.k + (size_t)(r0 + r) * p.ldk + head * p.dim;
      const bool live = in && r < nr;
      q[r] = live ? to_f(qr[d]) : 0.f;
      k[r] = live ? to_f(kr[d]) : 0.f;
      if (live && turn) {
        qo[r] = to_f(qr[pd]);
        ko[r] = to_f(kr[pd]);
        cs[r] = p.rope[(size_t)(pos0 + r0 + r) * half + (low ? d : d - half)];
      }
    }
#pragma unroll
    for (int r = 0; r < SP_ROWS; ++r) {
      if (r >= nr) continue;
      if (WKV) {
        bonus[r] = fmaf(q[r] * u, k[r], bonus[r]);
      } else {
        if (turn) {
          q[r] = low ? q[r] * cs[r].x - qo[r] * cs[r].y : q[r] * cs[r].x + qo[r] * cs[r].y;
          k[r] = low ? k[r] * cs[r].x - ko[r] * cs[r].y : k[r] * cs[r].x + ko[r] * cs[r].y;
        }
        k[r] *= p.kscale;
      }
      float* o = out + (size_t)r * z.stride;
      o[d] = q[r];
      o[z.dimp + d] = k[r];
      if (WKV && !in) o[2 * z.dimp + d] = 0.f;  // (the other channels' decays are written by their own kernel)
    }
  }
#pragma unroll
  for (int r = 0; r < SP_ROWS; ++r) {
    const float b = warp_sum(bonus[r]);
    if (lane < 4 && r < nr) out[(size_t)r * z.stride + z.stride - 4 + lane] = lane == 0 && WKV ? b : 0.f;
  }
  float* v = p.packed_v + (size_t)head * z.blocks * m * z.cols;
  for (int j = lane; j < z.blocks * z.cols; j += 32) {
    const int b = j / z.cols, c = j - b * z.cols;
    float x[SP_ROWS];
#pragma unroll
    for (int r = 0; r < SP_ROWS; ++r) x[r] = j < p.vdim && r < nr ? to_f(p.v[(size_t)(r0 + r) * p.ldv + head * p.vdim + j]) : 0.f;
#pragma unroll
    for (int r = 0; r < SP_ROWS; ++r)
      if (r < nr) v[((size_t)b * m + r0 + r) * z.cols + c] = x[r];
  }
}

struct scan_args {  // what the second launch needs of scan_rows
  const float *packed, *packed_v, *decay;
  float *state, *out;
  int dim, vdim, ldo;
  int* err;
};

template <int KC, int G, bool WKV>
__global__ void __launch_bounds__(SC_THREADS) scan_kernel(const scan_args p, const scan_shape z, int m, int pos0, int n_stages) {
  constexpr int RB = 4;                         // rows reduced together
  constexpr int SPREAD = G < 8 ? G : 8;         // lanes of a group that end up with results
  constexpr int KEEP = RB * SC_NC / SPREAD;     // results per such lane
  constexpr int DIMP = G * KC, STRIDE = (WKV ? 3 : 2) * DIMP + 4, COLS = SC_THREADS / G * SC_NC;
  extern __shared__ __align__(16) float sm[];
  __shared__ uint64_t bars[SC_MAX_STAGES];
  const int tid = threadIdx.x, sub = tid % G, grp = tid / G;
  const int head = blockIdx.x, v0 = blockIdx.y * COLS, D = p.dim, DV = p.vdim;
  constexpr int STAGE = SC_ROWS * (STRIDE + COLS);
  const int n_tiles = (m + SC_ROWS - 1) / SC_ROWS;
  if (tid == 0) {
    for (int i = 0; i < n_stages; ++i) mbar_init(smem_u32(&bars[i]), 1);
    fence_mbar_init();
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  const float* rows = p.packed + (size_t)head * m * STRIDE;
  const float* vals = p.packed_v + ((size_t)head * z.blocks + blockIdx.y) * m * COLS;
  auto fetch = [&](int tile) {
    const int s = tile % n_stages, nr = min(SC_ROWS, m - tile * SC_ROWS);
    const uint32_t bar = smem_u32(&bars[s]), dst = smem_u32(sm + s * STAGE);
    const uint32_t b0 = (uint32_t)(nr * STRIDE) * 4, b1 = (uint32_t)(nr * COLS) * 4;
    mbar_arrive_expect_tx(bar, b0 + b1);
    bulk_g2s(dst, rows + (size_t)tile * SC_ROWS * STRIDE, b0, bar);
    bulk_g2s(dst + SC_ROWS * STRIDE * 4, vals + (size_t)tile * SC_ROWS * COLS, b1, bar);
  };
  if (tid == 0)
    for (int t = 0; t < n_stages && t < n_tiles; ++t) fetch(t);

  float S[SC_NC][KC];
  float* st = p.state + (size_t)head * D * DV;
  const int c0 = v0 + grp * SC_NC;  // first of this group's columns
#pragma unroll
  for (int n = 0; n < SC_NC; ++n)
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int i = (c >> 2) * 4 * G + 4 * sub + (c & 3);
      S[n][c] = pos0 > 0 && c0 + n < DV && i < D ? st[(size_t)i * DV + c0 + n] : 0.f;
    }
  const float dec = WKV ? 0.f : p.decay[head];
  const bool odd = sub & 1;

  // one row: updates the state, leaves this lane's share of both columns' results in o
  auto advance = [&](const float* row, const float* val, float (&o)[SC_NC]) {
    const float2 v = *reinterpret_cast<const float2*>(val);
    o[0] = o[1] = 0.f;
#pragma unroll
    for (int c4 = 0; c4 < KC / 4; ++c4) {
      const int at = c4 * 4 * G + 4 * sub;
      const float4 q4 = *reinterpret_cast<const float4*>(row + at), k4 = *reinterpret_cast<const float4*>(row + DIMP + at);
      float4 w4 = make_float4(dec, dec, dec, dec);
      if (WKV) w4 = *reinterpret_cast<const float4*>(row + 2 * DIMP + at);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = c4 * 4 + e;
        const float q = reinterpret_cast<const float*>(&q4)[e], k = reinterpret_cast<const float*>(&k4)[e], w = reinterpret_cast<const float*>(&w4)[e];
        if (WKV) {
          o[0] = fmaf(q, S[0][c], o[0]);
          o[1] = fmaf(q, S[1][c], o[1]);
        }
        S[0][c] = fmaf(w, S[0][c], k * v.x);
        S[1][c] = fmaf(w, S[1][c], k * v.y);
        if (!WKV) {
          o[0] = fmaf(q, S[0][c], o[0]);
          o[1] = fmaf(q, S[1][c], o[1]);
        }
      }
    }
  };
  for (int tile = 0; tile < n_tiles; ++tile) {
    const int s = tile % n_stages, nr = min(SC_ROWS, m - tile * SC_ROWS);
    mbar_wait(smem_u32(&bars[s]), (uint32_t)(tile / n_stages) & 1u, p.err, DEV_ERR_FULL_WAIT);  // (expired: the error word is set, results are not used)
    const float* rs = sm + s * STAGE;
    const float* vs = rs + SC_ROWS * STRIDE + grp * SC_NC;
    float* out = p.out + (size_t)tile * SC_ROWS * p.ldo + head * DV;
    // results of RB rows: lanes exchange halves - bit 0 of `sub` keeps one column, bit 1 one row of a pair, bit 2 one pair
    auto finish = [&](const float (&o)[RB][SC_NC], int r) {
      float x[RB];
#pragma unroll
      for (int b = 0; b < RB; ++b) x[b] = (odd ? o[b][1] : o[b][0]) + __shfl_xor_sync(0xffffffffu, odd ? o[b][0] : o[b][1], 1);
      if (G >= 4) {
        const bool up = sub & 2;
#pragma unroll
        for (int b = 0; b < RB / 2; ++b) x[b] = (up ? x[2 * b + 1] : x[2 * b]) + __shfl_xor_sync(0xffffffffu, up ? x[2 * b] : x[2 * b + 1], 2);
      }
      if (G >= 8) {
        const bool up = sub & 4;
        x[0] = (up ? x[1] : x[0]) + __shfl_xor_sync(0xffffffffu, up ? x[0] : x[1], 4);
      }
#pragma unroll
      for (int y = 8; y < G; y <<= 1) x[0] += __shfl_xor_sync(0xffffffffu, x[0], y);
      if (sub < SPREAD && c0 + (sub & 1) < DV) {
#pragma unroll
        for (int e = 0; e < KEEP; ++e) {
          const int b = G >= 8 ? ((sub >> 1) & 1) + 2 * ((sub >> 2) & 1) : G >= 4 ? ((sub >> 1) & 1) + 2 * e : e;
          float y = x[e];
          if (WKV) y = fmaf(rs[(r + b) * STRIDE + STRIDE - 4], vs[(r + b) * COLS + (sub & 1)], y);
          out[(size_t)(r + b) * p.ldo + c0 + (sub & 1)] = y;
        }
      }
    };
    int r = 0;
    if (nr == SC_ROWS) {  // whole tiles: the exchange of one row block runs beside the next block's arithmetic
      float o[2][RB][SC_NC];
#pragma unroll
      for (; r < SC_ROWS; r += RB) {
        const int cur = (r / RB) & 1;
#pragma unroll
        for (int b = 0; b < RB; ++b) advance(rs + (r + b) * STRIDE, vs + (r + b) * COLS, o[cur][b]);
        if (r > 0) finish(o[cur ^ 1], r - RB);
      }
      finish(o[(SC_ROWS / RB - 1) & 1], SC_ROWS - RB);
    }
#pragma unroll 1
    for (; r < nr; ++r) {
      float o[SC_NC];
      advance(rs + r * STRIDE, vs + r * COLS, o);
      float y = (odd ? o[1] : o[0]) + __shfl_xor_sync(0xffffffffu, odd ? o[0] : o[1], 1);
#pragma unroll
      for (int b = 2; b < G; b <<= 1) y += __shfl_xor_sync(0xffffffffu, y, b);
      if (sub < 2 && c0 + sub < DV) {
        if (WKV) y = fmaf(rs[r * STRIDE + STRIDE - 4], vs[r * COLS + sub], y);
        out[(size_t)r * p.ldo + c0 + sub] = y;
      }
    }
    __syncthreads();  // the stage may be overwritten
    if (tid == 0 && tile + n_stages < n_tiles) fetch(tile + n_stages);
  }
#pragma unroll
  for (int n = 0; n < SC_NC; ++n)
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int i = (c >> 2) * 4 * G + 4 * sub + (c & 3);
      if (c0 + n < DV && i < D) st[(size_t)i * DV + c0 + n] = S[n][c];
    }
}

template <int KC, int G, bool WKV>
int launch_scan_shape(const scan_args& a, const scan_shape& z, int heads, int m, int pos0, cudaStream_t stream) {
  const size_t stage = (size_t)SC_ROWS * (z.stride + z.cols) * sizeof(float);
  const int n_stages = (int)std::min<size_t>(SC_MAX_STAGES, (200 * 1024) / stage);
  static bool attr_done[16] = {};
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  if (dev < 16 && !attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute((scan_kernel<KC, G, WKV>), cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_done[dev] = true;
  }
  LCU_CUDA(launch_after(scan_kernel<KC, G, WKV>, dim3(heads, z.blocks), dim3(SC_THREADS), stage * n_stages, stream, a, z, m, pos0, n_stages));
  return LCU_OK;
}

template <bool WKV>
int launch_scan_kernel(const scan_args& a, const scan_shape& z, int heads, int m, int pos0, cudaStream_t stream) {
#define LCU_SCAN(KC, GG) if (z.kc == KC && z.G == GG) return launch_scan_shape<KC, GG, WKV>(a, z, heads, m, pos0, stream)
  LCU_SCAN(4, 2);
  LCU_SCAN(4, 4);
  LCU_SCAN(4, 8);
  LCU_SCAN(4, 16);
  LCU_SCAN(4, 32);
  LCU_SCAN(8, 32);
  LCU_SCAN(16, 32);
#undef LCU_SCAN
  LCU_REQUIRE(false, "scan: head size %d", a.dim);
}

// ------------------------------------------------------------------ one token, all branches
constexpr int ST_CLUSTER = 8;

// sum over the cluster of a value every thread of a CTA holds; `slot` is a shared float that stays valid until the next
// cluster barrier
__device__ __forceinline__ float cluster_total(float v, float* slot) {
  if (threadIdx.x == 0) *slot = v;
  cluster_sync();
  float t = 0.f;
#pragma unroll
  for (int r = 0; r < ST_CLUSTER; ++r) t += ld_dsmem_f32(mapa(smem_u32(slot), r));
  return t;
}

template <typename T>
__device__ void step_attention(const step_branch<T>& b, int head, int rank, int pos, float* sm, float* red) {
  const attn_rows<T>& p = b.attn;
  const int tid = threadIdx.x, per = p.heads / p.kv_heads, kvh = head / per;
  const int ldk = p.cache.ldk, ldv = p.cache.ldv;
  T* cur_k = reinterpret_cast<T*>(sm);  // [ldk], [ldv]: the token's key and value as the cache will hold them
  T* cur_v = cur_k + ldk;
  float* q = sm + ldk + ldv;
  float* part = q + ldk;
  float* res = part + PART_FLOATS;
  float* sc = res + 2 + round_up_dev(p.vdim + 2, 4);
  for (int d = tid; d < ldk; d += MX_THREADS) cur_k[d] = d < p.dim ? p.k[kvh * p.dim + d] : from_f<T>(0.f);
  for (int d = tid; d < ldv; d += MX_THREADS) cur_v[d] = d < p.vdim ? p.v[kvh * p.vdim + d] : from_f<T>(0.f);
  __syncthreads();
  attend_slice(p, p.q, head, pos, rank, ST_CLUSTER, cur_k, cur_v, q, sc, part, red, res);
  // the first query head of a group keeps the token: its cache rows, and the means of the block it completes (which no
  // position sees before the next step)
  if (head % per == 0 && rank == 0) {
    const size_t row = (size_t)kvh * p.cache.ctx_len + pos;
    for (int d = tid; d < p.dim; d += MX_THREADS) p.cache.k[row * ldk + d] = cur_k[d];
    for (int d = tid; d < p.vdim; d += MX_THREADS) p.cache.v[row * ldv + d] = cur_v[d];
    if (p.pool > 0 && (pos + 1) % p.pool == 0) {
      const size_t first = row - (p.pool - 1), dst = (size_t)kvh * p.cache.n_blocks + pos / p.pool;
      pool_block(p.cache.k + first * ldk, ldk, p.pool, cur_k, p.cache.kp + dst * ldk, p.dim);
      pool_block(p.cache.v + first * ldv, ldv, p.pool, cur_v, p.cache.vp + dst * ldv, p.vdim);
    }
  }
  cluster_sync();
  float mx = -CUDART_INF_F, sum = 0.f, f[ST_CLUSTER];
#pragma unroll
  for (int r = 0; r < ST_CLUSTER; ++r) mx = fmaxf(mx, ld_dsmem_f32(mapa(smem_u32(res), r)));
#pragma unroll
  for (int r = 0; r < ST_CLUSTER; ++r) {
    const float m = ld_dsmem_f32(mapa(smem_u32(res), r));
    f[r] = m > -CUDART_INF_F ? expf(m - mx) : 0.f;
    if (f[r] > 0.f) sum += f[r] * ld_dsmem_f32(mapa(smem_u32(res + 1), r));
  }
  float inv = p.out_scale / sum;
  if (p.sink) {
    const float top = fmaxf(mx, p.sink[head]), g = expf(mx - top);
    inv = p.out_scale * g / (sum * g + expf(p.sink[head] - top));
  }
  if (p.gate) inv *= sigmoid_f(to_f(p.gate[head]));
  const int d1 = p.vdim * (rank + 1) / ST_CLUSTER;
  for (int d = p.vdim * rank / ST_CLUSTER + tid; d < d1; d += MX_THREADS) {
    float v = 0.f;
#pragma unroll
    for (int r = 0; r < ST_CLUSTER; ++r)
      if (f[r] > 0.f) v += f[r] * ld_dsmem_f32(mapa(smem_u32(res + 2 + d), r));
    b.out[head * p.vdim + d] = from_f<T>(v * inv);
  }
  cluster_sync();
}

template <typename T, bool WKV>
__device__ void step_recurrence(const step_branch<T>& b, int head, int rank, int pos, float* sm, float* red) {
  const scan_rows<T>& p = b.scan;
  const int tid = threadIdx.x, D = p.dim, DV = p.vdim;
  float* q = sm;
  float* k = q + D;
  float* w = k + D;        // wkv: decays
  float* part = w + D;     // [MX_THREADS]
  float* lows = part + MX_THREADS;
  __shared__ float s_slot;
  const int half = p.rot_dims >> 1;
  for (int d = tid; d < D; d += MX_THREADS) {
    const T *qr = p.q + head * D, *kr = p.k + head * D;
    float qv = to_f(qr[d]), kv = to_f(kr[d]);
    if (!WKV) {
      if (d < p.rot_dims) {
        const bool low = d < half;
        const float2 cs = p.rope[(size_t)pos * half + (low ? d : d - half)];
        const int pd = low ? d + half : d - half;
        const float qo = to_f(qr[pd]), ko = to_f(kr[pd]);
        qv = low ? qv * cs.x - qo * cs.y : qv * cs.x + qo * cs.y;
        kv = low ? kv * cs.x - ko * cs.y : kv * cs.x + ko * cs.y;
      }
      kv *= p.kscale;
    }
    q[d] = qv;
    k[d] = kv;
  }
  if (WKV) {
    for (int j = tid; j < b.rank; j += MX_THREADS) lows[j] = tanhf(b.low[j]);
    __syncthreads();
    const int ch_all = p.heads * D;
    const int ng = max(1, MX_THREADS / D), grp = tid / D, c0 = tid - grp * D;
    if (ng > 1) {  // groups of threads share the rank
      float a = 0.f;
      if (grp < ng)
#pragma unroll 8
        for (int j = grp; j < b.rank; j += ng) a = fmaf(b.w2t[(size_t)j * ch_all + head * D + c0], lows[j], a);
      part[tid] = a;
      __syncthreads();
      if (tid < D) {
        float z = b.w0[head * D + tid];
        for (int g = 0; g < ng; ++g) z += part[g * D + tid];
        w[tid] = expf(-expf(z));
      }
    } else {
      for (int c = tid; c < D; c += MX_THREADS) {
        float z = b.w0[head * D + c];
        for (int j = 0; j < b.rank; ++j) z = fmaf(b.w2t[(size_t)j * ch_all + head * D + c], lows[j], z);
        w[c] = expf(-expf(z));
      }
    }
  }
  __syncthreads();
  const int v0 = DV * rank / ST_CLUSTER, nv = DV * (rank + 1) / ST_CLUSTER - v0;  // (at most 64 columns)
  float* st = p.state + (size_t)head * D * DV;
  const float dec = WKV ? 0.f : p.decay[head];
  const float* u = WKV ? p.u + head * D : nullptr;
  float o = 0.f;
  if (nv > 0) {
    const int ng = MX_THREADS / nv, grp = tid / nv, j = tid - grp * nv;
    float acc = 0.f;
    if (grp < ng) {
      const float v = to_f(p.v[head * DV + v0 + j]);
#pragma unroll 4
      for (int i = grp; i < D; i += ng) {
        float* s = st + (size_t)i * DV + v0 + j;
        float S = pos > 0 ? *s : 0.f;
        const float kv = k[i] * v;
        if (WKV) {
          acc = fmaf(q[i], fmaf(u[i], kv, S), acc);
          S = fmaf(w[i], S, kv);
        } else {
          S = fmaf(dec, S, kv);
          acc = fmaf(q[i], S, acc);
        }
        *s = S;
      }
    }
    part[tid] = acc;
    __syncthreads();
    if (tid < nv)
      for (int g = 0; g < ng; ++g) o += part[g * nv + tid];
  }
  const float ss = cluster_total(block_sum(o * o, red), &s_slot);
  const float inv = 1.0f / sqrtf(ss / (float)DV + b.eps);
  if (tid < nv) {
    const int c = head * DV + v0 + tid;
    float v = o * inv;
    if (b.norm) v *= b.norm[c];
    b.out[c] = from_f<T>(v * silu_f(to_f(b.g[c])) * b.out_scale);
  }
  cluster_sync();
}

// lines of the caches, states and weights this CTA will read, requested while the kernel before it ends
template <typename T>
__device__ __forceinline__ void step_lines(const step_branch<T>& b, int head, int rank, const int* pos_ptr) {
  const int tid = threadIdx.x;
  if (b.kind == BRANCH_WINDOW_ATTN) {
    const attn_rows<T>& p = b.attn;
    const int pos = min(*(volatile const int*)pos_ptr, p.cache.ctx_len - 1);  // (may be the step before's: only lines are asked for)
    int lo, blocks;
    window_of(pos, p.window, p.pool, lo, blocks);
    const int kvh = head / (p.heads / p.kv_heads), total = blocks + pos + 1 - lo;
    const int t0 = (int)((long long)total * rank / ST_CLUSTER), n = (int)((long long)total * (rank + 1) / ST_CLUSTER) - t0;
    constexpr int LINE = 128 / sizeof(T);
    const int lk = (p.cache.ldk + LINE - 1) / LINE, lv = (p.cache.ldv + LINE - 1) / LINE;
    for (int i = tid; i < n * (lk + lv); i += MX_THREADS) {
      const int t = t0 + i / (lk + lv), l = i % (lk + lv);
      const bool pooled = t < blocks, key = l < lk;
      const size_t row = pooled ? (size_t)kvh * p.cache.n_blocks + t : (size_t)kvh * p.cache.ctx_len + lo + t - blocks;
      const T* base = key ? (pooled ? p.cache.kp : p.cache.k) : (pooled ? p.cache.vp : p.cache.v);
      l2_line(base + row * (key ? p.cache.ldk : p.cache.ldv) + (key ? l : l - lk) * LINE);
    }
  } else {
    const scan_rows<T>& p = b.scan;
    const int v0 = p.vdim * rank / ST_CLUSTER, nv = p.vdim * (rank + 1) / ST_CLUSTER - v0;
    if (nv > 0)
      for (int i = tid; i < p.dim; i += MX_THREADS) l2_line(p.state + ((size_t)head * p.dim + i) * p.vdim + v0);
    if (b.kind == BRANCH_WKV) {
      const int per = (p.dim + 31) / 32;
      for (int i = tid; i < b.rank * per; i += MX_THREADS)
        l2_line(b.w2t + (size_t)(i / per) * p.heads * p.dim + head * p.dim + min(32 * (i % per), p.dim - 1));
      if (tid < per) {
        l2_line(b.w0 + head * p.dim + 32 * tid);
        l2_line(p.u + head * p.dim + 32 * tid);
        l2_line(b.norm + head * p.dim + 32 * tid);
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(MX_THREADS) mixer_step_kernel(const __grid_constant__ mixer_step<T> p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[MX_THREADS / 32];
  pdl_launch_dependents();
  const int cl = blockIdx.x / ST_CLUSTER, rank = blockIdx.x % ST_CLUSTER;
  const int bi = p.n_branches > 1 && cl >= p.b[1].first ? 1 : 0;
  const step_branch<T>& b = p.b[bi];
  const int head = cl - b.first;
  step_lines(b, head, rank, p.pos);
  pdl_wait();
  const int pos = *p.pos;
  if (b.kind == BRANCH_WINDOW_ATTN) step_attention(b, head, rank, pos, sm, red);
  else if (b.kind == BRANCH_RETENTION) step_recurrence<T, false>(b, head, rank, pos, sm, red);
  else step_recurrence<T, true>(b, head, rank, pos, sm, red);
}

template <typename T>
size_t attention_smem(const attn_rows<T>& p, int keys, bool step) {
  return ((step ? p.cache.ldk + p.cache.ldv : 0) + query_cols(p) + PART_FLOATS + 2 + round_up(p.vdim + 2, 4) + keys + 8) * sizeof(float);
}
template <typename T>
int most_keys(const attn_rows<T>& p, int last_pos) {
  int lo, blocks;
  window_of(last_pos, p.window, p.pool, lo, blocks);
  return blocks + std::min(p.window, last_pos + 1);
}

}  // namespace

int& window_mma_mode() {
  static int mode = 1;
  return mode;
}

template <typename T>
int launch_window_append(const attn_rows<T>& p, int m, int pos0, cudaStream_t stream) {
  LCU_REQUIRE(pos0 >= 0 && pos0 + m <= p.cache.ctx_len, "window attention: rows %d..%d outside the cache of %d", pos0, pos0 + m, p.cache.ctx_len);
  LCU_CUDA(launch_after(window_append_kernel<T>, dim3(m), dim3(256), 0, stream, p, m, pos0));
  if (p.pool > 0) {
    const int b0 = pos0 / p.pool, b1 = (pos0 + m) / p.pool;
    if (b1 > b0) LCU_CUDA(launch_after(window_pool_kernel<T>, dim3(b1 - b0, p.kv_heads), dim3(128), 0, stream, p, b0));
  }
  return LCU_OK;
}

template <typename T>
int launch_window_attention(const attn_rows<T>& p, int m, int pos0, cudaStream_t stream) {
  if constexpr (sizeof(T) == 2)
    if (window_mma_mode() && window_mma_supported(p.dim, p.key2 ? p.dim2 : 0, p.vdim)) return launch_window_mma(p, m, pos0, stream);
  const int keys = most_keys(p, pos0 + m - 1);
  const size_t smem = attention_smem(p, keys, false);
  LCU_REQUIRE(smem <= 220 * 1024, "window attention: %d visible keys", keys);
  static bool attr_done[16] = {};
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  if (dev < 16 && !attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute(window_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    attr_done[dev] = true;
  }
  LCU_CUDA(launch_after(window_rows_kernel<T>, dim3(p.heads, m), dim3(MX_THREADS), smem, stream, p, pos0, keys));
  return LCU_OK;
}

template <typename T>
int launch_scan(const scan_rows<T>& p, bool wkv, int m, int pos0, cudaStream_t stream) {
  const scan_shape z = scan_shape_of(p.dim, p.vdim, wkv);
  const dim3 grid((m + SP_ROWS - 1) / SP_ROWS, (p.heads + 7) / 8);
  if (wkv) LCU_CUDA(launch_after(scan_prepare_kernel<T, true>, grid, dim3(256), 0, stream, p, z, m, pos0));
  else LCU_CUDA(launch_after(scan_prepare_kernel<T, false>, grid, dim3(256), 0, stream, p, z, m, pos0));
  const scan_args a{p.packed, p.packed_v, p.decay, p.state, p.out, p.dim, p.vdim, p.ldo, p.err};
  return wkv ? launch_scan_kernel<true>(a, z, p.heads, m, pos0, stream) : launch_scan_kernel<false>(a, z, p.heads, m, pos0, stream);
}

void scan_scratch(int heads, int dim, int vdim, bool wkv, size_t rows, size_t* packed_floats, size_t* value_floats) {
  const scan_shape z = scan_shape_of(dim, vdim, wkv);
  *packed_floats = heads * rows * z.stride;
  *value_floats = heads * rows * z.blocks * z.cols;
}
void scan_decay_layout(int dim, int vdim, int m, size_t* head_stride, size_t* row_stride, size_t* offset) {
  const scan_shape z = scan_shape_of(dim, vdim, true);
  *head_stride = (size_t)m * z.stride;
  *row_stride = z.stride;
  *offset = 2 * (size_t)z.dimp;
}

template <typename T>
int launch_mixer_step(const mixer_step<T>& p, int ctx_len, cudaStream_t stream) {
  size_t smem = 0;
  for (int i = 0; i < p.n_branches; ++i) {
    const step_branch<T>& b = p.b[i];
    if (b.kind == BRANCH_WINDOW_ATTN) smem = std::max(smem, attention_smem(b.attn, most_keys(b.attn, ctx_len - 1) / ST_CLUSTER + 2, true));
    else smem = std::max(smem, (3 * (size_t)b.scan.dim + MX_THREADS + b.rank + 8) * sizeof(float));
  }
  LCU_REQUIRE(smem <= 220 * 1024, "mixer step: %zu bytes of shared memory", smem);
  static bool attr_done[16] = {};
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  if (dev < 16 && !attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute(mixer_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    attr_done[dev] = true;
  }
  return launch_clustered(mixer_step_kernel<T>, p.n_clusters * ST_CLUSTER, ST_CLUSTER, MX_THREADS, smem, stream, p);
}

#define LCU_BLOCK_MIXERS(T)                                                                    \
  template int launch_window_append<T>(const attn_rows<T>&, int, int, cudaStream_t);           \
  template int launch_window_attention<T>(const attn_rows<T>&, int, int, cudaStream_t);  \
  template int launch_scan<T>(const scan_rows<T>&, bool, int, int, cudaStream_t);              \
  template int launch_mixer_step<T>(const mixer_step<T>&, int, cudaStream_t);
LCU_BLOCK_MIXERS(__nv_bfloat16)
LCU_BLOCK_MIXERS(float)

}  // namespace lcu
