// Row-wise kernels of the block models: embedding, hyper-connected residual, token shift, decays, head gates, weight
// placement, and the binary32 products.
#include <algorithm>

#include "block_ops.cuh"
#include "elem.cuh"

namespace lcu {
namespace {

// ------------------------------------------------------------------ embedding
// V: elements per thread and step (rows a multiple of V)
template <typename T, int V>
__global__ void __launch_bounds__(512) block_embed_kernel(const embed_params<T> p) {
  struct __align__(V * sizeof(T)) pack { T e[V]; };
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  __shared__ long long s_row;
  const int tok = p.ids[r];
  if (threadIdx.x == 0) {
    const int pos = (p.pos ? *p.pos : p.pos_value) + r;
    long long row = p.buckets;
    const int prev = r > 0 ? (int)p.ids[r - 1] : *p.prev_token;
    if (pos > 0 && p.buckets > 0) row = ((long long)prev * p.mul_prev + (long long)tok * p.mul_cur) % p.buckets;
    s_row = row;
    if (r == 0) *p.prev_token = p.ids[p.m - 1];  // (only row 0 reads it, just above)
  }
  __syncthreads();
  const T* e = p.table + (size_t)tok * p.width;
  const T* b = p.buckets > 0 ? p.bigram + (size_t)s_row * p.width : nullptr;
  float* x = p.xs + (size_t)r * p.streams * p.width;
  for (int c = threadIdx.x * V; c < p.width; c += 512 * V) {
    const pack ev = *reinterpret_cast<const pack*>(e + c);
    pack bv = {};
    if (b) bv = *reinterpret_cast<const pack*>(b + c);
    __align__(16) float v[V];
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = b ? fmaf(to_f(ev.e[k]), p.scale, to_f(bv.e[k])) : to_f(ev.e[k]) * p.scale;
    for (int s = 0; s < p.streams; ++s) {
      float* dst = x + (size_t)s * p.width + c;
      if (V == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(v);
      else dst[0] = v[0];
    }
    if (p.copy) {
      pack o;
#pragma unroll
      for (int k = 0; k < V; ++k) o.e[k] = from_f<T>(v[k]);
      *reinterpret_cast<pack*>(p.copy + (size_t)r * p.ld_copy + c) = o;
    }
  }
}

// ------------------------------------------------------------------ hyper-connected residual + norm
constexpr int HY_THREADS = 256;
constexpr int HY_MIX = 5;       // inputs of a token-shifted mixer
constexpr int HY_CLUSTER = 8;  // CTAs that share one long row when there is only one

// SM: room for the streams (p.streams <= SM); CL: CTAs per row; PRE: y is gathered and normed first
template <typename T, int SM, int CL, bool PRE>
__global__ void __launch_bounds__(HY_THREADS) hyper_rows_kernel(const hyper_params<T> p, const int per) {
  extern __shared__ __align__(16) float u_row[];  // this CTA's columns of u (PRE: first of y), then a router's partial sums
  __shared__ float s_red[2][HY_THREADS / 32], s_part[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int i_row = blockIdx.x / CL, rank = blockIdx.x % CL;
  pdl_launch_dependents();
  if (gridDim.x == CL) {  // a single row: what the columns' last step needs from the weights is on its way while the kernel before ends
    const int first = min(p.width, rank * per), n = min(p.width, first + per) - first;
    if (p.router) {
      constexpr int LINE = 128 / sizeof(T);
      const int lines = (n + LINE - 1) / LINE;
      for (int i = tid; i < p.experts * lines; i += HY_THREADS) l2_line(p.router + (size_t)(i / lines) * p.ld_router + first + i % lines * LINE);
    }
    for (int i = 32 * tid; i < n; i += 32 * HY_THREADS) {
      if (p.norm_w) l2_line(p.norm_w + first + i);
      if (PRE && p.post_w) l2_line(p.post_w + first + i);
      if (p.mix)
        for (int k = 0; k < p.n_mix; ++k) l2_line(p.mu + (size_t)k * p.width + first + i);
    }
  }
  pdl_wait();
  const int row = p.rows ? p.rows[i_row] : i_row;
  const int S = p.streams, W = p.width;
  const int c0 = min(W, rank * per), c1 = min(W, c0 + per);
  float in[SM], up[SM], mix[SM][SM];
#pragma unroll
  for (int s = 0; s < SM; ++s) {
    in[s] = s < S ? p.in[s] : 0.f;
    up[s] = p.y && s < S ? p.up_out[s] : 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) mix[s][t] = p.y && s < S && t < S ? p.up_mix[s * S + t] : 0.f;
  }
  float* x = p.xs + (size_t)row * S * W;
  const float* y = p.y ? p.y + (PRE && p.y_rows ? 0 : (size_t)row * p.ldy) : nullptr;
  auto row_total = [&](float v, int which) {  // over the CTA's threads, then the row's CTAs
    v = warp_sum(v);
    if (lane == 0) s_red[which][warp] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < HY_THREADS / 32; ++w) t += s_red[which][w];
    if (CL > 1) {
      if (tid == 0) s_part[which] = t;
      cluster_sync();
      t = 0.f;
#pragma unroll
      for (int r = 0; r < CL; ++r) t += ld_dsmem_f32(mapa(smem_u32(&s_part[which]), r));
    }
    return t;
  };
  constexpr int KEEP = PRE && SM == 1 ? (CL > 1 ? 1 : 4) : 0;  // vectors of the residual row held per thread from the start
  float4 kept[KEEP > 0 ? KEEP : 1];
  float inv_y = 1.f;
  if (PRE && y) {  // (a thread reads back only columns it has written itself)
    const int* yr = p.y_rows ? p.y_rows + (size_t)row * p.n_y : nullptr;
    const int pieces = yr ? p.n_y : 1;
    float sy = 0.f;
    if ((W & 3) == 0) {
      auto gather4 = [&](int c) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < pieces; ++k) {
          const float4 v = *reinterpret_cast<const float4*>(y + (yr ? (size_t)yr[k] * p.ldy : 0) + c);
          a = make_float4(a.x + v.x, a.y + v.y, a.z + v.z, a.w + v.w);
        }
        *reinterpret_cast<float4*>(u_row + c - c0) = a;
        sy = fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, sy))));
      };
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {  // the residual's columns are on their way meanwhile
        const int c = c0 + 4 * (tid + i * HY_THREADS);
        kept[i] = c < c1 ? *reinterpret_cast<const float4*>(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = c0 + 4 * (tid + i * HY_THREADS);
        if (c < c1) gather4(c);
      }
      for (int c = c0 + 4 * (tid + KEEP * HY_THREADS); c < c1; c += 4 * HY_THREADS) gather4(c);
    } else {
      for (int c = c0 + tid; c < c1; c += HY_THREADS) {
        float a = 0.f;
        for (int k = 0; k < pieces; ++k) a += y[(yr ? (size_t)yr[k] * p.ldy : 0) + c];
        u_row[c - c0] = a;
        sy = fmaf(a, a, sy);
      }
    }
    if (p.post_w) inv_y = 1.0f / sqrtf(row_total(sy, 0) / (float)W + p.eps);
  }
  auto y_at = [&](int c, float v) {  // PRE: the column's part in the sum
    if (!PRE || !p.post_w) return v;
    return v * (inv_y * p.post_w[c]);
  };
  float ss = 0.f;
  auto column = [&](float (&v)[SM], float yv) {  // new streams in v, returns u
    if (y) {
      float n[SM];
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        float a = up[t] * yv;
#pragma unroll
        for (int s = 0; s < SM; ++s) a = fmaf(mix[s][t], v[s], a);
        n[t] = a;
      }
#pragma unroll
      for (int t = 0; t < SM; ++t) v[t] = n[t];
    }
    float u = 0.f;
#pragma unroll
    for (int s = 0; s < SM; ++s) u = fmaf(in[s], v[s], u);
    return u;
  };
  auto columns4 = [&](int c, float4 (&xv)[SM]) {  // (per is a multiple of 4: rows and slices start 16-byte aligned)
    float4 yv = y ? *reinterpret_cast<const float4*>(PRE ? u_row + c - c0 : y + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (PRE && y) yv = make_float4(y_at(c, yv.x), y_at(c + 1, yv.y), y_at(c + 2, yv.z), y_at(c + 3, yv.w));
    float4 u;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float v[SM];
#pragma unroll
      for (int s = 0; s < SM; ++s) v[s] = reinterpret_cast<const float*>(&xv[s])[e];
      const float ue = column(v, reinterpret_cast<const float*>(&yv)[e]);
      reinterpret_cast<float*>(&u)[e] = ue;
      ss = fmaf(ue, ue, ss);
#pragma unroll
      for (int s = 0; s < SM; ++s) reinterpret_cast<float*>(&xv[s])[e] = v[s];
    }
    *reinterpret_cast<float4*>(u_row + c - c0) = u;
    if (y && p.store) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) *reinterpret_cast<float4*>(x + (size_t)s * W + c) = xv[s];
    }
  };
  if ((W & 3) == 0) {
    if (y) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = c0 + 4 * (tid + i * HY_THREADS);
        float4 xv[SM] = {kept[i]};
        if (c < c1) columns4(c, xv);
      }
    }
    for (int c = c0 + 4 * (tid + (y ? KEEP * HY_THREADS : 0)); c < c1; c += 4 * HY_THREADS) {
      float4 xv[SM];
#pragma unroll
      for (int s = 0; s < SM; ++s) xv[s] = s < S ? *reinterpret_cast<const float4*>(x + (size_t)s * W + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      columns4(c, xv);
    }
  } else {
    for (int c = c0 + tid; c < c1; c += HY_THREADS) {
      float v[SM];
#pragma unroll
      for (int s = 0; s < SM; ++s) v[s] = s < S ? x[(size_t)s * W + c] : 0.f;
      const float u = column(v, y ? y_at(c, PRE ? u_row[c - c0] : y[c]) : 0.f);
      u_row[c - c0] = u;
      ss = fmaf(u, u, ss);
      if (y && p.store) {
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) x[(size_t)s * W + c] = v[s];
      }
    }
  }
  const float inv = 1.0f / sqrtf(row_total(ss, 1) / (float)W + p.eps);
  T* h = p.h + (size_t)i_row * p.ldh;
  const bool start = p.mix && *p.pos == 0;
  if ((W & 3) == 0 && !p.mix) {  // (a thread's own columns)
    struct __align__(4 * sizeof(T)) pack { T e[4]; };
#pragma unroll 4
    for (int c = c0 + 4 * tid; c < c1; c += 4 * HY_THREADS) {
      const float4 u = *reinterpret_cast<const float4*>(u_row + c - c0);
      if (p.u_out) *reinterpret_cast<float4*>(p.u_out + (size_t)i_row * W + c) = u;
      const float4 w = p.norm_w ? *reinterpret_cast<const float4*>(p.norm_w + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      pack o;
      float4 back;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float ue = reinterpret_cast<const float*>(&u)[e];
        o.e[e] = from_f<T>(p.norm_w ? ue * inv * (p.norm_base + reinterpret_cast<const float*>(&w)[e]) : ue);
        reinterpret_cast<float*>(&back)[e] = to_f(o.e[e]);
      }
      *reinterpret_cast<pack*>(h + c) = o;
      if (p.router) *reinterpret_cast<float4*>(u_row + c - c0) = back;
    }
  } else for (int c = c0 + tid; c < c1; c += HY_THREADS) {
    const float u = u_row[c - c0];
    if (p.u_out) p.u_out[(size_t)i_row * W + c] = u;
    const T hv = from_f<T>(p.norm_w ? u * inv * (p.norm_base + p.norm_w[c]) : u);
    h[c] = hv;
    if (p.router) u_row[c - c0] = to_f(hv);
    if (p.mix) {
      const float hf = to_f(hv), d = (start ? 0.f : to_f(p.prev[c])) - hf;
      float mu[HY_MIX];
#pragma unroll
      for (int i = 0; i < HY_MIX; ++i) mu[i] = p.mu[(size_t)i * W + c];
#pragma unroll
      for (int i = 0; i < HY_MIX; ++i) p.mix[i * p.mix_stride + c] = from_f<T>(fmaf(d, mu[i], hf));
      p.prev[c] = hv;
    }
  }
  if (p.router) {  // z = router . h: this CTA's columns of every expert, then the sum over the CTAs in rank 0
    __syncthreads();
    float* z = u_row + per;
    for (int e = warp; e < p.experts; e += HY_THREADS / 32) {
      const T* w = p.router + (size_t)e * p.ld_router + c0;
      float a = 0.f;
      if ((W & 3) == 0) {
        struct __align__(4 * sizeof(T)) pack { T e[4]; };
#pragma unroll 4
        for (int c = 4 * lane; c < c1 - c0; c += 128) {
          const pack wv = *reinterpret_cast<const pack*>(w + c);
          const float4 hv = *reinterpret_cast<const float4*>(u_row + c);
          a = fmaf(to_f(wv.e[0]), hv.x, fmaf(to_f(wv.e[1]), hv.y, fmaf(to_f(wv.e[2]), hv.z, fmaf(to_f(wv.e[3]), hv.w, a))));
        }
      } else {
        for (int c = lane; c < c1 - c0; c += 32) a = fmaf(to_f(w[c]), u_row[c], a);
      }
      a = warp_sum(a);
      if (lane == 0) z[e] = a;
    }
    if (CL > 1) cluster_sync();
    else __syncthreads();
    if (rank == 0) {
      if (CL > 1) {
        for (int e = tid; e < p.experts; e += HY_THREADS) {
          float a = 0.f;
#pragma unroll
          for (int r = 0; r < CL; ++r) a += ld_dsmem_f32(mapa(smem_u32(z + e), r));
          z[p.experts + e] = a;
        }
        __syncthreads();
      }
      if (warp == 0)
        pick_largest(CL > 1 ? z + p.experts : z, p.experts, p.top, [&](int k, int e, float v) {
          p.pick[k] = e;
          p.pick_weight[k] = sigmoid_f(v);
        });
    }
  }
  if (CL > 1) cluster_sync();  // nobody leaves while its partial sum may still be read
}

template <typename T, int SM, int CL, bool PRE>
int launch_hyper_one(const hyper_params<T>& p, int n_rows, cudaStream_t stream) {
  const int per = (int)round_up(ceil_div(p.width, CL), 4);
  const size_t smem = ((size_t)per + (p.router ? 2 * p.experts : 0)) * sizeof(float);
  LCU_REQUIRE(smem <= 200 * 1024, "hyper_rows: a row of %d does not fit in shared memory", p.width);
  static bool attr_done[16] = {};
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  if (dev < 16 && !attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute((hyper_rows_kernel<T, SM, CL, PRE>), cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_done[dev] = true;
  }
  return launch_clustered(hyper_rows_kernel<T, SM, CL, PRE>, n_rows * CL, CL, HY_THREADS, smem, stream, p, per);
}

// ------------------------------------------------------------------ token shift
// A thread keeps V columns (width a multiple of V) and their mu over TS_ROWS rows.
constexpr int TS_ROWS = 8, TS_MIX = 5;
template <typename T, int V>
__global__ void __launch_bounds__(128) token_shift_kernel(const T* h, int ldh, T* prev, const float* mu, T* mix, size_t mix_stride, int m, int width,
                                                          int pos0) {
  struct __align__(V * sizeof(T)) pack { T e[V]; };
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, r0 = blockIdx.y * TS_ROWS, r1 = min(m, r0 + TS_ROWS);
  if (c >= width) return;
  float mv[TS_MIX][V];
#pragma unroll
  for (int i = 0; i < TS_MIX; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) mv[i][e] = mu[(size_t)i * width + c + e];
  pack pv;
  if (r0 > 0) {
    pv = *reinterpret_cast<const pack*>(h + (size_t)(r0 - 1) * ldh + c);
  } else {
    pv = *reinterpret_cast<const pack*>(prev + c);
    if (pos0 == 0)
#pragma unroll
      for (int e = 0; e < V; ++e) pv.e[e] = from_f<T>(0.f);
    *reinterpret_cast<pack*>(prev + c) = *reinterpret_cast<const pack*>(h + (size_t)(m - 1) * ldh + c);  // (only row 0 touches prev)
  }
#pragma unroll 2
  for (int r = r0; r < r1; ++r) {
    const pack hv = *reinterpret_cast<const pack*>(h + (size_t)r * ldh + c);
#pragma unroll
    for (int i = 0; i < TS_MIX; ++i) {
      pack o;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float hf = to_f(hv.e[e]);
        o.e[e] = from_f<T>(fmaf(to_f(pv.e[e]) - hf, mv[i][e], hf));
      }
      *reinterpret_cast<pack*>(mix + i * mix_stride + (size_t)r * ldh + c) = o;
    }
    pv = hv;
  }
}

__global__ void rotation_table_kernel(float2* table, int n_pos, int half, double base) {
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= n_pos * half) return;
  const int pos = idx / half, i = idx - pos * half;
  const double a = (double)pos * pow(base, -(double)i / half);
  table[idx] = make_float2((float)cos(a), (float)sin(a));
}

// ------------------------------------------------------------------ wkv decays
// A thread forms CH neighbouring channels of WD_ROWS rows (CH 4: whole 16-byte vectors of the matrix).
constexpr int WD_ROWS = 8;
template <int CH>
__global__ void __launch_bounds__(128) wkv_decay_kernel(float* w, size_t head_stride, size_t row_stride, const float* low, int ld_low, const float* w2t,
                                                        const float* w0, int rank, int heads, int dim, int m) {
  extern __shared__ __align__(16) float th[];  // [WD_ROWS][rank rounded up to 4]
  pdl_launch_dependents();
  pdl_wait();
  const int r0 = blockIdx.y * WD_ROWS, nr = min(WD_ROWS, m - r0), rp = (rank + 3) / 4 * 4, channels = heads * dim;
  for (int i = threadIdx.x; i < WD_ROWS * rp; i += 128) {
    const int r = i / rp, j = i - r * rp;
    th[i] = r < nr && j < rank ? tanhf(low[(size_t)(r0 + r) * ld_low + j]) : 0.f;
  }
  __syncthreads();
  const int ch = (blockIdx.x * 128 + threadIdx.x) * CH;
  if (ch >= channels) return;
  float acc[WD_ROWS][CH];
#pragma unroll
  for (int r = 0; r < WD_ROWS; ++r)
#pragma unroll
    for (int c = 0; c < CH; ++c) acc[r][c] = w0[ch + c];
#pragma unroll 2
  for (int j = 0; j < rank; j += 4) {
    float a[4][CH];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float* src = w2t + (size_t)(j + e) * channels + ch;
      if (CH == 4) {
        const float4 v = j + e < rank ? *reinterpret_cast<const float4*>(src) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int c = 0; c < CH; ++c) a[e][c] = reinterpret_cast<const float*>(&v)[c];
      } else {
        a[e][0] = j + e < rank ? src[0] : 0.f;
      }
    }
#pragma unroll
    for (int r = 0; r < WD_ROWS; ++r) {
      const float4 t = *reinterpret_cast<const float4*>(th + r * rp + j);
#pragma unroll
      for (int c = 0; c < CH; ++c) acc[r][c] = fmaf(a[3][c], t.w, fmaf(a[2][c], t.z, fmaf(a[1][c], t.y, fmaf(a[0][c], t.x, acc[r][c]))));
    }
  }
  const int head = ch / dim, d = ch - head * dim;  // (CH 4: the head size is a multiple of 4)
  float* out = w + head * head_stride + r0 * row_stride + d;
#pragma unroll
  for (int r = 0; r < WD_ROWS; ++r)
    if (r < nr) {
      __align__(16) float y[CH];
#pragma unroll
      for (int c = 0; c < CH; ++c) y[c] = expf(-expf(acc[r][c]));
      if (CH == 4) *reinterpret_cast<float4*>(out + r * row_stride) = *reinterpret_cast<const float4*>(y);
      else out[r * row_stride] = y[0];
    }
}

// ------------------------------------------------------------------ normalised, gated heads (one warp per row and head)
// LPH lanes share one (row, head), N vectors of VEC elements each; a group takes HG_ITEMS of them, loads first.  VEC 4: head
// sizes that are multiples of 4 with aligned rows; VEC 1: anything.
constexpr int HG_ITEMS = 4;
template <typename T, int VEC, int LPH, int N>
__global__ void __launch_bounds__(256) head_gate_kernel(T* out, int ldo, const float* o, int ld_raw, const T* g, int ldg, const float* norm, int heads,
                                                        int vdim, float eps, float out_scale, int m) {
  constexpr int GROUPS = 256 / LPH, I = N > 1 ? 1 : HG_ITEMS;
  pdl_launch_dependents();
  pdl_wait();
  const int grp = threadIdx.x / LPH, sub = threadIdx.x % LPH, total = m * heads;
  const int first = blockIdx.x * GROUPS * I + grp;
  __align__(16) float xv[I][N][VEC];
  __align__(16) T gv[I][N][VEC];
#pragma unroll
  for (int i = 0; i < I; ++i) {
    const int idx = first + i * GROUPS, r = idx / heads, hd = idx - r * heads;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (n * LPH + sub) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv[i][n][e] = 0.f;
      if (idx < total && j < vdim) {
        const float* x = o + (size_t)r * ld_raw + hd * vdim + j;
        const T* gr = g + (size_t)r * ldg + hd * vdim + j;
        if (VEC == 4) {
          *reinterpret_cast<float4*>(xv[i][n]) = *reinterpret_cast<const float4*>(x);
          if (sizeof(T) == 2) *reinterpret_cast<uint2*>(gv[i][n]) = *reinterpret_cast<const uint2*>(gr);
          else *reinterpret_cast<uint4*>(gv[i][n]) = *reinterpret_cast<const uint4*>(gr);
        } else {
          xv[i][n][0] = x[0];
          gv[i][n][0] = gr[0];
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < I; ++i) {
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(xv[i][n][e], xv[i][n][e], ss);
#pragma unroll
    for (int x = LPH / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
    const int idx = first + i * GROUPS, r = idx / heads, hd = idx - r * heads;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (n * LPH + sub) * VEC;
      if (idx < total && j < vdim) {
        __align__(16) T y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          float v = xv[i][n][e] * inv;
          if (norm) v *= norm[hd * vdim + j + e];
          y[e] = from_f<T>(v * silu_f(to_f(gv[i][n][e])) * out_scale);
        }
        T* dst = out + (size_t)r * ldo + hd * vdim + j;
        if (VEC == 4) {
          if (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(y);
          else *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(y);
        } else {
          dst[0] = y[0];
        }
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gate_rows_kernel(T* out, const T* ab, int m, int f, const float* row_scale, int block) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int V = 16 / sizeof(T);
  const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
  const int fv = f / V;
  if (i >= (size_t)m * fv) return;
  const size_t r = i / fv, jv = i - r * fv;
  const size_t j = jv * V, ja = block ? j / block * 2 * block + j % block : j, jb = ja + (block ? block : f);
  const uint4 av = *reinterpret_cast<const uint4*>(ab + r * 2 * f + ja), bv = *reinterpret_cast<const uint4*>(ab + r * 2 * f + jb);
  const float s = row_scale ? row_scale[r] : 1.0f;
  __align__(16) T o[V];
#pragma unroll
  for (int e = 0; e < V; ++e) o[e] = from_f<T>(silu_f(s * to_f(reinterpret_cast<const T*>(&av)[e])) * (s * to_f(reinterpret_cast<const T*>(&bv)[e])));
  reinterpret_cast<uint4*>(out + r * f)[jv] = *reinterpret_cast<const uint4*>(o);
}

template <typename T>
__global__ void place_kernel(T* dst, int ld, const void* src, int f32, int rows, int cols, int transpose, const row_groups g) {
  const size_t n = (size_t)rows * cols;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t from = i / cols, c = i - from * cols, w = from % g.group;
    const size_t r = from / g.group * g.stride + w + (w >= g.split ? g.gap : 0);
    const float v = f32 ? reinterpret_cast<const float*>(src)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(src)[i]);
    dst[transpose ? c * ld + r : r * ld + c] = from_f<T>(v);
  }
}

// ------------------------------------------------------------------ binary32 products
// few rows: one warp per output column, all rows of x at once
constexpr int MF_ROWS = 8;
__global__ void __launch_bounds__(256) matmul_f32_few_kernel(float* out, const float* x, int ldx, const float* w, int m, int N, int K) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, r0 = blockIdx.y * MF_ROWS;
  if (n >= N) return;
  const int nr = min(MF_ROWS, m - r0);
  float acc[MF_ROWS] = {};
  for (int k = lane * 4; k < K; k += 128) {
    const float4 a = *reinterpret_cast<const float4*>(w + (size_t)n * K + k);
#pragma unroll
    for (int r = 0; r < MF_ROWS; ++r)
      if (r < nr) {
        const float4 b = *reinterpret_cast<const float4*>(x + (size_t)(r0 + r) * ldx + k);
        acc[r] = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc[r]))));
      }
  }
#pragma unroll
  for (int r = 0; r < MF_ROWS; ++r) {
    const float v = warp_sum(acc[r]);
    if (lane == 0 && r < nr) out[(size_t)(r0 + r) * N + n] = v;
  }
}
// 64 x 64 tiles, 4 x 4 results per thread
__global__ void __launch_bounds__(256) matmul_f32_tile_kernel(float* out, const float* x, int ldx, const float* w, int m, int N, int K, const int4* tiles,
                                                              const int* n_tiles) {
  __shared__ float xs[16][68], ws[16][68];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, n0 = blockIdx.x * 64;
  int m0 = blockIdx.y * 64;
  if (tiles) {
    if ((int)blockIdx.y >= *n_tiles) return;
    const int4 t = tiles[blockIdx.y];
    m0 = t.x;
    m = t.y;
    w += (size_t)t.z * N * K;
  }
  float acc[4][4] = {};
  const int lr = tid >> 2, lk = (tid & 3) * 4;  // loader: row of the tile, four k
  for (int k0 = 0; k0 < K; k0 += 16) {
    const float4 a = m0 + lr < m ? *reinterpret_cast<const float4*>(x + (size_t)(m0 + lr) * ldx + k0 + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 b = n0 + lr < N ? *reinterpret_cast<const float4*>(w + (size_t)(n0 + lr) * K + k0 + lk) : make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      xs[lk + e][lr] = reinterpret_cast<const float*>(&a)[e];
      ws[lk + e][lr] = reinterpret_cast<const float*>(&b)[e];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&xs[k][ty * 4]), bv = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(reinterpret_cast<const float*>(&av)[i], reinterpret_cast<const float*>(&bv)[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (m0 + ty * 4 + i < m)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n0 + tx * 4 + j < N) out[(size_t)(m0 + ty * 4 + i) * N + n0 + tx * 4 + j] = acc[i][j];
}

}  // namespace

template <typename T>
int launch_block_embed(const embed_params<T>& p, cudaStream_t stream) {
  if (p.width % 4 == 0) LCU_CUDA(launch_after(block_embed_kernel<T, 4>, dim3(p.m), dim3(512), 0, stream, p));
  else LCU_CUDA(launch_after(block_embed_kernel<T, 1>, dim3(p.m), dim3(512), 0, stream, p));
  return LCU_OK;
}

int& hyper_row_one_cta() {
  static int width = 2048;
  return width;
}

template <typename T>
int launch_hyper_rows(const hyper_params<T>& p, int n_rows, cudaStream_t stream) {
  if (n_rows < 1) return LCU_OK;
  LCU_REQUIRE(p.streams >= 1 && p.streams <= 8, "hyper_rows: %d streams", p.streams);
  LCU_REQUIRE(p.mix == nullptr || (n_rows == 1 && p.n_mix == HY_MIX), "hyper_rows: the token shift is fused for a single row of %d inputs", HY_MIX);
  LCU_REQUIRE(p.router == nullptr || n_rows == 1, "hyper_rows: experts are picked for a single row");
  const bool pre = p.y && (p.post_w || p.y_rows);
  const int most = hyper_row_one_cta();  // (measured: 7 % of a step at 1024 columns, lost again where a CTA has four vectors per thread to load twice)
  const bool spread = n_rows == 1 && (p.width > most || p.width * p.streams > 2 * most);
#define LCU_HYPER(SM)                                                                                                                        \
  if (pre) return spread ? launch_hyper_one<T, SM, HY_CLUSTER, true>(p, n_rows, stream) : launch_hyper_one<T, SM, 1, true>(p, n_rows, stream); \
  return spread ? launch_hyper_one<T, SM, HY_CLUSTER, false>(p, n_rows, stream) : launch_hyper_one<T, SM, 1, false>(p, n_rows, stream)
  if (p.streams == 1) { LCU_HYPER(1); }
  if (p.streams == 2) { LCU_HYPER(2); }
  if (p.streams <= 4) { LCU_HYPER(4); }
  LCU_HYPER(8);
#undef LCU_HYPER
}

template <typename T>
int launch_token_shift(const T* h, int ldh, T* prev, const float* mu, T* mix, size_t mix_stride, int n_mix, int m, int width, int pos0,
                       cudaStream_t stream) {
  LCU_REQUIRE(n_mix == TS_MIX, "token_shift: %d mixes", n_mix);
  const dim3 grid((width + 511) / 512, (m + TS_ROWS - 1) / TS_ROWS);
  if (width % 4 == 0) LCU_CUDA(launch_after(token_shift_kernel<T, 4>, grid, dim3(128), 0, stream, h, ldh, prev, mu, mix, mix_stride, m, width, pos0));
  else LCU_CUDA(launch_after(token_shift_kernel<T, 1>, dim3((width + 127) / 128, grid.y), dim3(128), 0, stream, h, ldh, prev, mu, mix, mix_stride, m, width, pos0));
  return LCU_OK;
}

int launch_rotation_table(float2* table, int n_pos, int dims, double base, cudaStream_t stream) {
  const int half = dims / 2;
  rotation_table_kernel<<<(unsigned)ceil_div((size_t)n_pos * half, 256), 256, 0, stream>>>(table, n_pos, half, base);
  LCU_CUDA(cudaGetLastError());
  return LCU_OK;
}

int launch_wkv_decay(float* w, size_t head_stride, size_t row_stride, const float* low, int ld_low, const float* w2t, const float* w0, int rank, int heads,
                     int dim, int m, cudaStream_t stream) {
  const size_t smem = (size_t)WD_ROWS * round_up(rank, 4) * 4;
  LCU_REQUIRE(smem <= 160 * 1024, "wkv_decay: rank %d", rank);
  const bool vec = dim % 4 == 0 && ((uintptr_t)w & 15) == 0 && ((uintptr_t)w2t & 15) == 0 && head_stride % 4 == 0 && row_stride % 4 == 0;
  auto kernel = vec ? wkv_decay_kernel<4> : wkv_decay_kernel<1>;
  if (smem > 48 * 1024) LCU_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  LCU_CUDA(launch_after(kernel, dim3((heads * dim / (vec ? 4 : 1) + 127) / 128, (m + WD_ROWS - 1) / WD_ROWS), dim3(128), smem, stream, w, head_stride,
                        row_stride, low, ld_low, w2t, w0, rank, heads, dim, m));
  return LCU_OK;
}

template <typename T>
int launch_head_gate(T* out, int ldo, const float* o, int ld_raw, const T* g, int ldg, const float* norm, int heads, int vdim, float eps,
                     float out_scale, int m, cudaStream_t stream) {
  LCU_REQUIRE(vdim <= 512, "head_gate: head size %d", vdim);
  const size_t al = 4 * sizeof(T) - 1;
  const bool vec = vdim % 4 == 0 && ldo % 4 == 0 && ldg % 4 == 0 && ld_raw % 4 == 0 && (((uintptr_t)out | (uintptr_t)g) & al) == 0 && ((uintptr_t)o & 15) == 0;
  const size_t total = (size_t)m * heads;
#define LCU_GATE(VEC, LPH, N)                                                                                                                     \
  LCU_CUDA(launch_after(head_gate_kernel<T, VEC, LPH, N>, dim3((unsigned)ceil_div(total, (256 / LPH) * (N > 1 ? 1 : HG_ITEMS))), dim3(256), 0, stream, \
                        out, ldo, o, ld_raw, g, ldg, norm, heads, vdim, eps, out_scale, m))
  if (!vec) LCU_GATE(1, 32, 16);
  else if (vdim <= 64) LCU_GATE(4, 16, 1);
  else if (vdim <= 128) LCU_GATE(4, 32, 1);
  else LCU_GATE(4, 32, 4);
#undef LCU_GATE
  return LCU_OK;
}

template <typename T>
int launch_gate_rows(T* out, const T* ab, int m, int f, cudaStream_t stream, const float* row_scale, int block) {
  LCU_REQUIRE(f % 8 == 0 && block % 8 == 0 && (block == 0 || f % block == 0), "gate_rows: rows of %d elements (blocks of %d) are not 16-byte vectors", f, block);
  LCU_CUDA(launch_after(gate_rows_kernel<T>, dim3((unsigned)ceil_div((size_t)m * f * sizeof(T) / 16, 256)), dim3(256), 0, stream, out, ab, m, f, row_scale, block));
  return LCU_OK;
}

template <typename T>
int launch_place(T* dst, int ld, const void* src, place_source type, int rows, int cols, bool transpose, cudaStream_t stream, const row_groups& groups) {
  const size_t n = (size_t)rows * cols;
  if (n == 0) return LCU_OK;
  place_kernel<T><<<(unsigned)std::min<size_t>(ceil_div(n, 256), 148 * 16), 256, 0, stream>>>(dst, ld, src, type == PLACE_F32, rows, cols, transpose, groups);
  LCU_CUDA(cudaGetLastError());
  return LCU_OK;
}

__global__ void scale_vector_kernel(float* dst, const float* src, int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) dst[i] *= src[i];
}
int launch_scale_vector(float* dst, const float* src, int n, cudaStream_t stream) {
  scale_vector_kernel<<<(n + 255) / 256, 256, 0, stream>>>(dst, src, n);
  LCU_CUDA(cudaGetLastError());
  return LCU_OK;
}

int launch_matmul_f32(float* out, const float* x, int ldx, const float* w, int m, int N, int K, cudaStream_t stream) {
  LCU_REQUIRE(m >= 1 && K % 16 == 0 && ldx % 4 == 0, "matmul_f32: unsupported shape m=%d K=%d", m, K);
  if (m <= MF_ROWS) LCU_CUDA(launch_after(matmul_f32_few_kernel, dim3((N + 7) / 8, 1), dim3(256), 0, stream, out, x, ldx, w, m, N, K));
  else LCU_CUDA(launch_after(matmul_f32_tile_kernel, dim3((N + 63) / 64, (m + 63) / 64), dim3(256), 0, stream, out, x, ldx, w, m, N, K, (const int4*)nullptr,
                             (const int*)nullptr));
  return LCU_OK;
}
int launch_matmul_f32_grouped(float* out, const float* x, int ldx, const float* w, int N, int K, const int4* tiles, const int* n_tiles, int most_tiles,
                              cudaStream_t stream) {
  LCU_REQUIRE(most_tiles >= 1 && K % 16 == 0 && ldx % 4 == 0, "matmul_f32: unsupported shape of %d tiles, K=%d", most_tiles, K);
  LCU_CUDA(launch_after(matmul_f32_tile_kernel, dim3((N + 63) / 64, most_tiles), dim3(256), 0, stream, out, x, ldx, w, 0, N, K, tiles, n_tiles));
  return LCU_OK;
}

#define LCU_BLOCK_OPS(T)                                                                                                             \
  template int launch_block_embed<T>(const embed_params<T>&, cudaStream_t);                                                          \
  template int launch_hyper_rows<T>(const hyper_params<T>&, int, cudaStream_t);                                                      \
  template int launch_token_shift<T>(const T*, int, T*, const float*, T*, size_t, int, int, int, int, cudaStream_t);                 \
  template int launch_head_gate<T>(T*, int, const float*, int, const T*, int, const float*, int, int, float, float, int, cudaStream_t); \
  template int launch_gate_rows<T>(T*, const T*, int, int, cudaStream_t, const float*, int);                                                            \
  template int launch_place<T>(T*, int, const void*, place_source, int, int, bool, cudaStream_t, const row_groups&);
LCU_BLOCK_OPS(__nv_bfloat16)
LCU_BLOCK_OPS(float)

}  // namespace lcu
