// Latent attention, rows of a pass: norm of the latents, rotation of the query and key parts, cache rows, and the dense copy
// of every latent the rows see, from which one product forms the keys and values of all heads.  A single token is one launch that
// works on the cached latents themselves.
#include <algorithm>

#include "block_ops.cuh"
#include "elem.cuh"
#include "gemv.cuh"

namespace lcu {
namespace {

constexpr int LR_THREADS = 256;

// one CTA per position: the first n_old copy cached latents, the others work on a new row
template <typename T>
__global__ void __launch_bounds__(LR_THREADS) latent_rows_kernel(const latent_rows<T> p, int n_old, int pos0) {
  __shared__ float s_red[LR_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, rp = p.cache.rot, ld = p.cache.ld;
  T* staged = p.staged + (size_t)blockIdx.x * p.ld_staged;
  for (int d = rp + tid; d < p.ld_staged; d += LR_THREADS) staged[d] = from_f<T>(0.f);
  if ((int)blockIdx.x < n_old) {
    constexpr int VEC = 16 / sizeof(T);
    const T* src = p.cache.rows + (size_t)(pos0 - n_old + blockIdx.x) * ld;
    for (int d = tid * VEC; d < rp; d += LR_THREADS * VEC) *reinterpret_cast<uint4*>(staged + d) = *reinterpret_cast<const uint4*>(src + d);
    return;
  }
  const int r = blockIdx.x - n_old, pos = pos0 + r, half = p.rot_dims >> 1;
  const T *c = p.c + (size_t)r * p.ld, *k = p.k + (size_t)r * p.ld;
  T* row = p.cache.rows + (size_t)pos * ld;
  const float2* cs = p.rope + (size_t)pos * half;
  float ss = 0.f;
  for (int d = tid; d < p.kv_rank; d += LR_THREADS) {
    const float x = to_f(c[d]);
    ss = fmaf(x, x, ss);
  }
  // the shared key part, and the heads' rotated query parts in place
  for (int d = tid; d < ld - rp; d += LR_THREADS) {
    float v = d < p.rot_dim ? to_f(k[d]) : 0.f;
    if (d < p.rot_dims) v = v * cs[d >> 1].x + to_f(k[d ^ 1]) * (d & 1 ? cs[d >> 1].y : -cs[d >> 1].y);
    row[rp + d] = from_f<T>(v);
  }
  const int kp = round_up_dev(p.dim, 8), q_head = kp + ld - rp;
  T* q = p.q + (size_t)r * p.ld;
  for (int i = tid; i < p.heads * half; i += LR_THREADS) {
    const int h = i / half, j = i - h * half;
    T* at = q + (size_t)h * q_head + kp + 2 * j;
    const float u = to_f(at[0]), v = to_f(at[1]);
    at[0] = from_f<T>(u * cs[j].x - v * cs[j].y);
    at[1] = from_f<T>(v * cs[j].x + u * cs[j].y);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int w = 0; w < LR_THREADS / 32; ++w) total += s_red[w];
  const float inv = 1.0f / sqrtf(total / (float)p.kv_rank + p.eps);
  for (int d = tid; d < rp; d += LR_THREADS) {
    const T v = from_f<T>(d < p.kv_rank ? to_f(c[d]) * inv * p.norm[d] : 0.f);
    row[d] = v;
    staged[d] = v;
  }
}

// ------------------------------------------------------------------ one token
// A cluster of 8 CTAs serves up to LS_HEADS heads: the CTAs share the columns of the query-times-key-matrix product, the visible
// cache rows and the rows of the value matrix; partial results meet in distributed shared memory.  A CTA's cache rows come in
// by bulk copies, chunk by chunk through two stages, and are read there twice, for the scores and for the sums, with a running
// maximum over the chunks.
//
// bfloat16 rows take the tensor cores without giving up binary32 queries and weights: a 16-row operand has room for three
// bfloat16 parts of every head's value (rows 3 h .. 3 h + 2, together 24 bits), products with bfloat16 rows are exact, sums are
// binary32.  Binary32 rows take plain multiply-adds, one head per cluster.
constexpr int LS_CLUSTER = 8, LS_THREADS = 256, LS_WARPS = LS_THREADS / 32, LS_STAGES = 2;
constexpr int LS_CHUNK = 64;      // rows of a chunk at most
constexpr int LS_HEADS = 5, LS_PARTS = 3;
constexpr int LS_GROUPS = 32;     // groups of threads that share the rows of the key matrices
constexpr int LS_SMEM = 220 * 1024;

struct latent_layout {  // bytes from the start of shared memory
  int ld, rp, kp, res_stride, row, steps;  // row: bytes between staged rows (an odd number of 16-byte units: no bank conflicts)
  int cur, qh, q, oc, sc, w, f, part, res, stages, total;
  __host__ __device__ latent_layout(int dim, int kv_rank, int cache_ld, int rot, int elem, int nh, int chunk) {
    auto up = [](int n) { return (n + 15) / 16 * 16; };
    ld = cache_ld;
    rp = rot;
    kp = (dim + 7) / 8 * 8;
    res_stride = 4 + (kv_rank + 3) / 4 * 4;
    row = ((ld * elem / 16) | 1) * 16;
    steps = (ld + 31) / 32 * 2;
    cur = 64;
    qh = cur + up(ld * elem);
    q = qh + up(nh * kp * 4);
    oc = q + up(nh * ld * 4);
    sc = oc + up(nh * rp * 4);
    w = sc + 16 * LS_CHUNK * 4;
    f = w + 16 * (LS_CHUNK + 8) * 2;
    part = f + up((LS_HEADS * LS_CLUSTER + 16) * 4);
    const int parts = elem == 2 ? (nh * LS_PARTS + 1) * (steps * 16 + 8) * 2 : 0, sums = LS_THREADS * 8 * 4;  // (the second is gone when the first is made)
    res = part + up(parts > sums ? parts : sums);
    stages = res + up(nh * res_stride * 4);
    const int rows = LS_STAGES * chunk * row, out = elem == 2 ? nh * LS_PARTS * rp * 4 : 0;  // (likewise)
    total = stages + (rows > out ? rows : out);
  }
};

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// N values as sums of bfloat16 parts, each the nearest to what the parts before leave; parts lie `stride` apart
template <int N>
__device__ __forceinline__ void store_parts(__nv_bfloat16* at, int stride, const float* x) {
  struct __align__(2 * N) pack { __nv_bfloat16 e[N]; };
  float left[N];
#pragma unroll
  for (int i = 0; i < N; ++i) left[i] = x[i];
#pragma unroll
  for (int t = 0; t < LS_PARTS; ++t) {
    pack v;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      v.e[i] = __float2bfloat16(left[i]);
      left[i] -= __bfloat162float(v.e[i]);
    }
    *reinterpret_cast<pack*>(at + t * stride) = v;
  }
}
__device__ __forceinline__ float4 ld_dsmem_f4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}
// i / n for i below LS_HEADS * n
__device__ __forceinline__ int head_of(int i, int n) { return (i >= n) + (i >= 2 * n) + (i >= 3 * n) + (i >= 4 * n); }

// QF: a cache row has up to 32 QF columns
template <typename T, int QF>
__global__ void __launch_bounds__(LS_THREADS, 1) latent_step_kernel(const __grid_constant__ latent_step<T> a, const int clusters, const int most_heads,
                                                                   const int chunk) {
  constexpr bool TC = sizeof(T) == 2;
  constexpr int MOST = QF * 32 > 2048 ? 2048 : QF * 32;  // columns of a latent at most
  struct __align__(16) vec8 { T e[8]; };
  extern __shared__ __align__(128) uint8_t ls_smem[];
  __shared__ float red[LS_WARPS];
  const latent_rows<T>& p = a.rows;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cl = blockIdx.x / LS_CLUSTER, rank = blockIdx.x % LS_CLUSTER;
  const int h0 = p.heads * cl / clusters, nh = p.heads * (cl + 1) / clusters - h0;
  const latent_layout z(p.dim, p.kv_rank, p.cache.ld, p.cache.rot, sizeof(T), most_heads, chunk);
  const int ld = z.ld, rp = z.rp, kp = z.kp, rotp = ld - rp, vp = round_up_dev(p.vdim, 8), half = p.rot_dims >> 1;
  uint64_t* bars = reinterpret_cast<uint64_t*>(ls_smem);
  T* cur = reinterpret_cast<T*>(ls_smem + z.cur);           // [ld] the token's row as the cache will hold it
  float* qh = reinterpret_cast<float*>(ls_smem + z.qh);     // [nh][kp] queries against unrotated keys
  float* q = reinterpret_cast<float*>(ls_smem + z.q);       // [nh][ld] queries against cache rows
  float* oc = reinterpret_cast<float*>(ls_smem + z.oc);     // [nh][rp] sums of cache rows
  float* sc = reinterpret_cast<float*>(ls_smem + z.sc);     // [16][LS_CHUNK] scores (of parts)
  __nv_bfloat16* wt = reinterpret_cast<__nv_bfloat16*>(ls_smem + z.w);  // [16][LS_CHUNK + 8] weights in parts
  float* fac = reinterpret_cast<float*>(ls_smem + z.f);     // [nh] factor of what the chunks before have added up
  float* share = fac + 16;                                  // [nh][LS_CLUSTER] factors of the CTAs' sums of rows
  float* part = reinterpret_cast<float*>(ls_smem + z.part); // partial sums of the queries
  __nv_bfloat16* qp = reinterpret_cast<__nv_bfloat16*>(ls_smem + z.part);  // [nh * LS_PARTS][ldq] queries in parts, a row of zeros
  const int ldq = z.steps * 16 + 8;
  float* res = reinterpret_cast<float*>(ls_smem + z.res);   // [nh][res_stride]: maximum, sum, sum of rows
  uint8_t* stages = ls_smem + z.stages;
  const int vecs = rp >> 3, v0 = vecs * rank / LS_CLUSTER, nv = vecs * (rank + 1) / LS_CLUSTER - v0;
  const int j0 = p.vdim * rank / LS_CLUSTER, nj = p.vdim * (rank + 1) / LS_CLUSTER - j0;

  pdl_launch_dependents();
  if (tid == 0) {
    for (int i = 0; i < LS_STAGES; ++i) mbar_init(smem_u32(&bars[i]), 1);
    fence_mbar_init();
  }
  {  // lines of the matrices and the cache, requested while the kernel before this one ends
    constexpr int LINE = 128 / sizeof(T);
    const int lc = (nv * 8 + LINE - 1) / LINE, lr = (rp + LINE - 1) / LINE, lk = (ld + LINE - 1) / LINE;
    for (int i = tid; i < nh * p.dim * lc; i += LS_THREADS) {
      const int r = i / lc, h = r / p.dim;
      l2_line(a.up + ((size_t)(h0 + h) * kp + r - h * p.dim) * a.ld_up + min(v0 * 8 + (i - r * lc) * LINE, rp - 1));
    }
    for (int i = tid; i < nh * nj * lr; i += LS_THREADS) {
      const int r = i / lr, h = r / nj;
      l2_line(a.up + ((size_t)a.up_v + (size_t)(h0 + h) * vp + j0 + r - h * nj) * a.ld_up + (i - r * lr) * LINE);
    }
    const int at = min(*(volatile const int*)a.pos, p.cache.ctx_len - 1);  // (may be the step before's: only lines are asked for)
    const int lo = window_first(at, p.window), total = at + 1 - lo;
    const int t0 = (int)((long long)total * rank / LS_CLUSTER), n = (int)((long long)total * (rank + 1) / LS_CLUSTER) - t0;
    for (int i = tid + LS_THREADS * cl; i < n * lk; i += LS_THREADS * clusters)  // (the clusters share the cache rows)
      l2_line(p.cache.rows + (size_t)(lo + t0 + i / lk) * ld + min(i % lk * LINE, ld - 1));
  }
  if (TC)
    for (int i = tid; i < 16 * (LS_CHUNK + 8); i += LS_THREADS) wt[i] = __float2bfloat16(0.f);
  __syncthreads();
  pdl_wait();
  const int pos = *a.pos, lo = window_first(pos, p.window), total = pos + 1 - lo;
  const int t0 = (int)((long long)total * rank / LS_CLUSTER), n = (int)((long long)total * (rank + 1) / LS_CLUSTER) - t0;
  const int chunks = (n + chunk - 1) / chunk;
  const bool has_token = rank == LS_CLUSTER - 1;  // its slice ends with the token itself, which is not in the cache yet
  auto fetch = [&](int c) {  // by one warp, a copy per row
    const int s = c % LS_STAGES, rows = min(chunk, n - c * chunk) - (has_token && c == chunks - 1);
    const uint32_t bar = smem_u32(&bars[s]), bytes = (uint32_t)(ld * sizeof(T));
    if (lane == 0) mbar_arrive_expect_tx(bar, rows * bytes);
    __syncwarp();
    for (int r = lane; r < rows; r += 32)
      bulk_g2s(smem_u32(stages + (size_t)(s * chunk + r) * z.row), p.cache.rows + (size_t)(lo + t0 + c * chunk + r) * ld, bytes, bar);
  };
  if (warp == LS_WARPS - 1)
    for (int c = 0; c < chunks && c < LS_STAGES; ++c) fetch(c);

  // the token's cache row, and the heads' queries
  float ss = 0.f;
  for (int d = tid; d < rp; d += LS_THREADS) {
    const float x = d < p.kv_rank ? to_f(p.c[d]) : 0.f;
    oc[d] = x;
    ss = fmaf(x, x, ss);
  }
  for (int i = tid; i < nh * kp; i += LS_THREADS) {
    const int h = head_of(i, kp), d = i - h * kp;
    qh[i] = to_f(p.q[(size_t)(h0 + h) * (kp + rotp) + d]);
  }
  for (int i = tid; i < (nh + 1) * rotp; i += LS_THREADS) {  // heads, then the shared key part
    const int h = i < nh * rotp ? head_of(i, rotp) : nh, d = i - h * rotp;
    const T* src = h < nh ? p.q + (size_t)(h0 + h) * (kp + rotp) + kp : p.k;
    float v = d < p.rot_dim ? to_f(src[d]) : 0.f;
    if (d < p.rot_dims) {
      const float2 cs = p.rope[(size_t)pos * half + (d >> 1)];
      v = v * cs.x + to_f(src[d ^ 1]) * (d & 1 ? cs.y : -cs.y);
    }
    if (h < nh) q[h * ld + rp + d] = v;
    else cur[rp + d] = from_f<T>(v);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float all = 0.f;
#pragma unroll
  for (int w = 0; w < LS_WARPS; ++w) all += red[w];
  const float inv_c = 1.0f / sqrtf(all / (float)p.kv_rank + p.eps);
  for (int d = tid; d < rp; d += LS_THREADS) cur[d] = from_f<T>(d < p.kv_rank ? oc[d] * inv_c * p.norm[d] : 0.f);
  if (nv > 0) {  // this CTA's columns of the queries against latents, in vectors of 8; the heads share the groups of threads
    const int per = max(1, min(LS_THREADS / nv, LS_GROUPS) / nh), grp = tid / nv, j = tid - grp * nv, h = grp / per;
    if (h < nh) {
      float acc[8] = {};
      const T* w = a.up + (size_t)(h0 + h) * kp * a.ld_up + (v0 + j) * 8;
#pragma unroll 4
      for (int d = grp - h * per; d < p.dim; d += per) {
        const vec8 x = *reinterpret_cast<const vec8*>(w + (size_t)d * a.ld_up);
        const float qd = qh[h * kp + d];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(qd, to_f(x.e[e]), acc[e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) part[(grp * nv + j) * 8 + e] = acc[e];
    }
    __syncthreads();
    for (int i = tid; i < nh * nv * 8; i += LS_THREADS) {
      const int hd = head_of(i, nv * 8), c = i - hd * nv * 8;
      float v = 0.f;
#pragma unroll 4
      for (int g = 0; g < per; ++g) v += part[(hd * per + g) * nv * 8 + c];
      q[hd * ld + v0 * 8 + c] = v;
    }
  }
  cluster_sync();
  // (four columns at a time; owner: whose vectors hold them)
#pragma unroll 2
  for (int i = tid; i < nh * (ld >> 2); i += LS_THREADS) {
    const int h = head_of(i, ld >> 2), c = 4 * (i - h * (ld >> 2)), owner = ((c >> 3) * LS_CLUSTER + LS_CLUSTER - 1) / vecs;
    float* at = q + h * ld + c;
    const float4 x = c < rp && owner != rank ? ld_dsmem_f4(mapa(smem_u32(at), owner)) : *reinterpret_cast<const float4*>(at);
    if (TC) {
      const float y[4] = {x.x * a.scale, x.y * a.scale, x.z * a.scale, x.w * a.scale};
      store_parts<4>(qp + h * LS_PARTS * ldq + c, ldq, y);
    } else {
      *reinterpret_cast<float4*>(at) = x;
    }
  }
  if (TC) {  // columns past the row, and the row of zeros
    for (int r = warp; r <= nh * LS_PARTS; r += LS_WARPS)
      for (int c = (r < nh * LS_PARTS ? ld : 0) + lane; c < ldq; c += 32) qp[r * ldq + c] = __float2bfloat16(0.f);
  }
  if (cl == 0 && rank == 0)
    for (int d = tid; d < ld; d += LS_THREADS) p.cache.rows[(size_t)pos * ld + d] = cur[d];
  __syncthreads();

  float mx = -CUDART_INF_F, sum = 0.f;  // of head `warp` (one head in binary32: of every warp)
  const int g = lane >> 2, c2 = (lane & 3) * 2;  // tensor-core lanes: rows g and g + 8, columns c2 and c2 + 1
  constexpr int TILES = TC ? MOST / 64 : 1;      // column tiles of 8 per warp
  constexpr int NV = QF / 4, NC = TC ? 1 : (MOST + 2 * LS_THREADS - 1) / (2 * LS_THREADS);
  float o[TILES][4] = {}, qr[TC ? 1 : QF], acc[NC][2] = {};
  if (!TC) {
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int d = (v * 32 + lane) * 4;
#pragma unroll
      for (int e = 0; e < 4; ++e) qr[TC ? 0 : v * 4 + e] = d < ld ? q[d + e] * a.scale : 0.f;
    }
  }
  for (int c = 0; c < chunks; ++c) {
    const int s = c % LS_STAGES, rows = min(chunk, n - c * chunk);
    uint8_t* st = stages + (size_t)s * chunk * z.row;
    mbar_wait(smem_u32(&bars[s]), (uint32_t)(c / LS_STAGES) & 1u, a.err, DEV_ERR_FULL_WAIT);  // (expired: the error word is set, results are not used)
    if (has_token && c == chunks - 1) {
      for (int d = tid; d < ld; d += LS_THREADS) reinterpret_cast<T*>(st + (size_t)(rows - 1) * z.row)[d] = cur[d];
      __syncthreads();
    }
    if constexpr (TC) {
      for (int k0 = warp * 8; k0 < rows; k0 += LS_WARPS * 8) {  // 8 rows x all columns
        float d0[4] = {}, d1[4] = {};
        const uint32_t base = smem_u32(st + (size_t)min(k0 + (lane & 7), rows - 1) * z.row);
        const uint32_t qbase = smem_u32(qp + min(lane & 15, nh * LS_PARTS) * ldq) + (lane >> 4) * 16;
#pragma unroll 6
        for (int k = 0; k < z.steps; k += 2) {
          uint32_t b[4], a0[4], a1[4];
          const int col = k * 16 + (lane >> 3) * 8;
          ldsm4(base + (col < ld ? col * 2 : 0), b);  // (columns past the row meet queries of 0)
          ldsm4(qbase + k * 32, a0);
          ldsm4(qbase + k * 32 + 32, a1);
          mma_16816_bf16(d0, a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
          mma_16816_bf16(d1, a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
        }
        sc[g * LS_CHUNK + k0 + c2] = d0[0] + d1[0];
        sc[g * LS_CHUNK + k0 + c2 + 1] = d0[1] + d1[1];
        sc[(g + 8) * LS_CHUNK + k0 + c2] = d0[2] + d1[2];
        sc[(g + 8) * LS_CHUNK + k0 + c2 + 1] = d0[3] + d1[3];
      }
      __syncthreads();
      if (warp < nh) {  // a warp per head: running maximum and sum, weights of the chunk in parts
        const float* mine = sc + warp * LS_PARTS * LS_CHUNK;
        float x[LS_CHUNK / 32], top = mx;
#pragma unroll
        for (int i = 0; i < LS_CHUNK / 32; ++i) {
          const int k = lane + 32 * i;
          x[i] = k < rows ? mine[k] + (mine[LS_CHUNK + k] + mine[2 * LS_CHUNK + k]) : -CUDART_INF_F;
          top = fmaxf(top, x[i]);
        }
        top = warp_max(top);
        const float f = expf(mx - top);
        sum *= f;
#pragma unroll
        for (int i = 0; i < LS_CHUNK / 32; ++i) {
          const float e = expf(x[i] - top);
          sum += e;  // (this lane's rows; the lanes are added at the end)
          store_parts<1>(wt + warp * LS_PARTS * (LS_CHUNK + 8) + lane + 32 * i, LS_CHUNK + 8, &e);
        }
        mx = top;
        if (lane == 0) fac[warp] = f;
      }
      __syncthreads();
      const float f0 = g / LS_PARTS < nh ? fac[g / LS_PARTS] : 0.f, f1 = (g + 8) / LS_PARTS < nh ? fac[(g + 8) / LS_PARTS] : 0.f;
#pragma unroll
      for (int t = 0; t < TILES; ++t) {
        o[t][0] *= f0;
        o[t][1] *= f0;
        o[t][2] *= f1;
        o[t][3] *= f1;
      }
      for (int k0 = 0; k0 < rows; k0 += 16) {  // (weights past the last row are 0)
        const __nv_bfloat16 *lo_row = wt + g * (LS_CHUNK + 8) + k0 + c2, *hi_row = lo_row + 8 * (LS_CHUNK + 8);
        const uint32_t a0 = *reinterpret_cast<const uint32_t*>(lo_row), a1 = *reinterpret_cast<const uint32_t*>(hi_row);
        const uint32_t a2 = *reinterpret_cast<const uint32_t*>(lo_row + 8), a3 = *reinterpret_cast<const uint32_t*>(hi_row + 8);
        const uint32_t base = smem_u32(st + (size_t)min(k0 + (lane & 7) + ((lane >> 3) & 1) * 8, rows - 1) * z.row) + (lane >> 4) * 16;
#pragma unroll
        for (int t = 0; t < TILES; t += 2) {  // tiles of the warp: pairs (t / 2) * LS_WARPS + warp
          const int col = ((t >> 1) * LS_WARPS + warp) * 16;
          if (col < rp) {
            uint32_t b[4];
            ldsm4_trans(base + (col + (lane >> 4) * 8 < ld ? col * 2 : 0), b);
            mma_16816_bf16(o[t], a0, a1, a2, a3, b[0], b[1]);
            mma_16816_bf16(o[t + 1 < TILES ? t + 1 : t], a0, a1, a2, a3, b[2], b[3]);
          }
        }
      }
    } else {
      for (int k = warp; k < rows; k += LS_WARPS) {
        const T* row = reinterpret_cast<const T*>(st + (size_t)k * z.row);
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < NV; ++w) {
          const int d = (w * 32 + lane) * 4;
          if (d < ld) {
#pragma unroll
            for (int e = 0; e < 4; ++e) v = fmaf(qr[TC ? 0 : w * 4 + e], to_f(row[d + e]), v);
          }
        }
        v = warp_sum(v);
        if (lane == 0) sc[k] = v;
      }
      __syncthreads();
      float top = mx;
      for (int k = lane; k < rows; k += 32) top = fmaxf(top, sc[k]);
      top = warp_max(top);
      const float f = expf(mx - top);
      mx = top;
      sum *= f;
      for (int k = lane; k < rows; k += 32) sum += expf(sc[k] - top);
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int d = min(2 * (tid + i * LS_THREADS), rp - 2);  // (threads past the last column repeat it and keep nothing)
        acc[i][0] *= f;
        acc[i][1] *= f;
        for (int k = 0; k < rows; ++k) {
          const T* row = reinterpret_cast<const T*>(st + (size_t)k * z.row);
          const float w = expf(sc[k] - top);
          acc[i][0] = fmaf(w, to_f(row[d]), acc[i][0]);
          acc[i][1] = fmaf(w, to_f(row[d + 1]), acc[i][1]);
        }
      }
    }
    __syncthreads();  // the stage and the scores are used again
    if (warp == LS_WARPS - 1 && c + LS_STAGES < chunks) fetch(c + LS_STAGES);
  }
  sum = warp_sum(sum);
  if (warp < nh && lane == 0) {
    res[warp * z.res_stride] = mx;
    res[warp * z.res_stride + 1] = sum;
  }
  if constexpr (TC) {  // parts meet in shared memory (the stages are free)
    float* out = reinterpret_cast<float*>(stages);  // [nh * LS_PARTS][rp]
#pragma unroll
    for (int t = 0; t < TILES; ++t) {
      const int col = ((t >> 1) * LS_WARPS + warp) * 16 + (t & 1) * 8 + c2;
      if (col < rp) {
        if (g < nh * LS_PARTS) *reinterpret_cast<float2*>(out + g * rp + col) = make_float2(o[t][0], o[t][1]);
        if (g + 8 < nh * LS_PARTS) *reinterpret_cast<float2*>(out + (g + 8) * rp + col) = make_float2(o[t][2], o[t][3]);
      }
    }
    __syncthreads();
    for (int i = tid; i < nh * (z.res_stride - 4); i += LS_THREADS) {
      const int h = head_of(i, z.res_stride - 4), d = i - h * (z.res_stride - 4);
      const float* x = out + h * LS_PARTS * rp + d;
      res[h * z.res_stride + 4 + d] = x[0] + (x[rp] + x[2 * rp]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = 2 * (tid + i * LS_THREADS) + e;
        if (d < z.res_stride - 4) res[4 + d] = acc[i][e];
      }
  }
  cluster_sync();
  if (tid < nh * LS_CLUSTER) {  // eight lanes per head, one per CTA
    const int h = tid / LS_CLUSTER, r = tid % LS_CLUSTER;
    const unsigned lanes = 0xffu << (lane & 24);
    const uint32_t from = mapa(smem_u32(res + h * z.res_stride), r);
    const float m = ld_dsmem_f32(from), l = ld_dsmem_f32(from + 4), sink = a.sink ? a.sink[h0 + h] : -CUDART_INF_F;
    float top = fmaxf(m, sink);
#pragma unroll
    for (int y = 4; y > 0; y >>= 1) top = fmaxf(top, __shfl_xor_sync(lanes, top, y));
    const float f = expf(m - top);  // (0 for a CTA without rows)
    float t = f * l;
#pragma unroll
    for (int y = 4; y > 0; y >>= 1) t += __shfl_xor_sync(lanes, t, y);
    if (a.sink) t += expf(sink - top);
    share[tid] = f * (a.out_scale / t) * (a.gate ? sigmoid_f(to_f(a.gate[h0 + h])) : 1.f);
  }
  __syncthreads();
  const int quads = (z.res_stride - 4) >> 2;  // (columns past the rank, up to a multiple of 4, are sums of zeros)
#pragma unroll 2
  for (int i = tid; i < nh * (rp >> 2); i += LS_THREADS) {
    const int h = head_of(i, rp >> 2), d4 = i - h * (rp >> 2);
    float v[4] = {};
    if (d4 < quads) {
      const uint32_t from = smem_u32(res + h * z.res_stride + 4 + 4 * d4);
#pragma unroll
      for (int r = 0; r < LS_CLUSTER; ++r) {
        const float4 x = ld_dsmem_f4(mapa(from, r));
        const float w = share[h * LS_CLUSTER + r];
        v[0] = fmaf(w, x.x, v[0]);
        v[1] = fmaf(w, x.y, v[1]);
        v[2] = fmaf(w, x.z, v[2]);
        v[3] = fmaf(w, x.w, v[3]);
      }
    }
    if (TC) store_parts<4>(qp + h * LS_PARTS * ldq + 4 * d4, ldq, v);
    else *reinterpret_cast<float4*>(oc + h * rp + 4 * d4) = make_float4(v[0], v[1], v[2], v[3]);
  }
  __syncthreads();
  // this CTA's rows of the value matrices
  if constexpr (TC) {
    // 16 rows of a head are an operand; the warps share the heads, then the columns.  A lane's 16 bytes - columns 8 (lane % 4)
    // .. + 7 of 32 - serve two products, with the same columns of the other operand (parts of the sum of rows) in their places.
    const int tiles = (nj + 15) / 16, units = nh * tiles, kg = max(1, LS_WARPS / max(units, 1)), steps = (rp + 31) / 32;
    for (int u = warp / kg; u < units; u += LS_WARPS / kg) {
      const int h = head_of(u, tiles), r0 = (u - h * tiles) * 16;
      const T* w0 = a.up + ((size_t)a.up_v + (size_t)(h0 + h) * vp + j0 + min(r0 + g, nj - 1)) * a.ld_up + c2 * 4;
      const T* w1 = a.up + ((size_t)a.up_v + (size_t)(h0 + h) * vp + j0 + min(r0 + g + 8, nj - 1)) * a.ld_up + c2 * 4;
      const __nv_bfloat16* b = qp + (h * LS_PARTS + min(g, LS_PARTS - 1)) * ldq + c2 * 4;
      float d0[4] = {}, d1[4] = {};
#pragma unroll 4
      for (int k = warp % kg; k < steps; k += kg) {
        const bool in = k * 32 + c2 * 4 < rp;  // (a column past the latent counts as 0)
        const uint4 none = make_uint4(0, 0, 0, 0);
        const uint4 x0 = in ? *reinterpret_cast<const uint4*>(w0 + k * 32) : none, x1 = in ? *reinterpret_cast<const uint4*>(w1 + k * 32) : none;
        const uint4 y = in && g < LS_PARTS ? *reinterpret_cast<const uint4*>(b + k * 32) : none;
        mma_16816_bf16(d0, x0.x, x1.x, x0.y, x1.y, y.x, y.y);
        mma_16816_bf16(d1, x0.z, x1.z, x0.w, x1.w, y.z, y.w);
      }
      // columns 0 .. 2 hold the parts' products
      float lo = c2 == 0 ? (d0[0] + d1[0]) + (d0[1] + d1[1]) : c2 == 2 ? d0[0] + d1[0] : 0.f;
      float hi = c2 == 0 ? (d0[2] + d1[2]) + (d0[3] + d1[3]) : c2 == 2 ? d0[2] + d1[2] : 0.f;
      lo += __shfl_xor_sync(0xffffffffu, lo, 1);
      hi += __shfl_xor_sync(0xffffffffu, hi, 1);
      if (c2 == 0) {
        sc[(u * kg + warp % kg) * 16 + g] = lo;
        sc[(u * kg + warp % kg) * 16 + g + 8] = hi;
      }
    }
    __syncthreads();
    for (int i = tid; i < units * 16; i += LS_THREADS) {
      const int u = i >> 4, h = head_of(u, tiles), j = (u - h * tiles) * 16 + (i & 15);
      float v = 0.f;
      for (int k = 0; k < kg; ++k) v += sc[(u * kg + k) * 16 + (i & 15)];
      if (j < nj) a.out[(size_t)(h0 + h) * p.vdim + j0 + j] = from_f<T>(v);
    }
  } else {
    for (int i = warp; i < nh * nj; i += LS_WARPS) {
      const int h = i / nj, j = j0 + i - h * nj;
      const T* w = a.up + ((size_t)a.up_v + (size_t)(h0 + h) * vp + j) * a.ld_up;
      float v = 0.f;
      for (int d = lane; d < rp; d += 32) v = fmaf(oc[h * rp + d], to_f(w[d]), v);
      v = warp_sum(v);
      if (lane == 0) a.out[(size_t)(h0 + h) * p.vdim + j] = from_f<T>(v);
    }
  }
  cluster_sync();  // nobody leaves while its partial sums may still be read
}

template <typename T, int QF>
int launch_step(const latent_step<T>& p, cudaStream_t stream) {
  const latent_rows<T>& r = p.rows;
  auto bytes = [&](int heads, int chunk) { return latent_layout(r.dim, r.kv_rank, r.cache.ld, r.cache.rot, sizeof(T), heads, chunk).total; };
  static bool attr_done[16] = {};
  static int room[16] = {};  // clusters that run at the same time with a CTA per SM
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  LCU_REQUIRE(dev < 16, "latent attention: device %d", dev);
  auto kernel = latent_step_kernel<T, QF>;
  if (!attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LS_SMEM));
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(LS_CLUSTER);
    cfg.blockDim = dim3(LS_THREADS);
    cfg.dynamicSmemBytes = LS_SMEM;
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = LS_CLUSTER;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    LCU_CUDA(cudaOccupancyMaxActiveClusters(&room[dev], kernel, &cfg));
    LCU_REQUIRE(room[dev] >= 1, "latent attention: no room for a cluster of %d", LS_CLUSTER);
    attr_done[dev] = true;
  }
  // heads per cluster: as few as still let all clusters run at once
  int clusters = sizeof(T) == 2 ? std::min(r.heads, room[dev]) : r.heads;
  clusters = std::max(clusters, (r.heads + LS_HEADS - 1) / LS_HEADS);
  const int most = (r.heads + clusters - 1) / clusters;
  int chunk = std::min(LS_CHUNK, std::min(r.window, r.cache.ctx_len) / LS_CLUSTER + 1);
  while (chunk > 1 && bytes(most, chunk) > LS_SMEM) --chunk;
  LCU_REQUIRE(bytes(most, chunk) <= LS_SMEM, "latent attention: %d bytes of shared memory", bytes(most, chunk));
  return launch_clustered(kernel, clusters * LS_CLUSTER, LS_CLUSTER, LS_THREADS, bytes(most, chunk), stream, p, clusters, most, chunk);
}

}  // namespace

template <typename T>
int launch_latent_step(const latent_step<T>& p, cudaStream_t stream) {
  const int ld = p.rows.cache.ld;
  if (ld <= 256) return launch_step<T, 8>(p, stream);
  if (ld <= 512) return launch_step<T, 16>(p, stream);
  if (ld <= 768) return launch_step<T, 24>(p, stream);
  if (ld <= 1280) return launch_step<T, 40>(p, stream);
  LCU_REQUIRE(ld <= 2560, "latent attention: cache rows of %d", ld);
  return launch_step<T, 80>(p, stream);
}

template <typename T>
int launch_latent_rows(const latent_rows<T>& p, int m, int pos0, cudaStream_t stream) {
  LCU_REQUIRE(pos0 >= 0 && pos0 + m <= p.cache.ctx_len, "latent attention: rows %d..%d outside the cache of %d", pos0, pos0 + m, p.cache.ctx_len);
  const int n_old = pos0 - window_first(pos0, p.window);
  LCU_CUDA(launch_after(latent_rows_kernel<T>, dim3(n_old + m), dim3(LR_THREADS), 0, stream, p, n_old, pos0));
  return LCU_OK;
}

template int launch_latent_rows<__nv_bfloat16>(const latent_rows<__nv_bfloat16>&, int, int, cudaStream_t);
template int launch_latent_rows<float>(const latent_rows<float>&, int, int, cudaStream_t);
template int launch_latent_step<__nv_bfloat16>(const latent_step<__nv_bfloat16>&, cudaStream_t);
template int launch_latent_step<float>(const latent_step<float>&, cudaStream_t);

}  // namespace lcu
