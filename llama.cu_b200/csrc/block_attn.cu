// Attention over a sliding window and pooled blocks for several rows, bfloat16 caches, on warp-level tensor-core tiles.
//
// One CTA takes 64 query rows of one head (4 warps of 16 rows) and walks the visible keys in tiles of 64: first the block
// means any of its rows sees, then the tokens from the first row's window start to the last row.  Keys and values come in
// by asynchronous copies into two alternating stages; scores and the running softmax (maximum and sum per row) are
// binary32, probabilities enter the second product as bfloat16.  Keys may come in two parts (a head's own and one that all
// heads share); up to 256 key and 128 value columns.  Rows in memory are padded to multiples of 8 with zeros, smaller heads
// are zero-filled to the tile width in shared memory.
#include <math_constants.h>

#include "block_ops.cuh"
#include "elem.cuh"

namespace lcu {
namespace {

constexpr int WA_Q = 64, WA_K = 64, WA_THREADS = 128;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void copy16_or_zero(uint32_t dst, const void* src, bool valid) {
  const uint32_t n = valid ? 16u : 0u;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// HK, HV: columns of the key (both parts) and value tiles
template <int HK, int HV>
__global__ void __launch_bounds__(WA_THREADS, HK == 64 ? 4 : HK == 128 ? 3 : 2) window_mma_kernel(const attn_rows<__nv_bfloat16> p, int m, int pos0) {
  using T = __nv_bfloat16;
  constexpr int LDK = HK + 8, LDV = HV + 8, STAGE = WA_K * (LDK + LDV), CK = HK / 8, CV = HV / 8;
  extern __shared__ __align__(16) T wa_smem[];  // [2 stages][keys | values]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
  // row tiles in descending order (the last ones see the most keys), heads of a key/value group next to each other
  const int head = blockIdx.x, q0 = (gridDim.y - 1 - blockIdx.y) * WA_Q;
  const int kvh = head / (p.heads / p.kv_heads);
  const int ldk = p.cache.ldk, ldv = p.cache.ldv;
  const T* kc = p.cache.k + kvh * p.cache.k_head;
  const T* vc = p.cache.v + kvh * p.cache.v_head;
  // columns of a staged row: the first key part (padded to 8), the second, zeros
  const int k_cols = (p.dim + 7) / 8 * 8, v_cols = (p.vdim + 7) / 8 * 8, k2_end = k_cols + (p.key2 ? (p.dim2 + 7) / 8 * 8 : 0);
  const int q_cols = p.key2 ? k2_end : p.dim;
  const T* kp = p.cache.kp + (size_t)kvh * p.cache.n_blocks * ldk;
  const T* vp = p.cache.vp + (size_t)kvh * p.cache.n_blocks * ldv;
  pdl_launch_dependents();
  pdl_wait();

  const int rows_here = min(WA_Q, m - q0);
  const int first_pos = pos0 + q0, last_pos = first_pos + rows_here - 1;
  auto blocks_of = [&](int pos) {
    const int past = pos + 1 - p.window;
    return p.pool > 0 && past > 0 ? past / p.pool : 0;
  };
  const int n_blocks = blocks_of(last_pos), lo = max(0, first_pos + 1 - p.window);
  const int pool_tiles = (n_blocks + WA_K - 1) / WA_K, tok_tiles = (last_pos - lo + WA_K) / WA_K, n_tiles = pool_tiles + tok_tiles;

  // query fragments (16 rows x HD per warp): rows g and g + 8
  const int r_lo = q0 + warp * 16 + g, r_hi = r_lo + 8;
  uint32_t qa[HK / 16][4];
  {
    auto pair = [&](int r, int d) {
      const T* q = p.q + (size_t)r * p.ld + head * p.q_head + d;
      const T zero = __float2bfloat16(0.f);
      __nv_bfloat162 h;
      h.x = r < m && d < q_cols ? q[0] : zero;
      h.y = r < m && d + 1 < q_cols ? q[1] : zero;
      return *reinterpret_cast<const uint32_t*>(&h);
    };
#pragma unroll
    for (int ks = 0; ks < HK / 16; ++ks) {
      const int d = ks * 16 + 2 * c;
      qa[ks][0] = pair(r_lo, d);
      qa[ks][1] = pair(r_hi, d);
      qa[ks][2] = pair(r_lo, d + 8);
      qa[ks][3] = pair(r_hi, d + 8);
    }
  }
  const int pos_lo = pos0 + r_lo, pos_hi = pos0 + r_hi;
  const int blk_lo = blocks_of(pos_lo), blk_hi = blocks_of(pos_hi);
  const int win_lo = pos_lo + 1 - p.window, win_hi = pos_hi + 1 - p.window;  // first token of the window (may be negative)
  const int warp_first = pos0 + q0 + warp * 16, warp_last = warp_first + 15;

  auto stage_tile = [&](int tile, int stage) {
    T* ks = wa_smem + (size_t)stage * STAGE;
    T* vs = ks + WA_K * LDK;
    const bool pooled = tile < pool_tiles;
    const int t0 = pooled ? tile * WA_K : lo + (tile - pool_tiles) * WA_K, end = pooled ? n_blocks : last_pos + 1;
    const T *kb = pooled ? kp : kc, *vb = pooled ? vp : vc;
    const int shift = pooled ? 0 : p.cache.first;
    for (int i = tid; i < WA_K * CK; i += WA_THREADS) {
      const int r = i / CK, ch = (i % CK) * 8;
      const bool live = t0 + r < end;
      const size_t row = live ? t0 + r - shift : 0;
      const bool second = ch >= k_cols, kv = live && ch < k2_end;
      const T* src = !kv ? kb : second ? p.key2 + (size_t)(t0 + r - p.first2) * p.ld2 + ch - k_cols : kb + row * ldk + ch;
      copy16_or_zero(smem_u32(ks + r * LDK + ch), src, kv);
    }
    for (int i = tid; i < WA_K * CV; i += WA_THREADS) {
      const int r = i / CV, ch = (i % CV) * 8;
      const bool live = t0 + r < end;
      const size_t row = live ? t0 + r - shift : 0;
      const bool vv = live && ch < v_cols;
      copy16_or_zero(smem_u32(vs + r * LDV + ch), vv ? vb + row * ldv + ch : vb, vv);
    }
    cp_async_commit();
  };

  float o[HV / 8][4];
#pragma unroll
  for (int j = 0; j < HV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float mx_lo = -CUDART_INF_F, mx_hi = -CUDART_INF_F, sum_lo = 0.f, sum_hi = 0.f;
  const float scale2 = p.scale * LOG2E;

  stage_tile(0, 0);
  for (int tile = 0; tile < n_tiles; ++tile) {
    if (tile + 1 < n_tiles) {
      stage_tile(tile + 1, (tile + 1) & 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bool pooled = tile < pool_tiles;
    const int t0 = pooled ? tile * WA_K : lo + (tile - pool_tiles) * WA_K;
    // nothing of the tile is visible to this warp's rows
    const bool skip = pooled ? t0 >= blocks_of(warp_last) : (t0 > warp_last || t0 + WA_K - 1 < warp_first + 1 - p.window);
    if (!skip) {
      const T* ks = wa_smem + (size_t)(tile & 1) * STAGE;
      const T* vs = ks + WA_K * LDK;
      float s[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < HK / 16; kk += 2) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(smem_u32(ks + (j * 8 + (lane & 7)) * LDK + kk * 16 + (lane >> 3) * 8), b0, b1, b2, b3);
          mma_16816_bf16(s[j], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b0, b1);
          mma_16816_bf16(s[j], qa[kk + 1][0], qa[kk + 1][1], qa[kk + 1][2], qa[kk + 1][3], b2, b3);
        }
      }
      // every key of the tile visible to every row of the warp?
      const bool full = pooled ? t0 + WA_K <= blocks_of(warp_first) : (t0 + WA_K - 1 <= warp_first && t0 >= warp_last + 1 - p.window);
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] *= scale2;
      if (!full) {
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int t = t0 + j * 8 + 2 * c + (e & 1);
            const bool hi = e >= 2;
            const bool seen = pooled ? t < (hi ? blk_hi : blk_lo) : t >= (hi ? win_hi : win_lo) && t <= (hi ? pos_hi : pos_lo);
            if (!seen) s[j][e] = -CUDART_INF_F;
          }
      }
      float tm_lo = -CUDART_INF_F, tm_hi = -CUDART_INF_F;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        tm_lo = fmaxf(tm_lo, fmaxf(s[j][0], s[j][1]));
        tm_hi = fmaxf(tm_hi, fmaxf(s[j][2], s[j][3]));
      }
      tm_lo = fmaxf(tm_lo, __shfl_xor_sync(0xffffffffu, tm_lo, 1));
      tm_lo = fmaxf(tm_lo, __shfl_xor_sync(0xffffffffu, tm_lo, 2));
      tm_hi = fmaxf(tm_hi, __shfl_xor_sync(0xffffffffu, tm_hi, 1));
      tm_hi = fmaxf(tm_hi, __shfl_xor_sync(0xffffffffu, tm_hi, 2));
      const float nm_lo = fmaxf(mx_lo, tm_lo), nm_hi = fmaxf(mx_hi, tm_hi);
      // a row that has seen nothing yet keeps sum 0 and output 0 (its maximum is still -inf)
      const float ref_lo = nm_lo > -CUDART_INF_F ? nm_lo : 0.f, ref_hi = nm_hi > -CUDART_INF_F ? nm_hi : 0.f;
      const float f_lo = ex2(mx_lo - ref_lo), f_hi = ex2(mx_hi - ref_hi);
      mx_lo = nm_lo;
      mx_hi = nm_hi;
      float ts_lo = 0.f, ts_hi = 0.f;
      uint32_t pa[4][4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int j = 2 * kk + b;
          const float e0 = ex2(s[j][0] - ref_lo), e1 = ex2(s[j][1] - ref_lo), e2 = ex2(s[j][2] - ref_hi), e3 = ex2(s[j][3] - ref_hi);
          ts_lo += e0 + e1;
          ts_hi += e2 + e3;
          pa[kk][2 * b] = pack2(e0, e1);
          pa[kk][2 * b + 1] = pack2(e2, e3);
        }
      }
      sum_lo = sum_lo * f_lo + ts_lo;  // (this lane's keys; the lanes of a row are added at the end)
      sum_hi = sum_hi * f_hi + ts_hi;
#pragma unroll
      for (int j = 0; j < HV / 8; ++j) {
        o[j][0] *= f_lo;
        o[j][1] *= f_lo;
        o[j][2] *= f_hi;
        o[j][3] *= f_hi;
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
#pragma unroll
        for (int dj = 0; dj < HV / 16; ++dj) {
          const int mrow = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          const int mcol = dj * 16 + (lane >> 4) * 8;
          uint32_t b0, b1, b2, b3;
          ldsm_x4_trans(smem_u32(vs + mrow * LDV + mcol), b0, b1, b2, b3);
          mma_16816_bf16(o[2 * dj], pa[kk][0], pa[kk][1], pa[kk][2], pa[kk][3], b0, b1);
          mma_16816_bf16(o[2 * dj + 1], pa[kk][0], pa[kk][1], pa[kk][2], pa[kk][3], b2, b3);
        }
      }
    }
    __syncthreads();  // the stage is overwritten two tiles later
  }
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 1);
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 2);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 1);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 2);
  float inv_lo = p.out_scale / sum_lo, inv_hi = p.out_scale / sum_hi;
  if (p.sink) {  // one more term of the denominator, against the larger of it and the row's maximum
    const float s2 = p.sink[head] * LOG2E;
    auto with_sink = [&](float mx, float sum) {
      const float top = fmaxf(mx, s2), f = ex2(mx - top);
      return p.out_scale * f / (sum * f + ex2(s2 - top));
    };
    inv_lo = with_sink(mx_lo, sum_lo);
    inv_hi = with_sink(mx_hi, sum_hi);
  }
  if (p.gate) {
    if (r_lo < m) inv_lo *= sigmoid_f(to_f(p.gate[(size_t)r_lo * p.ldg + head]));
    if (r_hi < m) inv_hi *= sigmoid_f(to_f(p.gate[(size_t)r_hi * p.ldg + head]));
  }
#pragma unroll
  for (int j = 0; j < HV / 8; ++j) {
    const int d = j * 8 + 2 * c;
    if (d >= p.vdim) continue;
    T* a = p.out + (size_t)r_lo * p.ldo + head * p.vdim + d;
    T* b = p.out + (size_t)r_hi * p.ldo + head * p.vdim + d;
    const bool two = d + 1 < p.vdim;
    if (r_lo < m) {
      a[0] = __float2bfloat16(o[j][0] * inv_lo);
      if (two) a[1] = __float2bfloat16(o[j][1] * inv_lo);
    }
    if (r_hi < m) {
      b[0] = __float2bfloat16(o[j][2] * inv_hi);
      if (two) b[1] = __float2bfloat16(o[j][3] * inv_hi);
    }
  }
}

template <int HK, int HV>
int launch_hd(const attn_rows<__nv_bfloat16>& p, int m, int pos0, cudaStream_t stream) {
  const size_t smem = (size_t)2 * WA_K * (HK + HV + 16) * 2;
  static bool attr_done[16] = {};
  int dev = 0;
  LCU_CUDA(cudaGetDevice(&dev));
  if (dev < 16 && !attr_done[dev]) {
    LCU_CUDA(cudaFuncSetAttribute((window_mma_kernel<HK, HV>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr_done[dev] = true;
  }
  LCU_CUDA(launch_after(window_mma_kernel<HK, HV>, dim3(p.heads, (m + WA_Q - 1) / WA_Q), dim3(WA_THREADS), smem, stream, p, m, pos0));
  return LCU_OK;
}

}  // namespace

bool window_mma_supported(int dim, int dim2, int vdim) { return round_up(dim, 8) + round_up(dim2, 8) <= 256 && vdim <= 128; }

int launch_window_mma(const attn_rows<__nv_bfloat16>& p, int m, int pos0, cudaStream_t stream) {
  const int dim2 = p.key2 ? p.dim2 : 0, hk = (int)(round_up(p.dim, 8) + round_up(dim2, 8));
  LCU_REQUIRE(window_mma_supported(p.dim, dim2, p.vdim), "window attention: head size %d + %d x %d", p.dim, dim2, p.vdim);
  if (hk <= 64 && p.vdim <= 64) return launch_hd<64, 64>(p, m, pos0, stream);
  if (hk <= 128) return launch_hd<128, 128>(p, m, pos0, stream);
  if (hk <= 192) return launch_hd<192, 128>(p, m, pos0, stream);
  return launch_hd<256, 128>(p, m, pos0, stream);
}

}  // namespace lcu
