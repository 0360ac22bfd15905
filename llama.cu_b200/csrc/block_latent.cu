// Latent attention, rows of a pass: norm of the latents, rotation of the query and key parts, cache rows, and the dense copy
// of every latent the rows see, from which one product forms the keys and values of all heads.
#include "block_ops.cuh"
#include "elem.cuh"

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

}  // namespace

template <typename T>
int launch_latent_rows(const latent_rows<T>& p, int m, int pos0, cudaStream_t stream) {
  LCU_REQUIRE(pos0 >= 0 && pos0 + m <= p.cache.ctx_len, "latent attention: rows %d..%d outside the cache of %d", pos0, pos0 + m, p.cache.ctx_len);
  const int n_old = pos0 - window_first(pos0, p.window);
  LCU_CUDA(launch_after(latent_rows_kernel<T>, dim3(n_old + m), dim3(LR_THREADS), 0, stream, p, n_old, pos0));
  return LCU_OK;
}

template int launch_latent_rows<__nv_bfloat16>(const latent_rows<__nv_bfloat16>&, int, int, cudaStream_t);
template int launch_latent_rows<float>(const latent_rows<float>&, int, int, cudaStream_t);

}  // namespace lcu
