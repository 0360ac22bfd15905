// Routed feed-forward, rows of a pass: every row picks its experts, then the rows are laid out expert by expert for products
// with one matrix per group.  Both launches work on chunks of ROUTE_CHUNK rows: the first picks and counts a chunk's rows per
// expert, the second turns the counts of all chunks into the chunk's first place in every expert's run and copies its rows.
#include "block_ops.cuh"
#include "elem.cuh"

namespace lcu {
namespace {

constexpr int ROUTE_CHUNK = 16, ROUTE_THREADS = 256, ROUTE_WARPS = ROUTE_THREADS / 32;
constexpr int ROUTE_SLICES = 8;  // CTAs that share the columns of a chunk's copies

// scratch: pick [rows * top], pick_weight [rows * top] (float), counts [chunks][experts]
template <typename T>
__global__ void __launch_bounds__(ROUTE_THREADS) route_pick_kernel(const route_rows<T> p) {
  extern __shared__ float z_sm[];  // [ROUTE_WARPS][experts], then counts [experts]
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, E = p.experts;
  int* count = reinterpret_cast<int*>(z_sm + ROUTE_WARPS * E);
  int* pick = p.scratch;
  float* weight = reinterpret_cast<float*>(p.scratch + (size_t)p.rows * p.top);
  int* counts = p.scratch + 2 * (size_t)p.rows * p.top + (size_t)blockIdx.x * E;
  for (int e = tid; e < E; e += ROUTE_THREADS) count[e] = 0;
  __syncthreads();
  float* z = z_sm + warp * E;
  for (int i = warp; i < ROUTE_CHUNK; i += ROUTE_WARPS) {
    const int r = blockIdx.x * ROUTE_CHUNK + i;
    if (r >= p.rows) break;
    for (int e = lane; e < E; e += 32) z[e] = p.z[(size_t)r * p.ldz + e];
    __syncwarp();
    pick_largest(z, E, p.top, [&](int k, int e, float v) {
      pick[(size_t)r * p.top + k] = e;
      weight[(size_t)r * p.top + k] = sigmoid_f(v);
      atomicAdd(&count[e], 1);
    });
  }
  __syncthreads();
  for (int e = tid; e < E; e += ROUTE_THREADS) counts[e] = count[e];
}

// grid (chunks, slices of the columns); the first slice also writes what the later launches read
template <typename T>
__global__ void __launch_bounds__(ROUTE_THREADS) route_place_kernel(const route_rows<T> p, int chunks) {
  extern __shared__ int r_sm[];  // first [E]: the chunk's place in every expert's run; size [E]
  __shared__ int s_at[ROUTE_CHUNK * MAX_TOP], s_pick[ROUTE_CHUNK * MAX_TOP];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, E = p.experts, top = p.top;
  int *first = r_sm, *size = r_sm + E;
  const int* pick = p.scratch;
  const float* weight = reinterpret_cast<const float*>(p.scratch + (size_t)p.rows * top);
  const int* counts = p.scratch + 2 * (size_t)p.rows * top;
  const int r0 = blockIdx.x * ROUTE_CHUNK, n = min(ROUTE_CHUNK, p.rows - r0) * top;
  const size_t at0 = (size_t)r0 * top;
  for (int e = tid; e < 2 * E; e += ROUTE_THREADS) r_sm[e] = 0;
  for (int i = tid; i < n; i += ROUTE_THREADS) s_pick[i] = pick[at0 + i];
  __syncthreads();
  // (threads that share an expert take chunks in turn)
  const int per = E >= ROUTE_THREADS ? 1 : ROUTE_THREADS / E;
  for (int i = tid; i < E * per; i += ROUTE_THREADS) {
    const int e = i % E, g = i / E;
    int all = 0, before = 0;
#pragma unroll 4
    for (int c = g; c < chunks; c += per) {
      const int n = counts[(size_t)c * E + e];
      all += n;
      if (c < (int)blockIdx.x) before += n;
    }
    atomicAdd(&size[e], all);
    atomicAdd(&first[e], before);
  }
  __syncthreads();
  if (tid < 32) {  // starts of the experts' runs; the first CTA also writes the tiles
    int run = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + tid, n = e < E ? size[e] : 0, t = (n + p.tile_rows - 1) / p.tile_rows;
      int ns = n, ts = t;  // inclusive sums over the lanes
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, ns, o), b = __shfl_up_sync(0xffffffffu, ts, o);
        if (tid >= o) {
          ns += a;
          ts += b;
        }
      }
      const int start = run + ns - n;
      if (e < E) {
        first[e] += start;
        if (blockIdx.x == 0 && blockIdx.y == 0)
          for (int j = 0; j < t; ++j) p.tiles[tiles + ts - t + j] = make_int4(start + j * p.tile_rows, min(start + (j + 1) * p.tile_rows, start + n), e, 0);
      }
      run += __shfl_sync(0xffffffffu, ns, 31);
      tiles += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (blockIdx.x == 0 && blockIdx.y == 0 && tid == 0) *p.n_tiles = tiles;
  }
  __syncthreads();
  for (int i = tid; i < n; i += ROUTE_THREADS) {  // place of entry i: entries of the chunk before it with the same expert
    const int e = s_pick[i];
    int at = first[e];
    for (int j = 0; j < i; ++j) at += s_pick[j] == e;
    s_at[i] = at;
    if (blockIdx.y > 0) continue;
    p.at[at0 + i] = at;
    p.weight[at] = weight[at0 + i];
  }
  __syncthreads();
  constexpr int VEC = 16 / sizeof(T);
  // a row is read once and written to the places of all its experts
  const int all = p.cols / VEC, first_vec = all * blockIdx.y / gridDim.y, vecs = all * (blockIdx.y + 1) / gridDim.y - first_vec, rows = n / top;
#pragma unroll 4
  for (int i = tid; i < rows * vecs; i += ROUTE_THREADS) {
    const int r = i / vecs, c = (first_vec + i - r * vecs) * VEC;
    const uint4 v = *reinterpret_cast<const uint4*>(p.h + (size_t)(r0 + r) * p.ldh + c);
    for (int k = 0; k < top; ++k) *reinterpret_cast<uint4*>(p.packed + (size_t)s_at[r * top + k] * p.ldh + c) = v;
  }
}

}  // namespace

size_t route_scratch(int rows, int experts, int top) {
  return 2 * (size_t)rows * top + ceil_div(rows, ROUTE_CHUNK) * experts;
}

template <typename T>
int launch_route(const route_rows<T>& p, cudaStream_t stream) {
  LCU_REQUIRE(p.experts >= 1 && p.experts <= MAX_EXPERTS && p.top >= 1 && p.top <= MAX_TOP && p.top <= p.experts, "route: top %d of %d experts", p.top,
              p.experts);
  LCU_REQUIRE(p.cols % 8 == 0 && p.ldh % 8 == 0, "route: rows of %d columns are not 16-byte vectors", p.cols);
  const int chunks = (int)ceil_div(p.rows, ROUTE_CHUNK);
  LCU_CUDA(launch_after(route_pick_kernel<T>, dim3(chunks), dim3(ROUTE_THREADS), (ROUTE_WARPS + 1) * (size_t)p.experts * 4, stream, p));
  LCU_CUDA(launch_after(route_place_kernel<T>, dim3(chunks, ROUTE_SLICES), dim3(ROUTE_THREADS), 2 * (size_t)p.experts * 4, stream, p, chunks));
  return LCU_OK;
}

template int launch_route<__nv_bfloat16>(const route_rows<__nv_bfloat16>&, cudaStream_t);
template int launch_route<float>(const route_rows<float>&, cudaStream_t);

}  // namespace lcu
