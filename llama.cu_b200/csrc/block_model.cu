// Weights of the block models: layout in the arena, loading, synthetic values.
#include "block_model.cuh"

#include <cstring>

#include "block_ops.cuh"
#include "context.cuh"
#include "loader.cuh"
#include "ops.cuh"

namespace lcu {

int block_model::create(std::unique_ptr<block_model>& out, const block_spec& spec, block_dtype dtype, const std::vector<int>& wkv_rank) {
  auto m = std::make_unique<block_model>();
  m->spec = spec;
  m->dtype = dtype;
  LCU_CUDA(cudaGetDevice(&m->device));
  const int W = spec.width, S = spec.streams;
  m->k_width = pad_k(W);
  m->n_width = pad_rows(W);
  m->n_vocab_pad = pad_rows(spec.vocab);
  m->layers.resize(spec.layers.size());
  const size_t es = m->elem_bytes();
  // pass 0 sizes the arena, pass 1 hands out addresses
  char* base = nullptr;
  for (int pass = 0; pass < 2; ++pass) {
    carve cv;
    auto mat = [&](void*& p, size_t rows, size_t cols) { p = base + cv.take(rows * cols * es); };
    auto vec = [&](float*& p, size_t n) { p = reinterpret_cast<float*>(base + cv.take(n * 4)); };
    mat(m->embed, spec.vocab, W);
    if (spec.buckets > 0) mat(m->bigram, spec.buckets + 1, W);
    mat(m->head, m->n_vocab_pad, m->k_width);
    vec(m->final_norm, W);
    vec(m->ones, S);
    vec(m->zeros, S * S);
    if (spec.loop_input) {
      m->k_loop = pad_k(2 * W);
      mat(m->loop_in, m->n_width, m->k_loop);
    }
    const hyper_weights plain{m->ones, m->ones, m->ones};  // (one stream: the plain sum)
    auto residual = [&](hyper_weights& hc, float*& post, float*& scale) {
      if (spec.sandwich) {
        hc = plain;
        vec(post, W);
        vec(scale, W);
        return;
      }
      vec(hc.in, S);
      vec(hc.out, S);
      vec(hc.mix, S * S);
    };
    for (size_t i = 0; i < m->layers.size(); ++i) {
      const layer_spec& ls = spec.layers[i];
      block_layer& L = m->layers[i];
      L.branches.assign(ls.branches.size(), branch_weights{});
      vec(L.norm1, W);
      residual(L.hc1, L.norm1b, L.scale1);
      int rows = 0, cols = 0;
      for (size_t b = 0; b < ls.branches.size(); ++b) {
        const branch_spec& bs = ls.branches[b];
        branch_weights& bw = L.branches[b];
        bw.out_col = cols;
        cols += bs.out_cols();
        if (bs.kind == BRANCH_WKV) continue;
        bw.q = rows;
        if (bs.kind == BRANCH_LATENT_ATTN) {
          rows += bs.heads * (bs.dim_pad() + bs.rot_pad());
          bw.k = rows;
          rows += bs.rank_pad();
          bw.v = rows;
          rows += bs.rot_pad();
          bw.g = rows;
          rows += round_up(bs.heads, 8);
          vec(bw.sink, bs.heads);
          vec(bw.latent_norm, bs.kv_rank);
          bw.up_v = bs.heads * bs.dim_pad();
          bw.up_rows = pad_stack(bw.up_v + bs.heads * bs.vdim_pad());
          bw.up_k = pad_k(bs.kv_rank);
          mat(bw.up, bw.up_rows, bw.up_k);
          continue;
        }
        rows += bs.heads * bs.dim;
        bw.k = rows;
        rows += bs.kv_heads * bs.dim;
        bw.v = rows;
        rows += bs.kv_heads * bs.vdim;
        if (bs.kind == BRANCH_RETENTION) {
          bw.g = rows;
          rows += bs.out_cols();
          vec(bw.decay, bs.heads);
        }
      }
      if (ls.is_wkv()) {
        const int ch = ls.branches[0].out_cols();
        L.rank = wkv_rank[i];
        for (int j = 0; j < 5; ++j) {
          L.shifted_rows[j] = pad_rows(j < 4 ? ch : L.rank);
          mat(L.shifted[j], L.shifted_rows[j], m->k_width);
        }
        vec(L.mu, (size_t)5 * W);
        vec(L.w2t, (size_t)L.rank * ch);
        vec(L.w0, ch);
        vec(L.u, ch);
        vec(L.head_norm, ch);
      } else {
        L.proj_rows = pad_stack(rows);
        mat(L.proj, L.proj_rows, m->k_width);
      }
      L.out_k = pad_k(cols);
      mat(L.out, m->n_width, L.out_k);
      if (ls.ff > 0) {
        vec(L.norm2, W);
        residual(L.hc2, L.norm2b, L.scale2);
        L.ff_pad = pad_k(ls.ff);
        if (ls.experts > 0) {
          expert_weights& x = L.experts;
          x.router_rows = pad_rows(ls.experts);
          x.gate_up_stride = 2 * (size_t)L.ff_pad * m->k_width;
          x.down_stride = (size_t)m->n_width * L.ff_pad;
          mat(x.router, x.router_rows, m->k_width);
          mat(x.gate_up, ls.experts * 2 * (size_t)L.ff_pad, m->k_width);
          mat(x.down, ls.experts * (size_t)m->n_width, L.ff_pad);
          continue;
        }
        mat(L.gate_up, 2 * (size_t)L.ff_pad, m->k_width);
        mat(L.down, m->n_width, L.ff_pad);
      }
    }
    if (pass == 0) {
      void* p = nullptr;
      LCU_CUDA(cudaMalloc(&p, cv.off));
      m->arenas.push_back({m->device, p});
      m->weight_bytes_total = cv.off;
      LCU_CUDA(cudaMemset(p, 0, cv.off));
      base = (char*)p;
    }
  }
  // constants of the description
  std::vector<float> ones(S, 1.0f);
  LCU_CUDA(cudaMemcpy(m->ones, ones.data(), S * 4, cudaMemcpyHostToDevice));
  for (size_t i = 0; i < m->layers.size(); ++i)
    for (size_t b = 0; b < spec.layers[i].branches.size(); ++b) {
      const branch_spec& bs = spec.layers[i].branches[b];
      if (!bs.decay.empty()) LCU_CUDA(cudaMemcpy(m->layers[i].branches[b].decay, bs.decay.data(), bs.decay.size() * 4, cudaMemcpyHostToDevice));
    }
  LCU_CUDA(cudaStreamSynchronize(0));
  out = std::move(m);
  return LCU_OK;
}

std::vector<block_model::slot> block_model::slots() const {
  std::vector<slot> out;
  const int W = spec.width, S = spec.streams;
  const size_t es = elem_bytes();
  auto mat = [&](const std::string& name, void* base, int row0, int col0, int ld, int rows, int cols) {
    slot s;
    s.name = name;
    s.rows = rows;
    s.cols = cols;
    s.dst = (char*)base + ((size_t)row0 * ld + col0) * es;
    s.ld = ld;
    s.f32 = dtype == BLOCK_F32;
    out.push_back(s);
  };
  auto vec = [&](const std::string& name, float* dst, int rows, int cols, slot::fill_t fill, bool transpose = false, bool optional = false) {
    slot s;
    s.name = name;
    s.rows = rows;
    s.cols = cols;
    s.dst = dst;
    s.ld = transpose ? rows : cols;
    s.f32 = true;
    s.transpose = transpose;
    s.fill = fill;
    s.optional = optional;
    out.push_back(s);
  };
  auto grouped = [&](int group, int stride, int split = 1 << 30, int gap = 0) {  // of the matrix just listed
    out.back().groups = row_groups{group, stride, split, gap};
  };
  auto hyper = [&](const std::string& name, const hyper_weights& h) {
    const bool plain = S == 1;  // a single stream without tensors of its own is the plain residual sum
    vec(name + ".in", h.in, 1, S, slot::MEAN, false, plain);
    vec(name + ".out", h.out, 1, S, slot::ONES, false, plain);
    vec(name + ".mix", h.mix, S, S, slot::IDENTITY, false, plain);
  };
  mat("embed", embed, 0, 0, W, spec.vocab, W);
  if (spec.buckets > 0) mat("bigram", bigram, 0, 0, W, spec.buckets + 1, W);
  if (spec.loop_input) mat("loop.in", loop_in, 0, 0, k_loop, W, 2 * W);
  const slot::fill_t norm_fill = spec.sandwich ? slot::ONES : slot::ZEROS;
  for (size_t i = 0; i < layers.size(); ++i) {
    const layer_spec& ls = spec.layers[i];
    const block_layer& L = layers[i];
    const std::string l = "l" + std::to_string(i) + ".", mx = l + "mix.";
    vec(l + "norm1", L.norm1, 1, W, norm_fill);
    if (spec.sandwich) {
      vec(l + "norm1b", L.norm1b, 1, W, slot::ONES);
      vec(l + "ls1", L.scale1, 1, W, slot::ONES);
    } else {
      hyper(l + "hc1", L.hc1);
    }
    for (size_t b = 0; b < ls.branches.size(); ++b) {
      const branch_spec& bs = ls.branches[b];
      const branch_weights& bw = L.branches[b];
      const std::string p = mx + bs.prefix;
      const int ch = bs.out_cols();
      if (bs.kind == BRANCH_WKV) {
        const char* names[5] = {"r", "k", "v", "g", "w"};
        for (int j = 0; j < 5; ++j) vec(p + "mu." + names[j], L.mu + (size_t)j * W, 1, W, slot::UNIFORM);
        for (int j = 0; j < 4; ++j) mat(p + names[j], L.shifted[j], 0, 0, k_width, ch, W);
        mat(p + "w1", L.shifted[4], 0, 0, k_width, L.rank, W);
        vec(p + "w2", L.w2t, ch, L.rank, slot::UNIFORM, true);
        vec(p + "w0", L.w0, 1, ch, slot::UNIFORM);
        vec(p + "u", L.u, bs.heads, bs.dim, slot::UNIFORM);
        vec(p + "norm", L.head_norm, 1, ch, slot::ONES);
      } else if (bs.kind == BRANCH_LATENT_ATTN) {
        const int dk = bs.dim + bs.rot_dim;
        mat(p + "q", L.proj, bw.q, 0, k_width, bs.heads * dk, W);
        grouped(dk, bs.dim_pad() + bs.rot_pad(), bs.dim, bs.dim_pad() - bs.dim);
        mat(p + "dkv", L.proj, bw.k, 0, k_width, bs.kv_rank + bs.rot_dim, W);
        grouped(bs.kv_rank + bs.rot_dim, 0, bs.kv_rank, bs.rank_pad() - bs.kv_rank);
        vec(p + "dkv.norm", bw.latent_norm, 1, bs.kv_rank, slot::ONES);
        mat(p + "uk", bw.up, 0, 0, bw.up_k, bs.heads * bs.dim, bs.kv_rank);
        grouped(bs.dim, bs.dim_pad());
        mat(p + "uv", bw.up, bw.up_v, 0, bw.up_k, bs.heads * bs.vdim, bs.kv_rank);
        grouped(bs.vdim, bs.vdim_pad());
        vec(p + "sink", bw.sink, 1, bs.heads, slot::ZEROS);
        mat(p + "g", L.proj, bw.g, 0, k_width, bs.heads, W);
      } else {
        mat(p + "q", L.proj, bw.q, 0, k_width, bs.heads * bs.dim, W);
        mat(p + "k", L.proj, bw.k, 0, k_width, bs.kv_heads * bs.dim, W);
        mat(p + "v", L.proj, bw.v, 0, k_width, bs.kv_heads * bs.vdim, W);
        if (bs.kind == BRANCH_RETENTION) mat(p + "g", L.proj, bw.g, 0, k_width, ch, W);
      }
      mat(p + "o", L.out, 0, bw.out_col, L.out_k, W, ch);
    }
    if (ls.ff > 0) {
      vec(l + "norm2", L.norm2, 1, W, norm_fill);
      if (spec.sandwich) {
        vec(l + "norm2b", L.norm2b, 1, W, slot::ONES);
        vec(l + "ls2", L.scale2, 1, W, slot::ONES);
      } else {
        hyper(l + "hc2", L.hc2);
      }
      if (ls.experts > 0) {
        const expert_weights& x = L.experts;
        constexpr int G = EXPERT_GATE_BLOCK;
        mat(l + "mlp.router", x.router, 0, 0, k_width, ls.experts, W);
        for (int e = 0; e < ls.experts; ++e) {
          const std::string n = l + "mlp.e" + std::to_string(e);
          mat(n + ".gate", (char*)x.gate_up + e * x.gate_up_stride * es, 0, 0, k_width, ls.ff, W);
          grouped(G, 2 * G);
          mat(n + ".up", (char*)x.gate_up + e * x.gate_up_stride * es, G, 0, k_width, ls.ff, W);
          grouped(G, 2 * G);
          mat(n + ".down", (char*)x.down + e * x.down_stride * es, 0, 0, L.ff_pad, W, ls.ff);
        }
        continue;
      }
      mat(l + "mlp.gate", L.gate_up, 0, 0, k_width, ls.ff, W);
      mat(l + "mlp.up", L.gate_up, L.ff_pad, 0, k_width, ls.ff, W);
      mat(l + "mlp.down", L.down, 0, 0, L.ff_pad, W, ls.ff);
    }
  }
  vec("final.norm", final_norm, 1, W, norm_fill);
  mat("head", head, 0, 0, k_width, spec.vocab, W);
  return out;
}

// values of a vector that is not read from a file
int block_model::set_default(const slot& s) {
  std::vector<float> v((size_t)s.rows * s.cols, 0.f);
  for (size_t i = 0; i < v.size(); ++i) {
    const size_t r = i / s.cols, c = i % s.cols;
    switch (s.fill) {
      case slot::ONES: v[i] = 1.f; break;
      case slot::IDENTITY: v[i] = r == c ? 1.f : 0.f; break;
      case slot::MEAN: v[i] = 1.f / spec.streams; break;
      case slot::UNIFORM: v[i] = (float)((i * 2654435761u >> 8) & 0xffff) / 65536.f; break;  // spread over [0, 1)
      default: break;
    }
  }
  LCU_CUDA(cudaMemcpy(s.dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
  LCU_CUDA(cudaStreamSynchronize(0));
  return LCU_OK;
}

// every output norm and the channel scale behind it become one factor (products of two bfloat16 values are exact)
int block_model::fold_scales() {
  for (auto& L : layers) {
    if (L.scale1) LCU_TRY(launch_scale_vector(L.norm1b, L.scale1, spec.width, 0));
    if (L.scale2) LCU_TRY(launch_scale_vector(L.norm2b, L.scale2, spec.width, 0));
  }
  LCU_CUDA(cudaDeviceSynchronize());
  return LCU_OK;
}

int block_model::fill_synthetic(uint64_t seed, float scale) {
  device_guard g(device);
  size_t most = 0;
  const auto all = slots();
  for (auto& s : all) most = std::max(most, (size_t)s.rows * s.cols);
  __half* tmp = nullptr;
  float* wide = nullptr;
  LCU_CUDA(cudaMalloc(&tmp, most * 2));
  cudaError_t e = cudaMalloc(&wide, most * 4);
  int rc = e == cudaSuccess ? LCU_OK : LCU_ERR_CUDA;
  for (auto& s : all) {
    if (rc) break;
    if (s.fill != slot::MATRIX) {
      rc = set_default(s);
      continue;
    }
    const size_t n = (size_t)s.rows * s.cols;
    rc = launch_synth_fill(tmp, n, seed, fnv1a64(s.name.c_str()), scale, 0, 0);
    if (!rc) rc = launch_half_to_f32(wide, tmp, n, 0);
    if (!rc)
      rc = s.f32 ? launch_place<float>((float*)s.dst, s.ld, wide, PLACE_F32, s.rows, s.cols, s.transpose, 0, s.groups)
                 : launch_place<__nv_bfloat16>((__nv_bfloat16*)s.dst, s.ld, wide, PLACE_F32, s.rows, s.cols, s.transpose, 0, s.groups);
  }
  e = cudaDeviceSynchronize();
  cudaFree(tmp);
  cudaFree(wide);
  if (rc) return rc;
  LCU_CUDA(e);
  return fold_scales();
}

int block_model::load(std::unique_ptr<block_model>& out, const std::string& dir, block_dtype dtype) {
  std::string text;
  LCU_TRY(read_text_file(dir + "/config.json", text));
  block_spec spec;
  LCU_TRY(read_block_config(text, spec));
  tensor_file file;
  LCU_TRY(file.open(dir + "/model.safetensors"));
  std::vector<int> rank(spec.layers.size(), 0);
  for (size_t i = 0; i < spec.layers.size(); ++i)
    if (spec.layers[i].is_wkv()) {  // the low-rank size of the decays is the tensor's
      const std::string name = "l" + std::to_string(i) + ".mix." + spec.layers[i].branches[0].prefix + "w1";
      const tensor_entry* t = file.find(name);
      LCU_REQUIRE(t && t->shape.size() == 2, "%s: no matrix '%s'", file.path.c_str(), name.c_str());
      rank[i] = (int)t->shape[0];
    }
  std::unique_ptr<block_model> m;
  LCU_TRY(create(m, spec, dtype, rank));
  device_guard g(m->device);
  const auto all = m->slots();
  size_t most = 0;
  for (auto& s : all) {
    const tensor_entry* t = file.find(s.name);
    if (!t) {
      LCU_REQUIRE(s.optional, "%s: tensor '%s' is missing", file.path.c_str(), s.name.c_str());
      continue;
    }
    long long n = 1;
    for (long long d : t->shape) n *= d;
    LCU_REQUIRE(n == (long long)s.rows * s.cols && (s.rows == 1 || (t->shape.size() == 2 && t->shape[0] == s.rows)),
                "%s: tensor '%s' is not %d x %d", file.path.c_str(), s.name.c_str(), s.rows, s.cols);
    LCU_REQUIRE((t->dtype == "BF16" && t->bytes == (size_t)n * 2) || (t->dtype == "F32" && t->bytes == (size_t)n * 4),
                "%s: tensor '%s' has type %s", file.path.c_str(), s.name.c_str(), t->dtype.c_str());
    most = std::max(most, t->bytes);
  }
  // staged through pinned memory into a device buffer, then placed (padded, stacked, converted) by a kernel
  staged_loader loader;
  LCU_TRY(loader.init(m->device));
  void* tmp = nullptr;
  LCU_CUDA(cudaMalloc(&tmp, most + 16));
  int rc = LCU_OK;
  for (auto& s : all) {
    const tensor_entry* t = file.find(s.name);
    if (!t) {
      rc = m->set_default(s);
    } else {
      const place_source src = t->dtype == "F32" ? PLACE_F32 : PLACE_BF16;
      rc = loader.copy_file(file.path, tmp, t->bytes, t->offset, file.file_bytes);
      if (!rc)
        rc = s.f32 ? launch_place<float>((float*)s.dst, s.ld, tmp, src, s.rows, s.cols, s.transpose, loader.stream, s.groups)
                   : launch_place<__nv_bfloat16>((__nv_bfloat16*)s.dst, s.ld, tmp, src, s.rows, s.cols, s.transpose, loader.stream, s.groups);
    }
    if (rc) break;
  }
  if (!rc) rc = loader.finish();
  cudaFree(tmp);
  if (!rc) rc = m->fold_scales();
  if (rc) return rc;
  out = std::move(m);
  return LCU_OK;
}

}  // namespace lcu
