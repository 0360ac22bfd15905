// Configuration reader and architecture registry of the block models, safetensors header reader.
#include "block_spec.cuh"

#include <cmath>
#include <cstdio>
#include <cstring>

#include "common.cuh"

namespace lcu {
namespace {

// ---- typed access with the path of what is missing in the message
int need(const json_value& o, const char* key, json_value::kind_t kind, const json_value** out) {
  const json_value* v = o.get(key);
  LCU_REQUIRE(v != nullptr && v->kind == kind, "config.json: '%s' is missing or of the wrong kind", key);
  *out = v;
  return LCU_OK;
}
int need_int(const json_value& o, const char* key, int* out, int lowest = 1) {
  const json_value* v = nullptr;
  int rc = need(o, key, json_value::NUMBER, &v);
  if (rc) return rc;
  LCU_REQUIRE(v->number == std::floor(v->number) && v->number >= lowest && v->number <= 1 << 30, "config.json: '%s' = %g is not a usable size", key,
              v->number);
  *out = (int)v->number;
  return LCU_OK;
}
int need_float(const json_value& o, const char* key, float* out) {
  const json_value* v = nullptr;
  int rc = need(o, key, json_value::NUMBER, &v);
  if (rc) return rc;
  *out = (float)v->number;
  return LCU_OK;
}
// an integer factor of a sum that is taken modulo `mod`
int need_residue(const json_value& o, const char* key, int mod, long long* out) {
  const json_value* v = nullptr;
  int rc = need(o, key, json_value::NUMBER, &v);
  if (rc) return rc;
  LCU_REQUIRE(v->number == std::floor(v->number) && std::fabs(v->number) <= 9007199254740992.0, "config.json: '%s' = %g is not an integer", key, v->number);
  *out = ((long long)v->number % mod + mod) % mod;
  return LCU_OK;
}
#define SPEC_TRY(expr)   \
  do {                   \
    int _rc = (expr);    \
    if (_rc) return _rc; \
  } while (0)

// ---- parts an architecture is put together from
int read_window_attention(const json_value& m, branch_spec& b) {
  b.kind = BRANCH_WINDOW_ATTN;
  SPEC_TRY(need_int(m, "heads", &b.heads));
  b.kv_heads = b.heads;
  if (m.get("kv_heads")) SPEC_TRY(need_int(m, "kv_heads", &b.kv_heads));
  SPEC_TRY(need_int(m, "dim", &b.dim));
  b.vdim = b.dim;
  if (m.get("vdim")) SPEC_TRY(need_int(m, "vdim", &b.vdim));
  SPEC_TRY(need_float(m, "scale", &b.score_scale));
  const json_value* mask = nullptr;
  SPEC_TRY(need(m, "mask", json_value::OBJECT, &mask));
  SPEC_TRY(need_int(*mask, "size", &b.window));
  if (mask->get("pool")) SPEC_TRY(need_int(*mask, "pool", &b.pool));
  LCU_REQUIRE(b.heads % b.kv_heads == 0, "config.json: %d heads are not a multiple of %d key/value heads", b.heads, b.kv_heads);
  return LCU_OK;
}

int read_rotation(const json_value& m, branch_spec& b, int most) {
  const json_value *rot = nullptr, *base = nullptr;
  SPEC_TRY(need(m, "rot", json_value::OBJECT, &rot));
  SPEC_TRY(need_int(*rot, "dims", &b.rot_dims));
  SPEC_TRY(need(*rot, "base", json_value::NUMBER, &base));
  b.rot_base = base->number;
  LCU_REQUIRE(b.rot_dims % 2 == 0 && b.rot_dims <= most, "config.json: %d rotated dimensions of %d", b.rot_dims, most);
  return LCU_OK;
}

int read_latent_attention(const json_value& m, branch_spec& b) {
  b.kind = BRANCH_LATENT_ATTN;
  SPEC_TRY(need_int(m, "heads", &b.heads));
  b.kv_heads = b.heads;
  SPEC_TRY(need_int(m, "dim", &b.dim));
  SPEC_TRY(need_int(m, "vdim", &b.vdim));
  SPEC_TRY(need_int(m, "kv_rank", &b.kv_rank));
  SPEC_TRY(need_int(m, "rot_dim", &b.rot_dim));
  SPEC_TRY(need_float(m, "scale", &b.score_scale));
  const json_value* mask = nullptr;
  SPEC_TRY(need(m, "mask", json_value::OBJECT, &mask));
  SPEC_TRY(need_int(*mask, "size", &b.window));
  b.sink = b.head_gate = true;
  return read_rotation(m, b, b.rot_dim);
}

int read_retention(const json_value& m, branch_spec& b) {
  b.kind = BRANCH_RETENTION;
  SPEC_TRY(need_int(m, "heads", &b.heads));
  b.kv_heads = b.heads;
  SPEC_TRY(need_int(m, "dim", &b.dim));
  b.vdim = b.dim;
  if (m.get("vdim")) SPEC_TRY(need_int(m, "vdim", &b.vdim));
  if (m.get("rot")) SPEC_TRY(read_rotation(m, b, b.dim));
  const json_value* decay = nullptr;
  SPEC_TRY(need(m, "decay", json_value::ARRAY, &decay));
  LCU_REQUIRE((int)decay->items.size() == b.heads, "config.json: %zu decays for %d heads", decay->items.size(), b.heads);
  for (auto& d : decay->items) b.decay.push_back((float)d.number);
  return LCU_OK;
}

int read_wkv(const json_value& m, branch_spec& b) {
  b.kind = BRANCH_WKV;
  SPEC_TRY(need_int(m, "heads", &b.heads));
  b.kv_heads = b.heads;
  SPEC_TRY(need_int(m, "dim", &b.dim));
  b.vdim = b.dim;
  return LCU_OK;
}

int read_stack(const json_value& c, block_spec& s) {
  SPEC_TRY(need_int(c, "vocab", &s.vocab));
  SPEC_TRY(need_int(c, "width", &s.width));
  if (c.get("streams")) SPEC_TRY(need_int(c, "streams", &s.streams));
  const json_value* norm = nullptr;
  SPEC_TRY(need(c, "norm", json_value::OBJECT, &norm));
  SPEC_TRY(need_float(*norm, "eps", &s.eps));
  if (const json_value* e = c.get("embedding")) {
    if (e->get("scale")) SPEC_TRY(need_float(*e, "scale", &s.embed_scale));
    if (const json_value* b = e->get("bigram")) {
      SPEC_TRY(need_int(*b, "buckets", &s.buckets));
      SPEC_TRY(need_residue(*b, "mul_cur", s.buckets, &s.mul_cur));
      SPEC_TRY(need_residue(*b, "mul_prev", s.buckets, &s.mul_prev));
    }
  }
  return LCU_OK;
}

int read_mlp(const json_value& layer, layer_spec& l) {
  const json_value* mlp = layer.get("mlp");
  if (!mlp) return LCU_OK;
  const json_value* kind = mlp->get("kind");
  if (kind && kind->text == "moe") {
    const json_value *router = nullptr, *expert = nullptr;
    SPEC_TRY(need(*mlp, "router", json_value::OBJECT, &router));
    SPEC_TRY(need_int(*router, "experts", &l.experts));
    SPEC_TRY(need_int(*router, "top", &l.top));
    LCU_REQUIRE(l.experts <= MAX_EXPERTS, "config.json: %d experts (up to %d)", l.experts, MAX_EXPERTS);
    LCU_REQUIRE(l.top <= l.experts && l.top <= MAX_TOP, "config.json: top %d of %d experts (up to %d)", l.top, l.experts, MAX_TOP);
    SPEC_TRY(need(*mlp, "expert", json_value::OBJECT, &expert));
    return need_int(*expert, "ff", &l.ff);
  }
  LCU_REQUIRE(!kind || kind->text == "dense", "config.json: feed-forward kind '%s' is not known", kind->text.c_str());
  return need_int(*mlp, "ff", &l.ff);
}

// order of layer runs: layers start .. stop-1 run `times` times in a row, the others once
int read_runs(const json_value& c, block_spec& s) {
  const int n = (int)s.layers.size();
  int start = 0, stop = 0, times = 1;
  if (const json_value* loop = c.get("loop")) {
    SPEC_TRY(need_int(*loop, "start", &start, 0));
    SPEC_TRY(need_int(*loop, "stop", &stop, 0));
    SPEC_TRY(need_int(*loop, "times", &times, 0));
    LCU_REQUIRE(start <= stop && stop <= n, "config.json: loop over layers %d..%d of %d", start, stop, n);
  }
  auto add = [&](int layer, bool first) {
    s.runs.push_back(layer);
    s.pass_start.push_back(first);
  };
  for (int i = 0; i < start; ++i) add(i, false);
  for (int t = 0; t < times; ++t)
    for (int i = start; i < stop; ++i) add(i, i == start);
  for (int i = stop; i < n; ++i) add(i, false);
  return LCU_OK;
}

// ---- architectures
// Filulix: window-and-blocks attention beside retention ('parallel'), or a wkv recurrence, per layer; hyper-connected
// residual streams; bigram embedding; looped layers.
int read_filulix(const json_value& c, block_spec& s) {
  SPEC_TRY(read_stack(c, s));
  const json_value* layers = nullptr;
  SPEC_TRY(need(c, "layers", json_value::ARRAY, &layers));
  for (auto& jl : layers->items) {
    layer_spec l;
    const json_value *type = nullptr, *mixer = nullptr;
    SPEC_TRY(need(jl, "type", json_value::STRING, &type));
    SPEC_TRY(need(jl, "mixer", json_value::OBJECT, &mixer));
    if (type->text == "parallel") {
      const json_value *left = nullptr, *right = nullptr;
      SPEC_TRY(need(*mixer, "left", json_value::OBJECT, &left));
      SPEC_TRY(need(*mixer, "right", json_value::OBJECT, &right));
      l.branches.resize(2);
      SPEC_TRY(read_window_attention(*left, l.branches[0]));
      SPEC_TRY(read_retention(*right, l.branches[1]));
      l.branches[0].prefix = "left.";
      l.branches[1].prefix = "right.";
      SPEC_TRY(need_float(*mixer, "left_scale", &l.branches[0].out_scale));
      SPEC_TRY(need_float(*mixer, "right_scale", &l.branches[1].out_scale));
    } else if (type->text == "wkv") {
      l.branches.resize(1);
      SPEC_TRY(read_wkv(*mixer, l.branches[0]));
    } else {
      LCU_REQUIRE(false, "config.json: mixer type '%s' is not known", type->text.c_str());
    }
    SPEC_TRY(read_mlp(jl, l));
    s.layers.push_back(std::move(l));
  }
  return read_runs(c, s);
}

// Zibovik: latent attention with a sink and gated heads, mixture of experts; norms before and after every sublayer, its
// result scaled channel by channel; looped layers that start every pass from the residual and the embedding.
int read_zibovik(const json_value& c, block_spec& s) {
  SPEC_TRY(read_stack(c, s));
  s.sandwich = true;
  s.loop_input = c.get("loop") != nullptr;
  const json_value* layers = nullptr;
  SPEC_TRY(need(c, "layers", json_value::ARRAY, &layers));
  for (auto& jl : layers->items) {
    layer_spec l;
    const json_value *type = nullptr, *mixer = nullptr;
    SPEC_TRY(need(jl, "type", json_value::STRING, &type));
    SPEC_TRY(need(jl, "mixer", json_value::OBJECT, &mixer));
    LCU_REQUIRE(type->text == "latent_attention", "config.json: mixer type '%s' is not known", type->text.c_str());
    l.branches.resize(1);
    SPEC_TRY(read_latent_attention(*mixer, l.branches[0]));
    SPEC_TRY(read_mlp(jl, l));
    s.layers.push_back(std::move(l));
  }
  return read_runs(c, s);
}

const architecture ARCHITECTURES[] = {
    {"Filulix", read_filulix},
    {"Zibovik", read_zibovik},
};

}  // namespace

const architecture* find_architecture(const std::string& name) {
  for (auto& a : ARCHITECTURES)
    if (name == a.name) return &a;
  return nullptr;
}
std::string architecture_names() {
  std::string s;
  for (auto& a : ARCHITECTURES) s += (s.empty() ? "" : ", ") + std::string(a.name);
  return s;
}

int read_block_config(const std::string& text, block_spec& out) {
  json_value c;
  json_reader r(text.data(), text.data() + text.size());
  LCU_REQUIRE(r.parse(c) && c.is(json_value::OBJECT), "config.json: malformed at byte %zu", (size_t)(r.fault_at() - text.data()));
  const json_value* name = nullptr;
  SPEC_TRY(need(c, "architecture", json_value::STRING, &name));
  const architecture* a = find_architecture(name->text);
  LCU_REQUIRE(a != nullptr, "config.json: architecture '%s' is not known (known: %s)", name->text.c_str(), architecture_names().c_str());
  out = block_spec{};
  out.architecture = name->text;
  SPEC_TRY(a->read(c, out));
  LCU_REQUIRE(out.vocab >= 2 && out.vocab <= 32768, "config.json: vocabulary of %d does not fit 16-bit token ids", out.vocab);
  LCU_REQUIRE(out.streams >= 1 && out.streams <= 8, "config.json: %d residual streams (1 to 8)", out.streams);
  LCU_REQUIRE(!out.layers.empty() && !out.runs.empty(), "config.json: no layers");
  for (auto& l : out.layers)
    for (auto& b : l.branches) {
      LCU_REQUIRE(b.dim <= 512 && b.vdim <= 512, "config.json: head size %d x %d (up to 512)", b.dim, b.vdim);
      LCU_REQUIRE(b.kv_rank <= 2048 && b.rot_dim <= 512, "config.json: latent of %d with %d rotated dimensions (up to 2048 and 512)", b.kv_rank, b.rot_dim);
      LCU_REQUIRE(b.kind != BRANCH_WKV || l.branches.size() == 1, "config.json: a wkv mixer does not share its layer");
    }
  return LCU_OK;
}

int read_text_file(const std::string& path, std::string& out) {
  FILE* f = fopen(path.c_str(), "rb");
  if (!f) {
    set_last_error("cannot open %s", path.c_str());
    return LCU_ERR_IO;
  }
  out.clear();
  char buf[65536];
  size_t n;
  while ((n = fread(buf, 1, sizeof buf, f)) > 0) out.append(buf, n);
  const bool bad = ferror(f);
  fclose(f);
  if (bad) {
    set_last_error("cannot read %s", path.c_str());
    return LCU_ERR_IO;
  }
  return LCU_OK;
}

int tensor_file::open(const std::string& p) {
  path = p;
  tensors.clear();
  FILE* f = fopen(p.c_str(), "rb");
  if (!f) {
    set_last_error("cannot open %s", p.c_str());
    return LCU_ERR_IO;
  }
  uint64_t head = 0;
  fseek(f, 0, SEEK_END);
  const long long size = ftell(f);
  fseek(f, 0, SEEK_SET);
  std::string text;
  bool ok = size >= 8 && fread(&head, 8, 1, f) == 1 && head <= (uint64_t)size - 8 && head < (1u << 28);
  if (ok) {
    text.resize(head);
    ok = fread(&text[0], 1, head, f) == head;
  }
  fclose(f);
  if (!ok) {
    set_last_error("%s is not a safetensors file", p.c_str());
    return LCU_ERR_IO;
  }
  file_bytes = (size_t)size;
  json_value h;
  json_reader r(text.data(), text.data() + text.size());
  // (the header may be padded with blanks)
  LCU_REQUIRE(r.parse(h) && h.is(json_value::OBJECT), "%s: malformed header", p.c_str());
  for (auto& m : h.members) {
    if (m.first == "__metadata__") continue;
    tensor_entry t;
    const json_value *dt = m.second.get("dtype"), *sh = m.second.get("shape"), *off = m.second.get("data_offsets");
    LCU_REQUIRE(dt && sh && off && off->items.size() == 2, "%s: malformed entry '%s'", p.c_str(), m.first.c_str());
    t.dtype = dt->text;
    for (auto& d : sh->items) t.shape.push_back((long long)d.number);
    const double lo = off->items[0].number, hi = off->items[1].number;
    LCU_REQUIRE(lo >= 0 && hi >= lo && hi + 8 + (double)head <= (double)file_bytes, "%s: '%s' lies outside the file", p.c_str(), m.first.c_str());
    t.offset = 8 + head + (size_t)lo;
    t.bytes = (size_t)(hi - lo);
    tensors.emplace(m.first, std::move(t));
  }
  return LCU_OK;
}

}  // namespace lcu
