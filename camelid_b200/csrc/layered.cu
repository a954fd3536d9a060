// Layered designs behind the engine: a model described layer by layer (mixer type and sizes, feed-forward), with a
// residual held as several streams or as one with norms on the sublayers' outputs, and, optionally, a run of layers that is
// passed several times.
//
// The engine's own parts stay in charge: the token-driven calls, rows and slots, CUDA graphs of decode steps, argmax
// and sampling (csrc/engine.cu).  This file owns the description, the named tensors, the caches and states, and the
// step: which kernels run for `rows` rows.
//
// Three forms of a step share the kernels between the linear layers:
//   one or two rows    fused matrix-vector products (csrc/lin_mv.cu), 32-bit activations
//   more rows, bf16    tcgen05 products (csrc/lin_tc5.cu), bfloat16 activations, 32-bit residual, norms and scores
//   more rows, f32     FP32 products (csrc/lin_f32.cu)
//
// Cache and state: per layer run (a looped layer counts once per pass) and slot, a latent layer keeps max_pos rows, a
// lightning layer one state, a parallel layer one state and a ring of the window and one step's rows.  A sequence that starts at position 0 starts from nothing, whatever the slot held before;
// any other start must be where the slot's sequence ends, because a state cannot be rewound.
#include <cmath>
#include <cstring>
#include <tuple>

#include "engine.cuh"
#include "layered.cuh"

namespace cmld {

namespace {

struct HyperW {
  float *in = nullptr, *out = nullptr, *mix = nullptr;
};
struct NormW {
  float *w = nullptr, *b = nullptr;
};
struct LayerDef {
  cmld_layer_desc d{};
  // in: the projections that read the mixer's input, stacked; up: with a SwiGLU feed-forward gate and up, row by row in turn
  LinW in, uq, ukv, uk, uv, o, up, down;
  // parallel: output matrices of the branches, the second factor of the decay's projection, bias of `in`
  LinW o_window, o_gated, decay;
  float *in_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *decay_bias = nullptr, *gated_norm = nullptr, *window_out = nullptr, *gated_out = nullptr;
  WindowShape win{};
  int32_t cap = 0;  // positions of the ring
  NormW norm1, norm2;
  float *dq_norm = nullptr, *dkv_norm = nullptr, *mix_norm = nullptr;
  HyperW hc[2];
  float *powers = nullptr, *cs = nullptr;
  LatentShape lat{};
};
struct Named {
  std::string name;
  int64_t rows = 0, cols = 0;  // rows == 0: a vector of cols f32 values (cols may itself be a product)
  bf16 *m = nullptr;           // matrix destination, row stride ld
  int64_t ld = 0;
  float *v = nullptr;
  float add = 0.0f;            // vectors: added to the stored values (norm weights stored around zero)
  bool set = false;
};

constexpr int kLatentRows = 256;    // rows whose queries are in latent space at a time
constexpr int kExpandRows = 32;     // portions of this many rows expand keys and values
constexpr int kTileRows = 16;       // portions of this many rows run the tiled forms of a parallel layer's branches
constexpr int kPortionRows = 2048;  // rows of one step of a portion

// What the last sublayer left behind for the next boundary.
struct Pending {
  const HyperW *hyper = nullptr;     // streams
  const LayerDef *branches = nullptr;  // two results to merge
  const float *out_norm = nullptr;   // norm of the sublayer's output
  bool any = false;
};

}  // namespace

struct LayeredModel {
  cmld_layered_config cfg{};
  bool f32 = false;
  std::vector<LayerDef> layers;
  std::vector<int> order;       // layer of every run
  std::vector<void *> store;    // per run: cache or state
  std::vector<void *> state;    // per run: a parallel layer's state (its cache is in store)
  LinW embed, head;
  NormW embed_norm, final_norm;
  std::vector<Named> named;
  std::vector<int64_t> filled;  // per slot: tokens its sequence holds; -1: a call on it failed half-way
  int64_t part_floats = 0;
  // scratch, f32 unless noted
  float *x[2] = {}, *y = nullptr, *proj = nullptr, *q = nullptr, *qa = nullptr, *part = nullptr, *taps = nullptr;
  void *act = nullptr, *wide = nullptr, *mixed = nullptr, *hidden = nullptr;  // bf16 or f32
  bf16 *kv = nullptr;
  float *y2 = nullptr, *linear_out = nullptr;  // parallel: the second branch's result; what its recurrence gave
  uint8_t *chunks = nullptr;                   // parallel: scratch of the chunked recurrence
  int32_t *row_map = nullptr;
};

namespace {

int64_t cache_ld(const LayerDef &L) { return (L.d.kv_rank + L.d.rot_dim + 7) & ~7; }

struct Builder {
  cmld_engine *e;
  LayeredModel *m;
  int32_t rc = CMLD_OK;
  void matrix(LinW &w, int64_t rows, int64_t cols) {
    if (rc != CMLD_OK) return;
    bf16 *p = nullptr;
    w.rows = (int32_t)rows;
    w.cols = (int32_t)cols;
    w.ld = lin_ld(cols);
    rc = dev_alloc(e, &p, rows * w.ld);  // zeroed: the padding stays zero
    w.w = p;
  }
  // rows [row0, row0 + rows) of w under `name`
  void name_rows(const std::string &name, const LinW &w, int64_t row0, int64_t rows) {
    Named n;
    n.name = name;
    n.rows = rows;
    n.cols = w.cols;
    n.m = const_cast<bf16 *>(w.w) + row0 * w.ld;
    n.ld = w.ld;
    m->named.push_back(n);
  }
  void named_matrix(const std::string &name, LinW &w, int64_t rows, int64_t cols) {
    matrix(w, rows, cols);
    if (rc == CMLD_OK) name_rows(name, w, 0, rows);
  }
  void vector(const std::string &name, float *&v, int64_t n) {
    if (rc != CMLD_OK) return;
    rc = dev_alloc(e, &v, n);
    Named d;
    d.name = name;
    d.cols = n;
    d.v = v;
    m->named.push_back(d);
  }
  // n values of a vector at v under `name`
  void name_values(const std::string &name, float *v, int64_t n) {
    Named d;
    d.name = name;
    d.cols = n;
    d.v = v;
    m->named.push_back(d);
  }
  // every second row of w, from row `first` on, under `name`
  void name_alternate_rows(const std::string &name, const LinW &w, int64_t first) {
    name_rows(name, w, first, w.rows / 2);
    m->named.back().ld = 2 * w.ld;
  }
  bool post_norm() const { return m->cfg.residual == CMLD_RESIDUAL_POST_NORM; }
  void norm(const std::string &name, NormW &n) {
    vector(name, n.w, m->cfg.width);
    if (rc != CMLD_OK) return;
    if (post_norm()) m->named.back().add = 1.0f;
    else vector(name + ".b", n.b, m->cfg.width);
  }
  void hyper(const std::string &name, HyperW &h) {
    if (post_norm()) return;
    vector(name + ".in", h.in, m->cfg.streams);
    vector(name + ".out", h.out, m->cfg.streams);
    vector(name + ".mix", h.mix, (int64_t)m->cfg.streams * m->cfg.streams);
  }
};

WindowShape window_shape(const cmld_window_desc &w, float eps) {
  return WindowShape{w.heads, w.kv_heads, w.dim, w.vdim, w.rot_dims, w.window, w.scale, eps};
}

int32_t check_layer(const cmld_layer_desc &d, int i) {
  if (d.type == CMLD_LAYER_LATENT) {
    const LatentShape s{d.heads, d.dim, d.rot_dim, d.rot_dims, d.vdim, d.kv_rank, d.scale, 0.0f};
    if (d.q_rank < 1 || !latent_shape_ok(s)) return fail(CMLD_ERR_SHAPE, "layer %d: latent attention sizes not supported", i);
    if (d.rot_dims > 0 && !(d.rot_base > 0.0)) return fail(CMLD_ERR_INVALID, "layer %d: rotation base must be positive", i);
  } else if (d.type == CMLD_LAYER_LIGHTNING) {
    if (!lightning_shape_ok(d.heads, d.dim, d.vdim)) return fail(CMLD_ERR_SHAPE, "layer %d: lightning attention sizes not supported", i);
    if (!d.decay) return fail(CMLD_ERR_INVALID, "layer %d: decays are missing", i);
  } else if (d.type == CMLD_LAYER_PARALLEL) {
    const cmld_window_desc &w = d.window;
    const cmld_gated_desc &g = d.gated;
    if (!window_shape_ok(window_shape(w, 0.0f))) return fail(CMLD_ERR_SHAPE, "layer %d: window attention sizes not supported", i);
    if (!gated_shape_ok(g.heads, g.dim, g.vdim, g.rank)) return fail(CMLD_ERR_SHAPE, "layer %d: gated linear attention sizes not supported", i);
    if (w.rot_dims > 0 && !(w.rot_base > 0.0)) return fail(CMLD_ERR_INVALID, "layer %d: rotation base must be positive", i);
    if (w.rot_factor > 0.0 && !(w.rot_original > 0.0 && w.rot_fast > 0.0 && w.rot_slow > 0.0 && w.rot_base > 1.0))
      return fail(CMLD_ERR_INVALID, "layer %d: rotation scaling needs positive constants and a base above 1", i);
    if (!(g.tau > 0.0)) return fail(CMLD_ERR_INVALID, "layer %d: tau must be positive", i);
  } else {
    return fail(CMLD_ERR_UNSUPPORTED, "layer %d: mixer type %d", i, d.type);
  }
  if (d.ff < 0) return fail(CMLD_ERR_SHAPE, "layer %d: feed-forward width %d", i, d.ff);
  if (d.mlp != CMLD_MLP_RELU2 && d.mlp != CMLD_MLP_SWIGLU) return fail(CMLD_ERR_UNSUPPORTED, "layer %d: feed-forward type %d", i, d.mlp);
  return CMLD_OK;
}

// Frequencies of a rotation: base^(-2i / dims), with YaRN scaling (factor > 0) divided by `factor` for the pairs that turn
// less than `slow` times over `original` positions, as they are for those that turn more than `fast` times, mixed in between;
// cosine and sine then carry a factor of 0.1 ln(factor) + 1.
struct Rotation {
  int dims;
  double base, factor, original, fast, slow;
  bool operator<(const Rotation &o) const {
    return std::tie(dims, base, factor, original, fast, slow) < std::tie(o.dims, o.base, o.factor, o.original, o.fast, o.slow);
  }
};

// Cosine and sine of position * frequency, formed in 64-bit on the host: [position][pair][2] in 32-bit.
int32_t rotation_table(cmld_engine *e, int64_t max_pos, const Rotation &r, float **out) {
  const int dims = r.dims, half = dims / 2;
  std::vector<double> f(half);
  std::vector<float> t((size_t)max_pos * dims);
  double lo = 0.0, hi = 0.0, gain = 1.0;
  if (r.factor > 0.0) {
    auto place = [&](double turns) { return dims * std::log(r.original / (2.0 * M_PI * turns)) / (2.0 * std::log(r.base)); };
    lo = std::max(std::floor(place(r.fast)), 0.0);
    hi = std::min(std::ceil(place(r.slow)), dims - 1.0);
    gain = 0.1 * std::log(r.factor) + 1.0;
  }
  for (int i = 0; i < half; ++i) {
    double v = std::pow(r.base, -2.0 * i / dims);
    if (r.factor > 0.0) {
      const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
      v = v / r.factor * ramp + v * (1.0 - ramp);
    }
    f[i] = v;
  }
  for (int64_t p = 0; p < max_pos; ++p)
    for (int i = 0; i < half; ++i) {
      const double a = (double)p * f[i];
      t[(size_t)p * dims + 2 * i] = (float)(gain * std::cos(a));
      t[(size_t)p * dims + 2 * i + 1] = (float)(gain * std::sin(a));
    }
  CMLD_TRY(dev_alloc(e, out, (int64_t)t.size(), false));
  CMLD_CUDA(cudaMemcpyAsync(*out, t.data(), t.size() * 4, cudaMemcpyHostToDevice, e->stream));
  CMLD_CUDA(cudaStreamSynchronize(e->stream));
  return CMLD_OK;
}

int32_t build(cmld_engine *e, LayeredModel *m) {
  const cmld_layered_config &c = m->cfg;
  Builder b{e, m};
  const int64_t slots = std::max(1, c.max_seqs);
  const int64_t R = std::max<int64_t>(slots, std::min<int64_t>(c.max_pos, c.portion > 0 ? c.portion : kPortionRows));  // rows of a step
  b.named_matrix("embed", m->embed, c.vocab, c.width);
  if (!b.post_norm()) b.norm("embed.norm", m->embed_norm);
  std::map<Rotation, float *> tables;
  auto table = [&](const Rotation &r, float **cs) -> int32_t {
    if (r.dims == 0) return CMLD_OK;
    float *&t = tables[r];
    if (!t) CMLD_TRY(rotation_table(e, c.max_pos, r, &t));
    *cs = t;
    return CMLD_OK;
  };
  for (int i = 0; i < c.n_layers; ++i) {
    LayerDef &L = m->layers[i];
    const cmld_layer_desc &d = L.d;
    const std::string p = "l" + std::to_string(i) + ".", mx = p + "mix.";
    const int64_t H = d.heads;
    b.norm(p + "norm1", L.norm1);
    if (d.type == CMLD_LAYER_LATENT) {
      b.matrix(L.in, d.q_rank + d.kv_rank + d.rot_dim + H * d.vdim, c.width);
      b.matrix(L.ukv, H * (d.dim + d.vdim), d.kv_rank);
      CMLD_TRY(b.rc);
      b.name_rows(mx + "dq", L.in, 0, d.q_rank);
      b.name_rows(mx + "dkv", L.in, d.q_rank, d.kv_rank + d.rot_dim);
      b.name_rows(mx + "g", L.in, d.q_rank + d.kv_rank + d.rot_dim, H * d.vdim);
      b.vector(mx + "dq.norm", L.dq_norm, d.q_rank);
      b.vector(mx + "dkv.norm", L.dkv_norm, d.kv_rank);
      b.named_matrix(mx + "uq", L.uq, H * (d.dim + d.rot_dim), d.q_rank);
      b.name_rows(mx + "uk", L.ukv, 0, H * d.dim);
      b.name_rows(mx + "uv", L.ukv, H * d.dim, H * d.vdim);
      L.uk = L.uv = L.ukv;
      L.uk.rows = (int32_t)(H * d.dim);
      L.uv.rows = (int32_t)(H * d.vdim);
      L.uv.w = L.ukv.w + H * d.dim * L.ukv.ld;
      L.lat = LatentShape{d.heads, d.dim, d.rot_dim, d.rot_dims, d.vdim, d.kv_rank, d.scale, c.eps};
      CMLD_TRY(table(Rotation{d.rot_dims, d.rot_base, 0.0, 0.0, 0.0, 0.0}, &L.cs));
    } else if (d.type == CMLD_LAYER_PARALLEL) {
      const cmld_window_desc &w = d.window;
      const cmld_gated_desc &g = d.gated;
      const std::string l = mx + "left.", r = mx + "right.";
      const int64_t wq = (int64_t)w.heads * w.dim, wk = (int64_t)w.kv_heads * w.dim, wv = (int64_t)w.kv_heads * w.vdim, gk = (int64_t)g.heads * g.dim,
                    gv = (int64_t)g.heads * g.vdim;
      b.matrix(L.in, wq + wk + wv + 2 * gk + 2 * gv + g.rank, c.width);
      CMLD_TRY(b.rc);
      CMLD_TRY(dev_alloc(e, &L.in_bias, L.in.rows));
      int64_t at = 0;
      auto part = [&](const std::string &name, int64_t rows, bool bias) {
        b.name_rows(name, L.in, at, rows);
        if (bias) b.name_values(name + ".b", L.in_bias + at, rows);
        at += rows;
      };
      part(l + "q", wq, true);
      part(l + "k", wk, true);
      part(l + "v", wv, true);
      part(r + "q", gk, false);
      part(r + "k", gk, false);
      part(r + "v", gv, false);
      part(r + "g", gv, false);
      part(r + "a1", g.rank, false);
      b.vector(l + "q.norm", L.q_norm, w.dim);
      b.vector(l + "k.norm", L.k_norm, w.dim);
      b.named_matrix(l + "o", L.o_window, c.width, (int64_t)w.heads * w.vdim);
      b.named_matrix(r + "a2", L.decay, gk, g.rank);
      b.vector(r + "a2.b", L.decay_bias, gk);
      b.vector(r + "norm", L.gated_norm, g.vdim);
      b.named_matrix(r + "o", L.o_gated, c.width, gv);
      b.vector(l + "out", L.window_out, c.width);
      b.vector(r + "out", L.gated_out, c.width);
      L.win = window_shape(w, c.eps);
      // every position that a row of a step sees is in the ring when the whole step has been appended
      L.cap = (int32_t)std::min<int64_t>(c.max_pos, w.window > 0 ? (int64_t)w.window - 1 + R : c.max_pos);
      CMLD_TRY(table(Rotation{w.rot_dims, w.rot_base, w.rot_factor, w.rot_original, w.rot_fast, w.rot_slow}, &L.cs));
    } else {
      b.matrix(L.in, H * (2 * d.dim + 2 * d.vdim), c.width);
      CMLD_TRY(b.rc);
      b.name_rows(mx + "q", L.in, 0, H * d.dim);
      b.name_rows(mx + "k", L.in, H * d.dim, H * d.dim);
      b.name_rows(mx + "v", L.in, 2 * H * d.dim, H * d.vdim);
      b.name_rows(mx + "g", L.in, 2 * H * d.dim + H * d.vdim, H * d.vdim);
      b.vector(mx + "norm", L.mix_norm, H * d.vdim);
      std::vector<float> pw((size_t)H * (kLightningChunk + 1));
      for (int h = 0; h < d.heads; ++h)
        for (int j = 0; j <= kLightningChunk; ++j) pw[(size_t)h * (kLightningChunk + 1) + j] = (float)std::pow((double)d.decay[h], (double)j);
      CMLD_TRY(dev_alloc(e, &L.powers, (int64_t)pw.size(), false));
      CMLD_CUDA(cudaMemcpyAsync(L.powers, pw.data(), pw.size() * 4, cudaMemcpyHostToDevice, e->stream));
      CMLD_CUDA(cudaStreamSynchronize(e->stream));
    }
    if (d.type != CMLD_LAYER_PARALLEL) b.named_matrix(mx + "o", L.o, c.width, H * d.vdim);
    b.hyper(p + "hc1", L.hc[0]);
    if (d.ff > 0) {
      b.norm(p + "norm2", L.norm2);
      if (d.mlp == CMLD_MLP_SWIGLU) {
        b.matrix(L.up, 2ll * d.ff, c.width);
        CMLD_TRY(b.rc);
        b.name_alternate_rows(p + "mlp.gate", L.up, 0);
        b.name_alternate_rows(p + "mlp.up", L.up, 1);
      } else {
        b.named_matrix(p + "mlp.up", L.up, d.ff, c.width);
      }
      b.named_matrix(p + "mlp.down", L.down, c.width, d.ff);
      b.hyper(p + "hc2", L.hc[1]);
    }
    L.d.decay = nullptr;  // the caller's memory
    CMLD_TRY(b.rc);
  }
  b.norm("final.norm", m->final_norm);
  b.named_matrix("head", m->head, c.vocab, c.width);
  CMLD_TRY(b.rc);

  // order of runs
  const int times = std::max(1, c.loop_times);
  for (int i = 0; i < c.loop_start; ++i) m->order.push_back(i);
  for (int t = 0; t < times; ++t)
    for (int i = c.loop_start; i < c.loop_stop; ++i) m->order.push_back(i);
  for (int i = c.loop_stop; i < c.n_layers; ++i) m->order.push_back(i);

  // caches and states
  m->filled.assign(slots, 0);
  const int64_t es = m->f32 ? 4 : 2;
  for (int li : m->order) {
    const LayerDef &L = m->layers[li];
    uint8_t *p = nullptr;
    m->state.push_back(nullptr);
    if (L.d.type == CMLD_LAYER_PARALLEL) {
      const cmld_gated_desc &g = L.d.gated;
      CMLD_TRY(dev_alloc(e, &p, slots * L.win.kv_heads * L.cap * (window_pad(L.win.dim) + window_pad(L.win.vdim)) * es));
      m->store.push_back(p);
      CMLD_TRY(dev_alloc(e, &p, slots * g.heads * (int64_t)g.dim * g.vdim * 4));
      m->state.back() = p;
      continue;
    }
    const int64_t bytes = L.d.type == CMLD_LAYER_LATENT ? slots * c.max_pos * cache_ld(L) * es : slots * L.d.heads * (int64_t)L.d.dim * L.d.vdim * 4;
    CMLD_TRY(dev_alloc(e, &p, bytes));
    m->store.push_back(p);
  }

  // scratch for the widest layer
  CMLD_TRY(init_rows(e, R, std::max<int64_t>(slots, 32), c.vocab));
  int64_t proj = 1, q = 1, wide = 1, mixed = 1, ff = 1, kv = 0, qa = 1, part = 1, linear = 0, chunks = 0;
  for (const LayerDef &L : m->layers) {
    const cmld_layer_desc &d = L.d;
    const int64_t H = d.heads;
    ff = std::max(ff, lin_ld(std::max(d.ff, 1)));
    if (d.type == CMLD_LAYER_PARALLEL) {
      const cmld_gated_desc &g = d.gated;
      proj = std::max(proj, lin_ld(L.in.rows));
      q = std::max(q, (int64_t)L.win.heads * window_pad(L.win.dim));
      mixed = std::max(mixed, lin_ld((int64_t)L.win.heads * L.win.vdim));
      wide = std::max(wide, lin_ld((int64_t)g.heads * g.vdim));
      linear = std::max(linear, (int64_t)g.heads * g.vdim);
      if (!m->f32 && gated_chunk_fits(g.dim, g.rank)) chunks = std::max(chunks, gated_scratch_bytes(g.heads, g.dim, g.vdim, R));
      continue;
    }
    mixed = std::max(mixed, lin_ld(H * d.vdim));
    if (d.type == CMLD_LAYER_LATENT) {
      proj = std::max<int64_t>(proj, L.in.rows);
      q = std::max(q, H * (d.dim + d.rot_dim));
      wide = std::max(wide, lin_ld(d.q_rank));
      const int64_t kv_ld = lin_ld(H * (d.dim + d.vdim));
      if (!m->f32 && latent_prefill_fits(L.lat, cache_ld(L), kv_ld)) kv = std::max(kv, kv_ld);
      qa = std::max(qa, H * (d.kv_rank + d.rot_dim));
      part = std::max(part, (int64_t)(2 * e->sm_count * 16 + std::min<int64_t>(R, kLatentRows) * H) * (d.kv_rank + 2));
    } else {
      wide = std::max(wide, lin_ld(L.in.rows));
      proj = std::max<int64_t>(proj, H * d.vdim);
    }
  }
  m->part_floats = part;
  for (float *&x : m->x) CMLD_TRY(dev_alloc(e, &x, R * c.streams * c.width));
  CMLD_TRY(dev_alloc(e, &m->y, R * c.width));
  CMLD_TRY(dev_alloc(e, &m->proj, R * proj));
  CMLD_TRY(dev_alloc(e, &m->q, R * q));
  CMLD_TRY(dev_alloc(e, &m->qa, std::min<int64_t>(R, kLatentRows) * qa));
  CMLD_TRY(dev_alloc(e, &m->part, part));
  float *f = nullptr;  // sized for f32 rows: steps of one or two rows keep 32-bit activations in either precision
  CMLD_TRY(dev_alloc(e, &f, R * lin_ld(c.width)));
  m->act = f;
  CMLD_TRY(dev_alloc(e, &f, R * wide));
  m->wide = f;
  CMLD_TRY(dev_alloc(e, &f, R * mixed));
  m->mixed = f;
  CMLD_TRY(dev_alloc(e, &f, R * ff));
  m->hidden = f;
  if (kv > 0) CMLD_TRY(dev_alloc(e, &m->kv, c.max_pos * kv));
  if (linear > 0) {
    CMLD_TRY(dev_alloc(e, &m->linear_out, R * linear));
    CMLD_TRY(dev_alloc(e, &m->y2, R * c.width));
  }
  if (chunks > 0) CMLD_TRY(dev_alloc(e, &m->chunks, chunks));
  CMLD_TRY(dev_alloc(e, &m->row_map, std::max<int64_t>(slots, 32)));
  CMLD_CUDA(cudaStreamSynchronize(e->stream));
  return CMLD_OK;
}

int32_t validate(const cmld_layered_config &c) {
  if (c.n_layers < 1 || c.streams < 1 || c.width < 1 || c.vocab < 1 || c.max_pos < 1 || !c.layers) return fail(CMLD_ERR_SHAPE, "layered model: dimensions must be positive");
  if (c.max_pos > (1 << 24)) return fail(CMLD_ERR_SHAPE, "max_pos too large");
  if (c.width > 16384) return fail(CMLD_ERR_SHAPE, "width %d, at most 16384", c.width);
  if (c.loop_start < 0 || c.loop_stop < c.loop_start || c.loop_stop > c.n_layers || c.loop_times < 0)
    return fail(CMLD_ERR_INVALID, "loop %d..%d x %d does not fit %d layers", c.loop_start, c.loop_stop, c.loop_times, c.n_layers);
  if (c.residual != CMLD_RESIDUAL_STREAMS && c.residual != CMLD_RESIDUAL_POST_NORM) return fail(CMLD_ERR_UNSUPPORTED, "residual type %d", c.residual);
  if (c.residual == CMLD_RESIDUAL_POST_NORM && c.streams != 1) return fail(CMLD_ERR_INVALID, "norms on the sublayers' outputs go with one stream");
  if (c.portion < 0) return fail(CMLD_ERR_INVALID, "portion of %d rows", c.portion);
  if (c.dtype != CMLD_BF16 && c.dtype != CMLD_F32) return fail(CMLD_ERR_UNSUPPORTED, "layered models compute in bfloat16 or 32-bit");
  for (int i = 0; i < c.n_layers; ++i) {
    CMLD_TRY(check_layer(c.layers[i], i));
    if (c.layers[i].type == CMLD_LAYER_PARALLEL && c.residual != CMLD_RESIDUAL_POST_NORM)
      return fail(CMLD_ERR_UNSUPPORTED, "layer %d: a parallel layer goes with norms on the sublayers' outputs", i);
  }
  return CMLD_OK;
}

// ---------------------------------------------------------------- the step

struct Step {
  cmld_engine *e;
  LayeredModel *m;
  const StepOpts &o;
  int32_t R;
  bool mv, pdl, half;        // matrix-vector form; programmatic dependent launches; bf16 activations
  int cur = 0;
  Pending pending{};

  Pending after_mixer(const LayerDef &L) const { return after(L, 0); }
  Pending after_mlp(const LayerDef &L) const { return after(L, 1); }
  Pending after(const LayerDef &L, int sublayer) const {
    Pending p{};
    p.any = true;
    if (m->cfg.residual == CMLD_RESIDUAL_POST_NORM) {
      p.out_norm = (sublayer ? L.norm2 : L.norm1).w;
      if (!sublayer && L.d.type == CMLD_LAYER_PARALLEL) p.branches = &L;
    } else {
      p.hyper = &L.hc[sublayer];
    }
    return p;
  }
  // the norm in front of a sublayer; a design with norms on the outputs has none
  NormW before(const NormW &n) const { return m->cfg.residual == CMLD_RESIDUAL_POST_NORM ? NormW{} : n; }
  // A step's first kernel starts when the step before it has ended: kernels that look at rows and cache without waiting for
  // their predecessor rely on it.
  bool chained() const { return pdl && pending.any; }

  StreamMix boundary(const float *in, const NormW &n) {
    StreamMix s{};
    s.streams = m->cfg.streams;
    s.width = m->cfg.width;
    s.eps = m->cfg.eps;
    s.in = in;
    s.norm_w = n.w;
    s.norm_b = n.b;
    s.embed_scale = m->cfg.embed_scale != 0.0f ? m->cfg.embed_scale : 1.0f;
    if (!pending.any) {
      s.embed = m->embed.w;
      s.embed_ld = m->embed.ld;
      s.tokens = e->d_tokens;
      s.enorm_w = m->embed_norm.w;
      s.enorm_b = m->embed_norm.b;
    } else {
      s.x_in = m->x[cur];
      s.y = m->y;
      if (pending.hyper) {
        s.mix = pending.hyper->mix;
        s.out = pending.hyper->out;
      }
      s.out_norm = pending.out_norm;
      if (pending.branches) {
        s.y2 = m->y2;
        s.y_norm = pending.branches->window_out;
        s.y2_norm = pending.branches->gated_out;
      }
    }
    s.x_out = m->x[cur ^ 1];
    cur ^= 1;
    return s;
  }
  ActBuf buf(void *p, int64_t cols) const { return ActBuf{p, half ? 1 : 0, lin_ld(cols)}; }

  int32_t vec(LinMvArgs a) {
    a.batch = R;
    e->launches += 1;
    return launch_lin_mv(a, chained() || a.prologue != kProStreams ? pdl : false, e->stream);
  }
  int32_t lin(const LinW &w, ActBuf x, void *out, bool out_half, int64_t out_ld, int act = kActNone, int act_rows = 0, int32_t rows = -1,
              const float *bias = nullptr, float scale = 1.0f) {
    LinArgs a{};
    a.w = w;
    a.x = x.p;
    a.x_ld = x.ld;
    a.rows = rows < 0 ? R : rows;
    a.out = out;
    a.out_half = out_half;
    a.out_ld = out_ld;
    a.act = act;
    a.act_rows = act_rows;
    a.bias = bias;
    a.scale = scale;
    e->launches += 1;
    return x.half ? launch_lin_tc5(a, e->sm_count, e->d_status, pdl, e->stream) : launch_lin_f32(a, e->stream);
  }
  // The sublayer boundary followed by the linear layer that reads it.
  int32_t read_in(const StreamMix &s, const LinW &w, void *out, bool out_half, int64_t out_ld, int act, int act_rows, const float *bias = nullptr) {
    if (mv) {
      LinMvArgs a{};
      a.w = w;
      a.prologue = kProStreams;
      a.mix = s;
      a.y = static_cast<float *>(out);
      a.y_ld = out_ld;
      a.act = act;
      a.act_rows = act_rows;
      a.bias = bias;
      return vec(a);
    }
    const ActBuf h = buf(m->act, m->cfg.width);
    e->launches += 1;
    CMLD_TRY(launch_stream_mix(s, R, h, chained(), e->stream));
    return lin(w, h, out, out_half, out_ld, act, act_rows, -1, bias);
  }
  int32_t vec_plain(const LinW &w, const float *x, int64_t x_ld, float *y, int64_t y_ld) {
    LinMvArgs a{};
    a.w = w;
    a.x = x;
    a.x_ld = x_ld;
    a.y = y;
    a.y_ld = y_ld;
    return vec(a);
  }

  int32_t latent(const LayerDef &L, void *store, const StreamMix &s) {
    const cmld_layer_desc &d = L.d;
    const int64_t pl = L.in.rows, kv0 = d.q_rank, g0 = d.q_rank + d.kv_rank + d.rot_dim, ql = L.uq.rows, ov = (int64_t)d.heads * d.vdim;
    CMLD_TRY(read_in(s, L.in, m->proj, false, pl, kActNone, 0));
    if (mv) {
      LinMvArgs a{};
      a.w = L.uq;
      a.prologue = kProRms;
      a.x = m->proj;
      a.x_ld = pl;
      a.norm_w = L.dq_norm;
      a.eps = m->cfg.eps;
      a.y = m->q;
      a.y_ld = ql;
      CMLD_TRY(vec(a));
    } else {
      const ActBuf cq = buf(m->wide, d.q_rank);
      CMLD_TRY(launch_rms_rows(m->proj, pl, L.dq_norm, d.q_rank, m->cfg.eps, ActBuf{}, cq, R, pdl, e->stream));
      e->launches += 1;
      CMLD_TRY(lin(L.uq, cq, m->q, false, ql));
    }
    LatentArgs a{};
    a.m = L.lat;
    a.cs = L.cs;
    a.cache = store;
    a.cache_half = m->f32 ? 0 : 1;
    a.cache_ld = cache_ld(L);
    a.max_pos = m->cfg.max_pos;
    a.low_ld = pl;
    a.latent_norm = L.dkv_norm;
    a.uk = L.uk;
    a.uv = L.uv;
    a.qa = m->qa;
    a.part = m->part;
    a.gate_ld = pl;
    const ActBuf out = buf(m->mixed, ov);
    const int64_t kv_ld = lin_ld(L.ukv.rows);
    const bool expand = half && o.shared_slots && R >= kExpandRows && latent_prefill_fits(L.lat, a.cache_ld, kv_ld);
    // every row's cache entry goes in before any row attends
    const bool append_first = expand || R > kLatentRows;
    auto rows_from = [&](int r0, int n) {
      a.rows = n;
      a.positions = e->d_positions + r0;
      a.slots = e->d_slots + r0;
      a.low = m->proj + (int64_t)r0 * pl + kv0;
      a.q = m->q + (int64_t)r0 * ql;
      a.gate = m->proj + (int64_t)r0 * pl + g0;
      a.out = out;
      a.out.p = static_cast<uint8_t *>(out.p) + (int64_t)r0 * out.ld * (out.half ? 2 : 4);
    };
    if (append_first) {
      rows_from(0, R);
      CMLD_TRY(launch_latent_prep(a, false, pdl, e->stream));
      e->launches += 1;
    }
    if (expand) {
      const int64_t total = o.seq_start + R;
      const bf16 *c = static_cast<const bf16 *>(store) + (int64_t)o.seq_slot * a.max_pos * a.cache_ld;
      CMLD_TRY(lin(L.ukv, ActBuf{const_cast<bf16 *>(c), 1, a.cache_ld}, m->kv, true, kv_ld, kActNone, 0, (int32_t)total));
      LatentPrefillArgs p{};
      p.m = L.lat;
      p.rows = R;
      p.start = o.seq_start;
      p.cs = L.cs;
      p.cache = c;
      p.cache_ld = a.cache_ld;
      p.kv = m->kv;
      p.kv_ld = kv_ld;
      p.q = m->q;
      p.gate = m->proj + g0;
      p.gate_ld = pl;
      p.out = static_cast<bf16 *>(out.p);
      p.out_ld = out.ld;
      CMLD_TRY(launch_latent_prefill(p, pdl, e->stream));
      e->launches += 1;
    } else {
      const int groups = latent_attention_groups(a);
      const int64_t cap = o.attn_cap > 0 ? o.attn_cap : m->cfg.max_pos;
      for (int r0 = 0; r0 < R; r0 += kLatentRows) {
        const int n = std::min(kLatentRows, R - r0);
        rows_from(r0, n);
        a.splits = (int)std::max<int64_t>(1, std::min<int64_t>({64, (2 * e->sm_count) / (n * groups), cap / 32}));
        if ((int64_t)n * d.heads * a.splits * (d.kv_rank + 2) > m->part_floats) return fail(CMLD_ERR_STATE, "latent attention: partials exceed the scratch");
        CMLD_TRY(launch_latent_prep(a, true, pdl, e->stream));
        CMLD_TRY(launch_latent_attention(a, pdl, e->stream));
        CMLD_TRY(launch_latent_output(a, pdl, e->stream));
        e->launches += 3;
      }
    }
    if (mv) return vec_plain(L.o, static_cast<float *>(out.p), out.ld, m->y, m->cfg.width);
    return lin(L.o, out, m->y, false, m->cfg.width);
  }

  int32_t lightning(const LayerDef &L, void *store, const StreamMix &s) {
    const cmld_layer_desc &d = L.d;
    const int64_t ld = lin_ld(L.in.rows), ov = (int64_t)d.heads * d.vdim, g0 = (int64_t)d.heads * (2 * d.dim + d.vdim);
    CMLD_TRY(read_in(s, L.in, m->wide, half, ld, kActSilu, (int)g0));
    LightningArgs a{};
    a.heads = d.heads;
    a.dim = d.dim;
    a.vdim = d.vdim;
    a.powers = L.powers;
    a.state = static_cast<float *>(store);
    a.qkv = m->wide;
    a.half = half;
    a.ld = ld;
    a.out = m->proj;
    a.positions = e->d_positions;
    a.slots = e->d_slots;
    a.rows = R;
    a.one_sequence = o.shared_slots;
    e->launches += 1;
    if (R >= kLightningChunk / 4 && lightning_chunk_fits(a)) CMLD_TRY(launch_lightning_chunks(a, pdl, e->stream));
    else CMLD_TRY(launch_lightning_steps(a, pdl, e->stream));
    if (mv) {
      LinMvArgs v{};
      v.w = L.o;
      v.prologue = kProRmsGate;
      v.x = m->proj;
      v.x_ld = ov;
      v.norm_w = L.mix_norm;
      v.eps = m->cfg.eps;
      v.gate = static_cast<float *>(m->wide) + g0;
      v.gate_ld = ld;
      v.y = m->y;
      v.y_ld = m->cfg.width;
      return vec(v);
    }
    const ActBuf out = buf(m->mixed, ov);
    ActBuf gate{static_cast<uint8_t *>(m->wide) + g0 * (half ? 2 : 4), half ? 1 : 0, ld};
    CMLD_TRY(launch_rms_rows(m->proj, ov, L.mix_norm, (int)ov, m->cfg.eps, gate, out, R, pdl, e->stream));
    e->launches += 1;
    return lin(L.o, out, m->y, false, m->cfg.width);
  }

  // Sliding-window attention of the rows in m->proj (columns from 0) into m->mixed.
  int32_t window_attention(const LayerDef &L, void *store, int64_t ld, ActBuf out) {
    WindowArgs a{};
    a.m = L.win;
    a.rows = R;
    a.positions = e->d_positions;
    a.slots = e->d_slots;
    a.cs = L.cs;
    a.q_norm = L.q_norm;
    a.k_norm = L.k_norm;
    a.qkv = m->proj;
    a.ld = ld;
    a.cache = store;
    a.cache_half = m->f32 ? 0 : 1;
    a.cap = L.cap;
    a.q = m->q;
    a.out = out;
    const bool tiled = half && o.shared_slots && R >= kTileRows;
    a.q_half = tiled ? 1 : 0;
    if (tiled && window_prefill_fits(a)) {
      e->launches += 2;
      CMLD_TRY(launch_window_prep(a, true, pdl, e->stream));
      return launch_window_prefill(a, pdl, e->stream);
    }
    a.q_half = 0;
    if (!window_decode_fits(a)) {
      e->launches += 2;
      CMLD_TRY(launch_window_prep(a, true, pdl, e->stream));
      return launch_window_attention(a, pdl, e->stream);
    }
    // rows of one sequence see one another: their keys and values go in first
    a.append = o.shared_slots ? 0 : 1;
    if (!a.append) {
      CMLD_TRY(launch_window_prep(a, false, pdl, e->stream));
      e->launches += 1;
    }
    const int64_t ctx = o.attn_cap > 0 ? o.attn_cap : m->cfg.max_pos, seen = L.win.window > 0 ? std::min<int64_t>(ctx, L.win.window) : ctx;
    const int64_t ctas = (int64_t)R * window_decode_groups(a);
    while (a.splits < 8 && ctas * a.splits * 2 <= e->sm_count && seen >= 256 * a.splits) a.splits *= 2;
    e->launches += 1;
    return launch_window_decode(a, pdl, e->stream);
  }

  // Gated linear attention of the rows in m->proj (columns from `at`) into m->linear_out.
  int32_t gated_linear(const LayerDef &L, void *state, int64_t ld, int64_t at) {
    const cmld_gated_desc &g = L.d.gated;
    const int64_t gk = (int64_t)g.heads * g.dim, gv = (int64_t)g.heads * g.vdim;
    LightningArgs a{};
    a.heads = g.heads;
    a.dim = g.dim;
    a.vdim = g.vdim;
    a.channel.w = L.decay;
    a.channel.b = L.decay_bias;
    a.channel.x = m->proj + at + 2 * gk + 2 * gv;
    a.channel.inv_tau = (float)(1.0 / g.tau);
    a.q_scale = (float)(1.0 / std::sqrt((double)g.dim));
    a.state = static_cast<float *>(state);
    a.qkv = m->proj + at;
    a.ld = ld;
    a.out = m->linear_out;
    a.positions = e->d_positions;
    a.slots = e->d_slots;
    a.rows = R;
    a.one_sequence = o.shared_slots;
    // the attention before it waits for the projections and lets this kernel start only then: both run side by side
    a.late_wait = 1;
    if (half && o.shared_slots && R >= kTileRows && gated_chunk_fits(g.dim, g.rank)) {
      e->launches += 2;
      return launch_gated_chunks(a, m->chunks, pdl, e->stream);
    }
    e->launches += 1;
    return launch_lightning_steps(a, pdl, e->stream);
  }

  int32_t parallel(const LayerDef &L, void *store, void *state, const StreamMix &s) {
    const cmld_gated_desc &g = L.d.gated;
    const int64_t pl = lin_ld(L.in.rows), wv = (int64_t)L.win.heads * L.win.vdim, gv = (int64_t)g.heads * g.vdim, gk = (int64_t)g.heads * g.dim;
    const int64_t at = (int64_t)(L.win.heads + L.win.kv_heads) * L.win.dim + (int64_t)L.win.kv_heads * L.win.vdim;
    const float *gate = m->proj + at + 2 * gk + gv;
    CMLD_TRY(read_in(s, L.in, m->proj, false, pl, kActNone, 0, L.in_bias));
    const ActBuf left = buf(m->mixed, wv), right = buf(m->wide, gv);
    CMLD_TRY(window_attention(L, store, pl, left));
    CMLD_TRY(gated_linear(L, state, pl, at));
    if (mv) {
      LinMvArgs a{}, b{};
      a.w = L.o_window;
      a.x = static_cast<float *>(left.p);
      a.x_ld = left.ld;
      a.y = m->y;
      b.w = L.o_gated;
      b.prologue = kProRmsGroups;
      b.group = g.vdim;
      b.x = m->linear_out;
      b.x_ld = gv;
      b.norm_w = L.gated_norm;
      b.eps = m->cfg.eps;
      b.gate = gate;
      b.gate_ld = pl;
      b.y = m->y2;
      a.y_ld = b.y_ld = m->cfg.width;
      a.batch = b.batch = R;
      e->launches += 1;
      return launch_lin_mv_pair(a, b, pdl, e->stream);
    }
    e->launches += 1;
    CMLD_TRY(launch_rms_groups(m->linear_out, gv, L.gated_norm, (int)gv, g.vdim, m->cfg.eps, gate, pl, right, R, pdl, e->stream));
    CMLD_TRY(lin(L.o_window, left, m->y, false, m->cfg.width));
    return lin(L.o_gated, right, m->y2, false, m->cfg.width);
  }

  int32_t mlp(const LayerDef &L, const StreamMix &s) {
    const ActBuf h = buf(m->hidden, L.d.ff);
    CMLD_TRY(read_in(s, L.up, h.p, half, h.ld, L.d.mlp == CMLD_MLP_SWIGLU ? kActSwiGlu : kActRelu2, 0));
    if (mv) return vec_plain(L.down, static_cast<float *>(h.p), h.ld, m->y, m->cfg.width);
    return lin(L.down, h, m->y, false, m->cfg.width);
  }

  int32_t head() {
    StreamMix s = boundary(nullptr, m->final_norm);
    s.x_out = nullptr;
    const float scale = m->cfg.logit_scale != 0.0f ? m->cfg.logit_scale : 1.0f;
    const int32_t n = o.n_want < 0 ? R : o.n_want;
    if (o.n_want >= 0) s.row_map = m->row_map;
    if (n <= 2 && lin_mv_fits(m->cfg.width, n)) {
      LinMvArgs a{};
      a.w = m->head;
      a.batch = n;
      a.prologue = kProStreams;
      a.mix = s;
      a.y = e->logits;
      a.y_ld = m->cfg.vocab;
      a.scale = scale;
      e->launches += 1;
      return launch_lin_mv(a, pdl, e->stream);
    }
    const ActBuf h{m->act, m->f32 ? 0 : 1, lin_ld(m->cfg.width)};
    CMLD_TRY(launch_stream_mix(s, n, h, pdl, e->stream));
    e->launches += 1;
    return lin(m->head, h, e->logits, false, m->cfg.vocab, kActNone, 0, n, nullptr, scale);
  }
};

bool all_fit_mv(const LayeredModel *m, int32_t R) {
  if (!lin_mv_fits(m->cfg.width, R)) return false;
  for (const LayerDef &L : m->layers)
    for (int64_t cols : {(int64_t)L.d.heads * L.d.vdim, (int64_t)L.d.ff, (int64_t)L.d.q_rank, (int64_t)L.o_window.cols, (int64_t)L.o_gated.cols})
      if (cols > 0 && !lin_mv_fits((int32_t)cols, R)) return false;
  return true;
}

}  // namespace

int32_t layered_step(cmld_engine *e, const StepOpts &o) {
  LayeredModel *m = e->lay;
  const int32_t R = o.batch;
  if (R < 1 || R > e->max_rows) return fail(CMLD_ERR_INVALID, "step of %d rows exceeds the engine's %d", R, e->max_rows);
  const int32_t n_logits = !o.logits ? 0 : o.n_want < 0 ? R : o.n_want;
  if (n_logits > e->logit_rows) return fail(CMLD_ERR_INVALID, "logits of %d rows exceed the engine's %d", n_logits, e->logit_rows);
  const bool mv = all_fit_mv(m, R);
  Step st{e, m, o, R, mv, !(e->cfg.flags & CMLD_FLAG_NO_PDL), !mv && !m->f32};
  const int64_t W = m->cfg.width;
  for (size_t run = 0; run < m->order.size(); ++run) {
    const LayerDef &L = m->layers[m->order[run]];
    const StreamMix s = st.boundary(L.hc[0].in, st.before(L.norm1));
    switch (L.d.type) {
      case CMLD_LAYER_LATENT: CMLD_TRY(st.latent(L, m->store[run], s)); break;
      case CMLD_LAYER_LIGHTNING: CMLD_TRY(st.lightning(L, m->store[run], s)); break;
      default: CMLD_TRY(st.parallel(L, m->store[run], m->state[run], s)); break;
    }
    st.pending = st.after_mixer(L);
    if (L.d.ff > 0) {
      CMLD_TRY(st.mlp(L, st.boundary(L.hc[1].in, st.before(L.norm2))));
      st.pending = st.after_mlp(L);
    }
    if (o.taps_out) {
      const int cur = st.cur;
      StreamMix t = st.boundary(nullptr, NormW{});
      t.x_out = nullptr;
      st.cur = cur;
      CMLD_TRY(launch_stream_tap(t, R, o.taps_out + (int64_t)run * R * W, e->stream));
    }
  }
  if (n_logits > 0) {
    CMLD_TRY(st.head());
    if (o.argmax) {
      CMLD_TRY(launch_argmax(e->logits, m->cfg.vocab, n_logits, e->am_val, e->am_idx, e->am_ticket, e->out_idx, o.feed_back ? e->d_tokens : nullptr,
                             e->d_positions, e->d_history, e->stream));
      e->launches += 1;
    }
  }
  return CMLD_OK;
}

int32_t layered_ready(const cmld_engine *e, bool report) {
  for (const Named &n : e->lay->named)
    if (!n.set) {
      if (report) fail(CMLD_ERR_STATE, "tensor %s is not set", n.name.c_str());
      return 0;
    }
  return 1;
}

// Before a call touches the rows' slots: each row starts a sequence (position 0) or continues the slot's, one row per slot.
int32_t layered_claim(cmld_engine *e, int32_t n, const int32_t *seqs, const int64_t *positions) {
  LayeredModel *m = e->lay;
  for (int i = 0; i < n; ++i) {
    for (int j = 0; j < i; ++j)
      if (seqs[i] == seqs[j]) return fail(CMLD_ERR_INVALID, "slot %d appears twice in a step (use cmld_engine_extend for several tokens of a sequence)", seqs[i]);
    if (positions[i] != 0 && m->filled[seqs[i]] != positions[i])
      return fail(CMLD_ERR_STATE, "slot %d holds %lld tokens: its sequence cannot continue at position %lld", seqs[i], (long long)m->filled[seqs[i]],
                  (long long)positions[i]);
  }
  for (int i = 0; i < n; ++i) m->filled[seqs[i]] = -1;  // until the call has succeeded
  return CMLD_OK;
}

void layered_advance(cmld_engine *e, int32_t n, const int32_t *seqs, const int64_t *positions, int64_t steps) {
  for (int i = 0; i < n; ++i) e->lay->filled[seqs[i]] = positions[i] + steps;
}

int32_t layered_extend(cmld_engine *e, int32_t seq, const int32_t *tokens, int64_t n, int64_t start, const int32_t *want, int32_t n_want,
                       float *logits_out, float *taps_out) {
  LayeredModel *m = e->lay;
  const cmld_layered_config &c = m->cfg;
  if (seq < 0 || seq >= (int32_t)m->filled.size()) return fail(CMLD_ERR_INVALID, "sequence slot %d out of range (max_seqs %zu)", seq, m->filled.size());
  if (start < 0 || start + n > c.max_pos) return fail(CMLD_ERR_STATE, "positions %lld..%lld exceed max_pos %d", (long long)start, (long long)(start + n - 1), c.max_pos);
  for (int64_t i = 0; i < n; ++i)
    if (tokens[i] < 0 || tokens[i] >= c.vocab) return fail(CMLD_ERR_INVALID, "token id %d out of range", tokens[i]);
  CMLD_TRY(layered_claim(e, 1, &seq, &start));
  const int64_t runs = (int64_t)m->order.size();
  int32_t w = 0;
  for (int64_t i = 0; i < n; i += e->max_rows) {
    const int rows = (int)std::min<int64_t>(e->max_rows, n - i);
    std::vector<int32_t> pos(rows), slots(rows, seq);
    for (int r = 0; r < rows; ++r) pos[r] = (int32_t)(start + i + r);
    CMLD_TRY(stage_rows(e, rows, tokens + i, pos.data(), slots.data()));
    StepOpts o;
    o.batch = rows;
    o.shared_slots = rows > 1;
    o.from_tokens = true;
    o.seq_start = start + i;
    o.seq_slot = seq;
    o.attn_cap = 512;
    while (o.attn_cap <= start + i + rows - 1) o.attn_cap *= 2;
    float *taps = nullptr;
    if (taps_out) {
      CMLD_CUDA(cudaMalloc(&taps, (size_t)runs * rows * c.width * 4));
      o.taps_out = taps;
    }
    // The rows whose logits are wanted, as many at a time as the logits buffer holds; after the last token always its own.
    const bool last = i + rows >= n;
    std::vector<int32_t> ask;
    while (w + (int32_t)ask.size() < n_want && want[w + ask.size()] < i + rows) ask.push_back((int32_t)(want[w + ask.size()] - i));
    const int32_t live = (int32_t)ask.size();
    if (last && (ask.empty() || ask.back() != rows - 1)) ask.push_back(rows - 1);
    if (rows == 1 && !taps && last) {
      // the shape of a decode step, and its graph
      CMLD_TRY(run_step(e, o));
      e->last_logit_row = 0;
      if (live) CMLD_CUDA(cudaMemcpyAsync(logits_out + (int64_t)w * c.vocab, e->logits, (size_t)c.vocab * 4, cudaMemcpyDeviceToHost, e->stream));
    } else {
      o.logits = false;
      int32_t rc = layered_step(e, o);
      // the stream after the last layer is still in place: read it out for the rows asked for
      Step st{e, m, o, rows, all_fit_mv(m, rows), !(e->cfg.flags & CMLD_FLAG_NO_PDL), false};
      int flips = 0;
      for (int li : m->order) flips += m->layers[li].d.ff > 0 ? 2 : 1;
      const LayerDef &tail = m->layers[m->order.back()];
      for (size_t a = 0; a < ask.size() && rc == CMLD_OK; a += e->logit_rows) {
        const int32_t k = (int32_t)std::min<size_t>(e->logit_rows, ask.size() - a);
        cudaError_t ce = cudaMemcpyAsync(m->row_map, ask.data() + a, (size_t)k * 4, cudaMemcpyHostToDevice, e->stream);
        o.n_want = k;
        st.pending = tail.d.ff > 0 ? st.after_mlp(tail) : st.after_mixer(tail);
        st.cur = flips & 1;
        if (ce == cudaSuccess) rc = st.head();
        if (rc == CMLD_OK && ce == cudaSuccess)
          rc = launch_argmax(e->logits, c.vocab, k, e->am_val, e->am_idx, e->am_ticket, e->out_idx, nullptr, e->d_positions, e->d_history, e->stream);
        const int32_t give = std::max(0, std::min<int32_t>(k, live - (int32_t)a));
        if (rc == CMLD_OK && ce == cudaSuccess && give > 0)
          ce = cudaMemcpyAsync(logits_out + (int64_t)(w + a) * c.vocab, e->logits, (size_t)give * c.vocab * 4, cudaMemcpyDeviceToHost, e->stream);
        if (ce != cudaSuccess) rc = fail(CMLD_ERR_CUDA, "extend: %s", cudaGetErrorString(ce));
        e->launches += 1;
        e->last_logit_row = k - 1;
      }
      if (taps && rc == CMLD_OK) {
        for (int64_t r = 0; r < runs && rc == CMLD_OK; ++r)
          if (cudaMemcpyAsync(taps_out + (r * n + i) * c.width, taps + r * rows * c.width, (size_t)rows * c.width * 4, cudaMemcpyDeviceToHost, e->stream) != cudaSuccess)
            rc = fail(CMLD_ERR_CUDA, "extend: copying the residual stream failed");
      }
      if (taps) {
        cudaStreamSynchronize(e->stream);
        cudaFree(taps);
      }
      CMLD_TRY(rc);
    }
    w += live;
  }
  return CMLD_OK;
}

void layered_free(cmld_engine *e) {
  delete e->lay;
  e->lay = nullptr;
}

// f32 or bfloat16 values -> a padded bfloat16 matrix, or an f32 vector
__global__ void named_from_f32_kernel(const float *src, int64_t rows, int64_t cols, bf16 *m, int64_t ld, float *v, float mean, float add) {
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < rows * cols; i += (int64_t)gridDim.x * blockDim.x) {
    if (m) m[i / cols * ld + i % cols] = __float2bfloat16_rn(src[i] + mean);
    else v[i] = __bfloat162float(__float2bfloat16_rn(src[i] + mean)) + add;
  }
}

static Named *find_named(cmld_engine *e, const char *name) {
  for (Named &n : e->lay->named)
    if (n.name == name) return &n;
  return nullptr;
}

}  // namespace cmld

using namespace cmld;

extern "C" {

int32_t cmld_engine_create_layered(const cmld_layered_config *cfg, cmld_engine **out) {
  if (!cfg || !out) return fail(CMLD_ERR_INVALID, "config or out pointer is null");
  *out = nullptr;
  CMLD_TRY(validate(*cfg));
  int ndev = 0;
  if (cudaGetDeviceCount(&ndev) != cudaSuccess || ndev == 0) {
    cudaGetLastError();
    return fail(CMLD_ERR_CUDA, "no CUDA device: this engine has no CPU path");
  }
  int dev = cfg->device;
  if (dev < 0) CMLD_CUDA(cudaGetDevice(&dev));
  if (dev >= ndev) return fail(CMLD_ERR_INVALID, "device %d out of range (%d present)", dev, ndev);
  cudaDeviceProp prop{};
  CMLD_CUDA(cudaGetDeviceProperties(&prop, dev));
  if (prop.major != 10) return fail(CMLD_ERR_UNSUPPORTED, "device %d is sm_%d%d; this library is built for sm_100a only", dev, prop.major, prop.minor);
  DeviceGuard guard(dev);
  if (!guard.ok) return fail(CMLD_ERR_CUDA, "cannot select CUDA device %d", dev);
  cmld_engine *e = new cmld_engine();
  e->lay = new LayeredModel();
  e->lay->cfg = *cfg;
  e->lay->f32 = cfg->dtype == CMLD_F32;
  e->lay->layers.resize(cfg->n_layers);
  for (int i = 0; i < cfg->n_layers; ++i) e->lay->layers[i].d = cfg->layers[i];
  e->lay->cfg.layers = nullptr;
  e->cfg.n_layers = cfg->n_layers;
  e->cfg.hidden = cfg->width;
  e->cfg.head_dim = 1;
  e->cfg.vocab = cfg->vocab;
  e->cfg.max_pos = cfg->max_pos;
  e->cfg.max_seqs = std::max(1, cfg->max_seqs);
  e->cfg.eps = cfg->eps;
  e->cfg.flags = cfg->flags;
  e->full = e->cfg;
  e->vocab_local = cfg->vocab;
  e->device = dev;
  int32_t rc = engine_open(e, dev);
  if (rc == CMLD_OK) rc = build(e, e->lay);
  if (rc != CMLD_OK) {
    cmld_engine_destroy(e);
    return rc;
  }
  *out = e;
  return CMLD_OK;
}

int32_t cmld_engine_named_count(const cmld_engine *e) { return e && e->lay ? (int32_t)e->lay->named.size() : 0; }

int32_t cmld_engine_named_info(const cmld_engine *e, int32_t i, const char **name, int64_t *rows, int64_t *cols) {
  if (!e || !e->lay || i < 0 || i >= (int32_t)e->lay->named.size() || !name || !rows || !cols) return fail(CMLD_ERR_INVALID, "named_info: bad argument");
  const Named &n = e->lay->named[i];
  *name = n.name.c_str();
  *rows = n.rows;
  *cols = n.cols;
  return CMLD_OK;
}

int32_t cmld_engine_set_named(cmld_engine *e, const char *name, int32_t dtype, const void *data, uint64_t nbytes) {
  CMLD_ENGINE_ENTER(e);
  if (!e->lay) return fail(CMLD_ERR_UNSUPPORTED, "set_named: a llama-shaped engine takes its weights by layer");
  if (!name || !data) return fail(CMLD_ERR_INVALID, "set_named: null argument");
  Named *n = find_named(e, name);
  if (!n) return fail(CMLD_ERR_INVALID, "set_named: this model has no tensor %s", name);
  const int64_t rows = std::max<int64_t>(1, n->rows), count = rows * n->cols, es = dtype == CMLD_F32 ? 4 : 2;
  if (dtype != CMLD_BF16 && dtype != CMLD_F32) return fail(CMLD_ERR_UNSUPPORTED, "set_named(%s): type %d", name, dtype);
  if ((int64_t)nbytes != count * es)
    return fail(CMLD_ERR_SHAPE, "set_named(%s): %lld x %lld values need %lld bytes, got %llu", name, (long long)rows, (long long)n->cols, (long long)(count * es),
                (unsigned long long)nbytes);
  if (n->m && dtype == CMLD_BF16) {
    CMLD_CUDA(cudaMemcpy2DAsync(n->m, (size_t)n->ld * 2, data, (size_t)n->cols * 2, (size_t)n->cols * 2, (size_t)rows, cudaMemcpyDefault, e->stream));
  } else if (n->m) {
    return fail(CMLD_ERR_UNSUPPORTED, "set_named(%s): matrices are bfloat16", name);
  } else {
    std::vector<float> f(count);
    if (dtype == CMLD_F32) {
      CMLD_CUDA(cudaMemcpy(f.data(), data, (size_t)count * 4, cudaMemcpyDefault));
    } else {
      std::vector<uint16_t> h(count);
      CMLD_CUDA(cudaMemcpy(h.data(), data, (size_t)count * 2, cudaMemcpyDefault));
      for (int64_t i = 0; i < count; ++i) {
        const uint32_t u = (uint32_t)h[i] << 16;
        memcpy(&f[i], &u, 4);
      }
    }
    if (n->add != 0.0f)
      for (float &v : f) v += n->add;
    CMLD_CUDA(cudaMemcpyAsync(n->v, f.data(), (size_t)count * 4, cudaMemcpyHostToDevice, e->stream));
    CMLD_CUDA(cudaStreamSynchronize(e->stream));
  }
  CMLD_CUDA(cudaStreamSynchronize(e->stream));
  n->set = true;
  return CMLD_OK;
}

int32_t cmld_engine_synth_named(cmld_engine *e, const char *name, uint64_t seed, uint64_t stream, float mean, float sigma) {
  CMLD_ENGINE_ENTER(e);
  if (!e->lay || !name) return fail(CMLD_ERR_INVALID, "synth_named: bad argument");
  Named *n = find_named(e, name);
  if (!n) return fail(CMLD_ERR_INVALID, "synth_named: this model has no tensor %s", name);
  const int64_t rows = std::max<int64_t>(1, n->rows);
  // 64 Mi values at a time through an f32 slab
  const int64_t slab = std::max<int64_t>(1, std::min<int64_t>(rows, (64ll << 20) / n->cols));
  Weight w;
  CMLD_TRY(weight_alloc(w, CMLD_F32, slab, n->cols));
  int32_t rc = CMLD_OK;
  for (int64_t r0 = 0; r0 < rows && rc == CMLD_OK; r0 += slab) {
    w.rows = std::min(slab, rows - r0);
    rc = launch_synth(w, seed, stream, r0, sigma, e->stream);
    if (rc != CMLD_OK) break;
    named_from_f32_kernel<<<1024, 256, 0, e->stream>>>(reinterpret_cast<const float *>(w.data), w.rows, n->cols, n->m ? n->m + r0 * n->ld : nullptr, n->ld,
                                                       n->v, mean, n->add);
    if (cudaGetLastError() != cudaSuccess || cudaStreamSynchronize(e->stream) != cudaSuccess) rc = fail(CMLD_ERR_CUDA, "synth_named failed");
  }
  weight_free(w);
  if (rc == CMLD_OK) n->set = true;
  return rc;
}

int32_t cmld_linear(int32_t kernel, const void *w_dev, int64_t rows, int64_t cols, const void *x_dev, int32_t n, void *out_dev, int32_t out_bf16,
                    int32_t act, int32_t act_rows, const float *bias_dev, float scale, int32_t n_copies, int32_t iters, float *ms_out) {
  if (!w_dev || !x_dev || !out_dev || rows < 1 || cols < 1 || n < 1) return fail(CMLD_ERR_INVALID, "linear: bad argument");
  if (kernel < 0 || kernel > 2 || (kernel == 0 && (out_bf16 || !lin_mv_fits((int32_t)cols, n)))) return fail(CMLD_ERR_SHAPE, "linear: the kernel does not take this");
  cudaStream_t s = nullptr;
  int32_t *status = nullptr;
  CMLD_CUDA(cudaStreamCreateWithFlags(&s, cudaStreamNonBlocking));
  int32_t rc = CMLD_OK;
  cudaGraph_t graph = nullptr;
  cudaGraphExec_t exec = nullptr;
  cudaEvent_t e0 = nullptr, e1 = nullptr;
  auto cuda = [&](cudaError_t ce) {
    if (rc == CMLD_OK && ce != cudaSuccess) rc = fail(CMLD_ERR_CUDA, "linear: %s", cudaGetErrorString(ce));
  };
  cuda(cudaMalloc(&status, 4));
  if (rc == CMLD_OK) cuda(cudaMemsetAsync(status, 0, 4, s));
  int sms = 148, dev = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  auto once = [&](int i, bool pdl) -> int32_t {
    const int64_t ld = lin_ld(cols);
    const LinW w{static_cast<const bf16 *>(w_dev) + (int64_t)(i % std::max(1, n_copies)) * rows * ld, (int32_t)rows, (int32_t)cols, ld};
    if (kernel == 0) {
      LinMvArgs a{};
      a.w = w;
      a.batch = n;
      a.x = static_cast<const float *>(x_dev);
      a.x_ld = ld;
      a.y = static_cast<float *>(out_dev);
      a.y_ld = lin_outputs(rows, act);
      a.act = act;
      a.act_rows = act_rows;
      a.bias = bias_dev;
      a.scale = scale;
      return launch_lin_mv(a, pdl, s);
    }
    LinArgs a{};
    a.w = w;
    a.x = x_dev;
    a.x_ld = ld;
    a.rows = n;
    a.out = out_dev;
    a.out_half = out_bf16;
    a.out_ld = lin_outputs(rows, act);
    a.act = act;
    a.act_rows = act_rows;
    a.bias = bias_dev;
    a.scale = scale;
    return kernel == 1 ? launch_lin_tc5(a, sms, status, pdl, s) : launch_lin_f32(a, s);
  };
  if (rc == CMLD_OK) rc = once(0, false);
  if (rc == CMLD_OK && iters > 0) {
    cuda(cudaEventCreate(&e0));
    cuda(cudaEventCreate(&e1));
    for (int i = 0; i < 3 && rc == CMLD_OK; ++i) rc = once(i, true);
    cuda(cudaStreamBeginCapture(s, cudaStreamCaptureModeThreadLocal));
    for (int i = 0; i < iters && rc == CMLD_OK; ++i) rc = once(i, true);
    cuda(cudaStreamEndCapture(s, &graph));
    if (rc == CMLD_OK) cuda(cudaGraphInstantiate(&exec, graph, 0));
    for (int i = 0; i < 2 && rc == CMLD_OK; ++i) {  // the first replay warms up
      cuda(cudaEventRecord(e0, s));
      cuda(cudaGraphLaunch(exec, s));
      cuda(cudaEventRecord(e1, s));
      cuda(cudaStreamSynchronize(s));
    }
    float ms = 0.0f;
    if (rc == CMLD_OK) cuda(cudaEventElapsedTime(&ms, e0, e1));
    if (ms_out) *ms_out = ms / (float)iters;
  }
  int32_t st = 0;
  if (rc == CMLD_OK) {
    cuda(cudaMemcpyAsync(&st, status, 4, cudaMemcpyDeviceToHost, s));
    cuda(cudaStreamSynchronize(s));
    if (rc == CMLD_OK && st != 0) rc = fail(st, "linear: a bounded device-side wait gave up");
  }
  if (exec) cudaGraphExecDestroy(exec);
  if (graph) cudaGraphDestroy(graph);
  if (e0) cudaEventDestroy(e0);
  if (e1) cudaEventDestroy(e1);
  cudaFree(status);
  cudaStreamDestroy(s);
  return rc;
}

int32_t cmld_engine_slot_filled(const cmld_engine *e, int32_t slot, int64_t *tokens) {
  if (!e || !e->lay || !tokens) return fail(CMLD_ERR_INVALID, "slot_filled: bad argument");
  if (slot < 0 || slot >= (int32_t)e->lay->filled.size()) return fail(CMLD_ERR_INVALID, "sequence slot %d out of range", slot);
  *tokens = e->lay->filled[slot];
  return CMLD_OK;
}

}  // extern "C"
