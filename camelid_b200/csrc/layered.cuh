// Building blocks of layered models: designs described layer by layer (mixer type, sizes, feed-forward) instead of by
// the one llama shape.  Weights are bfloat16 matrices; activations are bfloat16 or 32-bit, sums always 32-bit.
// One launcher per mechanism, its sizes and constants as arguments; csrc/layered.cu strings them together.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace cmld {

typedef __nv_bfloat16 bf16;

// A bfloat16 matrix [rows][cols], row stride ld elements (a multiple of 8; the padding is zero).
struct LinW {
  const bf16 *w = nullptr;
  int32_t rows = 0, cols = 0;
  int64_t ld = 0;
};
inline int64_t lin_ld(int64_t cols) { return (cols + 7) & ~int64_t(7); }

// Activation rows: bf16 (half = 1) or f32.
struct ActBuf {
  void *p = nullptr;
  int32_t half = 0;
  int64_t ld = 0;  // elements
};

// What a linear layer does to its sums: SiLU on output rows below act_rows, the square of ReLU on all, SiLU of an even row's
// sum times the sum of the next row (half as many outputs as rows), or nothing.
enum LinAct { kActNone = 0, kActSilu = 1, kActRelu2 = 2, kActSwiGlu = 3 };
inline int64_t lin_outputs(int64_t rows, int act) { return act == kActSwiGlu ? rows / 2 : rows; }

// One boundary between two sublayers: the update of the residual with what the sublayer has just produced, then the read-out
// and norm that feed the next one.
//   y' = y, or 0.5 (rms(y) y_norm + rms(y2) y2_norm) where two branches ran side by side; with out_norm: y' <- rms(y') out_norm
//   several copies of the residual (hyper-connections):
//     x'_t = sum_s mix[s][t] x_s + out[t] y';   u = sum_t in[t] x'_t (in == null: the plain sum)
//   mix == null: one stream, u = x' = x + y'
//   result = LN(u) (norm_w and norm_b), rms(u) norm_w (norm_w alone), or u
// embed != null: the first boundary instead: x' = embed_scale * embed[token], layer-normed with enorm_w, in every stream.
// All of it in 32-bit.
struct StreamMix {
  const float *x_in = nullptr;  // [row][streams][width]
  float *x_out = nullptr;       // same layout, another buffer; null: the updated streams are not kept
  const float *y = nullptr;     // [row][width]
  const float *y2 = nullptr, *y_norm = nullptr, *y2_norm = nullptr, *out_norm = nullptr;  // mix == null only
  const float *mix = nullptr, *out = nullptr, *in = nullptr;
  const float *norm_w = nullptr, *norm_b = nullptr;
  float eps = 0.0f, embed_scale = 1.0f;
  const bf16 *embed = nullptr;
  int64_t embed_ld = 0;
  const int32_t *tokens = nullptr;
  const float *enorm_w = nullptr, *enorm_b = nullptr;  // null: no norm
  int32_t streams = 1, width = 0;
  const int32_t *row_map = nullptr;  // result row r comes from row row_map[r]; null: r
};

// stream_mix.cu
int32_t launch_stream_mix(const StreamMix &m, int32_t rows, ActBuf out, bool pdl, cudaStream_t s);
// residual after a layer, [rows][width] f32: the sum of the updated streams
int32_t launch_stream_tap(const StreamMix &m, int32_t rows, float *out, cudaStream_t s);
// out[r] = x[r] / rms(x[r]) * w (* sigmoid(gate[r])), x f32 [rows][x_ld]; gate f32 or bf16
int32_t launch_rms_rows(const float *x, int64_t x_ld, const float *w, int32_t cols, float eps, ActBuf gate, ActBuf out, int32_t rows,
                        bool pdl, cudaStream_t s);
// The same over groups of `group` columns that share the weights w[group], times silu(gate[r]) (f32).
int32_t launch_rms_groups(const float *x, int64_t x_ld, const float *w, int32_t cols, int32_t group, float eps, const float *gate, int64_t gate_ld,
                          ActBuf out, int32_t rows, bool pdl, cudaStream_t s);

// lin_mv.cu: up to two activation rows, one pass over the weights at HBM speed, with the operand's preparation fused
// into the prologue of every CTA.
enum LinPrologue { kProPlain = 0, kProRms = 1, kProRmsGate = 2, kProStreams = 3, kProRmsGroups = 4 };
struct LinMvArgs {
  LinW w;
  int32_t batch = 1;
  int32_t prologue = kProPlain;
  StreamMix mix;              // kProStreams
  const float *x = nullptr;   // the others: f32 rows
  int64_t x_ld = 0;
  const float *norm_w = nullptr;
  float eps = 0.0f;
  const float *gate = nullptr;  // kProRmsGate: f32 rows, multiplied by their sigmoid; kProRmsGroups: by their SiLU
  int64_t gate_ld = 0;
  int32_t group = 0;            // kProRmsGroups: columns of a group
  float *y = nullptr;
  int64_t y_ld = 0;
  int32_t act = kActNone, act_rows = 0;
  const float *bias = nullptr;  // [rows], added before the activation
  float scale = 1.0f;           // of the sums
};
bool lin_mv_fits(int32_t cols, int32_t batch);
int32_t launch_lin_mv(const LinMvArgs &a, bool pdl, cudaStream_t s);
// Two products that do not depend on each other in one launch, the CTAs split between them by their weights.
int32_t launch_lin_mv_pair(const LinMvArgs &a, const LinMvArgs &b, bool pdl, cudaStream_t s);

// lin_tc5.cu / lin_f32.cu: any number of rows.  out[r][o] = act(scale * sum_k w[o][k] x[r][k] + bias[o])
struct LinArgs {
  LinW w;
  const void *x = nullptr;  // bf16 rows (tcgen05) or f32 rows (f32 kernel), x_ld elements apart
  int64_t x_ld = 0;
  int32_t rows = 0;
  void *out = nullptr;
  int32_t out_half = 0;
  int64_t out_ld = 0;
  int32_t act = kActNone, act_rows = 0;
  const float *bias = nullptr;
  float scale = 1.0f;
};
int32_t launch_lin_tc5(const LinArgs &a, int32_t sm_count, int32_t *status, bool pdl, cudaStream_t s);
int32_t launch_lin_f32(const LinArgs &a, cudaStream_t s);

// latent_attn.cu: attention over a cache of one latent vector and one shared rotated key part per position.
struct LatentShape {
  int32_t heads, dim, rot_dim, rot_dims, vdim, rank;
  float scale, eps;
};
struct LatentArgs {
  LatentShape m;
  int32_t rows = 0;
  const int32_t *positions = nullptr, *slots = nullptr;  // per row
  const float *cs = nullptr;    // [position][rot_dims / 2][cos, sin]
  void *cache = nullptr;        // [slot][max_pos][cache_ld]: latent | rotated key part
  int32_t cache_half = 0;
  int64_t cache_ld = 0, max_pos = 0;
  const float *low = nullptr;   // [row][low_ld]: latent before its norm | key part before its rotation
  int64_t low_ld = 0;
  const float *latent_norm = nullptr;
  const float *q = nullptr;     // [row][heads * (dim + rot_dim)]
  LinW uk, uv;
  float *qa = nullptr;          // [row][heads][rank + rot_dim]: queries in latent space, scaled
  float *part = nullptr;        // [row][heads][splits][rank + 2]
  int32_t splits = 1;
  const float *gate = nullptr;  // [row][gate_ld]
  int64_t gate_ld = 0;
  ActBuf out;                   // [row][heads * vdim]
};
// Appends the rows' latents to the cache; with queries, also brings the queries into latent space.
int32_t launch_latent_prep(const LatentArgs &a, bool queries, bool pdl, cudaStream_t s);
int latent_attention_groups(const LatentArgs &a);  // CTAs the heads of a row are spread over
int32_t launch_latent_attention(const LatentArgs &a, bool pdl, cudaStream_t s);
int32_t launch_latent_output(const LatentArgs &a, bool pdl, cudaStream_t s);
bool latent_shape_ok(const LatentShape &m);
// A long portion of one sequence: keys and values already expanded to kv[position][heads * dim | heads * vdim] (bf16).
struct LatentPrefillArgs {
  LatentShape m;
  int32_t rows = 0;
  int64_t start = 0;            // position of row 0
  const float *cs = nullptr;
  const bf16 *cache = nullptr;  // this slot's cache rows, for the rotated key part
  int64_t cache_ld = 0;
  const bf16 *kv = nullptr;
  int64_t kv_ld = 0;
  const float *q = nullptr;
  const float *gate = nullptr;
  int64_t gate_ld = 0;
  bf16 *out = nullptr;
  int64_t out_ld = 0;
};
bool latent_prefill_fits(const LatentShape &m, int64_t cache_ld, int64_t kv_ld);
int32_t launch_latent_prefill(const LatentPrefillArgs &a, bool pdl, cudaStream_t s);

// window_attn.cu: attention of grouped heads over a sliding window.  A slot's keys (normed and rotated) and values lie in a
// ring of `cap` positions, position p in row p % cap, head by head: [slot][kv_head][cap][kp | vp], kp and vp the sizes
// rounded up to 16, the padding zero.
struct WindowShape {
  int32_t heads, kv_heads, dim, vdim, rot_dims;
  int32_t window;  // 0: every earlier position
  float scale, eps;
};
inline __host__ __device__ int window_pad(int n) { return (n + 15) & ~15; }
struct WindowArgs {
  WindowShape m;
  int32_t rows = 0;
  const int32_t *positions = nullptr, *slots = nullptr;  // per row
  const float *cs = nullptr;    // [position][rot_dims / 2][cos, sin]
  const float *q_norm = nullptr, *k_norm = nullptr;      // [dim]
  const float *qkv = nullptr;   // [row][ld]: q (heads x dim) | k (kv_heads x dim) | v (kv_heads x vdim)
  int64_t ld = 0;
  void *cache = nullptr;
  int32_t cache_half = 0, cap = 0;
  void *q = nullptr;            // prepared queries: [row][heads][dim] f32, or [row][heads][kp] bf16
  int32_t q_half = 0;
  int32_t append = 0;           // decode: the row's own key and value come from qkv and go into the cache
  int32_t splits = 1;           // decode: CTAs (one cluster) that share a row's positions
  ActBuf out;                   // [row][heads * vdim]
};
bool window_shape_ok(const WindowShape &m);
// Norms and rotations: keys and values of the rows into the cache; with `queries` also the queries into q.
int32_t launch_window_prep(const WindowArgs &a, bool queries, bool pdl, cudaStream_t s);
int32_t launch_window_attention(const WindowArgs &a, bool pdl, cudaStream_t s);      // FP32 units, any cache; reads q
bool window_decode_fits(const WindowArgs &a);
int window_decode_groups(const WindowArgs &a);                                       // CTAs of a row before splitting
int32_t launch_window_decode(const WindowArgs &a, bool pdl, cudaStream_t s);         // bf16 cache, tensor cores; prepares its queries
bool window_prefill_fits(const WindowArgs &a);
int32_t launch_window_prefill(const WindowArgs &a, bool pdl, cudaStream_t s);        // consecutive rows of one sequence, bf16; reads q

// A decay per key channel and token: sigmoid(w x + b)^(1 / tau), x the low-rank projection of the layer's input.
struct ChannelDecay {
  LinW w;                          // [heads * dim][rank]
  const float *b = nullptr;        // [heads * dim]
  const float *x = nullptr;        // [row][ld of qkv]
  float inv_tau = 1.0f;
};

// lightning.cu: linear attention, state [slot][heads][dim][vdim] in f32, with a fixed decay per head or one per channel.
struct LightningArgs {
  int32_t heads, dim, vdim;
  const float *powers = nullptr;   // [heads][kLightningChunk + 1]: decay^0, decay^1, ...; null: `channel` applies
  ChannelDecay channel;
  float q_scale = 1.0f;
  float *state = nullptr;
  const void *qkv = nullptr;       // [row][ld]: q (heads x dim) | k (heads x dim) | v (heads x vdim), f32 or bf16
  int32_t half = 0;
  int64_t ld = 0;
  float *out = nullptr;            // [row][heads * vdim]
  const int32_t *positions = nullptr, *slots = nullptr;
  int32_t rows = 0;
  int32_t one_sequence = 0;        // 1: the rows are consecutive tokens of one sequence; 0: one token of each row's own
  // 1: the inputs were complete before the predecessor let this kernel start; it waits for the predecessor only at its end
  int32_t late_wait = 0;
};
constexpr int kLightningChunk = 64;
bool lightning_shape_ok(int32_t heads, int32_t dim, int32_t vdim);
int32_t launch_lightning_steps(const LightningArgs &a, bool pdl, cudaStream_t s);   // token after token
bool lightning_chunk_fits(const LightningArgs &a);
int32_t launch_lightning_chunks(const LightningArgs &a, bool pdl, cudaStream_t s);  // 64 tokens at a time on the tensor cores

// gated_linear.cu: the recurrence with a decay per channel, 64 tokens at a time on the tensor cores (f32 rows of one sequence)
bool gated_shape_ok(int32_t heads, int32_t dim, int32_t vdim, int32_t rank);
bool gated_chunk_fits(int32_t dim, int32_t rank);
int64_t gated_scratch_bytes(int32_t heads, int32_t dim, int32_t vdim, int64_t rows);
int32_t launch_gated_chunks(const LightningArgs &a, void *scratch, bool pdl, cudaStream_t s);

#ifdef __CUDACC__

template <typename... KA, typename... A>
inline int32_t launch_kernel(void (*k)(KA...), dim3 grid, dim3 block, size_t smem, bool pdl, cudaStream_t s, A &&...args) {
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  CMLD_CUDA(cudaLaunchKernelEx(&cfg, k, static_cast<KA>(args)...));
  return CMLD_OK;
}
// Once per kernel: full shared memory.
template <typename K>
inline int32_t allow_smem(K k, size_t bytes) {
  CMLD_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
  return CMLD_OK;
}

__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float ld_peer(uint32_t local_addr, uint32_t rank) {
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ void cp16(void *dst, const void *src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
// log(sigmoid(z)) / tau
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return (fminf(z, 0.0f) - log1pf(expf(-fabsf(z)))) * inv_tau; }
__device__ __forceinline__ float lin_activate(float v, int act, bool in_range) {
  if (act == kActSilu && in_range) return v * sigmoid_f(v);
  if (act == kActRelu2) {
    const float p = fmaxf(v, 0.0f);
    return p * p;
  }
  return v;
}
__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ float act_load(const void *p, int half, int64_t i) {
  return half ? __bfloat162float(static_cast<const bf16 *>(p)[i]) : static_cast<const float *>(p)[i];
}
__device__ __forceinline__ void act_store(void *p, int half, int64_t i, float v) {
  if (half) static_cast<bf16 *>(p)[i] = __float2bfloat16_rn(v);
  else static_cast<float *>(p)[i] = v;
}

// Sum over the CTA; every thread gets it.  `red` holds at least blockDim.x / 32 floats.
__device__ __forceinline__ float cta_total(float v, float *red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, n = (blockDim.x + 31) >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[warp] = v;
  __syncthreads();
  float t = 0.0f;
  for (int i = 0; i < n; ++i) t += red[i];
  return t;
}

template <int S>
__device__ __forceinline__ void stream_update(const StreamMix &m, int64_t row, float *u, bool store) {
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    const bool live = s < m.streams;
    out[s] = live ? m.out[s] : 0.0f;
    in[s] = live ? (m.in ? m.in[s] : 1.0f) : 0.0f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = live && t < m.streams ? m.mix[s * m.streams + t] : 0.0f;
  }
  const float *x = m.x_in + row * m.streams * m.width, *y = m.y + row * m.width;
  float *xo = m.x_out ? m.x_out + row * m.streams * m.width : nullptr;
  for (int i = threadIdx.x; i < m.width; i += blockDim.x) {
    float xs[S];
#pragma unroll
    for (int s = 0; s < S; ++s) xs[s] = s < m.streams ? x[(int64_t)s * m.width + i] : 0.0f;
    const float yi = y[i];
    float acc = 0.0f;
#pragma unroll
    for (int t = 0; t < S; ++t) {
      float v = out[t] * yi;
#pragma unroll
      for (int s = 0; s < S; ++s) v = fmaf(mix[s][t], xs[s], v);
      if (store && xo && t < m.streams) xo[(int64_t)t * m.width + i] = v;
      acc = fmaf(in[t], v, acc);
    }
    u[i] = acc;
  }
}

// Any number of streams: one updated stream at a time.
__device__ __forceinline__ void stream_update_many(const StreamMix &m, int64_t row, float *u, bool store) {
  const float *x = m.x_in + row * m.streams * m.width, *y = m.y + row * m.width;
  float *xo = store && m.x_out ? m.x_out + row * m.streams * m.width : nullptr;
  for (int i = threadIdx.x; i < m.width; i += blockDim.x) {
    const float yi = y[i];
    float acc = 0.0f;
    for (int t = 0; t < m.streams; ++t) {
      float v = m.out[t] * yi;
      for (int s = 0; s < m.streams; ++s) v = fmaf(m.mix[s * m.streams + t], x[(int64_t)s * m.width + i], v);
      if (xo) xo[(int64_t)t * m.width + i] = v;
      acc = fmaf(m.in ? m.in[t] : 1.0f, v, acc);
    }
    u[i] = acc;
  }
}

// (u - mean) / sqrt(var + eps) * w + b in place over the CTA (u in shared memory).
__device__ __forceinline__ void layer_norm_cta(float *u, int n, const float *w, const float *b, float eps, float *red) {
  float s = 0.0f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) s += u[i];
  const float mean = cta_total(s, red) / (float)n;
  s = 0.0f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float d = u[i] - mean;
    s = fmaf(d, d, s);
  }
  const float r = 1.0f / sqrtf(cta_total(s, red) / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) u[i] = (u[i] - mean) * r * w[i] + b[i];
}

// Two sums over the CTA at once.
__device__ __forceinline__ float2 cta_total2(float2 v, float *red) {
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  const int warp = threadIdx.x >> 5, n = (blockDim.x + 31) >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) *reinterpret_cast<float2 *>(red + 2 * warp) = v;
  __syncthreads();
  float2 t = make_float2(0.0f, 0.0f);
  for (int i = 0; i < n; ++i) {
    const float2 p = *reinterpret_cast<const float2 *>(red + 2 * i);
    t.x += p.x;
    t.y += p.y;
  }
  return t;
}
__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }

// x + y' of a single stream, or its embedding row (see StreamMix); put(i, v) takes values 4i .. 4i + 3 of the result.  The row stays in registers,
// V times four values per thread (width a multiple of four, at most 4 V blockDim.x).  `red` holds 2 * blockDim.x / 32 floats.
template <int V, typename Put>
__device__ __forceinline__ void post_norm_row(const StreamMix &m, int64_t row, float *red, Put put) {
  const int n4 = m.width / 4;
  if (m.embed) {
    const uint2 *e = reinterpret_cast<const uint2 *>(m.embed + (int64_t)m.tokens[row] * m.embed_ld);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i >= n4) break;
      const uint2 v = e[i];
      put(i, make_float4(m.embed_scale * bf16_lo(v.x), m.embed_scale * bf16_hi(v.x), m.embed_scale * bf16_lo(v.y), m.embed_scale * bf16_hi(v.y)));
    }
    return;
  }
  const float4 *x = reinterpret_cast<const float4 *>(m.x_in + row * m.width), *y = reinterpret_cast<const float4 *>(m.y + row * m.width);
  float4 xv[V], yv[V];
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    yv[j] = i < n4 ? y[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (m.y2) {
    const float4 *z = reinterpret_cast<const float4 *>(m.y2 + row * m.width), *yw = reinterpret_cast<const float4 *>(m.y_norm);
    const float4 *zw = reinterpret_cast<const float4 *>(m.y2_norm);
    float4 zv[V];
    float2 s = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      zv[j] = i < n4 ? z[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      s.x += dot4(yv[j], yv[j]);
      s.y += dot4(zv[j], zv[j]);
      const int i = threadIdx.x + j * blockDim.x;
      if (i < n4) {  // the branches' weights do not wait for the sums
        const float4 a = yw[i], b = zw[i];
        yv[j] = make_float4(yv[j].x * a.x, yv[j].y * a.y, yv[j].z * a.z, yv[j].w * a.w);
        zv[j] = make_float4(zv[j].x * b.x, zv[j].y * b.y, zv[j].z * b.z, zv[j].w * b.w);
      }
    }
    s = cta_total2(s, red);
    const float ry = 0.5f / sqrtf(s.x / (float)m.width + m.eps), rz = 0.5f / sqrtf(s.y / (float)m.width + m.eps);
#pragma unroll
    for (int j = 0; j < V; ++j)
      yv[j] = make_float4(fmaf(yv[j].x, ry, zv[j].x * rz), fmaf(yv[j].y, ry, zv[j].y * rz), fmaf(yv[j].z, ry, zv[j].z * rz), fmaf(yv[j].w, ry, zv[j].w * rz));
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    xv[j] = i < n4 ? x[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  float r = 1.0f;
  if (m.out_norm) {
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < V; ++j) s += dot4(yv[j], yv[j]);
    r = 1.0f / sqrtf(cta_total2(make_float2(s, 0.0f), red).x / (float)m.width + m.eps);
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= n4) break;
    const float4 w = m.out_norm ? reinterpret_cast<const float4 *>(m.out_norm)[i] : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
    put(i, make_float4(fmaf(yv[j].x * r, w.x, xv[j].x), fmaf(yv[j].y * r, w.y, xv[j].y), fmaf(yv[j].z * r, w.z, xv[j].z), fmaf(yv[j].w * r, w.w, xv[j].w)));
  }
}

// The same for any width, through u.
__device__ __forceinline__ void post_norm_update(const StreamMix &m, int64_t row, float *u, float *red, bool store) {
  const float *x = m.x_in + row * m.width, *y = m.y + row * m.width;
  float *xo = store && m.x_out ? m.x_out + row * m.width : nullptr;
  if (m.width % 4 == 0 && m.width <= 8 * (int)blockDim.x) {
    if (!m.y2 && !m.out_norm) __syncthreads();  // no sum keeps the readers of an earlier row in u apart
    auto put = [&](int i, float4 v) {
      reinterpret_cast<float4 *>(u)[i] = v;
      if (xo) reinterpret_cast<float4 *>(xo)[i] = v;
    };
    if (m.width <= 4 * (int)blockDim.x) post_norm_row<1>(m, row, red, put);
    else post_norm_row<2>(m, row, red, put);
    __syncthreads();  // a thread's values in u are not those of its stride
    return;
  }
  if (m.y2) {
    const float *z = m.y2 + row * m.width;
    float2 s = make_float2(0.0f, 0.0f);
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) {
      s.x = fmaf(y[i], y[i], s.x);
      s.y = fmaf(z[i], z[i], s.y);
    }
    s = cta_total2(s, red);
    const float ry = 0.5f / sqrtf(s.x / (float)m.width + m.eps), rz = 0.5f / sqrtf(s.y / (float)m.width + m.eps);
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) u[i] = y[i] * m.y_norm[i] * ry + z[i] * m.y2_norm[i] * rz;
  } else {
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) u[i] = y[i];
  }
  float r = 1.0f;
  if (m.out_norm) {
    float s = 0.0f;
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) s = fmaf(u[i], u[i], s);
    r = 1.0f / sqrtf(cta_total(s, red) / (float)m.width + m.eps);
  }
  for (int i = threadIdx.x; i < m.width; i += blockDim.x) {
    const float v = x[i] + u[i] * r * (m.out_norm ? m.out_norm[i] : 1.0f);
    if (xo) xo[i] = v;
    u[i] = v;
  }
}

// u / rms(u) * w in place over the CTA.
__device__ __forceinline__ void rms_norm_cta(float *u, int n, const float *w, float eps, float *red) {
  float s = 0.0f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) s = fmaf(u[i], u[i], s);
  const float r = 1.0f / sqrtf(cta_total(s, red) / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) u[i] = u[i] * r * w[i];
}

// The whole boundary for one row; the result is left in u[width] (shared memory, 16-byte aligned; each thread may read its
// own stride).  `red` holds 2 * blockDim.x / 32 floats, 8-byte aligned.
__device__ __forceinline__ void stream_mix_row(const StreamMix &m, int r, float *u, float *red, bool store) {
  const int64_t row = m.row_map ? m.row_map[r] : r;
  if (m.embed) {
    const bf16 *e = m.embed + (int64_t)m.tokens[row] * m.embed_ld;
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) u[i] = m.embed_scale * __bfloat162float(e[i]);
    if (m.enorm_w) layer_norm_cta(u, m.width, m.enorm_w, m.enorm_b, m.eps, red);
    float in = 0.0f;
    for (int s = 0; s < m.streams; ++s) in += m.in ? m.in[s] : 1.0f;
    for (int i = threadIdx.x; i < m.width; i += blockDim.x) {
      const float x = u[i];
      if (store && m.x_out)
        for (int s = 0; s < m.streams; ++s) m.x_out[(row * m.streams + s) * m.width + i] = x;
      u[i] = in * x;
    }
  } else if (!m.mix) {
    post_norm_update(m, row, u, red, store);
  } else {
    switch (m.streams) {
      case 1: stream_update<1>(m, row, u, store); break;
      case 2: stream_update<2>(m, row, u, store); break;
      case 3: stream_update<3>(m, row, u, store); break;
      case 4: stream_update<4>(m, row, u, store); break;
      default: stream_update_many(m, row, u, store); break;
    }
  }
  if (m.norm_b) layer_norm_cta(u, m.width, m.norm_w, m.norm_b, m.eps, red);
  else if (m.norm_w) rms_norm_cta(u, m.width, m.norm_w, m.eps, red);
}

#endif  // __CUDACC__

}  // namespace cmld
