// Attention of grouped heads over a sliding window: query head h reads key/value head h / (heads / kv_heads); queries and keys
// are RMS-normed per head and rotated; the token at position i sees the positions i - window + 1 .. i.
//
// Keys (as they are scored) and values lie in a ring per slot, so that a slot holds the window and the rows of one step,
// whatever the length of the sequence.
//   window_prep_kernel     norms, rotations, cache rows; a warp per head
//   window_attn_kernel     one row and head per CTA, FP32 units, caches of either precision
//   window_decode_kernel   one row and the (up to 16) query heads of a key head per cluster, on the tensor cores: every warp
//                          takes 16 positions at a time with its own online softmax, queries and weights as two bfloat16
//                          terms; the warps and CTAs are merged at the end.  Prepares its own queries; in a decode step also
//                          the row's new key and value.
//   window_prefill_kernel  64 queries of one head, 64 positions at a time; scores, weights and sums in 32-bit (the weights
//                          enter the second product as two bfloat16 terms)
#include "layered.cuh"
#include "mma_sync.cuh"

namespace cmld {

namespace {

// Element j of a head after its norm and the rotation of its first `dims` elements.
__device__ __forceinline__ float head_value(const float *x, int j, float inv, const float *w, int dims, const float *cs) {
  const float v = x[j] * inv * w[j];
  if (j >= dims) return v;
  const int half = dims >> 1, p = j < half ? j : j - half, o = j < half ? j + half : j - half;
  const float c = cs[2 * p], s = cs[2 * p + 1], t = x[o] * inv * w[o];
  return j < half ? v * c - t * s : v * c + t * s;
}
// 1 / rms of a head, by one warp.
__device__ __forceinline__ float head_inv_rms(const float *x, int dim, float eps, int lane) {
  float s = 0.0f;
#pragma unroll 4
  for (int i = lane; i < dim; i += 32) s = fmaf(x[i], x[i], s);
  return 1.0f / sqrtf(warp_sum(s) / (float)dim + eps);
}
__device__ __forceinline__ int64_t cache_row(const WindowArgs &a, int slot, int g, int row) {
  return (((int64_t)slot * a.m.kv_heads + g) * a.cap + row) * (window_pad(a.m.dim) + window_pad(a.m.vdim));
}

__global__ void __launch_bounds__(256) window_prep_kernel(const WindowArgs a, int first) {
  pdl_wait();
  pdl_launch();
  const WindowShape &m = a.m;
  const int row = blockIdx.x, unit = first + blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= m.heads + 2 * m.kv_heads) return;
  const float *x = a.qkv + row * a.ld;
  const int pos = a.positions[row], kp = window_pad(m.dim);
  const float *cs = a.cs + (int64_t)pos * m.rot_dims;
  if (unit < m.heads) {
    x += unit * m.dim;
    const float inv = head_inv_rms(x, m.dim, m.eps, lane);
    const int n = a.q_half ? kp : m.dim;
    const int64_t at = ((int64_t)row * m.heads + unit) * n;
#pragma unroll 4
    for (int j = lane; j < n; j += 32) act_store(a.q, a.q_half, at + j, j < m.dim ? head_value(x, j, inv, a.q_norm, m.rot_dims, cs) : 0.0f);
  } else if (unit < m.heads + m.kv_heads) {
    const int g = unit - m.heads;
    x += unit * m.dim;
    const float inv = head_inv_rms(x, m.dim, m.eps, lane);
    const int64_t at = cache_row(a, a.slots[row], g, pos % a.cap);
#pragma unroll 4
    for (int j = lane; j < m.dim; j += 32) act_store(a.cache, a.cache_half, at + j, head_value(x, j, inv, a.k_norm, m.rot_dims, cs));
  } else {
    const int g = unit - m.heads - m.kv_heads;
    x += (m.heads + m.kv_heads) * m.dim + g * m.vdim;
    const int64_t at = cache_row(a, a.slots[row], g, pos % a.cap) + kp;
#pragma unroll 4
    for (int j = lane; j < m.vdim; j += 32) act_store(a.cache, a.cache_half, at + j, x[j]);
  }
}

// ---------------------------------------------------------------- FP32 units

// NV: value dimensions per lane (vdim <= 32 * NV)
template <int NV>
__global__ void __launch_bounds__(256) window_attn_kernel(const WindowArgs a) {
  extern __shared__ float sm[];
  const WindowShape &m = a.m;
  float *qs = sm, *part = sm + m.dim;  // [dim]; [8][vdim]
  __shared__ float pm[8], pl[8];
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x, h = blockIdx.y, g = h / (m.heads / m.kv_heads), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kp = window_pad(m.dim), pos = a.positions[row], lo = m.window > 0 ? max(0, pos - m.window + 1) : 0;
  const float *q = static_cast<const float *>(a.q) + ((int64_t)row * m.heads + h) * m.dim;
  for (int i = threadIdx.x; i < m.dim; i += 256) qs[i] = q[i];
  __syncthreads();
  const int64_t base = cache_row(a, a.slots[row], g, 0), ld = kp + window_pad(m.vdim);
  float mx = -INFINITY, sum = 0.0f, acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.0f;
  for (int p = lo + warp; p <= pos; p += 8) {
    const int64_t at = base + p % a.cap * ld;
    float s = 0.0f;
#pragma unroll 4
    for (int d = lane; d < m.dim; d += 32) s = fmaf(qs[d], act_load(a.cache, a.cache_half, at + d), s);
    s = warp_sum(s) * m.scale;
    const float nm = fmaxf(mx, s), c = expf(mx - nm), w = expf(s - nm);
    mx = nm;
    sum = fmaf(sum, c, w);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = lane + 32 * i;
      acc[i] = fmaf(acc[i], c, d < m.vdim ? w * act_load(a.cache, a.cache_half, at + kp + d) : 0.0f);
    }
  }
  if (lane == 0) {
    pm[warp] = mx;
    pl[warp] = sum;
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (lane + 32 * i < m.vdim) part[warp * m.vdim + lane + 32 * i] = acc[i];
  __syncthreads();
  float all = -INFINITY, l = 0.0f, w[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) all = fmaxf(all, pm[i]);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    w[i] = expf(pm[i] - all);  // a warp without positions: exp(-inf) = 0
    l = fmaf(w[i], pl[i], l);
  }
  for (int d = threadIdx.x; d < m.vdim; d += 256) {
    float o = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) o = fmaf(w[i], part[i * m.vdim + d], o);
    act_store(a.out.p, a.out.half, row * a.out.ld + h * m.vdim + d, o / l);
  }
}

// ---------------------------------------------------------------- decode on the tensor cores

constexpr int kDecWarps = 8, kDecThreads = kDecWarps * 32, kDecKeys = 16, kDecHeads = 16;

struct DecodeSmem {
  int q, row, stats, om, region, region_bytes, total;  // byte offsets
};
__host__ __device__ inline DecodeSmem decode_smem(int kp, int vp, int VP, int stages) {
  DecodeSmem s{};
  s.q = 0;                                                 // hi, lo [16][kp + 8] bf16
  s.row = s.q + 2 * kDecHeads * (kp + 8) * 2;              // the row's own key and value, bf16
  s.stats = s.row + (kp + vp) * 2;                         // [warp][16] maxima, [warp][16] sums, [16] maxima, [16] sums
  s.om = s.stats + (2 * kDecWarps * 16 + 32) * 4;          // [16][VP] f32
  s.region = s.om + kDecHeads * VP * 4;                    // per warp: stages of [16][kp + 8] and [16][VP + 8]; later [16][VP + 4] f32
  const int stage = kDecKeys * (kp + 8 + VP + 8) * 2, merge = kDecHeads * (VP + 4) * 4;
  s.region_bytes = stages * stage > merge ? stages * stage : merge;
  s.total = s.region + kDecWarps * s.region_bytes;
  return s;
}

// VP: value dimensions, padded to 32, 64, 128 or 256
template <int VP>
__global__ void __launch_bounds__(kDecThreads, 1) window_decode_kernel(const WindowArgs a, int stages) {
  extern __shared__ __align__(16) uint8_t raw[];
  const WindowShape &m = a.m;
  const int kp = window_pad(m.dim), vp = window_pad(m.vdim), KS = kp + 8;
  constexpr int VS = VP + 8, MS = VP + 4;
  const DecodeSmem L = decode_smem(kp, vp, VP, stages);
  bf16 *qh = reinterpret_cast<bf16 *>(raw + L.q), *ql = qh + kDecHeads * KS, *own = reinterpret_cast<bf16 *>(raw + L.row);
  float *wm = reinterpret_cast<float *>(raw + L.stats), *wl = wm + kDecWarps * 16, *cm = wl + kDecWarps * 16, *cl = cm + 16;
  float *om = reinterpret_cast<float *>(raw + L.om);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, tr = lane >> 2, tc = (lane & 3) * 2;
  const int rank = blockIdx.x, row = blockIdx.z;
  const int per = m.heads / m.kv_heads, blocks = (per + kDecHeads - 1) / kDecHeads;
  const int g = blockIdx.y / blocks, hb = blockIdx.y % blocks * kDecHeads, h0 = g * per + hb, nh = min(kDecHeads, per - hb);
  bf16 *stage = reinterpret_cast<bf16 *>(raw + L.region + warp * L.region_bytes);
  const int stage_elems = kDecKeys * (KS + VS);

  // rows, places and the cache rows of earlier steps were complete before this step began
  const bool early = a.append;
  if (!early) pdl_wait();
  const int pos = a.positions[row], slot = a.slots[row];
  const int lo = m.window > 0 ? max(0, pos - m.window + 1) : 0, cached = a.append ? pos : pos + 1;
  const int tiles = (pos - lo + kDecKeys) / kDecKeys, step = a.splits * kDecWarps;
  bf16 *cache = static_cast<bf16 *>(a.cache);
  const int64_t base = cache_row(a, slot, g, 0);
  auto load = [&](int t, bf16 *dst) {
    const int p0 = lo + t * kDecKeys, i0 = p0 % a.cap;
    for (int u = lane; u < (kp + vp) / 8; u += 32) {
      bf16 *d = u * 8 < kp ? dst + u * 8 : dst + kDecKeys * KS + u * 8 - kp;
      const int ds = u * 8 < kp ? KS : VS;
#pragma unroll
      for (int k = 0; k < kDecKeys; ++k) {
        const bool live = p0 + k < cached;
        const int i = i0 + k < a.cap ? i0 + k : i0 + k - a.cap;
        cp16(d + k * ds, cache + base + (live ? (int64_t)i * (kp + vp) : 0) + u * 8, live);
      }
    }
  };
  int t = rank * kDecWarps + warp;
  for (int i = 0; i < stages; ++i) {
    if (t + i * step < tiles) load(t + i * step, stage + i * stage_elems);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  if (early) pdl_wait();
  pdl_launch();

  const float *x = a.qkv + row * a.ld, *cs = a.cs + (int64_t)pos * m.rot_dims;
  for (int h = warp; h < kDecHeads; h += kDecWarps) {
    const float *q = x + (h0 + h) * m.dim;
    const float inv = h < nh ? head_inv_rms(q, m.dim, m.eps, lane) : 0.0f;
    for (int j = lane; j < kp; j += 32) {
      const float v = h < nh && j < m.dim ? m.scale * head_value(q, j, inv, a.q_norm, m.rot_dims, cs) : 0.0f;
      const bf16 hi = __float2bfloat16_rn(v);
      qh[h * KS + j] = hi;
      ql[h * KS + j] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
  }
  if (a.append && warp >= kDecWarps - 2) {
    const bool key = warp == kDecWarps - 1, keep = rank == 0 && hb == 0;
    const float *k = x + (m.heads + g) * m.dim, *v = x + (m.heads + m.kv_heads) * m.dim + g * m.vdim;
    const int64_t at = base + (int64_t)(pos % a.cap) * (kp + vp);
    const float inv = key ? head_inv_rms(k, m.dim, m.eps, lane) : 0.0f;
    for (int j = (key ? 0 : kp) + lane; j < (key ? kp : kp + vp); j += 32) {
      float f = 0.0f;
      if (key && j < m.dim) f = head_value(k, j, inv, a.k_norm, m.rot_dims, cs);
      if (!key && j - kp < m.vdim) f = v[j - kp];
      own[j] = __float2bfloat16_rn(f);
      if (keep) cache[at + j] = own[j];
    }
  }
  __syncthreads();

  float O[VP / 8][4];
#pragma unroll
  for (int n = 0; n < VP / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[n][e] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  for (int i = 0; t < tiles; t += step, i = i + 1 == stages ? 0 : i + 1) {
    bf16 *ks = stage + i * stage_elems, *vs = ks + kDecKeys * KS;
    if (stages == 2) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
    const int p0 = lo + t * kDecKeys;
    if (a.append && pos < p0 + kDecKeys) {  // the last tile
      for (int u = lane; u < (kp + vp) / 8; u += 32)
        *reinterpret_cast<uint4 *>(u * 8 < kp ? ks + (pos - p0) * KS + u * 8 : vs + (pos - p0) * VS + u * 8 - kp) = *reinterpret_cast<const uint4 *>(own + u * 8);
      __syncwarp();
    }
    float P[2][4] = {};
    for (int k = 0; k < kp; k += 16) {
      uint32_t A[4], B[4];
      ldsm4(B, ks + ((lane & 7) + ((lane >> 4) << 3)) * KS + k + ((lane >> 3) & 1) * 8);
      ldsm4(A, qh + (lane & 15) * KS + k + (lane >> 4) * 8);
      mma16816(P[0], A, B[0], B[1]);
      mma16816(P[1], A, B[2], B[3]);
      ldsm4(A, ql + (lane & 15) * KS + k + (lane >> 4) * 8);
      mma16816(P[0], A, B[0], B[1]);
      mma16816(P[1], A, B[2], B[3]);
    }
    float nm[2] = {mx[0], mx[1]}, ts[2] = {0.0f, 0.0f};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (p0 + n * 8 + tc + (e & 1) > pos) P[n][e] = -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], P[n][e]);
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 1));
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 2));
    }
    // a tile holds at least one visible position, so nm is finite
    const float c0 = expf(mx[0] - nm[0]), c1 = expf(mx[1] - nm[1]);
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        P[n][e] = expf(P[n][e] - nm[e >> 1]);
        ts[e >> 1] += P[n][e];
      }
    sum[0] = fmaf(sum[0], c0, ts[0]);
    sum[1] = fmaf(sum[1], c1, ts[1]);
    mx[0] = nm[0];
    mx[1] = nm[1];
    uint32_t H[4], Q[4];
    split_pair(P[0][0], P[0][1], H[0], Q[0]);
    split_pair(P[0][2], P[0][3], H[1], Q[1]);
    split_pair(P[1][0], P[1][1], H[2], Q[2]);
    split_pair(P[1][2], P[1][3], H[3], Q[3]);
#pragma unroll
    for (int n = 0; n < VP / 16; ++n) {
      if (n * 16 >= vp) break;
      uint32_t B[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float c = e < 2 ? c0 : c1;
        O[2 * n][e] *= c;
        O[2 * n + 1][e] *= c;
      }
      ldsm4t(B, vs + (lane & 15) * VS + n * 16 + (lane >> 4) * 8);
      mma16816(O[2 * n], H, B[0], B[1]);
      mma16816(O[2 * n + 1], H, B[2], B[3]);
      mma16816(O[2 * n], Q, B[0], B[1]);
      mma16816(O[2 * n + 1], Q, B[2], B[3]);
    }
    __syncwarp();
    if (t + stages * step < tiles) load(t + stages * step, ks);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncwarp();
  // the warps' results
  float *mine = reinterpret_cast<float *>(stage);  // [16][MS]
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
    sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
    if ((lane & 3) == 0) {
      wm[warp * 16 + tr + 8 * e] = mx[e];
      wl[warp * 16 + tr + 8 * e] = sum[e];
    }
  }
#pragma unroll
  for (int n = 0; n < VP / 8; ++n) {
    *reinterpret_cast<float2 *>(mine + tr * MS + n * 8 + tc) = make_float2(O[n][0], O[n][1]);
    *reinterpret_cast<float2 *>(mine + (tr + 8) * MS + n * 8 + tc) = make_float2(O[n][2], O[n][3]);
  }
  __syncthreads();
  if (tid < 16) {
    float all = -INFINITY, l = 0.0f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) all = fmaxf(all, wm[w * 16 + tid]);
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {
      const float v = wm[w * 16 + tid], f = v == -INFINITY ? 0.0f : expf(v - all);
      l = fmaf(f, wl[w * 16 + tid], l);
      wm[w * 16 + tid] = f;
    }
    cm[tid] = all;
    cl[tid] = l;
  }
  __syncthreads();
  const float *r0 = reinterpret_cast<const float *>(raw + L.region);
  const int rs = L.region_bytes / 4;
  for (int i = tid; i < nh * m.vdim; i += kDecThreads) {
    const int h = i / m.vdim, v = i % m.vdim;
    float o = 0.0f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) o = fmaf(wm[w * 16 + h], r0[w * rs + h * MS + v], o);
    if (a.splits == 1) act_store(a.out.p, a.out.half, row * a.out.ld + (h0 + h) * m.vdim + v, o / cl[h]);
    else om[h * VP + v] = o;
  }
  if (a.splits > 1) {
    cluster_sync();
    const uint32_t cm_s = (uint32_t)__cvta_generic_to_shared(cm), cl_s = (uint32_t)__cvta_generic_to_shared(cl), om_s = (uint32_t)__cvta_generic_to_shared(om);
    for (int i = rank * kDecThreads + tid; i < nh * m.vdim; i += a.splits * kDecThreads) {
      const int h = i / m.vdim, v = i % m.vdim;
      float all = -INFINITY, l = 0.0f, o = 0.0f;
      for (int p = 0; p < a.splits; ++p) all = fmaxf(all, ld_peer(cm_s + 4 * h, p));
      for (int p = 0; p < a.splits; ++p) {
        const float f = expf(ld_peer(cm_s + 4 * h, p) - all);  // a CTA without positions: exp(-inf) = 0
        l = fmaf(f, ld_peer(cl_s + 4 * h, p), l);
        o = fmaf(f, ld_peer(om_s + 4 * (h * VP + v), p), o);
      }
      act_store(a.out.p, a.out.half, row * a.out.ld + (h0 + h) * m.vdim + v, o / l);
    }
    cluster_sync();
  }
}

// ---------------------------------------------------------------- portions on the tensor cores

constexpr int kPfThreads = 128, kPfQ = 64, kPfK = 64;

__host__ __device__ inline int pf_smem(int kp, int dv) { return (kPfQ * (kp + 8) + 2 * kPfK * (kp + 8) + 2 * kPfK * (dv + 8)) * 2; }

// DV: value dimensions, padded to 32, 64, 128 or 256
template <int DV>
__global__ void __launch_bounds__(kPfThreads) window_prefill_kernel(const WindowArgs a) {
  extern __shared__ __align__(16) bf16 sh[];
  const WindowShape &m = a.m;
  const int kp = window_pad(m.dim), vp = window_pad(m.vdim), QS = kp + 8, VS = DV + 8;
  bf16 *q_s = sh, *k_s = q_s + kPfQ * QS, *v_s = k_s + 2 * kPfK * QS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, g = h / (m.heads / m.kv_heads);
  const int r0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kPfQ;  // the longest rows of all heads first
  pdl_wait();
  pdl_launch();
  const int start = a.positions[0] + r0, last = start + min(kPfQ, a.rows - r0) - 1;  // positions of this tile's queries
  const int first = m.window > 0 ? max(0, start - m.window + 1) : 0;
  const int t0 = first / kPfK, t1 = last / kPfK;
  const bf16 *cache = static_cast<const bf16 *>(a.cache) + cache_row(a, a.slots[0], g, 0);
  auto load_tile = [&](int t, int st) {
    bf16 *kd = k_s + st * kPfK * QS, *vd = v_s + st * kPfK * VS;
    const int p0 = t * kPfK, i0 = p0 % a.cap;
    // a warp takes every fourth position, its lanes the row's 16-byte units
    for (int u = lane; u < (kp + vp) / 8; u += 32) {
      bf16 *dst = u * 8 < kp ? kd + u * 8 : vd + u * 8 - kp;
      const int ds = u * 8 < kp ? QS : VS;
#pragma unroll 8
      for (int k = warp; k < kPfK; k += kPfThreads / 32) {
        const bool live = p0 + k >= first && p0 + k <= last;
        const int i = i0 + k < a.cap ? i0 + k : (i0 + k) % a.cap;
        cp16(dst + k * ds, cache + (live ? (int64_t)i * (kp + vp) : 0) + u * 8, live);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const bf16 *q = static_cast<const bf16 *>(a.q) + (int64_t)h * kp;
  for (int i = tid; i < kPfQ * (kp / 8); i += kPfThreads) {
    const int r = i / (kp / 8), u = i % (kp / 8);
    const bool live = r0 + r < a.rows;
    cp16(q_s + r * QS + u * 8, q + (live ? (int64_t)(r0 + r) * m.heads * kp : 0) + u * 8, live);
  }
  load_tile(t0, 0);
  float O[DV / 8][4];
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[n][e] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  const int tr = lane >> 2, tc = (lane & 3) * 2, i0 = warp * 16;
  const int pos0 = start + i0 + tr, span = m.window > 0 ? m.window : 1 << 30;
  for (int t = t0; t <= t1; ++t) {
    const int st = (t - t0) & 1;
    if (t < t1) {
      load_tile(t + 1, st ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16 *kt = k_s + st * kPfK * QS, *vt = v_s + st * kPfK * VS;
    float P[8][4] = {};
#pragma unroll 2
    for (int k = 0; k < kp; k += 16) {
      uint32_t A[4], B[4];
      ldsm4(A, q_s + (i0 + (lane & 15)) * QS + k + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        ldsm4(B, kt + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * QS + k + ((lane >> 3) & 1) * 8);
        mma16816(P[2 * n], A, B[0], B[1]);
        mma16816(P[2 * n + 1], A, B[2], B[3]);
      }
    }
    float nm[2] = {mx[0], mx[1]};
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int back = pos0 + (e >> 1) * 8 - (t * kPfK + n * 8 + tc + (e & 1));
        P[n][e] = back >= 0 && back < span ? P[n][e] * m.scale : -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], P[n][e]);
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 1));
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 2));
    }
    // a query may see nothing of a tile (and, past the portion's end, nothing at all): keep the exponents finite
    const float b0 = nm[0] == -INFINITY ? 0.0f : nm[0], b1 = nm[1] == -INFINITY ? 0.0f : nm[1];
    const float c0 = expf(mx[0] - b0), c1 = expf(mx[1] - b1);
    float ts[2] = {0.0f, 0.0f};
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        P[n][e] = expf(P[n][e] - (e < 2 ? b0 : b1));
        ts[e >> 1] += P[n][e];
      }
    sum[0] = fmaf(sum[0], c0, ts[0]);
    sum[1] = fmaf(sum[1], c1, ts[1]);
    mx[0] = nm[0];
    mx[1] = nm[1];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      O[n][0] *= c0;
      O[n][1] *= c0;
      O[n][2] *= c1;
      O[n][3] *= c1;
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t H[4], L[4], B[4];
      split_pair(P[2 * kk][0], P[2 * kk][1], H[0], L[0]);
      split_pair(P[2 * kk][2], P[2 * kk][3], H[1], L[1]);
      split_pair(P[2 * kk + 1][0], P[2 * kk + 1][1], H[2], L[2]);
      split_pair(P[2 * kk + 1][2], P[2 * kk + 1][3], H[3], L[3]);
#pragma unroll
      for (int n = 0; n < DV / 16; ++n) {
        if (n * 16 >= vp) break;
        ldsm4t(B, vt + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], H, B[0], B[1]);
        mma16816(O[2 * n + 1], H, B[2], B[3]);
        mma16816(O[2 * n], L, B[0], B[1]);
        mma16816(O[2 * n + 1], L, B[2], B[3]);
      }
    }
    __syncthreads();  // the stage is free for the tile after next
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
    sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
  }
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + i0 + tr + (e >> 1) * 8, v = n * 8 + tc + (e & 1);
      if (r < a.rows && v < m.vdim) act_store(a.out.p, a.out.half, r * a.out.ld + h * m.vdim + v, O[n][e] / sum[e >> 1]);
    }
}

constexpr int kMaxSmem = 227 * 1024;

int padded_values(int vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : 256; }

int decode_stages(const WindowShape &m) {
  for (int s : {2, 1})
    if (decode_smem(window_pad(m.dim), window_pad(m.vdim), padded_values(m.vdim), s).total <= kMaxSmem) return s;
  return 0;
}

template <int VP>
int32_t decode(const WindowArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(window_decode_kernel<VP>, kMaxSmem));
    ready = true;
  }
  const int stages = decode_stages(a.m);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(a.splits, window_decode_groups(a), a.rows);
  cfg.blockDim = dim3(kDecThreads);
  cfg.dynamicSmemBytes = decode_smem(window_pad(a.m.dim), window_pad(a.m.vdim), VP, stages).total;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (a.splits > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = (unsigned)a.splits;
    attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  CMLD_CUDA(cudaLaunchKernelEx(&cfg, window_decode_kernel<VP>, a, stages));
  return CMLD_OK;
}

template <int DV>
int32_t prefill(const WindowArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(window_prefill_kernel<DV>, kMaxSmem));
    ready = true;
  }
  return launch_kernel(window_prefill_kernel<DV>, dim3(a.m.heads, (a.rows + kPfQ - 1) / kPfQ), dim3(kPfThreads), pf_smem(window_pad(a.m.dim), DV), pdl, s, a);
}

size_t plain_smem(const WindowShape &m) { return (size_t)(m.dim + 8 * m.vdim) * 4; }

template <int NV>
int32_t plain(const WindowArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(window_attn_kernel<NV>, 64 * 1024));
    ready = true;
  }
  return launch_kernel(window_attn_kernel<NV>, dim3(a.rows, a.m.heads), dim3(256), plain_smem(a.m), pdl, s, a);
}

}  // namespace

bool window_shape_ok(const WindowShape &m) {
  return m.heads >= 1 && m.kv_heads >= 1 && m.heads % m.kv_heads == 0 && m.dim >= 1 && m.vdim >= 1 && m.vdim <= 1024 && m.dim <= 4096 && m.window >= 0 &&
         m.rot_dims >= 0 && m.rot_dims % 2 == 0 && m.rot_dims <= m.dim && plain_smem(m) <= 64 * 1024 && m.heads <= 65535;
}

int32_t launch_window_prep(const WindowArgs &a, bool queries, bool pdl, cudaStream_t s) {
  const int first = queries ? 0 : a.m.heads, units = a.m.heads + 2 * a.m.kv_heads - first;
  return launch_kernel(window_prep_kernel, dim3(a.rows, (units + 7) / 8), dim3(256), 0, pdl, s, a, first);
}

int32_t launch_window_attention(const WindowArgs &a, bool pdl, cudaStream_t s) {
  if (a.q_half) return fail(CMLD_ERR_INVALID, "window attention on the FP32 units takes f32 queries");
  if (a.m.vdim <= 128) return plain<4>(a, pdl, s);
  if (a.m.vdim <= 512) return plain<16>(a, pdl, s);
  return plain<32>(a, pdl, s);
}

bool window_decode_fits(const WindowArgs &a) { return a.cache_half && a.m.vdim <= 256 && decode_stages(a.m) > 0; }

int window_decode_groups(const WindowArgs &a) {
  const int per = a.m.heads / a.m.kv_heads;
  return a.m.kv_heads * ((per + kDecHeads - 1) / kDecHeads);
}

int32_t launch_window_decode(const WindowArgs &a, bool pdl, cudaStream_t s) {
  if (a.splits < 1 || a.splits > 8) return fail(CMLD_ERR_INVALID, "window attention: %d CTAs per row, at most 8", a.splits);
  switch (padded_values(a.m.vdim)) {
    case 32: return decode<32>(a, pdl, s);
    case 64: return decode<64>(a, pdl, s);
    case 128: return decode<128>(a, pdl, s);
    default: return decode<256>(a, pdl, s);
  }
}

bool window_prefill_fits(const WindowArgs &a) {
  return a.cache_half && a.q_half && a.m.vdim <= 256 && pf_smem(window_pad(a.m.dim), padded_values(a.m.vdim)) <= kMaxSmem;
}

int32_t launch_window_prefill(const WindowArgs &a, bool pdl, cudaStream_t s) {
  switch (padded_values(a.m.vdim)) {
    case 32: return prefill<32>(a, pdl, s);
    case 64: return prefill<64>(a, pdl, s);
    case 128: return prefill<128>(a, pdl, s);
    default: return prefill<256>(a, pdl, s);
  }
}

}  // namespace cmld
