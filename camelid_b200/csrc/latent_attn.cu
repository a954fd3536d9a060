// Multi-head attention over latents: a position's cache row is one latent vector c (rank values) and one rotated key
// part shared by all heads (rot_dim values); per head the unrotated key is W_uk c and the value W_uv c.
//
// Decoding and short portions work in latent space: the query is taken through W_uk^T once (q_nope . W_uk c =
// (W_uk^T q_nope) . c), the cache rows are scored and averaged as they are, and W_uv is applied to the average.
//   latent_prep_kernel    rotates and transforms the queries; norms, rotates and appends the new cache rows
//   latent_attn_kernel    a range of positions for eight heads of one row: online softmax, all in 32-bit (f32 cache)
//   latent_attn_mma_kernel  the same for 16 heads on the tensor cores (bfloat16 cache)
//   latent_output_kernel  merges the ranges, applies W_uv and the sigmoid gate
// Long portions expand keys and values with two matrix products and run a tiled attention on the tensor cores:
//   latent_prefill_kernel 64 queries of one head per CTA, 64 keys at a time; scores, weights and sums in 32-bit (the
//                         weights enter the second product as two bfloat16 terms)
#include "layered.cuh"
#include "mma_sync.cuh"

namespace cmld {

namespace {

// ---------------------------------------------------------------- queries into latent space, cache append

constexpr int kPrepThreads = 256, kPrepRanks = 128;

// The value at index j of a rotated vector whose pairs (2i, 2i + 1), i < dims / 2, turn by the angles behind cs.
__device__ __forceinline__ float rotated(const float *x, int j, int dims, const float *cs) {
  if (j >= dims) return x[j];
  const float c = cs[(j >> 1) * 2], s = cs[(j >> 1) * 2 + 1];
  const float u = x[j & ~1], v = x[j | 1];
  return (j & 1) ? v * c + u * s : u * c - v * s;
}

// One new cache row, by the whole CTA: the latent RMS-normed, the key part rotated.
__device__ __forceinline__ void latent_append(const LatentArgs &a, int r, float *red) {
  const LatentShape &m = a.m;
  const float *low = a.low + (int64_t)r * a.low_ld;
  const int64_t pos = a.positions[r];
  const int64_t at = ((int64_t)a.slots[r] * a.max_pos + pos) * a.cache_ld;
  float s = 0.0f;
  for (int i = threadIdx.x; i < m.rank; i += blockDim.x) s = fmaf(low[i], low[i], s);
  const float inv = 1.0f / sqrtf(cta_total(s, red) / (float)m.rank + m.eps);
  for (int i = threadIdx.x; i < m.rank; i += blockDim.x) act_store(a.cache, a.cache_half, at + i, low[i] * inv * a.latent_norm[i]);
  for (int i = threadIdx.x; i < m.rot_dim; i += blockDim.x)
    act_store(a.cache, a.cache_half, at + m.rank + i, rotated(low + m.rank, i, m.rot_dims, a.cs + pos * m.rot_dims));
}

__global__ void __launch_bounds__(128) latent_append_kernel(const LatentArgs a) {
  __shared__ float red[4];
  pdl_launch();
  pdl_wait();
  latent_append(a, blockIdx.x, red);
}

// grid: x = row groups, y = head * slices + slice of the latent; the last ROWS y append the new cache rows.
// ROWS: rows that share a CTA's pass over its weights.
template <int ROWS>
__global__ void __launch_bounds__(kPrepThreads, 2) latent_prep_kernel(const LatentArgs a, int slices, int query_ys) {
  __shared__ float red[kPrepThreads / 32];
  extern __shared__ float prep_sm[];
  float *qn = prep_sm, *part = prep_sm + ROWS * ((a.m.dim + 3) & ~3);  // [ROWS][dim]; [16][ROWS][kPrepRanks]
  pdl_launch();
  const LatentShape &m = a.m;
  const int tid = threadIdx.x, h = blockIdx.y / slices, sl = blockIdx.y % slices;
  // eight latent dimensions per thread, the head's dimensions over 16 groups of threads; the first 128 of them are asked
  // for before the predecessor's results (weights depend on no earlier kernel)
  const int dg = tid >> 4, r = sl * kPrepRanks + (tid & 15) * 8;
  const bf16 *w = a.uk.w + (int64_t)h * m.dim * a.uk.ld + r;
  const bool in = (int)blockIdx.y < query_ys && r < (int)a.uk.ld;
  uint4 pre[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) pre[j] = in && dg + 16 * j < m.dim ? ld_stream16(w + (int64_t)(dg + 16 * j) * a.uk.ld) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  if ((int)blockIdx.y >= query_ys) {
    for (int row = blockIdx.x + gridDim.x * (blockIdx.y - query_ys); row < a.rows; row += gridDim.x * ROWS) latent_append(a, row, red);
    return;
  }
  const int qd = m.dim + m.rot_dim, D = m.rank + m.rot_dim;
  const int n_groups = (a.rows + ROWS - 1) / ROWS;
  for (int g = blockIdx.x; g < n_groups; g += gridDim.x) {
    const int r0 = g * ROWS, nr = min(ROWS, a.rows - r0);
    __syncthreads();
    for (int i = tid; i < ROWS * m.dim; i += kPrepThreads) {
      const int rr = i / m.dim, d = i % m.dim;
      qn[i] = rr < nr ? a.q[((int64_t)(r0 + rr) * m.heads + h) * qd + d] : 0.0f;
    }
    __syncthreads();
    float acc[ROWS][8] = {};
    auto take = [&](uint4 v, int d) {
      const float f[8] = {bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y), bf16_lo(v.z), bf16_hi(v.z), bf16_lo(v.w), bf16_hi(v.w)};
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const float qv = qn[i * m.dim + d];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i][e] = fmaf(f[e], qv, acc[i][e]);
      }
    };
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (dg + 16 * j < m.dim) take(pre[j], dg + 16 * j);
    if (in)
      for (int d = dg + 128; d < m.dim; d += 16) take(ld_stream16(w + (int64_t)d * a.uk.ld), d);
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      float4 *o = reinterpret_cast<float4 *>(part + (dg * ROWS + i) * kPrepRanks + (tid & 15) * 8);
      o[0] = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
      o[1] = make_float4(acc[i][4], acc[i][5], acc[i][6], acc[i][7]);
    }
    __syncthreads();
#pragma unroll
    for (int o = tid; o < ROWS * kPrepRanks; o += kPrepThreads) {
      const int i = o / kPrepRanks, c = o % kPrepRanks;
      if (i < nr && sl * kPrepRanks + c < m.rank) {
        float t = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; ++k) t += part[(k * ROWS + i) * kPrepRanks + c];
        a.qa[((int64_t)(r0 + i) * m.heads + h) * D + sl * kPrepRanks + c] = m.scale * t;
      }
    }
    if (sl == 0)
      for (int i = tid; i < nr * m.rot_dim; i += kPrepThreads) {
        const int rr = i / m.rot_dim, j = i % m.rot_dim;
        const float *x = a.q + ((int64_t)(r0 + rr) * m.heads + h) * qd + m.dim;
        a.qa[((int64_t)(r0 + rr) * m.heads + h) * D + m.rank + j] =
            m.scale * rotated(x, j, m.rot_dims, a.cs + (int64_t)a.positions[r0 + rr] * m.rot_dims);
      }
  }
}

// ---------------------------------------------------------------- attention in latent space

constexpr int kAttThreads = 256, kAttHeads = 8, kAttKeys = 32;

__host__ __device__ inline int att_units(int D) {  // 16-byte units of a staged row: an odd count keeps lanes apart
  const int u = (D + 3) / 4;
  return u | 1;
}
__host__ __device__ inline int att_smem(int D) {
  return (kAttKeys + kAttHeads) * att_units(D) * 16 + (8 * kAttHeads * kAttKeys + kAttKeys * kAttHeads + kAttHeads) * 4;
}

// NR: pairs of latent dimensions per thread (rank <= 512 * NR)
template <int NR>
__global__ void __launch_bounds__(kAttThreads) latent_attn_kernel(const LatentArgs a) {
  extern __shared__ __align__(16) float sm[];
  pdl_launch();
  pdl_wait();
  const LatentShape &m = a.m;
  const int D = m.rank + m.rot_dim, U = att_units(D), ld = U * 4, used = (D + 3) / 4;
  float *ks = sm, *qs = ks + kAttKeys * ld, *sc = qs + kAttHeads * ld, *pr = sc + 8 * kAttHeads * kAttKeys, *corr = pr + kAttKeys * kAttHeads;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * kAttHeads, row = blockIdx.z, nh = min(kAttHeads, m.heads - h0);
  const int n = a.positions[row] + 1;
  const int tiles = (n + kAttKeys - 1) / kAttKeys, per = (tiles + a.splits - 1) / a.splits;
  const int lo = min(split * per, tiles) * kAttKeys, hi = min(min((split + 1) * per, tiles) * kAttKeys, n);
  const int64_t cache0 = (int64_t)a.slots[row] * a.max_pos * a.cache_ld;
  {
    const float *q = a.qa + ((int64_t)row * m.heads + h0 + warp) * D;  // a warp brings one head's query
#pragma unroll 4
    for (int d = lane; d < ld; d += 32) qs[warp * ld + d] = warp < nh && d < D ? q[d] : 0.0f;
  }
  float acc[kAttHeads][NR][2];
#pragma unroll
  for (int h = 0; h < kAttHeads; ++h)
#pragma unroll
    for (int j = 0; j < NR; ++j) acc[h][j][0] = acc[h][j][1] = 0.0f;
  float mx = -INFINITY, sum = 0.0f;  // of head `warp`
  const bool vec = a.cache_half && a.cache_ld % 8 == 0;
  for (int k0 = lo; k0 < hi; k0 += kAttKeys) {
    __syncthreads();
    if (vec) {
      const bf16 *c = static_cast<const bf16 *>(a.cache) + cache0;
      const int u8 = (ld + 7) / 8;
      // a warp takes every eighth key, its lanes 16 bytes each; the cache row's padding beyond D is zero
      for (int u = lane; u < u8; u += 32) {
        const int d = u * 8;
        uint4 v[kAttKeys / 8];
#pragma unroll
        for (int j = 0; j < kAttKeys / 8; ++j) {
          const int k = warp + 8 * j;
          v[j] = make_uint4(0, 0, 0, 0);
          if (k0 + k < hi && d < (int)a.cache_ld) v[j] = *reinterpret_cast<const uint4 *>(c + (int64_t)(k0 + k) * a.cache_ld + d);
        }
#pragma unroll
        for (int j = 0; j < kAttKeys / 8; ++j) {
          float *o = ks + (warp + 8 * j) * ld + d;
          *reinterpret_cast<float4 *>(o) = make_float4(bf16_lo(v[j].x), bf16_hi(v[j].x), bf16_lo(v[j].y), bf16_hi(v[j].y));
          if (d + 4 < ld) *reinterpret_cast<float4 *>(o + 4) = make_float4(bf16_lo(v[j].z), bf16_hi(v[j].z), bf16_lo(v[j].w), bf16_hi(v[j].w));
        }
      }
    } else {
      for (int i = tid; i < kAttKeys * ld; i += kAttThreads) {
        const int k = i / ld, d = i % ld;
        ks[i] = k0 + k < hi && d < D ? act_load(a.cache, a.cache_half, cache0 + (int64_t)(k0 + k) * a.cache_ld + d) : 0.0f;
      }
    }
    __syncthreads();
    // scores: lane = key, a warp takes every eighth 16-byte unit of the dimensions for all heads
    float s[kAttHeads];
#pragma unroll
    for (int h = 0; h < kAttHeads; ++h) s[h] = 0.0f;
    for (int u = warp; u < used; u += 8) {
      const float4 k = *reinterpret_cast<const float4 *>(ks + lane * ld + u * 4);
#pragma unroll
      for (int h = 0; h < kAttHeads; ++h) {
        const float4 q = *reinterpret_cast<const float4 *>(qs + h * ld + u * 4);
        s[h] = fmaf(k.x, q.x, fmaf(k.y, q.y, fmaf(k.z, q.z, fmaf(k.w, q.w, s[h]))));
      }
    }
#pragma unroll
    for (int h = 0; h < kAttHeads; ++h) sc[(warp * kAttHeads + h) * kAttKeys + lane] = s[h];
    __syncthreads();
    {
      float v = 0.0f;
#pragma unroll
      for (int w = 0; w < 8; ++w) v += sc[(w * kAttHeads + warp) * kAttKeys + lane];
      if (k0 + lane >= hi) v = -INFINITY;
      const float nm = fmaxf(mx, warp_max(v)), c = expf(mx - nm), p = expf(v - nm);
      sum = fmaf(sum, c, warp_sum(p));
      mx = nm;
      pr[lane * kAttHeads + warp] = p;
      if (lane == 0) corr[warp] = c;
    }
    __syncthreads();
    {
      float c[kAttHeads];
#pragma unroll
      for (int h = 0; h < kAttHeads; ++h) c[h] = corr[h];
#pragma unroll
      for (int j = 0; j < NR; ++j)
#pragma unroll
        for (int h = 0; h < kAttHeads; ++h) {
          acc[h][j][0] *= c[h];
          acc[h][j][1] *= c[h];
        }
    }
    const int nk = min(kAttKeys, hi - k0);
    if (2 * tid < m.rank) {
#pragma unroll 4
      for (int k = 0; k < nk; ++k) {
        const float4 p0 = *reinterpret_cast<const float4 *>(pr + k * kAttHeads), p1 = *reinterpret_cast<const float4 *>(pr + k * kAttHeads + 4);
        const float p[8] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
#pragma unroll
        for (int j = 0; j < NR; ++j) {
          const int d = 2 * tid + 512 * j;
          if (NR > 1 && d >= m.rank) break;
          const float2 v = *reinterpret_cast<const float2 *>(ks + k * ld + d);
#pragma unroll
          for (int h = 0; h < kAttHeads; ++h) {
            acc[h][j][0] = fmaf(p[h], v.x, acc[h][j][0]);
            acc[h][j][1] = fmaf(p[h], v.y, acc[h][j][1]);
          }
        }
      }
    }
  }
  // partials: maximum, sum, weighted latents
  const int64_t ps = m.rank + 2;
  float *out = a.part + (((int64_t)row * m.heads + h0) * a.splits + split) * ps;
  if (warp < nh && lane == 0) {
    out[(int64_t)warp * a.splits * ps] = mx;
    out[(int64_t)warp * a.splits * ps + 1] = sum;
  }
#pragma unroll
  for (int h = 0; h < kAttHeads; ++h)
    if (h < nh)
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int d = 2 * tid + 512 * j;
        float *o = out + (int64_t)h * a.splits * ps + 2;
        if (d < m.rank) o[d] = acc[h][j][0];
        if (d + 1 < m.rank) o[d + 1] = acc[h][j][1];
      }
}

// ---- the same on the tensor cores, for a bfloat16 cache: 16 heads, 32 keys at a time.  Queries and weights enter as two
// bfloat16 terms each, the cache rows as they are.

constexpr int kMmaHeads = 16, kMmaKeys = 32, kMmaThreads = 256;

__host__ __device__ inline int mma_dp(int D) { return (D + 15) & ~15; }
__host__ __device__ inline int mma_smem(int D) {
  return 2 * kMmaKeys * (mma_dp(D) + 8) * 2 + 8 * kMmaHeads * (kMmaKeys + 1) * 4 + 2 * kMmaHeads * (kMmaKeys + 8) * 2 + kMmaHeads * 4;
}

// NT: 8-wide tiles of the latent per warp in the second product (rank <= 64 * NT).  KS: 16-wide steps of the dimensions
// per warp in the first (D <= 128 * KS); a warp keeps its share of the queries in registers.
template <int NT, int KS>
__global__ void __launch_bounds__(kMmaThreads) latent_attn_mma_kernel(const LatentArgs a) {
  extern __shared__ __align__(16) uint8_t mraw[];
  const LatentShape &m = a.m;
  const int D = m.rank + m.rot_dim, DP = mma_dp(D), DS = DP + 8, PS = kMmaKeys + 8;
  bf16 *ks = reinterpret_cast<bf16 *>(mraw);                                // two stages of [32][DS]
  float *sc = reinterpret_cast<float *>(ks + 2 * kMmaKeys * DS);            // [8 shares of D][16][33]
  bf16 *ph = reinterpret_cast<bf16 *>(sc + 8 * kMmaHeads * (kMmaKeys + 1)), *pl = ph + kMmaHeads * PS;
  float *corr = reinterpret_cast<float *>(pl + kMmaHeads * PS);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * kMmaHeads, row = blockIdx.z, nh = min(kMmaHeads, m.heads - h0);
  const int tr = lane >> 2, tc = (lane & 3) * 2;
  pdl_launch();
  pdl_wait();
  const int n = a.positions[row] + 1;
  const int tiles = (n + kMmaKeys - 1) / kMmaKeys, per = (tiles + a.splits - 1) / a.splits;
  const int t_lo = min(split * per, tiles), t_hi = min(t_lo + per, tiles);
  const bf16 *cache = static_cast<const bf16 *>(a.cache) + (int64_t)a.slots[row] * a.max_pos * a.cache_ld;
  // the cache row's padding up to a multiple of eight is zero; beyond it the staged row is zero-filled
  auto load = [&](int t, bf16 *dst) {
    for (int u = lane; u < DP / 8; u += 32) {
#pragma unroll
      for (int k = warp; k < kMmaKeys; k += kMmaThreads / 32) {
        const int p = t * kMmaKeys + k;
        const bool live = p < n && u * 8 < (int)a.cache_ld;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst + k * DS + u * 8)),
                     "l"(cache + (live ? (int64_t)p * a.cache_ld + u * 8 : 0)), "r"(live ? 16 : 0)
                     : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t_lo < t_hi) load(t_lo, ks);
  uint32_t QH[KS][4], QL[KS][4];
  if (t_lo < t_hi) {
    const float *q = a.qa + ((int64_t)row * m.heads + h0) * D;
#pragma unroll
    for (int i = 0; i < KS; ++i)
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int h = tr + (f & 1) * 8, d = (warp * KS + i) * 16 + (f >> 1) * 8 + tc;
        split_pair(h < nh && d < D ? q[(int64_t)h * D + d] : 0.0f, h < nh && d + 1 < D ? q[(int64_t)h * D + d + 1] : 0.0f, QH[i][f], QL[i][f]);
      }
  }
  float O[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[i][e] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};  // of heads 2 * warp, 2 * warp + 1
  for (int t = t_lo; t < t_hi; ++t) {
    bf16 *k_s = ks + ((t - t_lo) & 1) * kMmaKeys * DS;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t + 1 < t_hi) load(t + 1, ks + ((t + 1 - t_lo) & 1) * kMmaKeys * DS);
    float P[4][4] = {};
#pragma unroll
    for (int i = 0; i < KS; ++i) {
      const int k = (warp * KS + i) * 16;
      if (k >= DP) break;
#pragma unroll
      for (int j = 0; j < 2; ++j) {  // 16 keys at a time
        uint32_t B[4];
        ldsm4(B, k_s + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * DS + k + ((lane >> 3) & 1) * 8);
        mma16816(P[2 * j], QH[i], B[0], B[1]);
        mma16816(P[2 * j + 1], QH[i], B[2], B[3]);
        mma16816(P[2 * j], QL[i], B[0], B[1]);
        mma16816(P[2 * j + 1], QL[i], B[2], B[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[(warp * kMmaHeads + tr + (e >> 1) * 8) * (kMmaKeys + 1) + j * 8 + tc + (e & 1)] = P[j][e];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int h = 2 * warp + i;
      float v = 0.0f;
#pragma unroll
      for (int w = 0; w < 8; ++w) v += sc[(w * kMmaHeads + h) * (kMmaKeys + 1) + lane];
      if (t * kMmaKeys + lane >= n) v = -INFINITY;
      const float nm = fmaxf(mx[i], warp_max(v)), c = expf(mx[i] - nm), p = expf(v - nm);
      sum[i] = fmaf(sum[i], c, warp_sum(p));
      mx[i] = nm;
      const bf16 hi = __float2bfloat16_rn(p);
      ph[h * PS + lane] = hi;
      pl[h * PS + lane] = __float2bfloat16_rn(p - __bfloat162float(hi));
      if (lane == 0) corr[h] = c;
    }
    __syncthreads();
    const float c0 = corr[tr], c1 = corr[tr + 8];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      O[i][0] *= c0;
      O[i][1] *= c0;
      O[i][2] *= c1;
      O[i][3] *= c1;
    }
#pragma unroll
    for (int k = 0; k < kMmaKeys; k += 16) {
      uint32_t A[4], L[4], B[4];
      ldsm4(A, ph + (lane & 15) * PS + k + (lane >> 4) * 8);
      ldsm4(L, pl + (lane & 15) * PS + k + (lane >> 4) * 8);
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        const int r = (warp * NT + i) * 8;
        if (r >= DP) break;  // a warp whose tiles lie past the latent
        ldsm4t(B, k_s + (k + (lane & 15)) * DS + min(r + (lane >> 4) * 8, DP - 8));
        mma16816(O[i], A, B[0], B[1]);
        mma16816(O[i + 1], A, B[2], B[3]);
        mma16816(O[i], L, B[0], B[1]);
        mma16816(O[i + 1], L, B[2], B[3]);
      }
    }
  }
  const int64_t ps = m.rank + 2;
  float *out = a.part + (((int64_t)row * m.heads + h0) * a.splits + split) * ps;
  if (lane == 0)
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (2 * warp + i < nh) {
        out[(int64_t)(2 * warp + i) * a.splits * ps] = mx[i];
        out[(int64_t)(2 * warp + i) * a.splits * ps + 1] = sum[i];
      }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = tr + (e >> 1) * 8, r = (warp * NT + i) * 8 + tc + (e & 1);
      if (h < nh && r < m.rank) out[(int64_t)h * a.splits * ps + 2 + r] = O[i][e];
    }
}

// ---------------------------------------------------------------- merge, W_uv, gate

constexpr int kOutThreads = 512, kOutCols = 32;

// grid: x = slices of a head's value dimensions, y = head, z = groups of ROWS rows (they share the weights in registers)
template <int ROWS>
__global__ void __launch_bounds__(kOutThreads, 2) latent_output_kernel(const LatentArgs a, int keys_per_tile) {
  extern __shared__ __align__(16) float ctx[];  // [ROWS][ld of W_uv]
  __shared__ float wgt[ROWS][64];
  __shared__ int ranges[ROWS];
  pdl_launch();
  const LatentShape &m = a.m;
  const int h = blockIdx.y, v0 = blockIdx.x * kOutCols, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int kPer = kOutCols / (kOutThreads / 32);  // value dimensions per warp
  uint4 w[kPer][2];  // the first 512 weights of each: they depend on no earlier kernel
#pragma unroll
  for (int j = 0; j < kPer; ++j)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int v = v0 + warp + j * (kOutThreads / 32), k = lane * 8 + q * 256;
      w[j][q] = v < m.vdim && k < (int)a.uv.ld ? ld_stream16(a.uv.w + ((int64_t)h * m.vdim + v) * a.uv.ld + k) : make_uint4(0, 0, 0, 0);
    }
  pdl_wait();
  const int64_t ps = m.rank + 2;
  const int row0 = blockIdx.z * ROWS, nr = min(ROWS, a.rows - row0), ld = (int)a.uv.ld;
  if (warp < nr) {
    // the ranges of the row that hold keys (the others are empty)
    const int tiles = a.positions[row0 + warp] / keys_per_tile + 1, per = (tiles + a.splits - 1) / a.splits, live = (tiles + per - 1) / per;
    if (lane == 0) ranges[warp] = live;
    const float *part = a.part + ((int64_t)(row0 + warp) * m.heads + h) * a.splits * ps;
    const float m0 = lane < live ? part[lane * ps] : -INFINITY, m1 = lane + 32 < live ? part[(lane + 32) * ps] : -INFINITY;
    const float l0 = lane < live ? part[lane * ps + 1] : 0.0f, l1 = lane + 32 < live ? part[(lane + 32) * ps + 1] : 0.0f;
    const float mx = warp_max(fmaxf(m0, m1));
    const float e0 = lane < live ? expf(m0 - mx) : 0.0f, e1 = lane + 32 < live ? expf(m1 - mx) : 0.0f;
    const float l = warp_sum(e0 * l0 + e1 * l1);
    wgt[warp][lane] = e0 / l;
    wgt[warp][lane + 32] = e1 / l;
  }
  __syncthreads();
  constexpr int kFlight = ROWS == 1 ? 16 : 4;  // partials of a row in flight
  for (int i = tid; i < ld; i += kOutThreads)
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      if (r >= nr) break;
      const int live = i < m.rank ? ranges[r] : 0;
      const float *part = a.part + ((int64_t)(row0 + r) * m.heads + h) * a.splits * ps + 2 + i;
      float c = 0.0f;
      for (int s0 = 0; s0 < live; s0 += kFlight, part += kFlight * (int)ps) {
        float p[kFlight];
#pragma unroll
        for (int j = 0; j < kFlight; ++j) p[j] = s0 + j < live ? part[j * (int)ps] : 0.0f;
#pragma unroll
        for (int j = 0; j < kFlight; ++j) c = fmaf(wgt[r][s0 + j], p[j], c);
      }
      ctx[r * ld + i] = c;
    }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < kPer; ++j) {
    const int v = v0 + warp + j * (kOutThreads / 32);
    if (v >= m.vdim) break;
    float s[ROWS] = {};
    for (int k = lane * 8, q = 0; k < ld; k += 256, ++q) {
      const uint4 x = q == 0 ? w[j][0] : q == 1 ? w[j][1] : ld_stream16(a.uv.w + ((int64_t)h * m.vdim + v) * ld + k);
#pragma unroll
      for (int r = 0; r < ROWS; ++r)
        if (r < nr) {
          const float4 c0 = *reinterpret_cast<const float4 *>(ctx + r * ld + k), c1 = *reinterpret_cast<const float4 *>(ctx + r * ld + k + 4);
          s[r] = fmaf(bf16_lo(x.x), c0.x, fmaf(bf16_hi(x.x), c0.y, s[r]));
          s[r] = fmaf(bf16_lo(x.y), c0.z, fmaf(bf16_hi(x.y), c0.w, s[r]));
          s[r] = fmaf(bf16_lo(x.z), c1.x, fmaf(bf16_hi(x.z), c1.y, s[r]));
          s[r] = fmaf(bf16_lo(x.w), c1.z, fmaf(bf16_hi(x.w), c1.w, s[r]));
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const float t = warp_sum(s[r]);
      const int64_t row = row0 + r;
      if (lane == 0 && r < nr) act_store(a.out.p, a.out.half, row * a.out.ld + h * m.vdim + v, t * sigmoid_f(a.gate[row * a.gate_ld + h * m.vdim + v]));
    }
  }
}

// ---------------------------------------------------------------- long portions on the tensor cores

constexpr int kPfThreads = 128, kPfQ = 64, kPfK = 64;

__host__ __device__ inline int pf_qd(const LatentShape &m) { return (m.dim + m.rot_dim + 15) & ~15; }
__host__ __device__ inline int pf_smem(int qd, int dv) { return (kPfQ * (qd + 8) + 2 * kPfK * (qd + 8) + 2 * kPfK * (dv + 8)) * 2; }

// DV: value dimensions, padded to 32, 64, 128 or 256
template <int DV>
__global__ void __launch_bounds__(kPfThreads) latent_prefill_kernel(const LatentPrefillArgs a) {
  extern __shared__ __align__(16) bf16 sh[];
  const LatentShape &m = a.m;
  const int qd = pf_qd(m), QS = qd + 8, VS = DV + 8;
  bf16 *q_s = sh, *k_s = q_s + kPfQ * QS, *v_s = k_s + 2 * kPfK * QS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  const int r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kPfQ;  // the longest rows first
  const int64_t last = a.start + min(r0 + kPfQ, a.rows) - 1;      // the last position this tile's queries see
  const int n_tiles = (int)(last / kPfK) + 1;
  pdl_launch();
  pdl_wait();
  auto load_tile = [&](int t, int st) {
    bf16 *kd = k_s + st * kPfK * QS, *vd = v_s + st * kPfK * VS;
    const int nu = m.dim / 8, ru = m.rot_dim / 8, ku = nu + ru, vu = m.vdim / 8;
    // a warp takes every fourth key, its lanes the key's 16-byte units: unrotated, rotated, values
    for (int u = lane; u < ku + vu; u += 32) {
      const bf16 *src = u < nu ? a.kv + h * m.dim + u * 8 : u < ku ? a.cache + m.rank + (u - nu) * 8 : a.kv + m.heads * m.dim + h * m.vdim + (u - ku) * 8;
      const int64_t ld = u >= nu && u < ku ? a.cache_ld : a.kv_ld;
      bf16 *dst = u < ku ? kd + u * 8 : vd + (u - ku) * 8;
      const int ds = u < ku ? QS : VS;
      const int64_t p0 = (int64_t)t * kPfK;
#pragma unroll 8
      for (int k = warp; k < kPfK; k += kPfThreads / 32) {
        const bool live = p0 + k <= last;
        cp16(dst + k * ds, src + (live ? p0 + k : 0) * ld, live);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // columns no copy touches: zero once
  for (int i = tid; i < 2 * kPfK * (qd - m.dim - m.rot_dim); i += kPfThreads) {
    const int w = qd - m.dim - m.rot_dim;
    k_s[(i / w) * QS + m.dim + m.rot_dim + i % w] = __float2bfloat16_rn(0.0f);
  }
  for (int i = tid; i < 2 * kPfK * (DV - m.vdim); i += kPfThreads) v_s[(i / (DV - m.vdim)) * VS + m.vdim + i % (DV - m.vdim)] = __float2bfloat16_rn(0.0f);
  load_tile(0, 0);
  const int q_ld = m.heads * (m.dim + m.rot_dim);
  {
    // queries, eight dimensions at a time (dim and rot_dim are multiples of eight; pairs do not straddle)
    const int units = qd / 8, live = (m.dim + m.rot_dim) / 8;
#pragma unroll 4
    for (int i = tid; i < kPfQ * units; i += kPfThreads) {
      const int r = i / units, u = i % units;
      float f[8] = {};
      if (r0 + r < a.rows && u < live) {
        const float4 *x = reinterpret_cast<const float4 *>(a.q + (int64_t)(r0 + r) * q_ld + h * (m.dim + m.rot_dim) + u * 8);
        const float4 x0 = x[0], x1 = x[1];
        f[0] = x0.x, f[1] = x0.y, f[2] = x0.z, f[3] = x0.w, f[4] = x1.x, f[5] = x1.y, f[6] = x1.z, f[7] = x1.w;
        const int j = u * 8 - m.dim;  // place in the rotated part
        if (j >= 0) {
          const float *cs = a.cs + (a.start + r0 + r) * m.rot_dims + j;
#pragma unroll
          for (int e = 0; e < 8; e += 2)
            if (j + e < m.rot_dims) {
              const float c = cs[e], s = cs[e + 1], x = f[e], y = f[e + 1];
              f[e] = x * c - y * s;
              f[e + 1] = y * c + x * s;
            }
        }
      }
      *reinterpret_cast<uint4 *>(q_s + r * QS + u * 8) =
          make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
    }
  }
  float O[DV / 8][4];
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[n][e] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  const int tr = lane >> 2, tc = (lane & 3) * 2, i0 = warp * 16;
  const int64_t pos0 = a.start + r0 + i0 + tr;
  for (int t = 0; t < n_tiles; ++t) {
    const int st = t & 1;
    if (t + 1 < n_tiles) {
      load_tile(t + 1, st ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16 *kt = k_s + st * kPfK * QS, *vt = v_s + st * kPfK * VS;
    float P[8][4] = {};
#pragma unroll 2
    for (int k = 0; k < qd; k += 16) {
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
        const int64_t key = (int64_t)t * kPfK + n * 8 + tc + (e & 1);
        P[n][e] = key <= pos0 + (e >> 1) * 8 ? P[n][e] * m.scale : -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], P[n][e]);
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 1));
      nm[e] = fmaxf(nm[e], __shfl_xor_sync(0xffffffffu, nm[e], 2));
    }
    // key 0 is visible to every query, so nm is finite from the first tile on
    const float c0 = expf(mx[0] - nm[0]), c1 = expf(mx[1] - nm[1]);
    float ts[2] = {0.0f, 0.0f};
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        P[n][e] = expf(P[n][e] - nm[e >> 1]);
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
      if (r < a.rows && v < m.vdim) {
        const float g = a.gate[(int64_t)r * a.gate_ld + h * m.vdim + v];
        a.out[(int64_t)r * a.out_ld + h * m.vdim + v] = __float2bfloat16_rn(O[n][e] / sum[e >> 1] * sigmoid_f(g));
      }
    }
}

template <int DV>
int32_t prefill(const LatentPrefillArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(latent_prefill_kernel<DV>, 227 * 1024));
    ready = true;
  }
  return launch_kernel(latent_prefill_kernel<DV>, dim3((a.rows + kPfQ - 1) / kPfQ, a.m.heads), dim3(kPfThreads), pf_smem(pf_qd(a.m), DV), pdl, s, a);
}

}  // namespace

bool latent_shape_ok(const LatentShape &m) {
  return m.heads >= 1 && m.dim >= 1 && m.vdim >= 1 && m.rank >= 1 && m.rank <= 1024 && m.rot_dim >= 0 && m.rot_dims >= 0 && m.rot_dims % 2 == 0 &&
         m.rot_dims <= m.rot_dim && att_smem(m.rank + m.rot_dim) <= 227 * 1024 && m.dim <= 4096;
}

template <int ROWS>
int32_t prep(const LatentArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(latent_prep_kernel<ROWS>, 160 * 1024));
    ready = true;
  }
  const int slices = (a.m.rank + kPrepRanks - 1) / kPrepRanks, ys = a.m.heads * slices;
  const size_t smem = (size_t)(ROWS * ((a.m.dim + 3) & ~3) + 16 * ROWS * kPrepRanks) * 4;
  return launch_kernel(latent_prep_kernel<ROWS>, dim3((a.rows + ROWS - 1) / ROWS, ys + ROWS), dim3(kPrepThreads), smem, pdl, s, a, slices, ys);
}

int32_t launch_latent_prep(const LatentArgs &a, bool queries, bool pdl, cudaStream_t s) {
  if (!queries) return launch_kernel(latent_append_kernel, dim3(a.rows), dim3(128), 0, pdl, s, a);
  return a.rows > 2 ? prep<4>(a, pdl, s) : prep<2>(a, pdl, s);
}

bool latent_attention_mma(const LatentArgs &a) { return a.cache_half && a.m.rank + a.m.rot_dim <= 1152 && mma_smem(a.m.rank + a.m.rot_dim) <= 227 * 1024; }

int latent_attention_groups(const LatentArgs &a) {
  const int g = latent_attention_mma(a) ? kMmaHeads : kAttHeads;
  return (a.m.heads + g - 1) / g;
}

int32_t launch_latent_attention(const LatentArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(latent_attn_kernel<1>, 227 * 1024));
    CMLD_TRY(allow_smem(latent_attn_kernel<2>, 227 * 1024));
    CMLD_TRY(allow_smem(latent_attn_mma_kernel<2, 2>, 227 * 1024));
    CMLD_TRY(allow_smem(latent_attn_mma_kernel<4, 3>, 227 * 1024));
    CMLD_TRY(allow_smem(latent_attn_mma_kernel<8, 5>, 227 * 1024));
    CMLD_TRY(allow_smem(latent_attn_mma_kernel<16, 9>, 227 * 1024));
    ready = true;
  }
  const dim3 grid(a.splits, latent_attention_groups(a), a.rows);
  const int D = a.m.rank + a.m.rot_dim;
  if (latent_attention_mma(a)) {
    const dim3 block(kMmaThreads);
    if (a.m.rank <= 128 && D <= 256) return launch_kernel(latent_attn_mma_kernel<2, 2>, grid, block, mma_smem(D), pdl, s, a);
    if (a.m.rank <= 256 && D <= 384) return launch_kernel(latent_attn_mma_kernel<4, 3>, grid, block, mma_smem(D), pdl, s, a);
    if (a.m.rank <= 512 && D <= 640) return launch_kernel(latent_attn_mma_kernel<8, 5>, grid, block, mma_smem(D), pdl, s, a);
    return launch_kernel(latent_attn_mma_kernel<16, 9>, grid, block, mma_smem(D), pdl, s, a);
  }
  if (a.m.rank <= 512) return launch_kernel(latent_attn_kernel<1>, grid, dim3(kAttThreads), att_smem(D), pdl, s, a);
  return launch_kernel(latent_attn_kernel<2>, grid, dim3(kAttThreads), att_smem(D), pdl, s, a);
}

int32_t launch_latent_output(const LatentArgs &a, bool pdl, cudaStream_t s) {
  if (a.splits > 64) return fail(CMLD_ERR_INVALID, "latent attention: %d ranges, at most 64", a.splits);
  static_assert(kMmaKeys == kAttKeys, "both attention kernels cut a range at the same keys");
  const dim3 grid((a.m.vdim + kOutCols - 1) / kOutCols, a.m.heads, a.rows <= 2 ? a.rows : (a.rows + 3) / 4);
  if (a.rows <= 2) return launch_kernel(latent_output_kernel<1>, grid, dim3(kOutThreads), (size_t)a.uv.ld * 4, pdl, s, a, kMmaKeys);
  return launch_kernel(latent_output_kernel<4>, grid, dim3(kOutThreads), (size_t)4 * a.uv.ld * 4, pdl, s, a, kMmaKeys);
}

bool latent_prefill_fits(const LatentShape &m, int64_t cache_ld, int64_t kv_ld) {
  if (m.dim % 8 || m.rot_dim % 8 || m.vdim % 8 || m.rank % 8 || cache_ld % 8 || kv_ld % 8 || m.vdim > 256) return false;
  const int dv = m.vdim <= 32 ? 32 : m.vdim <= 64 ? 64 : m.vdim <= 128 ? 128 : 256;
  return pf_smem(pf_qd(m), dv) <= 227 * 1024;
}

int32_t launch_latent_prefill(const LatentPrefillArgs &a, bool pdl, cudaStream_t s) {
  if (a.m.vdim <= 32) return prefill<32>(a, pdl, s);
  if (a.m.vdim <= 64) return prefill<64>(a, pdl, s);
  if (a.m.vdim <= 128) return prefill<128>(a, pdl, s);
  return prefill<256>(a, pdl, s);
}

}  // namespace cmld
