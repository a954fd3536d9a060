// Linear attention with a decay per key channel and token (gated linear attention), a portion of one sequence in chunks of
// 64 tokens.  With a_t the decays of token t, B_t = sum of log a over the chunk's tokens up to t, S the state before it:
//   o_t = (q_t exp(B_t))^T S + sum over s <= t of A_ts v_s,   A_ts = sum over channels of q_t k_s exp(B_t - B_s)
//   S'  = diag(exp(B_end)) S + sum over s of (k_s exp(B_end - B_s)) v_s^T
// Every exponent is <= 0.  exp(-B_s) alone would overflow under strong decays, so A is cut into blocks of 16 x 16 tokens
// (secondary chunks, as in "Gated Linear Attention Transformers with Hardware-Efficient Training", Yang et al.), those on the
// diagonal once more into 8 x 8: a block off the diagonal factors at the borders between the blocks and runs on the tensor
// cores, one on the diagonal takes the exponential of each pair's difference.
//
// gated_prep_kernel: everything that does not need the state, all chunks and heads at once: decays, A, the scaled queries
//   and keys, as two bfloat16 terms each.
// gated_scan_kernel: chunk after chunk for 32 value columns of a head: outputs and state, the state in registers in 32-bit
//   (two bfloat16 terms where it enters the tensor cores).  The step-by-step form is in lightning.cu.
#include "layered.cuh"
#include "mma_sync.cuh"

namespace cmld {

namespace {

constexpr int kC = 64, kSub = 16, kPrepThreads = 256, kCols = 32, kScanThreads = 128;

__host__ __device__ inline int pad16(int n) { return (n + 15) & ~15; }
__host__ __device__ inline int pad32(int n) { return (n + 31) & ~31; }

// One chunk of one head in scratch, in bf16 elements: q hi, q lo, k hi, k lo [64][dp]; A hi, A lo [64][64]; v [64][vp];
// then exp(B_end) [dp] f32.
struct ChunkLayout {
  int dp, vp;
  int64_t a, v, d, bytes;
};
__host__ __device__ inline ChunkLayout chunk_layout(int dim, int vdim) {
  ChunkLayout L{};
  L.dp = pad16(dim);
  L.vp = pad32(vdim);
  L.a = 4ll * kC * L.dp;
  L.v = L.a + 2 * kC * kC;
  L.d = L.v + (int64_t)kC * L.vp;
  L.bytes = L.d * 2 + L.dp * 4;
  return L;
}

__host__ __device__ inline int prep_w_ld(int rank) { return ((rank + 7) & ~7) + 8; }
__host__ __device__ inline int prep_u_ld(int rank) { return (rank + 3) & ~3; }
__host__ __device__ inline int prep_smem(int dim, int rank) {
  const int dp = pad16(dim), rows = kC * (dp + 8) * 4, w = dim * prep_w_ld(rank) * 2 + kC * prep_u_ld(rank) * 4;
  return 12 * dp * 4 + 2 * rows + (rows > w ? rows : w);
}

// 2^x, x <= 0 here
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// log2(sigmoid(z)); log(1 + e) by its series where e is small
__device__ __forceinline__ float log2_sigmoid(float z) {
  const float kLog2e = 1.44269504f, e = ex2(-fabsf(z) * kLog2e);
  const float l = e > 0.015625f ? __log2f(1.0f + e) : e * kLog2e * fmaf(-e, fmaf(-e, 0.33333334f, 0.5f), 1.0f);
  return fmaf(fminf(z, 0.0f), kLog2e, -l);
}

// Logarithms of decays are to base 2 in this kernel.
__global__ void __launch_bounds__(kPrepThreads, 2) gated_prep_kernel(const LightningArgs a, uint8_t *scratch) {
  extern __shared__ __align__(16) uint8_t raw[];
  const ChunkLayout L = chunk_layout(a.dim, a.vdim);
  const int dp = L.dp, ld = dp + 8, rank = a.channel.w.cols, wl = prep_w_ld(rank), ul = prep_u_ld(rank);
  float *T = reinterpret_cast<float *>(raw);         // [4][dp]: log decays summed over 16 tokens,
  float *before = T + 4 * dp, *rest = before + 4 * dp;  //   over the 16s before, over this one and those after it
  float *lb = T + 12 * dp;                    // [64][ld]: log decays summed since the 16 tokens began
  float *q = lb + kC * ld, *k = q + kC * ld;  // [64][ld]
  bf16 *w = reinterpret_cast<bf16 *>(k);      // first the decay weights [dim][wl] and the low-rank rows [64][ul]
  float *u = reinterpret_cast<float *>(w + a.dim * wl);
  const int h = blockIdx.x, c0 = blockIdx.y * kC, len = min(kC, a.rows - c0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  uint8_t *out = scratch + ((int64_t)blockIdx.y * a.heads + h) * L.bytes;
  bf16 *o16 = reinterpret_cast<bf16 *>(out);
  pdl_launch();
  const int units = (int)a.channel.w.ld / 8;
  for (int i = tid; i < a.dim * units; i += kPrepThreads)
    *reinterpret_cast<uint4 *>(w + (i / units) * wl + (i % units) * 8) =
        *reinterpret_cast<const uint4 *>(a.channel.w.w + (int64_t)(h * a.dim + i / units) * a.channel.w.ld + (i % units) * 8);
  if (!a.late_wait) pdl_wait();
  const int64_t hd = (int64_t)a.heads * a.dim;
  const float *x = static_cast<const float *>(a.qkv) + (int64_t)c0 * a.ld + h * a.dim, *xv = x + 2 * hd + h * (a.vdim - a.dim);
  const bool vec = ((a.ld | a.dim) & 3) == 0 && (reinterpret_cast<uintptr_t>(a.qkv) & 15) == 0;
  const bool vec_v = vec && (a.vdim & 3) == 0;
  // a head's rows of one chunk; what lies past the portion or the sizes is zero
  auto bring = [&](float *dst, const float *src) {
    if (vec) {
#pragma unroll 4
      for (int t = warp; t < kC; t += kPrepThreads / 32)
        for (int d = lane * 4; d < dp; d += 128) {
          const bool live = t < len && d < a.dim;
          cp16(dst + t * ld + d, live ? src + t * a.ld + d : src, live);
        }
    } else {
      for (int t = warp; t < kC; t += kPrepThreads / 32)
        for (int d = lane; d < dp; d += 32) dst[t * ld + d] = t < len && d < a.dim ? __ldcg(src + t * a.ld + d) : 0.0f;
    }
  };
  bring(q, x);
  asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll 4
  for (int i = tid; i < kC * ul; i += kPrepThreads) u[i] = i / ul < len && i % ul < rank ? __ldcg(a.channel.x + (c0 + i / ul) * a.ld + i % ul) : 0.0f;
  __syncthreads();
  // a thread sums a channel's log decays over 16 tokens
  for (int i = tid; i < 4 * dp; i += kPrepThreads) {
    const int d = i % dp, t0 = i / dp * kSub;
    const bool live = d < a.dim;
    const float b = live ? a.channel.b[h * a.dim + d] : 0.0f;
    float z[kSub];
#pragma unroll
    for (int t = 0; t < kSub; ++t) z[t] = b;
    if (live)
      for (int j = 0; j < rank; j += 4) {
        const uint2 v = *reinterpret_cast<const uint2 *>(w + d * wl + j);  // past the rank: zero
        const float w0 = bf16_lo(v.x), w1 = bf16_hi(v.x), w2 = bf16_lo(v.y), w3 = bf16_hi(v.y);
#pragma unroll
        for (int t = 0; t < kSub; ++t) {
          const float4 f = *reinterpret_cast<const float4 *>(u + (t0 + t) * ul + j);
          z[t] = fmaf(w0, f.x, fmaf(w1, f.y, fmaf(w2, f.z, fmaf(w3, f.w, z[t]))));
        }
      }
    float run = 0.0f;
#pragma unroll
    for (int t = 0; t < kSub; ++t) {
      if (live && t0 + t < len) run = fmaf(log2_sigmoid(z[t]), a.channel.inv_tau, run);
      lb[(t0 + t) * ld + d] = run;
    }
    T[i] = run;
  }
  __syncthreads();
  bring(k, x + hd);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (vec_v) {
#pragma unroll 8
    for (int t = warp; t < kC; t += kPrepThreads / 32)
      for (int c = lane * 4; c < L.vp; c += 128) {
        const float4 v = t < len && c < a.vdim ? __ldcg(reinterpret_cast<const float4 *>(xv + t * a.ld + c)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        *reinterpret_cast<uint2 *>(o16 + L.v + t * L.vp + c) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      }
  } else {
    for (int t = warp; t < kC; t += kPrepThreads / 32)
      for (int c = lane; c < L.vp; c += 32) o16[L.v + t * L.vp + c] = __float2bfloat16_rn(t < len && c < a.vdim ? __ldcg(xv + t * a.ld + c) : 0.0f);
  }
  for (int d = tid; d < dp; d += kPrepThreads) {
    const float s0 = T[d], s1 = T[dp + d], s2 = T[2 * dp + d], s3 = T[3 * dp + d];
    before[d] = 0.0f;
    before[dp + d] = s0;
    before[2 * dp + d] = s0 + s1;
    before[3 * dp + d] = s0 + s1 + s2;
    rest[3 * dp + d] = s3;
    rest[2 * dp + d] = s2 + s3;
    rest[dp + d] = s1 + (s2 + s3);
    rest[d] = s0 + (s1 + (s2 + s3));
    reinterpret_cast<float *>(o16 + L.d)[d] = ex2(rest[d]);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  bf16 *A = o16 + L.a;
  auto put = [&](int t, int s, float v) {
    const bf16 hi = __float2bfloat16_rn(v);
    A[t * kC + s] = hi;
    A[kC * kC + t * kC + s] = __float2bfloat16_rn(v - __bfloat162float(hi));
  };
  const int tr = lane >> 2, tc = (lane & 3) * 2;
  {
    // pairs within eight tokens: a warp takes eight, its lanes the channels
    const int t0 = warp * 8;
    float v[36] = {};
    for (int d = lane; d < dp; d += 32) {
      float kd[8], l[8];
#pragma unroll
      for (int s = 0; s < 8; ++s) {
        kd[s] = k[(t0 + s) * ld + d];
        l[s] = lb[(t0 + s) * ld + d];
      }
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        const float qd = q[(t0 + t) * ld + d];
#pragma unroll
        for (int s = 0; s <= t; ++s) v[t * (t + 1) / 2 + s] = fmaf(qd * kd[s], s < t ? ex2(l[t] - l[s]) : 1.0f, v[t * (t + 1) / 2 + s]);
      }
    }
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      float mine = 0.0f;
#pragma unroll
      for (int s = 0; s <= t; ++s) {
        const float f = warp_sum(v[t * (t + 1) / 2 + s]);
        if (lane == s) mine = f;
      }
      if (lane < 8) put(t0 + t, t0 + lane, a.q_scale * mine);  // zero above the diagonal
      if (lane >= 8 && lane < 16 && (warp & 1) == 0) put(t0 + t, t0 + lane, 0.0f);
    }
  }
  if (warp < 4) {
    // the second eight of 16 tokens against the first, factored at the last of those
    const int tk = warp * kSub, tq = tk + 8;
    const float *edge = lb + (tk + 7) * ld;
    float acc[4] = {};
#pragma unroll 2
    for (int d0 = 0; d0 < dp; d0 += 16) {
      uint32_t AH[4] = {}, AL[4] = {}, BH[2], BL[2];
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int d = d0 + f * 8 + tc;
        const float2 e = *reinterpret_cast<const float2 *>(edge + d);
        const float2 lq = *reinterpret_cast<const float2 *>(lb + (tq + tr) * ld + d), qv = *reinterpret_cast<const float2 *>(q + (tq + tr) * ld + d);
        const float2 lk = *reinterpret_cast<const float2 *>(lb + (tk + tr) * ld + d), kv = *reinterpret_cast<const float2 *>(k + (tk + tr) * ld + d);
        split_pair(qv.x * ex2(lq.x - e.x), qv.y * ex2(lq.y - e.y), AH[2 * f], AL[2 * f]);
        split_pair(kv.x * ex2(e.x - lk.x), kv.y * ex2(e.y - lk.y), BH[f], BL[f]);
      }
      mma16816(acc, AH, BH[0], BH[1]);
      mma16816(acc, AH, BL[0], BL[1]);
      mma16816(acc, AL, BH[0], BH[1]);
    }
    put(tq + tr, tk + tc, a.q_scale * acc[0]);
    put(tq + tr, tk + tc + 1, a.q_scale * acc[1]);
  }
  __syncthreads();
  // queries from the start of their 16 tokens, keys to the end of theirs: as two bf16 terms in place of the 32-bit rows
  // ([hi | lo] of dp each), and to the chunk's edges for the scan
#pragma unroll 2
  for (int t = warp; t < kC; t += kPrepThreads / 32) {
    const int sub = t / kSub;
    const float *Ts = T + sub * dp, *bt = before + sub * dp, *rt = rest + (sub + 1) * dp;
    bf16 *qt = reinterpret_cast<bf16 *>(q + t * ld), *kt = reinterpret_cast<bf16 *>(k + t * ld);
    for (int d0 = 0; d0 < dp; d0 += 256) {  // up to 256 channels in registers between the reads and the writes of a row
      uint32_t w[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int d = d0 + j * 64 + lane * 2;
        if (d >= dp) break;
        const float2 l = *reinterpret_cast<const float2 *>(lb + t * ld + d), qv = *reinterpret_cast<const float2 *>(q + t * ld + d);
        const float2 kv = *reinterpret_cast<const float2 *>(k + t * ld + d), e = *reinterpret_cast<const float2 *>(Ts + d);
        const float2 f = *reinterpret_cast<const float2 *>(bt + d), r = sub < 3 ? *reinterpret_cast<const float2 *>(rt + d) : make_float2(0.0f, 0.0f);
        const float2 qe = make_float2(a.q_scale * qv.x * ex2(l.x), a.q_scale * qv.y * ex2(l.y)), ke = make_float2(kv.x * ex2(e.x - l.x), kv.y * ex2(e.y - l.y));
        split_pair(qe.x, qe.y, w[j][0], w[j][1]);
        split_pair(ke.x, ke.y, w[j][2], w[j][3]);
        uint32_t hi, lo;
        uint32_t *o = reinterpret_cast<uint32_t *>(o16 + t * dp + d);
        split_pair(qe.x * ex2(f.x), qe.y * ex2(f.y), hi, lo);
        o[0] = hi;
        o[kC * dp / 2] = lo;
        split_pair(ke.x * ex2(r.x), ke.y * ex2(r.y), hi, lo);
        o[2 * kC * dp / 2] = hi;
        o[3 * kC * dp / 2] = lo;
      }
      __syncwarp();
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int d = d0 + j * 64 + lane * 2;
        if (d >= dp) break;
        *reinterpret_cast<uint32_t *>(qt + d) = w[j][0];
        *reinterpret_cast<uint32_t *>(qt + dp + d) = w[j][1];
        *reinterpret_cast<uint32_t *>(kt + d) = w[j][2];
        *reinterpret_cast<uint32_t *>(kt + dp + d) = w[j][3];
      }
    }
  }
  __syncthreads();
  // blocks of 16 x 16 below the diagonal: warp 0..5 = (1,0), (2,0), (2,1), (3,0), (3,1), (3,2)
  if (warp < 6) {
    const int bi = warp == 0 ? 1 : warp < 3 ? 2 : 3, bj = warp == 0 ? 0 : warp < 3 ? warp - 1 : warp - 3;
    const bf16 *q16 = reinterpret_cast<const bf16 *>(q + bi * kSub * ld), *k16 = reinterpret_cast<const bf16 *>(k + bj * kSub * ld);
    float acc[2][4] = {};
#pragma unroll 2
    for (int d0 = 0; d0 < dp; d0 += 16) {
      uint32_t AH[4], AL[4], BH[4], BL[4];
      const bf16 *qa = q16 + (lane & 15) * 2 * ld + d0 + (lane >> 4) * 8;
      const bf16 *kb = k16 + ((lane & 7) + ((lane >> 4) << 3)) * 2 * ld + d0 + ((lane >> 3) & 1) * 8;
      ldsm4(AH, qa);
      ldsm4(AL, qa + dp);
      ldsm4(BH, kb);
      ldsm4(BL, kb + dp);
      if (bi - bj > 1) {  // the 16s in between
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          float2 g = make_float2(0.0f, 0.0f);
          for (int s = bj + 1; s < bi; ++s) {
            const float2 e = *reinterpret_cast<const float2 *>(T + s * dp + d0 + (f >> 1) * 8 + tc);
            g.x += e.x;
            g.y += e.y;
          }
          split_pair((bf16_lo(AH[f]) + bf16_lo(AL[f])) * ex2(g.x), (bf16_hi(AH[f]) + bf16_hi(AL[f])) * ex2(g.y), AH[f], AL[f]);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma16816(acc[n], AH, BH[2 * n], BH[2 * n + 1]);
        mma16816(acc[n], AH, BL[2 * n], BL[2 * n + 1]);
        mma16816(acc[n], AL, BH[2 * n], BH[2 * n + 1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) put(bi * kSub + tr + (e >> 1) * 8, bj * kSub + n * 8 + tc + (e & 1), acc[n][e]);
  }
  if (a.late_wait) pdl_wait();
}

// MT: 16-row tiles of the state per warp (dim <= 64 * MT)
template <int MT>
struct Scan {
  static constexpr int DP = 64 * MT, QS = DP + 8, AS = kC + 8, VS = kCols + 8;
  static constexpr int kStage = 4 * kC * QS + 2 * kC * AS + kC * VS;  // elements
  static constexpr int kStages = MT <= 2 ? 2 : 1;
  static constexpr int kSmem = (kStages * kStage + 2 * DP * VS) * 2 + kStages * DP * 4;
};

template <int MT>
__global__ void __launch_bounds__(kScanThreads) gated_scan_kernel(const LightningArgs a, const uint8_t *scratch) {
  using C = Scan<MT>;
  constexpr int DP = C::DP, QS = C::QS, AS = C::AS, VS = C::VS;
  extern __shared__ __align__(16) uint8_t raw[];
  bf16 *stage = reinterpret_cast<bf16 *>(raw), *sh_s = stage + C::kStages * C::kStage, *sl_s = sh_s + DP * VS;
  float *dec = reinterpret_cast<float *>(sl_s + DP * VS);
  pdl_launch();
  pdl_wait();
  const ChunkLayout L = chunk_layout(a.dim, a.vdim);
  const int h = blockIdx.x, col0 = blockIdx.y * kCols, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float *st = a.state + ((int64_t)a.slots[0] * a.heads + h) * (int64_t)a.dim * a.vdim;
  const bool fresh = a.positions[0] == 0;
  const int tr = lane >> 2, tc = (lane & 3) * 2;
  float S[MT][4][4];  // rows (warp * MT + m) * 16 .., 32 columns
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp * MT + m) * 16 + tr + (e >> 1) * 8, c = col0 + n * 8 + tc + (e & 1);
        S[m][n][e] = !fresh && d < a.dim && c < a.vdim ? st[(int64_t)d * a.vdim + c] : 0.0f;
      }
  const int chunks = (a.rows + kC - 1) / kC;
  auto load = [&](int c, int sg) {
    const bf16 *src = reinterpret_cast<const bf16 *>(scratch + ((int64_t)c * a.heads + h) * L.bytes);
    bf16 *dst = stage + sg * C::kStage;
#pragma unroll 4
    for (int i = tid; i < 4 * kC * (DP / 8); i += kScanThreads) {
      const int r = i / (DP / 8), d = i % (DP / 8) * 8;
      cp16(dst + r * QS + d, src + (d < L.dp ? (int64_t)r * L.dp + d : 0), d < L.dp);
    }
    dst += 4 * kC * QS;
#pragma unroll 4
    for (int i = tid; i < 2 * kC * (kC / 8); i += kScanThreads) {
      const int r = i / (kC / 8), s = i % (kC / 8) * 8;
      cp16(dst + r * AS + s, src + L.a + r * kC + s, true);
    }
    dst += 2 * kC * AS;
#pragma unroll
    for (int i = tid; i < kC * (kCols / 8); i += kScanThreads) {
      const int r = i / (kCols / 8), s = i % (kCols / 8) * 8;
      cp16(dst + r * VS + s, src + L.v + (int64_t)r * L.vp + col0 + s, true);
    }
    for (int d = tid * 4; d < DP; d += kScanThreads * 4) cp16(dec + sg * DP + d, reinterpret_cast<const float *>(src + L.d) + (d < L.dp ? d : 0), d < L.dp);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0, 0);
  for (int c = 0; c < chunks; ++c) {
    const int sg = C::kStages == 2 ? c & 1 : 0, len = min(kC, a.rows - c * kC), i0 = warp * 16;
    const bf16 *qh = stage + sg * C::kStage, *ql = qh + kC * QS, *kh = ql + kC * QS, *kl = kh + kC * QS, *ah = kl + kC * QS, *al = ah + kC * AS, *v_s = al + kC * AS;
    // the state as two bf16 terms
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          uint32_t hi, lo;
          split_pair(S[m][n][2 * p], S[m][n][2 * p + 1], hi, lo);
          const int o = ((warp * MT + m) * 16 + tr + p * 8) * VS + n * 8 + tc;
          *reinterpret_cast<uint32_t *>(sh_s + o) = hi;
          *reinterpret_cast<uint32_t *>(sl_s + o) = lo;
        }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this chunk and the state have landed, and the previous chunk's readers are done
    if (C::kStages == 2 && c + 1 < chunks) load(c + 1, sg ^ 1);
    float O[4][4] = {};
#pragma unroll 2
    for (int k = 0; k < DP; k += 16) {
      if (k >= L.dp) break;
      uint32_t A[4], Q[4], B[4];
      ldsm4(A, qh + (i0 + (lane & 15)) * QS + k + (lane >> 4) * 8);
      ldsm4(Q, ql + (i0 + (lane & 15)) * QS + k + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 2; ++n) {  // 16 value columns at a time
        ldsm4t(B, sh_s + (k + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], A, B[0], B[1]);
        mma16816(O[2 * n + 1], A, B[2], B[3]);
        mma16816(O[2 * n], Q, B[0], B[1]);
        mma16816(O[2 * n + 1], Q, B[2], B[3]);
        ldsm4t(B, sl_s + (k + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], A, B[0], B[1]);
        mma16816(O[2 * n + 1], A, B[2], B[3]);
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {  // 16 earlier tokens; blocks above the diagonal do not exist
      if (kk > warp) break;
      uint32_t A[4], Q[4], B[4];
      ldsm4(A, ah + (i0 + (lane & 15)) * AS + kk * 16 + (lane >> 4) * 8);
      ldsm4(Q, al + (i0 + (lane & 15)) * AS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        ldsm4t(B, v_s + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], A, B[0], B[1]);
        mma16816(O[2 * n + 1], A, B[2], B[3]);
        mma16816(O[2 * n], Q, B[0], B[1]);
        mma16816(O[2 * n + 1], Q, B[2], B[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + tr + (e >> 1) * 8, col = col0 + n * 8 + tc + (e & 1);
        if (i < len && col < a.vdim) a.out[(int64_t)(c * kC + i) * a.heads * a.vdim + h * a.vdim + col] = O[n][e];
      }
    // the state: diag(exp(B_end)) S + K^T V
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int d = (warp * MT + m) * 16;
      const float d0 = dec[sg * DP + d + tr], d1 = dec[sg * DP + d + tr + 8];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        S[m][n][0] *= d0;
        S[m][n][1] *= d0;
        S[m][n][2] *= d1;
        S[m][n][3] *= d1;
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t A[4], Q[4], B[4];  // K^T: K is stored [token][d], hence the transposed loads
        const int o = (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * QS + d + ((lane >> 3) & 1) * 8;
        ldsm4t(A, kh + o);
        ldsm4t(Q, kl + o);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          ldsm4t(B, v_s + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
          mma16816(S[m][2 * n], A, B[0], B[1]);
          mma16816(S[m][2 * n + 1], A, B[2], B[3]);
          mma16816(S[m][2 * n], Q, B[0], B[1]);
          mma16816(S[m][2 * n + 1], Q, B[2], B[3]);
        }
      }
    }
    __syncthreads();  // the state's terms and, with one stage, the chunk have been read
    if (C::kStages == 1 && c + 1 < chunks) load(c + 1, 0);
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp * MT + m) * 16 + tr + (e >> 1) * 8, c = col0 + n * 8 + tc + (e & 1);
        if (d < a.dim && c < a.vdim) st[(int64_t)d * a.vdim + c] = S[m][n][e];
      }
}

template <int MT>
int32_t scan(const LightningArgs &a, const uint8_t *scratch, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(gated_scan_kernel<MT>, Scan<MT>::kSmem));
    ready = true;
  }
  return launch_kernel(gated_scan_kernel<MT>, dim3(a.heads, (a.vdim + kCols - 1) / kCols), dim3(kScanThreads), Scan<MT>::kSmem, pdl, s, a, scratch);
}

}  // namespace

bool gated_chunk_fits(int32_t dim, int32_t rank) { return dim <= 256 && prep_smem(dim, rank) <= 227 * 1024; }

int64_t gated_scratch_bytes(int32_t heads, int32_t dim, int32_t vdim, int64_t rows) {
  return (rows + kC - 1) / kC * heads * chunk_layout(dim, vdim).bytes;
}

int32_t launch_gated_chunks(const LightningArgs &a, void *scratch, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(gated_prep_kernel, 227 * 1024));
    ready = true;
  }
  if (a.half || !a.one_sequence || !gated_chunk_fits(a.dim, a.channel.w.cols)) return fail(CMLD_ERR_SHAPE, "gated linear attention: the chunked form does not take this");
  uint8_t *buf = static_cast<uint8_t *>(scratch);
  CMLD_TRY(launch_kernel(gated_prep_kernel, dim3(a.heads, (a.rows + kC - 1) / kC), dim3(kPrepThreads), prep_smem(a.dim, a.channel.w.cols), pdl, s, a, buf));
  if (a.dim <= 64) return scan<1>(a, buf, pdl, s);
  if (a.dim <= 128) return scan<2>(a, buf, pdl, s);
  return scan<4>(a, buf, pdl, s);
}

}  // namespace cmld
