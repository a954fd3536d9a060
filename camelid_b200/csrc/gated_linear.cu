// Linear attention with a decay per key channel and token (gated linear attention), a portion of one sequence in chunks of
// 64 tokens.  With a_t the decays of token t, B_t = sum of log a over the chunk's tokens up to t, S the state before it:
//   o_t = (q_t exp(B_t))^T S + sum over s <= t of A_ts v_s,   A_ts = sum over channels of q_t k_s exp(B_t - B_s)
//   S'  = diag(exp(B_end)) S + sum over s of (k_s exp(B_end - B_s)) v_s^T
// Every exponent is <= 0.  exp(-B_s) alone would overflow under strong decays, so A is cut into blocks of 16 x 16 tokens
// (secondary chunks, as in "Gated Linear Attention Transformers with Hardware-Efficient Training", Yang et al.): a block off
// the diagonal factors at the borders between the blocks and runs on the tensor cores, a block on the diagonal takes the
// exponential of each pair's difference.
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
__host__ __device__ inline int prep_smem(int dim, int rank) {
  const int dp = pad16(dim), rows = kC * (dp + 1) * 4, qk = 2 * rows, w = dim * prep_w_ld(rank) * 2 + kC * rank * 4;
  return 4 * dp * 4 + rows + (qk > w ? qk : w);
}

__global__ void __launch_bounds__(kPrepThreads) gated_prep_kernel(const LightningArgs a, uint8_t *scratch) {
  extern __shared__ __align__(16) uint8_t raw[];
  const ChunkLayout L = chunk_layout(a.dim, a.vdim);
  const int dp = L.dp, ld = dp + 1, rank = a.channel.w.cols, wl = prep_w_ld(rank);
  float *T = reinterpret_cast<float *>(raw);  // [4][dp]: sums of log decays over 16 tokens
  float *lb = T + 4 * dp;                     // [64][ld]: sums of log decays since the 16 tokens began
  float *q = lb + kC * ld, *k = q + kC * ld;  // [64][ld]
  bf16 *w = reinterpret_cast<bf16 *>(q);      // first the decay weights [dim][wl] and the low-rank rows [64][rank]
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
  for (int i = tid; i < kC * rank; i += kPrepThreads) u[i] = i / rank < len ? __ldcg(a.channel.x + (c0 + i / rank) * a.ld + i % rank) : 0.0f;
  __syncthreads();
  for (int i = tid; i < 4 * dp; i += kPrepThreads) {
    const int d = i % dp, sub = i / dp;
    const float b = d < a.dim ? a.channel.b[h * a.dim + d] : 0.0f;
    float run = 0.0f;
    for (int t = sub * kSub; t < (sub + 1) * kSub; ++t) {
      if (d < a.dim && t < len) {
        float z = 0.0f;
#pragma unroll 8
        for (int j = 0; j < rank; ++j) z = fmaf(__bfloat162float(w[d * wl + j]), u[t * rank + j], z);
        run += log_decay(z + b, a.channel.inv_tau);
      }
      lb[t * ld + d] = run;
    }
    T[i] = run;
  }
  __syncthreads();
  const int64_t hd = (int64_t)a.heads * a.dim;
  const float *x = static_cast<const float *>(a.qkv) + (int64_t)c0 * a.ld;
#pragma unroll 4
  for (int i = tid; i < kC * dp; i += kPrepThreads) {
    const int t = i / dp, d = i % dp;
    const bool live = t < len && d < a.dim;
    const float *p = x + t * a.ld + h * a.dim + d;
    q[t * ld + d] = live ? a.q_scale * __ldcg(p) : 0.0f;
    k[t * ld + d] = live ? __ldcg(p + hd) : 0.0f;
  }
#pragma unroll 4
  for (int i = tid; i < kC * L.vp; i += kPrepThreads) {
    const int t = i / L.vp, c = i % L.vp;
    o16[L.v + i] = __float2bfloat16_rn(t < len && c < a.vdim ? __ldcg(x + t * a.ld + 2 * hd + h * a.vdim + c) : 0.0f);
  }
  __syncthreads();
  // queries from the chunk's start, keys to its end
  for (int i = tid; i < kC * dp / 2; i += kPrepThreads) {
    const int t = i / (dp / 2), d = i % (dp / 2) * 2, sub = t / kSub;
    float qv[2], kv[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float l = lb[t * ld + d + e];
      float from = l, to = T[sub * dp + d + e] - l;
      for (int s = 0; s < 4; ++s) {
        if (s < sub) from += T[s * dp + d + e];
        if (s > sub) to += T[s * dp + d + e];
      }
      qv[e] = q[t * ld + d + e] * expf(from);
      kv[e] = k[t * ld + d + e] * expf(to);
    }
    uint32_t hi, lo;
    uint32_t *o = reinterpret_cast<uint32_t *>(o16 + t * dp + d);
    split_pair(qv[0], qv[1], hi, lo);
    o[0] = hi;
    o[kC * dp / 2] = lo;
    split_pair(kv[0], kv[1], hi, lo);
    o[2 * kC * dp / 2] = hi;
    o[3 * kC * dp / 2] = lo;
  }
  for (int d = tid; d < dp; d += kPrepThreads) reinterpret_cast<float *>(o16 + L.d)[d] = expf(T[d] + T[dp + d] + T[2 * dp + d] + T[3 * dp + d]);
  bf16 *A = o16 + L.a;
  auto put = [&](int t, int s, float v) {
    const bf16 hi = __float2bfloat16_rn(v);
    A[t * kC + s] = hi;
    A[kC * kC + t * kC + s] = __float2bfloat16_rn(v - __bfloat162float(hi));
  };
  // blocks on the diagonal, pair by pair
  constexpr int kPairs = kSub * (kSub + 1) / 2;
  for (int i = tid; i < 4 * kPairs; i += kPrepThreads) {
    const int sub = i / kPairs, r = i % kPairs;
    int t = (int)((sqrtf(8.0f * r + 1.0f) - 1.0f) * 0.5f);
    while (t * (t + 1) / 2 > r) --t;
    while ((t + 1) * (t + 2) / 2 <= r) ++t;
    const int s = sub * kSub + r - t * (t + 1) / 2;
    t += sub * kSub;
    float v = 0.0f;
#pragma unroll 4
    for (int d = 0; d < a.dim; ++d) v = fmaf(q[t * ld + d] * k[s * ld + d], expf(lb[t * ld + d] - lb[s * ld + d]), v);
    put(t, s, v);
  }
  for (int i = tid; i < 4 * kSub * kSub; i += kPrepThreads) {
    const int sub = i / (kSub * kSub), t = i / kSub % kSub, s = i % kSub;
    if (s > t) put(sub * kSub + t, sub * kSub + s, 0.0f);
  }
  // blocks below it: warp 0 (1,0), 1 (2,0), 2 (2,1), 3 (3,0), 4 (3,1), 5 (3,2)
  if (warp < 6) {
    const int bi = warp == 0 ? 1 : warp < 3 ? 2 : 3, bj = warp == 0 ? 0 : warp < 3 ? warp - 1 : warp - 3;
    const int tr = lane >> 2, tc = (lane & 3) * 2;
    float acc[2][4] = {};
    auto qe = [&](int t, int d) {
      float e = lb[t * ld + d];
      for (int s = bj + 1; s < bi; ++s) e += T[s * dp + d];
      return q[t * ld + d] * expf(e);
    };
    auto ke = [&](int s, int d) { return k[s * ld + d] * expf(T[bj * dp + d] - lb[s * ld + d]); };
    for (int d0 = 0; d0 < dp; d0 += 16) {
      uint32_t AH[4], AL[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int t = bi * kSub + tr + (f & 1) * 8, d = d0 + (f >> 1) * 8 + tc;
        split_pair(qe(t, d), qe(t, d + 1), AH[f], AL[f]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t BH[2], BL[2];
#pragma unroll
        for (int f = 0; f < 2; ++f) {
          const int s = bj * kSub + n * 8 + tr, d = d0 + f * 8 + tc;
          split_pair(ke(s, d), ke(s, d + 1), BH[f], BL[f]);
        }
        mma16816(acc[n], AH, BH[0], BH[1]);
        mma16816(acc[n], AH, BL[0], BL[1]);
        mma16816(acc[n], AL, BH[0], BH[1]);
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
