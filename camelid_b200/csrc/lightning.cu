// Linear attention, per head
//   S_t = diag(decay_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// with the state S [dim][vdim] in 32-bit, one per sequence slot, and the decay either fixed per head (lightning attention)
// or computed per token and key channel (gated linear attention).  A sequence starts from zero: the kernels ignore what
// the slot holds when a row's position is 0, so a slot can be handed to the next sequence as it is.
//
// linear_steps_kernel: token after token, the state in registers (32 value columns per CTA), either decay.
// lightning_chunk_kernel: the fixed decay, 64 tokens at a time.  With the tokens of a chunk numbered i, j = 0..63,
//   O = (Q K^T * [decay^(i-j), j <= i]) V + diag(decay^(i+1)) Q S,   S' = decay^64 S + K^T diag(decay^(63-j)) V.
// Q, K, V are bfloat16; the scores, the scaled values and the state enter the tensor cores as two bfloat16 terms each.
#include "layered.cuh"
#include "mma_sync.cuh"

namespace cmld {

namespace {

constexpr int kStepThreads = 256, kStepCols = 32, kStepGroups = kStepThreads / kStepCols;

// shared memory: q, k and, with a decay per channel, the decays of this row
inline size_t steps_smem(const LightningArgs &a) { return (size_t)(a.powers ? 2 : 3) * a.dim * 4; }

// Activations may have been written just before this kernel started (late_wait): they are read past the L1 cache.
__device__ __forceinline__ float act_load_cg(const void *p, int half, int64_t i) {
  if (half) return bf16_lo(__ldcg(reinterpret_cast<const unsigned short *>(p) + i));
  return __ldcg(static_cast<const float *>(p) + i);
}

template <int DPT, bool CHANNEL>
__global__ void __launch_bounds__(kStepThreads) linear_steps_kernel(const LightningArgs a) {
  extern __shared__ __align__(16) float sm[];
  float *qs = sm, *ks = sm + a.dim, *al = ks + a.dim;  // this row's q, k and decays of the head
  __shared__ float red[kStepGroups][kStepCols];
  const int h = blockIdx.x, c = threadIdx.x % kStepCols, g = threadIdx.x / kStepCols;
  const int rank = CHANNEL ? a.channel.w.cols : 0, wl = CHANNEL ? (int)a.channel.w.ld : 0, lane = threadIdx.x & 31;
  const bf16 *w = CHANNEL ? a.channel.w.w + (int64_t)h * a.dim * wl : nullptr;
  pdl_launch();
  // the first 16 decay weights of this thread's channel and its bias: they depend on no earlier kernel
  uint4 pre[2] = {};
  float bias = 0.0f;
  if (CHANNEL && (int)threadIdx.x < a.dim) {
    pre[0] = *reinterpret_cast<const uint4 *>(w + threadIdx.x * wl);
    if (wl > 8) pre[1] = *reinterpret_cast<const uint4 *>(w + threadIdx.x * wl + 8);
    bias = a.channel.b[h * a.dim + threadIdx.x];
  }
  if (!a.late_wait) pdl_wait();
  const int col = blockIdx.y * kStepCols + c;
  const bool live = col < a.vdim;
  const int r0 = a.one_sequence ? 0 : blockIdx.z, n = a.one_sequence ? a.rows : 1;
  float *st = a.state + (((int64_t)a.slots[r0] * a.heads + h) * a.dim) * a.vdim + col;
  const float decay = CHANNEL ? 0.0f : a.powers[(int64_t)h * (kLightningChunk + 1) + 1];
  const bool fresh = a.positions[r0] == 0;
  const int d0 = g * DPT;  // this thread's rows of the state
  float s[DPT];
#pragma unroll
  for (int j = 0; j < DPT; ++j) s[j] = live && !fresh && d0 + j < a.dim ? __ldcg(st + (int64_t)(d0 + j) * a.vdim) : 0.0f;
  const int64_t hd = (int64_t)a.heads * a.dim;
  for (int r = r0; r < r0 + n; ++r) {
    const int64_t row = (int64_t)r * a.ld;
    float u = CHANNEL && lane < rank ? __ldcg(a.channel.x + row + lane) : 0.0f;  // 32 of the low-rank values, one per lane
    for (int i = threadIdx.x; i < a.dim; i += kStepThreads) {
      qs[i] = a.q_scale * act_load_cg(a.qkv, a.half, row + h * a.dim + i);
      ks[i] = act_load_cg(a.qkv, a.half, row + hd + h * a.dim + i);
    }
    const float v = live ? act_load_cg(a.qkv, a.half, row + 2 * hd + h * a.vdim + col) : 0.0f;
    if (CHANNEL) {
      // whole warps, so that every lane can hand out its low-rank value
      for (int i = threadIdx.x; i - lane < a.dim; i += kStepThreads) {
        const bool mine = i < a.dim;
        float z = i == (int)threadIdx.x ? bias : mine ? a.channel.b[h * a.dim + i] : 0.0f;
        for (int j0 = 0; j0 < wl; j0 += 8) {
          if ((j0 & 31) == 0 && (j0 > 0 || i != (int)threadIdx.x)) u = j0 + lane < rank ? __ldcg(a.channel.x + row + j0 + lane) : 0.0f;
          uint4 p = make_uint4(0, 0, 0, 0);
          if (j0 < 16 && i == (int)threadIdx.x) p = j0 == 0 ? pre[0] : pre[1];
          else if (mine) p = *reinterpret_cast<const uint4 *>(w + (int64_t)i * wl + j0);
          const float f[8] = {bf16_lo(p.x), bf16_hi(p.x), bf16_lo(p.y), bf16_hi(p.y), bf16_lo(p.z), bf16_hi(p.z), bf16_lo(p.w), bf16_hi(p.w)};
#pragma unroll
          for (int j = 0; j < 8; ++j) z = fmaf(f[j], __shfl_sync(0xffffffffu, u, (j0 & 31) + j), z);
        }
        if (mine) al[i] = expf(log_decay(z, a.channel.inv_tau));
      }
    }
    __syncthreads();
    float o = 0.0f;
#pragma unroll
    for (int j = 0; j < DPT; ++j)
      if (d0 + j < a.dim) {
        s[j] = fmaf(CHANNEL ? al[d0 + j] : decay, s[j], ks[d0 + j] * v);
        o = fmaf(s[j], qs[d0 + j], o);
      }
    red[g][c] = o;
    __syncthreads();
    if (g == 0 && live) {
      float t = 0.0f;
#pragma unroll
      for (int i = 0; i < kStepGroups; ++i) t += red[i][c];
      a.out[(int64_t)r * a.heads * a.vdim + h * a.vdim + col] = t;
    }
  }
#pragma unroll
  for (int j = 0; j < DPT; ++j)
    if (live && d0 + j < a.dim) st[(int64_t)(d0 + j) * a.vdim] = s[j];
  if (a.late_wait) pdl_wait();
}

constexpr int kC = kLightningChunk, kChunkCols = 32, kChunkThreads = 128;

// shared memory: two stages of Q, K [64][dim + 8] and V [64][40]; V' hi, V' lo [64][40], S hi, S lo [dim][40] (all bf16);
// powers [65]
__host__ __device__ inline int chunk_smem(int dp) {
  return 2 * (2 * kC * (dp + 8) + kC * (kChunkCols + 8)) * 2 + 2 * kC * (kChunkCols + 8) * 2 + 2 * dp * (kChunkCols + 8) * 2 + (kC + 1) * 4 + 16;
}


// MT: 16-row tiles of the state per warp (dim <= 64 * MT)
template <int MT>
__global__ void __launch_bounds__(kChunkThreads) lightning_chunk_kernel(const LightningArgs a) {
  extern __shared__ __align__(16) uint8_t raw[];
  constexpr int DP = 64 * MT, QS = DP + 8, VS = kChunkCols + 8;
  constexpr int kStage = 2 * kC * QS + kC * VS;  // elements: Q, K, V of one chunk
  bf16 *stage = reinterpret_cast<bf16 *>(raw), *vh_s = stage + 2 * kStage, *vl_s = vh_s + kC * VS, *sh_s = vl_s + kC * VS, *sl_s = sh_s + DP * VS;
  float *pw = reinterpret_cast<float *>(sl_s + DP * VS);
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.x, col0 = blockIdx.y * kChunkCols, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i <= kC; i += kChunkThreads) pw[i] = a.powers[(int64_t)h * (kC + 1) + i];
  float *st = a.state + ((int64_t)a.slots[0] * a.heads + h) * (int64_t)a.dim * a.vdim;
  const bool fresh = a.positions[0] == 0;
  const bf16 *x = static_cast<const bf16 *>(a.qkv);
  const int64_t hd = (int64_t)a.heads * a.dim;
  const int tr = lane >> 2, tc = (lane & 3) * 2;  // accumulator fragment: rows tr, tr + 8, columns tc, tc + 1
  // state tiles of this warp: rows (warp * MT + m) * 16 .., 32 columns
  float S[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp * MT + m) * 16 + tr + (e >> 1) * 8, c = col0 + n * 8 + tc + (e & 1);
        S[m][n][e] = !fresh && d < a.dim && c < a.vdim ? st[(int64_t)d * a.vdim + c] : 0.0f;
      }
  const bool vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0;
  // a chunk's rows into a stage; rows past the end and columns past the sizes are zero
  auto load = [&](int c0, bf16 *q_s) {
    bf16 *k_s = q_s + kC * QS, *v_s = k_s + kC * QS;
    const int len = min(kC, a.rows - c0);
    const bf16 *x0 = x + (int64_t)c0 * a.ld;
    if (vec) {
#pragma unroll 4
      for (int i = tid; i < kC * (DP / 8); i += kChunkThreads) {
        const int r = i / (DP / 8), d = (i % (DP / 8)) * 8;
        const bool live = r < len && d < a.dim;
        const bf16 *p = live ? x0 + (int64_t)r * a.ld + h * a.dim + d : x;
        cp16(q_s + r * QS + d, p, live);
        cp16(k_s + r * QS + d, live ? p + hd : x, live);
      }
#pragma unroll
      for (int i = tid; i < kC * (kChunkCols / 8); i += kChunkThreads) {
        const int r = i / (kChunkCols / 8), c = (i % (kChunkCols / 8)) * 8;
        const bool live = r < len && col0 + c < a.vdim;
        cp16(v_s + r * VS + c, live ? x0 + (int64_t)r * a.ld + 2 * hd + h * a.vdim + col0 + c : x, live);
      }
    } else {
      const bf16 zero = __float2bfloat16_rn(0.0f);
      for (int i = tid; i < kC * DP; i += kChunkThreads) {
        const int r = i / DP, d = i % DP;
        const bool live = r < len && d < a.dim;
        const bf16 *p = x0 + (int64_t)r * a.ld + h * a.dim + d;
        q_s[r * QS + d] = live ? p[0] : zero;
        k_s[r * QS + d] = live ? p[hd] : zero;
      }
      for (int i = tid; i < kC * kChunkCols; i += kChunkThreads) {
        const int r = i / kChunkCols, c = i % kChunkCols;
        v_s[r * VS + c] = r < len && col0 + c < a.vdim ? x0[(int64_t)r * a.ld + 2 * hd + h * a.vdim + col0 + c] : zero;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0, stage);
  for (int c0 = 0; c0 < a.rows; c0 += kC) {
    const int len = min(kC, a.rows - c0), st = (c0 / kC) & 1;
    const bf16 *q_s = stage + st * kStage, *k_s = q_s + kC * QS, *v_s = k_s + kC * QS;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this chunk has landed, and the previous one's readers are done
    if (c0 + kC < a.rows) load(c0 + kC, stage + (st ^ 1) * kStage);
    // the state as two bf16 terms, for Q S
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
    // V' = diag(decay^(len-1-j)) V as two terms
#pragma unroll
    for (int i = tid; i < kC * kChunkCols / 2; i += kChunkThreads) {
      const int r = i / (kChunkCols / 2), c = (i % (kChunkCols / 2)) * 2;
      const uint32_t v = *reinterpret_cast<const uint32_t *>(v_s + r * VS + c);
      const float w = r < len ? pw[len - 1 - r] : 0.0f;
      uint32_t hi, lo;
      split_pair(bf16_lo(v) * w, bf16_hi(v) * w, hi, lo);
      *reinterpret_cast<uint32_t *>(vh_s + r * VS + c) = hi;
      *reinterpret_cast<uint32_t *>(vl_s + r * VS + c) = lo;
    }
    __syncthreads();

    // O for the warp's 16 tokens: first Q S, scaled by decay^(i+1)
    float O[4][4] = {};
    float P[8][4] = {};
    const int i0 = warp * 16;
#pragma unroll 2
    for (int k = 0; k < DP; k += 16) {
      uint32_t A[4], B[4];
      ldsm4(A, q_s + (i0 + (lane & 15)) * QS + k + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 2; ++n) {  // 16 value columns at a time
        ldsm4t(B, sh_s + (k + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], A, B[0], B[1]);
        mma16816(O[2 * n + 1], A, B[2], B[3]);
        ldsm4t(B, sl_s + (k + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], A, B[0], B[1]);
        mma16816(O[2 * n + 1], A, B[2], B[3]);
      }
#pragma unroll
      for (int n = 0; n < 4; ++n) {  // 16 keys at a time: rows n*16 + (0..15) of K
        ldsm4(B, k_s + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * QS + k + ((lane >> 3) & 1) * 8);
        mma16816(P[2 * n], A, B[0], B[1]);
        mma16816(P[2 * n + 1], A, B[2], B[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[n][e] *= pw[min(i0 + tr + (e >> 1) * 8 + 1, kC)];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + tr + (e >> 1) * 8, j = n * 8 + tc + (e & 1);
        P[n][e] = j <= i ? P[n][e] * pw[i - j] : 0.0f;
      }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {  // 16 keys
      uint32_t H[4], L[4], B[4];
      split_pair(P[2 * kk][0], P[2 * kk][1], H[0], L[0]);
      split_pair(P[2 * kk][2], P[2 * kk][3], H[1], L[1]);
      split_pair(P[2 * kk + 1][0], P[2 * kk + 1][1], H[2], L[2]);
      split_pair(P[2 * kk + 1][2], P[2 * kk + 1][3], H[3], L[3]);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        ldsm4t(B, v_s + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
        mma16816(O[2 * n], H, B[0], B[1]);
        mma16816(O[2 * n + 1], H, B[2], B[3]);
        mma16816(O[2 * n], L, B[0], B[1]);
        mma16816(O[2 * n + 1], L, B[2], B[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + tr + (e >> 1) * 8, c = col0 + n * 8 + tc + (e & 1);
        if (i < len && c < a.vdim) a.out[(int64_t)(c0 + i) * a.heads * a.vdim + h * a.vdim + c] = O[n][e];
      }
    // the state: decay^len S + K^T V'
    const float dl = pw[len];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= dl;
      const int d = (warp * MT + m) * 16;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        // A = K^T: rows d.., columns the keys; K is stored [key][d], hence the transposed load
        uint32_t A[4], B[4];
        ldsm4t(A, k_s + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * QS + d + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          ldsm4t(B, vh_s + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
          mma16816(S[m][2 * n], A, B[0], B[1]);
          mma16816(S[m][2 * n + 1], A, B[2], B[3]);
          ldsm4t(B, vl_s + (kk * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8);
          mma16816(S[m][2 * n], A, B[0], B[1]);
          mma16816(S[m][2 * n + 1], A, B[2], B[3]);
        }
      }
    }
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

template <int DPT>
int32_t steps(const LightningArgs &a, bool pdl, cudaStream_t s) {
  const dim3 grid(a.heads, (a.vdim + kStepCols - 1) / kStepCols, a.one_sequence ? 1 : a.rows);
  if (a.powers) return launch_kernel(linear_steps_kernel<DPT, false>, grid, dim3(kStepThreads), steps_smem(a), pdl, s, a);
  return launch_kernel(linear_steps_kernel<DPT, true>, grid, dim3(kStepThreads), steps_smem(a), pdl, s, a);
}

template <int MT>
int32_t chunks(const LightningArgs &a, bool pdl, cudaStream_t s) {
  const int smem = chunk_smem(64 * MT);
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(lightning_chunk_kernel<MT>, smem));
    ready = true;
  }
  return launch_kernel(lightning_chunk_kernel<MT>, dim3(a.heads, (a.vdim + kChunkCols - 1) / kChunkCols), dim3(kChunkThreads), smem, pdl, s, a);
}

}  // namespace

bool lightning_shape_ok(int32_t heads, int32_t dim, int32_t vdim) { return heads >= 1 && dim >= 1 && dim <= 512 && vdim >= 1; }

int32_t launch_lightning_steps(const LightningArgs &a, bool pdl, cudaStream_t s) {
  if (a.dim <= 64) return steps<8>(a, pdl, s);
  if (a.dim <= 128) return steps<16>(a, pdl, s);
  if (a.dim <= 256) return steps<32>(a, pdl, s);
  if (a.dim <= 512) return steps<64>(a, pdl, s);
  return fail(CMLD_ERR_SHAPE, "lightning attention: %d key dimensions, at most 512", a.dim);
}

bool gated_shape_ok(int32_t heads, int32_t dim, int32_t vdim, int32_t rank) {
  return lightning_shape_ok(heads, dim, vdim) && rank >= 1 && rank <= 16384;
}

bool lightning_chunk_fits(const LightningArgs &a) { return a.powers && a.half && a.one_sequence && a.dim <= 256; }

int32_t launch_lightning_chunks(const LightningArgs &a, bool pdl, cudaStream_t s) {
  if (a.dim <= 64) return chunks<1>(a, pdl, s);
  if (a.dim <= 128) return chunks<2>(a, pdl, s);
  return chunks<4>(a, pdl, s);
}

}  // namespace cmld
