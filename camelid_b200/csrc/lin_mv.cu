// Matrix-vector products with bfloat16 weights and 32-bit activations for one or two rows: one pass over the weights.
//
// Persistent grid, one CTA of 16 warps per SM.  A warp owns one or two output rows at a time; a lane reads 16 bytes
// (eight weights) of each, four steps of 256 columns in flight.  The first weights are asked for before the kernel
// waits for its predecessor (weights never depend on earlier kernels), then every CTA prepares the operand itself:
// the boundary between sublayers, an RMS norm (with a sigmoid gate, or over groups of columns with a SiLU gate), or a plain
// copy.  Two products that do not depend on each other can share a launch: the first `n_first` CTAs work on one.
// The prepared rows sit in shared memory as f32 in two planes (values 8j..8j+3 and 8j+4..8j+7), so that the lanes of
// a warp read consecutive 16-byte words.
#include "layered.cuh"

namespace cmld {

namespace {

constexpr int kMvThreads = 512, kMvUnroll = 4;
constexpr size_t kMvMaxSmem = 220 * 1024;

__host__ __device__ constexpr int mv_kpad(int cols) { return (cols + 255) & ~255; }

template <int R, int ROWS>
__device__ __forceinline__ void lin_mv_cta(const LinMvArgs &a, int cta, int ctas) {
  extern __shared__ __align__(16) float smem[];
  __shared__ __align__(8) float red[2 * kMvThreads / 32];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int K = a.w.cols, kp = mv_kpad(K), half = kp / 2, nit = kp / 256;
  float *xs = smem;              // [R][2][kp / 2]
  float *u = smem + R * kp;      // one row in plain order
  const int groups = (a.w.rows + ROWS - 1) / ROWS, stride = ctas * (kMvThreads / 32);
  int g = cta + ctas * warp;

  uint4 w[ROWS][kMvUnroll];
  auto fetch = [&](int grp, int it0) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int row = min(grp * ROWS + i, a.w.rows - 1);
      const bf16 *p = a.w.w + (int64_t)row * a.w.ld;
#pragma unroll
      for (int j = 0; j < kMvUnroll; ++j) {
        const int k = (it0 + j) * 256 + lane * 8;
        w[i][j] = k < a.w.ld ? ld_stream16(p + k) : make_uint4(0, 0, 0, 0);  // the row's padding is zero
      }
    }
  };
  pdl_launch();
  if (g < groups) fetch(g, 0);
  pdl_wait();

  auto put = [&](int r, int i, float v) { xs[r * kp + ((i >> 2) & 1) * half + (i >> 3) * 4 + (i & 3)] = v; };
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (a.prologue == kProStreams) {
      stream_mix_row(a.mix, r, u, red, cta == 0);
      for (int i = tid; i < kp; i += kMvThreads) put(r, i, i < K ? u[i] : 0.0f);
    } else if (a.prologue == kProRmsGroups) {
      // a warp per group of columns
      const float *x = a.x + r * a.x_ld, *gate = a.gate + r * a.gate_ld;
      for (int c0 = warp * a.group; c0 < K; c0 += (kMvThreads / 32) * a.group) {
        float s = 0.0f;
        for (int i = lane; i < a.group; i += 32) s = fmaf(x[c0 + i], x[c0 + i], s);
        const float inv = 1.0f / sqrtf(warp_sum(s) / (float)a.group + a.eps);
        for (int i = lane; i < a.group; i += 32) put(r, c0 + i, x[c0 + i] * inv * a.norm_w[i] * silu_f(gate[c0 + i]));
      }
      for (int i = K + tid; i < kp; i += kMvThreads) put(r, i, 0.0f);
    } else {
      const float *x = a.x + r * a.x_ld;
      float inv = 1.0f;
      if (a.prologue != kProPlain) {
        float s = 0.0f;
        for (int i = tid; i < K; i += kMvThreads) s = fmaf(x[i], x[i], s);
        inv = 1.0f / sqrtf(cta_total(s, red) / (float)K + a.eps);
      }
      for (int i = tid; i < kp; i += kMvThreads) {
        float v = i < K ? x[i] : 0.0f;
        if (a.prologue != kProPlain && i < K) {
          v = v * inv * a.norm_w[i];
          if (a.prologue == kProRmsGate) v *= sigmoid_f(a.gate[r * a.gate_ld + i]);
        }
        put(r, i, v);
      }
    }
  }
  __syncthreads();

  bool first = true;
  for (; g < groups; g += stride) {
    float acc[ROWS][R];
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
#pragma unroll
      for (int r = 0; r < R; ++r) acc[i][r] = 0.0f;
    for (int it0 = 0; it0 < nit; it0 += kMvUnroll) {
      if (!first) fetch(g, it0);
      first = false;
#pragma unroll
      for (int j = 0; j < kMvUnroll; ++j) {
        if (it0 + j >= nit) break;
        const int c = ((it0 + j) * 32 + lane) * 4;
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const float4 lo = *reinterpret_cast<const float4 *>(xs + r * kp + c), hi = *reinterpret_cast<const float4 *>(xs + r * kp + half + c);
#pragma unroll
          for (int i = 0; i < ROWS; ++i) {
            const uint4 v = w[i][j];
            float t = acc[i][r];
            t = fmaf(bf16_lo(v.x), lo.x, t);
            t = fmaf(bf16_hi(v.x), lo.y, t);
            t = fmaf(bf16_lo(v.y), lo.z, t);
            t = fmaf(bf16_hi(v.y), lo.w, t);
            t = fmaf(bf16_lo(v.z), hi.x, t);
            t = fmaf(bf16_hi(v.z), hi.y, t);
            t = fmaf(bf16_lo(v.w), hi.z, t);
            t = fmaf(bf16_hi(v.w), hi.w, t);
            acc[i][r] = t;
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      float v[ROWS];
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int row = g * ROWS + i;
        v[i] = fmaf(warp_sum(acc[i][r]), a.scale, a.bias && row < a.w.rows ? a.bias[row] : 0.0f);
        if (lane == 0 && row < a.w.rows && a.act != kActSwiGlu) a.y[r * a.y_ld + row] = lin_activate(v[i], a.act, row < a.act_rows);
      }
      if (ROWS == 2 && lane == 0 && a.act == kActSwiGlu) a.y[r * a.y_ld + g] = silu_f(v[0]) * v[ROWS - 1];
    }
  }
}

template <int R, int ROWS>
__global__ void __launch_bounds__(kMvThreads, 1) lin_mv_kernel(const __grid_constant__ LinMvArgs a) {
  lin_mv_cta<R, ROWS>(a, blockIdx.x, gridDim.x);
}

template <int R, int ROWS>
__global__ void __launch_bounds__(kMvThreads, 1) lin_mv_pair_kernel(const __grid_constant__ LinMvArgs a, const __grid_constant__ LinMvArgs b, int n_first) {
  if ((int)blockIdx.x < n_first) lin_mv_cta<R, ROWS>(a, blockIdx.x, n_first);
  else lin_mv_cta<R, ROWS>(b, blockIdx.x - n_first, gridDim.x - n_first);
}

size_t mv_smem(int cols, int batch) { return (size_t)(batch + 1) * mv_kpad(cols) * 4; }

int mv_sms() {
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  return sms;
}

template <int R, int ROWS>
int32_t mv_launch(const LinMvArgs &a, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(lin_mv_kernel<R, ROWS>, kMvMaxSmem));
    prefer_max_smem_carveout(lin_mv_kernel<R, ROWS>);
    ready = true;
  }
  const int groups = (a.w.rows + ROWS - 1) / ROWS;
  return launch_kernel(lin_mv_kernel<R, ROWS>, dim3(std::min(groups, mv_sms())), dim3(kMvThreads), mv_smem(a.w.cols, R), pdl, s, a);
}

template <int R, int ROWS>
int32_t mv_launch_pair(const LinMvArgs &a, const LinMvArgs &b, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(lin_mv_pair_kernel<R, ROWS>, kMvMaxSmem));
    prefer_max_smem_carveout(lin_mv_pair_kernel<R, ROWS>);
    ready = true;
  }
  const int sms = mv_sms();
  const double wa = (double)a.w.rows * a.w.ld, wb = (double)b.w.rows * b.w.ld;
  const int first = std::min(sms - 1, std::max(1, (int)(sms * wa / (wa + wb) + 0.5)));
  return launch_kernel(lin_mv_pair_kernel<R, ROWS>, dim3(sms), dim3(kMvThreads), mv_smem(std::max(a.w.cols, b.w.cols), R), pdl, s, a, b, first);
}

}  // namespace

bool lin_mv_fits(int32_t cols, int32_t batch) { return batch >= 1 && batch <= 2 && mv_smem(cols, batch) <= kMvMaxSmem; }

int32_t launch_lin_mv(const LinMvArgs &a, bool pdl, cudaStream_t s) {
  if (!lin_mv_fits(a.w.cols, a.batch)) return fail(CMLD_ERR_SHAPE, "matrix-vector product of %d columns and %d rows does not fit", a.w.cols, a.batch);
  if (a.act == kActSwiGlu) {
    if (a.w.rows % 2) return fail(CMLD_ERR_SHAPE, "linear: gated pairs need an even number of rows");
    return a.batch == 1 ? mv_launch<1, 2>(a, pdl, s) : mv_launch<2, 2>(a, pdl, s);
  }
  // one output row per warp while that is needed to give every warp of the machine something to do
  const bool single = a.w.rows <= 148 * (kMvThreads / 32) * 3 / 2;
  if (a.batch == 1) return single ? mv_launch<1, 1>(a, pdl, s) : mv_launch<1, 2>(a, pdl, s);
  return single ? mv_launch<2, 1>(a, pdl, s) : mv_launch<2, 2>(a, pdl, s);
}

int32_t launch_lin_mv_pair(const LinMvArgs &a, const LinMvArgs &b, bool pdl, cudaStream_t s) {
  if (a.batch != b.batch || a.act == kActSwiGlu || b.act == kActSwiGlu || !lin_mv_fits(a.w.cols, a.batch) || !lin_mv_fits(b.w.cols, b.batch))
    return fail(CMLD_ERR_SHAPE, "a pair of matrix-vector products does not fit one launch");
  return a.batch == 1 ? mv_launch_pair<1, 1>(a, b, pdl, s) : mv_launch_pair<2, 1>(a, b, pdl, s);
}

}  // namespace cmld
