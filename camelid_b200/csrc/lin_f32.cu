// Linear layers of layered models in true 32-bit: f32 rows times bfloat16 weights (exact as f32) on the FP32 units.
// 64 rows x 64 outputs per CTA, 16 columns of the inner dimension at a time, 4 x 4 results per thread.
#include "layered.cuh"

namespace cmld {

namespace {

constexpr int kT = 64, kKT = 16;

__global__ void __launch_bounds__(256) lin_f32_kernel(const LinArgs a) {
  __shared__ float xs[kKT][kT + 4], ws[kKT][kT + 4];
  pdl_wait();
  const float *x = static_cast<const float *>(a.x);
  const int tid = threadIdx.x, m0 = blockIdx.x * kT, n0 = blockIdx.y * kT;
  const int tm = (tid & 15) * 4, tn = (tid >> 4) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.w.cols; k0 += kKT) {
#pragma unroll
    for (int i = 0; i < kT * kKT / 256; ++i) {
      const int e = tid + i * 256, r = e / kKT, k = e % kKT;
      const bool kin = k0 + k < a.w.cols;
      xs[k][r] = kin && n0 + r < a.rows ? x[(int64_t)(n0 + r) * a.x_ld + k0 + k] : 0.0f;
      ws[k][r] = kin && m0 + r < a.w.rows ? __bfloat162float(a.w.w[(int64_t)(m0 + r) * a.w.ld + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kKT; ++k) {
      const float4 wv = *reinterpret_cast<const float4 *>(&ws[k][tm]), xv = *reinterpret_cast<const float4 *>(&xs[k][tn]);
      const float wa[4] = {wv.x, wv.y, wv.z, wv.w}, xa[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int m = 0; m < 4; ++m) acc[n][m] = fmaf(xa[n], wa[m], acc[n][m]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const int row = n0 + tn + n, o = m0 + tm + m;
      if (row >= a.rows || o >= a.w.rows) continue;
      acc[n][m] = fmaf(acc[n][m], a.scale, a.bias ? a.bias[o] : 0.0f);
      if (a.act != kActSwiGlu) act_store(a.out, a.out_half, (int64_t)row * a.out_ld + o, lin_activate(acc[n][m], a.act, o < a.act_rows));
      else if (m & 1) act_store(a.out, a.out_half, (int64_t)row * a.out_ld + (o >> 1), silu_f(acc[n][m - 1]) * acc[n][m]);
    }
}

}  // namespace

int32_t launch_lin_f32(const LinArgs &a, cudaStream_t s) {
  if (a.act == kActSwiGlu && a.w.rows % 2) return fail(CMLD_ERR_SHAPE, "linear: gated pairs need an even number of rows");
  return launch_kernel(lin_f32_kernel, dim3((a.w.rows + kT - 1) / kT, (a.rows + kT - 1) / kT), dim3(256), 0, false, s, a);
}

}  // namespace cmld
