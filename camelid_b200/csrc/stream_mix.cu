// Row operations of layered models: the boundary between sublayers (residual update, read-out, norm), the embedding, RMS
// norm with an optional gate, over whole rows or over groups of columns.
#include "layered.cuh"

namespace cmld {

namespace {

// One CTA per row: wide CTAs while the rows are too few to fill the machine.
constexpr int kMixThreads = 1024;
int mix_threads(int rows) { return rows >= 512 ? 256 : rows >= 256 ? 512 : kMixThreads; }

__global__ void __launch_bounds__(kMixThreads) stream_mix_kernel(const StreamMix m, ActBuf out) {
  extern __shared__ __align__(16) float u[];
  __shared__ __align__(8) float red[2 * kMixThreads / 32];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x;
  stream_mix_row(m, r, u, red, true);
  for (int i = threadIdx.x; i < m.width; i += blockDim.x) act_store(out.p, out.half, r * out.ld + i, u[i]);
}

// One stream with norms on the sublayers' outputs (or the embedding) and no norm in front of the next: the row stays in
// registers.
template <int V>
__global__ void __launch_bounds__(V == 4 ? 512 : kMixThreads) post_norm_kernel(const __grid_constant__ StreamMix m, ActBuf out) {
  __shared__ __align__(8) float red[2 * kMixThreads / 32];
  pdl_launch();
  pdl_wait();
  const int64_t row = blockIdx.x;
  post_norm_row<V>(m, row, red, [&](int i, float4 v) {
    if (m.x_out) reinterpret_cast<float4 *>(m.x_out + row * m.width)[i] = v;
    const int64_t at = row * out.ld + 4 * i;
    if (out.half) {
      __nv_bfloat162 p[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
      *reinterpret_cast<uint2 *>(static_cast<bf16 *>(out.p) + at) = *reinterpret_cast<const uint2 *>(p);
    } else {
      *reinterpret_cast<float4 *>(static_cast<float *>(out.p) + at) = v;
    }
  });
}

__global__ void __launch_bounds__(kMixThreads) stream_tap_kernel(const StreamMix m, float *out) {
  extern __shared__ __align__(16) float u[];
  __shared__ __align__(8) float red[2 * kMixThreads / 32];
  pdl_wait();
  stream_mix_row(m, blockIdx.x, u, red, false);
  for (int i = threadIdx.x; i < m.width; i += blockDim.x) out[(int64_t)blockIdx.x * m.width + i] = u[i];
}

__global__ void __launch_bounds__(kMixThreads) rms_rows_kernel(const float *x, int64_t x_ld, const float *w, int cols, float eps, ActBuf gate, ActBuf out) {
  __shared__ float red[kMixThreads / 32];
  pdl_launch();
  pdl_wait();
  const int64_t r = blockIdx.x;
  const float *xr = x + r * x_ld;
  float s = 0.0f;
#pragma unroll 4
  for (int i = threadIdx.x; i < cols; i += blockDim.x) s = fmaf(xr[i], xr[i], s);
  const float inv = 1.0f / sqrtf(cta_total(s, red) / (float)cols + eps);
#pragma unroll 4
  for (int i = threadIdx.x; i < cols; i += blockDim.x) {
    float v = xr[i] * inv * w[i];
    if (gate.p) v *= sigmoid_f(act_load(gate.p, gate.half, r * gate.ld + i));
    act_store(out.p, out.half, r * out.ld + i, v);
  }
}

// A warp per group of columns.
__global__ void __launch_bounds__(256) rms_groups_kernel(const float *x, int64_t x_ld, const float *w, int groups, int group, float eps, const float *gate,
                                                         int64_t gate_ld, ActBuf out, int rows) {
  pdl_launch();
  pdl_wait();
  const int64_t unit = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= (int64_t)rows * groups) return;
  const int64_t r = unit / groups, c0 = unit % groups * group;
  const float *xr = x + r * x_ld + c0, *gr = gate + r * gate_ld + c0;
  float s = 0.0f;
#pragma unroll 4
  for (int i = lane; i < group; i += 32) s = fmaf(xr[i], xr[i], s);
  const float inv = 1.0f / sqrtf(warp_sum(s) / (float)group + eps);
#pragma unroll 4
  for (int i = lane; i < group; i += 32) act_store(out.p, out.half, r * out.ld + c0 + i, xr[i] * inv * w[i] * silu_f(gr[i]));
}

}  // namespace

int32_t launch_stream_mix(const StreamMix &m, int32_t rows, ActBuf out, bool pdl, cudaStream_t s) {
  if (!m.mix && !m.enorm_w && m.streams == 1 && !m.in && !m.norm_w && !m.row_map && m.width % 4 == 0 && m.width <= 8192 && out.ld % 4 == 0) {
    // many rows: small CTAs, several values per thread
    const int n4 = m.width / 4, per = rows >= 256 ? 4 : 1, threads = std::min(per == 4 ? 512 : kMixThreads, ((n4 + per - 1) / per + 31) & ~31);
    const int v = (n4 + threads - 1) / threads;
    if (v == 1) return launch_kernel(post_norm_kernel<1>, dim3(rows), dim3(threads), 0, pdl, s, m, out);
    if (v == 2) return launch_kernel(post_norm_kernel<2>, dim3(rows), dim3(threads), 0, pdl, s, m, out);
    return launch_kernel(post_norm_kernel<4>, dim3(rows), dim3(threads), 0, pdl, s, m, out);
  }
  const size_t smem = (size_t)m.width * 4;
  if (smem > 48 * 1024) CMLD_TRY(allow_smem(stream_mix_kernel, smem));
  return launch_kernel(stream_mix_kernel, dim3(rows), dim3(mix_threads(rows)), smem, pdl, s, m, out);
}

int32_t launch_stream_tap(const StreamMix &m, int32_t rows, float *out, cudaStream_t s) {
  const size_t smem = (size_t)m.width * 4;
  if (smem > 48 * 1024) CMLD_TRY(allow_smem(stream_tap_kernel, smem));
  return launch_kernel(stream_tap_kernel, dim3(rows), dim3(mix_threads(rows)), smem, false, s, m, out);
}

int32_t launch_rms_rows(const float *x, int64_t x_ld, const float *w, int32_t cols, float eps, ActBuf gate, ActBuf out, int32_t rows,
                        bool pdl, cudaStream_t s) {
  return launch_kernel(rms_rows_kernel, dim3(rows), dim3(mix_threads(rows)), 0, pdl, s, x, x_ld, w, cols, eps, gate, out);
}

int32_t launch_rms_groups(const float *x, int64_t x_ld, const float *w, int32_t cols, int32_t group, float eps, const float *gate, int64_t gate_ld,
                          ActBuf out, int32_t rows, bool pdl, cudaStream_t s) {
  const int groups = cols / group;
  return launch_kernel(rms_groups_kernel, dim3((unsigned)(((int64_t)rows * groups + 7) / 8)), dim3(256), 0, pdl, s, x, x_ld, w, groups, group, eps, gate,
                       gate_ld, out, rows);
}

}  // namespace cmld
