// Linear layers on the 5th-generation tensor cores: out[r][o] = act(scale * sum_k w[o][k] x[r][k] + bias[o]), bfloat16
// operands, f32 accumulators in tensor memory.
//
// The weights are operand A (tiles of 128 output rows), the activation rows operand B (tiles of BN rows), both K-major
// and brought by TMA in 128-byte-swizzled boxes of 64 columns.  Persistent CTAs, one per SM; warp roles:
//   warp 0      TMA: operand stages (one elected lane)
//   warp 1      MMA issue (one elected lane), tensor-memory allocation
//   warps 2-9   epilogue: tcgen05.ld, activation, stores, two warps for each quarter of the accumulator lanes (every
//               other 16 columns); two accumulator slots, so that a tile's epilogue overlaps the next tile's products
// Few rows leave few tiles: then `split` CTAs of a thread-block cluster share a tile's inner dimension, leave their
// partial accumulators in shared memory, and each of them adds the partials of its share of the columns in rank order.
// The first weight boxes are asked for before the kernel waits for its predecessor.
// Every wait is bounded: one that runs out sets the status word and an abort flag, all roles leave their loops, tensor
// memory is freed and the kernel returns.
#include <cuda.h>

#include "layered.cuh"

namespace cmld {

namespace {

constexpr int kEpiWarps = 8, kThreads = (2 + kEpiWarps) * 32, kBM = 128, kBK = 64;
constexpr uint32_t kSpin = 1u << 22;
constexpr int kABytes = kBM * kBK * 2;

constexpr int b_bytes(int bn) { return bn * kBK * 2; }
constexpr int stages(int bn) { return bn == 256 ? 4 : bn == 128 ? 6 : 8; }
constexpr int off_bars(int bn) { return stages(bn) * (kABytes + b_bytes(bn)); }
constexpr int smem_bytes(int bn) { return off_bars(bn) + 256 + 1024; }  // + slack to align the base to 1024

struct TcLinArgs {
  int32_t m_rows, n_rows, n_k, tiles_m, tiles, split;
  void *out;
  int64_t out_ld;
  int32_t act, act_rows;
  const float *bias;
  float scale;
  int32_t *status;
};

__device__ __forceinline__ uint32_t s32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void bar_init(uint32_t bar, uint32_t count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count)); }
__device__ __forceinline__ void bar_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
__device__ __forceinline__ void bar_expect(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool bar_try(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
               : "=r"(ok)
               : "r"(bar), "r"(parity)
               : "memory");
  return ok != 0;
}
__device__ __forceinline__ bool bar_wait(uint32_t bar, uint32_t parity, volatile int *abort_flag, int32_t *status) {
  for (uint32_t i = 0; i < kSpin; ++i) {
    if (bar_try(bar, parity)) return true;
    if ((i & 255u) == 255u && *abort_flag) return false;
  }
  *abort_flag = 1;
  atomicExch(status, (int32_t)CMLD_ERR_TIMEOUT);
  return false;
}
__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cta.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst), "l"(map), "r"(x),
               "r"(y), "r"(bar)
               : "memory");
}
// K-major operand in 128-byte-swizzled rows: groups of eight rows are 1024 bytes apart (descriptor version 1, layout
// type 2 = 128-byte swizzle).
__device__ __forceinline__ uint64_t smem_desc(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void mma_bf16(uint32_t d, uint64_t da, uint64_t db, uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}" ::"r"(d),
      "l"(da), "l"(db), "r"(idesc), "r"(accumulate ? 1u : 0u), "r"(0u)
      : "memory");
}
__device__ __forceinline__ void mma_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tmem_ld16(uint32_t t, float (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n\t"
      "tcgen05.wait::ld.sync.aligned;"
      : "=&f"(r[0]), "=&f"(r[1]), "=&f"(r[2]), "=&f"(r[3]), "=&f"(r[4]), "=&f"(r[5]), "=&f"(r[6]), "=&f"(r[7]), "=&f"(r[8]), "=&f"(r[9]),
        "=&f"(r[10]), "=&f"(r[11]), "=&f"(r[12]), "=&f"(r[13]), "=&f"(r[14]), "=&f"(r[15])
      : "r"(t)
      : "memory");
}
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }

template <int BN, typename OutT>
__global__ void __launch_bounds__(kThreads, 1)
    lin_tc5_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, const TcLinArgs a) {
  constexpr int NS = stages(BN);
  constexpr int TSLOT = BN < 32 ? 32 : BN;                 // tensor-memory columns of one accumulator slot
  constexpr uint32_t TCOLS = 2 * TSLOT;
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kBM >> 4) << 24);
  extern __shared__ uint8_t raw[];
  uint8_t *smem = raw + ((1024u - (s32(raw) & 1023u)) & 1023u);
  const uint32_t base = s32(smem), bars = base + off_bars(BN);
  auto full = [&](int i) { return bars + 8u * i; };
  auto empty = [&](int i) { return bars + 8u * (NS + i); };
  auto acc_full = [&](int i) { return bars + 8u * (2 * NS + i); };
  auto acc_empty = [&](int i) { return bars + 8u * (2 * NS + 2 + i); };
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + off_bars(BN) + 8 * (2 * NS + 4));
  volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // a cluster of `split` CTAs works on one tile, each on its share of the inner dimension
  const int rank = (int)blockIdx.x % a.split, first = (int)blockIdx.x / a.split, step = (int)gridDim.x / a.split;
  const int per = (a.n_k + a.split - 1) / a.split, k_lo = min(rank * per, a.n_k), k_hi = min(k_lo + per, a.n_k), nk = k_hi - k_lo;

  if (tid == 0) {
    for (int i = 0; i < NS; ++i) {
      bar_init(full(i), 1);
      bar_init(empty(i), 1);
    }
    for (int i = 0; i < 2; ++i) {
      bar_init(acc_full(i), 1);
      bar_init(acc_empty(i), kEpiWarps);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(s32(tmem_slot)), "r"(TCOLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tbase = *tmem_slot;
  pdl_launch();

  if (warp == 0) {
    if (lane == 0) {
      const int n_mine = first < a.tiles ? (a.tiles - first + step - 1) / step : 0;
      const int total = n_mine * nk;
      auto load_w = [&](int q) {
        const int t = first + (q / nk) * step, kb = k_lo + q % nk, st = q % NS;
        bar_expect(full(st), kABytes + b_bytes(BN));
        tma_2d(base + st * (kABytes + b_bytes(BN)), &wmap, kb * kBK, (t % a.tiles_m) * kBM, full(st));
      };
      auto load_x = [&](int q) {
        const int t = first + (q / nk) * step, kb = k_lo + q % nk, st = q % NS;
        tma_2d(base + st * (kABytes + b_bytes(BN)) + kABytes, &xmap, kb * kBK, (t / a.tiles_m) * BN, full(st));
      };
      const int early = min(total, NS);
      for (int q = 0; q < early; ++q) load_w(q);
      pdl_wait();
      for (int q = 0; q < early; ++q) load_x(q);
      for (int q = early; q < total; ++q) {
        if (!bar_wait(empty(q % NS), (uint32_t)((q / NS - 1) & 1), abort_flag, a.status)) break;
        load_w(q);
        load_x(q);
      }
      if (*abort_flag) __nanosleep(1000000);  // copies in flight land before the shared memory is given back
    }
  } else if (warp == 1) {
    if (lane == 0 && nk > 0) {
      int q = 0, i = 0;
      bool ok = true;
      for (int t = first; t < a.tiles && ok; t += step, ++i) {
        const int slot = i & 1;
        if (i >= 2) ok = bar_wait(acc_empty(slot), (uint32_t)((i / 2 - 1) & 1), abort_flag, a.status);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int kb = 0; kb < nk && ok; ++kb, ++q) {
          const int st = q % NS;
          ok = bar_wait(full(st), (uint32_t)((q / NS) & 1), abort_flag, a.status);
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint64_t da = smem_desc(base + st * (kABytes + b_bytes(BN))), db = smem_desc(base + st * (kABytes + b_bytes(BN)) + kABytes);
#pragma unroll
          for (int k = 0; k < kBK / 16; ++k) mma_bf16(tbase + slot * TSLOT, da + 2 * k, db + 2 * k, kIdesc, kb > 0 || k > 0);
          mma_commit(empty(st));
        }
        if (ok) mma_commit(acc_full(slot));
      }
    }
    __syncwarp();
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2;  // the 32 accumulator lanes this warp may read; its column groups
    pdl_wait();                    // the output buffer may still be read by the predecessor
    int i = 0;
    OutT *out = static_cast<OutT *>(a.out);
    for (int t = first; t < a.tiles; t += step, ++i) {
      const int slot = i & 1, o = (t % a.tiles_m) * kBM + quarter * 32 + lane, n0 = (t / a.tiles_m) * BN;
      if (nk > 0) {
        if (!bar_wait(acc_full(slot), (uint32_t)((i / 2) & 1), abort_flag, a.status)) break;
      }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const int n_live = min(BN, a.n_rows - n0);
      float *part = reinterpret_cast<float *>(smem);  // [BN][128]: the operand stages are free by now
      const bool silu = a.act == kActSilu && o < a.act_rows, relu2 = a.act == kActRelu2, swiglu = a.act == kActSwiGlu;
      const float bias = a.bias && o < a.m_rows ? a.bias[o] : 0.0f;
      const bool odd = lane & 1;
      OutT *p = out + (int64_t)(n0 + 16 * half) * a.out_ld + (swiglu ? o >> 1 : o);
#pragma unroll 1
      for (int c = 16 * half; c < n_live; c += 32, p += 32 * a.out_ld) {
        float r[16];
        if (nk > 0) {
          tmem_ld16(tbase + slot * TSLOT + c + ((uint32_t)(quarter * 32) << 16), r);
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j) r[j] = 0.0f;
        }
        if (a.split > 1) {
#pragma unroll
          for (int j = 0; j < 16; ++j) part[(c + j) * kBM + quarter * 32 + lane] = r[j];
          continue;
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) r[j] = fmaf(r[j], a.scale, bias);
        if (swiglu) {
          // a lane holds the gate (even rows) or the other factor (odd rows); of two columns the even lane finishes one,
          // the odd lane the other
          OutT *w = p + (odd ? a.out_ld : 0);
#pragma unroll
          for (int j = 0; j < 16; j += 2, w += 2 * a.out_ld) {
            const float t = __shfl_xor_sync(0xffffffffu, odd ? r[j] : r[j + 1], 1);
            const float v = odd ? silu_f(t) * r[j + 1] : silu_f(r[j]) * t;
            if (o < a.m_rows && c + j + (odd ? 1 : 0) < n_live) put(w, v);
          }
          continue;
        }
        if (silu) {
#pragma unroll
          for (int j = 0; j < 16; ++j) r[j] = silu_f(r[j]);
        } else if (relu2) {
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float v = fmaxf(r[j], 0.0f);
            r[j] = v * v;
          }
        }
        if (o < a.m_rows) {
          OutT *w = p;
          if (c + 16 <= n_live) {
#pragma unroll
            for (int j = 0; j < 16; ++j, w += a.out_ld) put(w, r[j]);
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j, w += a.out_ld)
              if (c + j < n_live) put(w, r[j]);
          }
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) bar_arrive(acc_empty(slot));
    }
  }
  __syncwarp();
  if (a.split > 1) {
    // one tile per cluster: add the partial accumulators, column by column, in rank order
    cluster_sync();
    if (first < a.tiles && !*abort_flag) {
      OutT *out = static_cast<OutT *>(a.out);
      const int m0 = (first % a.tiles_m) * kBM, n0 = (first / a.tiles_m) * BN, n_live = min(BN, a.n_rows - n0);
      auto total = [&](int e, int o) {
        float v = 0.0f;
        for (int p = 0; p < a.split; ++p) v += ld_peer(base + 4u * e, p);
        return fmaf(v, a.scale, a.bias && o < a.m_rows ? a.bias[o] : 0.0f);
      };
      if (a.act == kActSwiGlu) {
        for (int e = 2 * (rank * kThreads + tid); e < n_live * kBM; e += 2 * a.split * kThreads) {
          const int o = m0 + e % kBM, n = e / kBM;
          const float v = silu_f(total(e, o)) * total(e + 1, o + 1);
          if (o < a.m_rows) put(out + (int64_t)(n0 + n) * a.out_ld + (o >> 1), v);
        }
      } else {
        for (int e = rank * kThreads + tid; e < n_live * kBM; e += a.split * kThreads) {
          const int o = m0 + e % kBM, n = e / kBM;
          const float v = total(e, o);
          if (o < a.m_rows) put(out + (int64_t)(n0 + n) * a.out_ld + o, lin_activate(v, a.act, o < a.act_rows));
        }
      }
    }
    cluster_sync();
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tbase), "r"(TCOLS) : "memory");
}

typedef CUresult (*EncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                             const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

int32_t make_map(CUtensorMap *map, const void *p, int64_t cols, int64_t rows, int64_t ld, int box_rows) {
  static EncodeFn encode = nullptr;
  if (!encode) {
    void *fn = nullptr;
    cudaDriverEntryPointQueryResult q{};
    CMLD_CUDA(cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q));
    if (!fn || q != cudaDriverEntryPointSuccess) return fail(CMLD_ERR_CUDA, "the driver does not offer cuTensorMapEncodeTiled");
    encode = reinterpret_cast<EncodeFn>(fn);
  }
  if ((reinterpret_cast<uintptr_t>(p) & 15) || (ld & 7)) return fail(CMLD_ERR_SHAPE, "tensor-core operand is not 16-byte aligned");
  const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {kBK, (cuuint32_t)box_rows}, es[2] = {1, 1};
  const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(p), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(CMLD_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d)", (int)r);
  return CMLD_OK;
}

template <int BN, typename OutT>
int32_t launch_bn(const LinArgs &L, int32_t sms, int32_t *status, bool pdl, cudaStream_t s) {
  static bool ready = false;
  if (!ready) {
    CMLD_TRY(allow_smem(lin_tc5_kernel<BN, OutT>, smem_bytes(BN)));
    prefer_max_smem_carveout(lin_tc5_kernel<BN, OutT>);
    ready = true;
  }
  CUtensorMap wmap, xmap;
  CMLD_TRY(make_map(&wmap, L.w.w, L.w.cols, L.w.rows, L.w.ld, kBM));
  CMLD_TRY(make_map(&xmap, L.x, L.w.cols, L.rows, L.x_ld, BN));
  TcLinArgs a{};
  a.m_rows = L.w.rows;
  a.n_rows = L.rows;
  a.n_k = (L.w.cols + kBK - 1) / kBK;
  a.tiles_m = (L.w.rows + kBM - 1) / kBM;
  a.tiles = a.tiles_m * ((L.rows + BN - 1) / BN);
  a.split = 1;
  if (BN <= 64)  // few rows: spread a tile's inner dimension until the machine is full
    while (a.split < 8 && a.tiles * a.split * 2 <= sms && a.n_k >= 4 * a.split) a.split *= 2;
  a.out = L.out;
  a.out_ld = L.out_ld;
  a.act = L.act;
  a.act_rows = L.act_rows;
  a.bias = L.bias;
  a.scale = L.scale;
  a.status = status;
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)(a.split > 1 ? a.tiles * a.split : std::min(a.tiles, sms)));
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem_bytes(BN);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (a.split > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = (unsigned)a.split;
    attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  CMLD_CUDA(cudaLaunchKernelEx(&cfg, lin_tc5_kernel<BN, OutT>, wmap, xmap, a));
  return CMLD_OK;
}

template <typename OutT>
int32_t launch_out(const LinArgs &a, int32_t sms, int32_t *status, bool pdl, cudaStream_t s) {
  if (a.rows <= 16) return launch_bn<16, OutT>(a, sms, status, pdl, s);
  if (a.rows <= 32) return launch_bn<32, OutT>(a, sms, status, pdl, s);
  const int64_t tm = (a.w.rows + kBM - 1) / kBM;
  if (a.rows <= 64 || tm * ((a.rows + 127) / 128) * 2 <= sms) return launch_bn<64, OutT>(a, sms, status, pdl, s);
  if (tm * ((a.rows + 255) / 256) <= sms / 2) return launch_bn<128, OutT>(a, sms, status, pdl, s);
  return launch_bn<256, OutT>(a, sms, status, pdl, s);
}

}  // namespace

int32_t launch_lin_tc5(const LinArgs &a, int32_t sms, int32_t *status, bool pdl, cudaStream_t s) {
  if (a.rows < 1) return CMLD_OK;
  if (a.act == kActSwiGlu && a.w.rows % 2) return fail(CMLD_ERR_SHAPE, "linear: gated pairs need an even number of rows");
  return a.out_half ? launch_out<bf16>(a, sms, status, pdl, s) : launch_out<float>(a, sms, status, pdl, s);
}

}  // namespace cmld
