// Unquantized linears:  out[t, n] = epilogue(sum_k x[t, k] w[n, k]),  bf16 x bf16 -> fp32 accumulate, or all fp32.
//
//   dense_gemm_kernel   tcgen05.mma.kind::f16, weights = A operand (128 rows), tokens = B operand (16 .. 256), both by TMA
//                       (128-byte swizzle) through a ring; ONE accumulator in TMEM for the whole K range.  The weight tiles
//                       of the first ring pass are requested before the programmatic-dependent-launch wait.  The fp32
//                       tile is then staged in the (by then free) ring as [token][128 rows], which makes every output
//                       store 16 bytes wide and gives the split-K form its exchange buffer: the splits of a tile are one
//                       thread-block cluster and sum each other's tiles through distributed shared memory in split order
//                       (deterministic), every CTA finishing a share of the items.
//   dense_gemv_kernel   up to 16 tokens: weight streaming without shared-memory staging.  A CTA owns 16 weight rows, eight
//                       warps take alternate 32-wide K blocks; a thread feeds 8 consecutive values of two weight rows to
//                       two m16n8k16 MMAs, the activation fragment uses the same K assignment, so the product is exact.
//   dense_sgemm_kernel  fp32 operands on the FMA units (64 x 64 tiles): the full-precision mode of a model.
//
// Two batched forms of the same kernels: G matrices [G, N, K] that each read their own columns of x and write their own columns of
// out (a matrix per head), and E matrices whose tokens are runs of rows of x sorted by matrix (experts), a tile list naming
// (matrix, token tile); the streaming kernel can read those rows through a row -> token map instead of a sorted copy.
//
// The output stage (bias, a gated unit over interleaved gate / up rows, GELU times a per-token table row, soft cap, squared ReLU,
// addition to the fp32 stream, plain fp32) is shared by the three kernels (dense_common.cuh).  Waits are bounded as everywhere (common.cuh).
#include "dense_common.cuh"

namespace mfq {

constexpr int kDnTileN = 128, kDnBlockK = 64, kDnThreads = 256;
constexpr int kDnABytes = kDnTileN * kDnBlockK * 2;

template <int BT>
struct DenseCfg {
  static constexpr int kStages = 4;
  static constexpr int kXBytes = BT * kDnBlockK * 2;
  static constexpr int kStageBytes = kDnABytes + kXBytes;
  static constexpr int kTmemCols = BT < 32 ? 32 : BT;
  static constexpr int kMinCtas = BT <= 64 ? 2 : 1;
  static constexpr int kSmemBytes = kStages * kStageBytes + 1024 + 256;
  static_assert(BT * kDnTileN * 4 <= kStages * kStageBytes, "the staged fp32 tile must fit the ring");
};

struct DenseParams {
  DenseEpilogue epi;
  int* status;
  int M, N, K, kb_per_split;
  int groups, x_step, out_step;  // matrices side by side; columns of x / of out between two of them
  const int2* tiles;             // expert form: (matrix, token tile) per blockIdx.y; matrix < 0: nothing
  const int* offsets;            // expert form: first row of every matrix, and the end
  const int* gather;             // expert form, streaming kernel: token of a sorted row (null: rows are sorted already)
};

// What a CTA works on.
struct DenseAt {
  int n0, w_row;      // first output row inside the matrix, and among all matrices' rows
  int x_col, t0, t1;  // first column of x; tokens t0 .. t1 - 1
  int out_col, bias;
};
// False: an unused entry of the tile list.
__device__ __forceinline__ bool dense_locate(const DenseParams& p, int tile_n, int tile_t, DenseAt& at) {
  const int per = (p.N + tile_n - 1) / tile_n, g = int(blockIdx.x) / per;  // per: CTAs along the rows of a matrix
  at.n0 = (int(blockIdx.x) - g * per) * tile_n;
  if (p.tiles) {
    const int2 m = p.tiles[blockIdx.y];
    if (m.x < 0) return false;
    at.w_row = m.x * p.N + at.n0;
    at.x_col = at.out_col = at.bias = 0;
    at.t0 = p.offsets[m.x] + m.y * tile_t;
    at.t1 = min(at.t0 + tile_t, p.offsets[m.x + 1]);
    return true;
  }
  at.w_row = g * p.N + at.n0;
  at.x_col = g * p.x_step;
  at.out_col = g * p.out_step;
  at.bias = g * p.N;
  at.t0 = blockIdx.y * tile_t;
  at.t1 = min(at.t0 + tile_t, p.M);
  return true;
}
template <typename T>
__device__ __forceinline__ DenseEpilogue dense_epilogue_at(const DenseParams& p, const DenseAt& at) {
  DenseEpilogue e = p.epi;
  const bool wide = e.kind == kDenseAdd || e.kind == kDenseFloat;
  e.out = static_cast<uint8_t*>(e.out) + size_t(at.out_col) * (wide ? 4 : sizeof(T));
  if (e.bias) e.bias += at.bias;
  return e;
}

__device__ __forceinline__ void dense_cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t dense_cluster_addr(uint32_t addr, uint32_t cta) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(cta));
  return r;
}
__device__ __forceinline__ float4 dense_cluster_load(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}

template <int BT>
__global__ void __launch_bounds__(kDnThreads, DenseCfg<BT>::kMinCtas)
dense_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, const DenseParams p) {
  using Cfg = DenseCfg<BT>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(base + Cfg::kStages * Cfg::kStageBytes);
  uint64_t* empty = full + Cfg::kStages;
  uint64_t* acc_done = empty + Cfg::kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (p.tiles) pdl_wait();  // the tile list comes from the kernel before
  DenseAt at;
  if (!dense_locate(p, kDnTileN, BT, at)) return;  // all CTAs of a cluster
  const int n0 = at.n0, t0 = at.t0;
  const int kb_total = (p.K + kDnBlockK - 1) / kDnBlockK;
  const int kb0 = blockIdx.z * p.kb_per_split;
  const int nkb = min(kb_total, kb0 + p.kb_per_split) - kb0;  // >= 1 by the host's choice of splits

  if (threadIdx.x == 0) {
    for (int i = 0; i < Cfg::kStages; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 1); }
    mbar_init(acc_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, Cfg::kTmemCols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_acc = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tmap_w);
      tma_prefetch_desc(&tmap_x);
      const int ahead = min(nkb, Cfg::kStages);
      for (int i = 0; i < ahead; ++i) {  // weights never depend on the previous kernel
        mbar_expect_tx(&full[i], Cfg::kStageBytes);
        tma_load_2d(base + i * Cfg::kStageBytes, &tmap_w, &full[i], (kb0 + i) * kDnBlockK, at.w_row);
      }
      pdl_wait();
      for (int i = 0; i < nkb; ++i) {
        const int s = i % Cfg::kStages;
        uint8_t* st = base + s * Cfg::kStageBytes;
        if (i >= ahead) {
          if (!mbar_wait(&empty[s], ((i / Cfg::kStages) & 1) ^ 1, abort_flag, p.status, kStatusTimeoutProducer)) break;
          mbar_expect_tx(&full[s], Cfg::kStageBytes);
          tma_load_2d(st, &tmap_w, &full[s], (kb0 + i) * kDnBlockK, at.w_row);
        }
        tma_load_2d(st + kDnABytes, &tmap_x, &full[s], at.x_col + (kb0 + i) * kDnBlockK, t0);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc(128, BT, 1, 1, 0, 0);
      for (int i = 0; i < nkb; ++i) {
        const int s = i % Cfg::kStages;
        if (!mbar_wait(&full[s], (i / Cfg::kStages) & 1, abort_flag, p.status, kStatusTimeoutMma)) break;
        tc_fence_after();
        const uint32_t a = smem_u32(base + s * Cfg::kStageBytes), b = a + kDnABytes;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          umma_f16(tmem_acc, umma_desc_k_sw128(a + ks * 32), umma_desc_k_sw128(b + ks * 32), idesc, (i | ks) != 0);
        tc_commit(&empty[s]);
      }
      tc_commit(acc_done);
    }
  }
  __syncwarp();
  pdl_wait();  // before this thread's first global access
  // ----- fp32 tile: TMEM -> shared memory [token][128 rows]; warp w reads lane quarter w % 4, half of the columns -----
  const bool ok = __all_sync(0xffffffffu, mbar_wait(acc_done, 0, abort_flag, p.status, kStatusTimeoutEpilogue));
  float* tile = reinterpret_cast<float*>(base);
  const int q = warp & 3, half = warp >> 2;
  if (ok) {
    tc_fence_after();
    constexpr int kHalfCols = BT >= 32 ? BT / 2 : BT;  // 16 columns: one warp per quarter takes them all
    if (BT >= 32 || half == 0) {
#pragma unroll 2
      for (int c = half * kHalfCols; c < half * kHalfCols + kHalfCols; c += 16) {
        uint32_t r[16];
        tmem_ld_32x16(tmem_acc + (uint32_t(q * 32) << 16) + c, r);
        tmem_wait_ld();
#pragma unroll
        for (int j = 0; j < 16; ++j) tile[(c + j) * kDnTileN + q * 32 + lane] = __uint_as_float(r[j]);
      }
    }
    tc_fence_before();
  }
  const int splits = gridDim.z;
  if (splits > 1) dense_cluster_barrier();
  else __syncthreads();
  const int tl = at.t1 - t0, nl = min(kDnTileN, p.N - n0);
  const DenseEpilogue epi = dense_epilogue_at<__nv_bfloat16>(p, at);
  const bool all_ok = splits > 1 || *abort_flag == 0;
  if (all_ok) {
    const int width = dense_is_glu(epi.kind) ? 16 : 8;  // N is a multiple of 16
    const int per = nl / width, items = tl * per;
    const uint32_t tile_addr = smem_u32(tile);
    for (int i = blockIdx.z * kDnThreads + threadIdx.x; i < items; i += splits * kDnThreads) {
      const int t = i / per, n = (i - t * per) * width;
      auto load = [&](int row, float(&v)[8]) {
        const int off = t * kDnTileN + row - n0;
        if (splits == 1) {
          load8<float>(tile + off, v);
          return;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = 0.f;
        for (int z = 0; z < splits; ++z) {
          const uint32_t a = dense_cluster_addr(tile_addr + uint32_t(off) * 4u, z);
          const float4 lo = dense_cluster_load(a), hi = dense_cluster_load(a + 16u);
          v[0] += lo.x; v[1] += lo.y; v[2] += lo.z; v[3] += lo.w;
          v[4] += hi.x; v[5] += hi.y; v[6] += hi.z; v[7] += hi.w;
        }
      };
      dense_store_item<__nv_bfloat16>(epi, t0 + t, n0 + n, load);
    }
  }
  __syncwarp();
  if (splits > 1) dense_cluster_barrier();  // nobody's shared memory goes away while a peer still reads it
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem_acc, Cfg::kTmemCols);
}

template <int BT>
static int launch_dense_gemm(const DenseParams& p0, const void* w, const void* x, int ldx, int matrices, int entries, int splits,
                             cudaStream_t stream) {
  using Cfg = DenseCfg<BT>;
  DenseParams p = p0;
  CUtensorMap tw, tx;
  if (make_tmap_2d(&tw, w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, uint64_t(p.N) * matrices, p.K, uint64_t(p.K) * 2, kDnTileN, kDnBlockK)) return -2;
  if (make_tmap_2d(&tx, x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.M, (p.groups - 1) * p.x_step + p.K, uint64_t(ldx) * 2, BT, kDnBlockK)) return -3;
  const int kb_total = (p.K + kDnBlockK - 1) / kDnBlockK;
  splits = max(1, min(min(splits, 8), kb_total));
  p.kb_per_split = (kb_total + splits - 1) / splits;
  splits = (kb_total + p.kb_per_split - 1) / p.kb_per_split;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(dense_gemm_kernel<BT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes) != cudaSuccess) return -6;
    attr = true;
  }
  const dim3 grid((p.N + kDnTileN - 1) / kDnTileN * p.groups, p.tiles ? entries : (p.M + BT - 1) / BT, splits);
  const cudaError_t rc = splits > 1
      ? launch_kernel_clustered(dense_gemm_kernel<BT>, grid, dim3(kDnThreads), dim3(1, 1, splits), Cfg::kSmemBytes, stream, tw, tx, p)
      : launch_kernel(dense_gemm_kernel<BT>, grid, dim3(kDnThreads), Cfg::kSmemBytes, stream, tw, tx, p);
  return rc == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// ---------------------------------------------------------------------------------------------
// Weight streaming for up to 8 * NT tokens.
// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int NT>
__global__ void __launch_bounds__(256)
dense_gemv_kernel(const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ x, int ldx, const DenseParams p) {
  pdl_trigger();
  constexpr int kBatch = 4;  // K blocks whose weights are requested before the first MMA of the batch
  __shared__ float red[8][16][8 * NT + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  if (p.tiles) pdl_wait();
  DenseAt at;
  if (!dense_locate(p, 16, 8 * NT, at)) return;
  const int n0 = at.n0, K = p.K, rows = at.t1 - at.t0;
  const int blocks = (K + 31) / 32;
  const __nv_bfloat16* w0 = w + size_t(at.w_row + g) * K;
  const __nv_bfloat16* w1 = w0 + size_t(8) * K;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 a[kBatch], b[kBatch];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const int k = (c0 + j * 8) * 32 + t4 * 8;
      a[j] = k < K ? __ldcs(reinterpret_cast<const uint4*>(w0 + k)) : zero;
      b[j] = k < K ? __ldcs(reinterpret_cast<const uint4*>(w1 + k)) : zero;
    }
  };
  fetch(warp);
  pdl_wait();
  const __nv_bfloat16* xr[NT];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int row = at.t0 + min(nt * 8 + g, rows - 1);
    xr[nt] = x + size_t(p.gather ? p.gather[row] : row) * ldx + at.x_col;
  }
  float acc[NT][4] = {};
  for (int c0 = warp; c0 < blocks; c0 += 8 * kBatch) {
    if (c0 != warp) fetch(c0);
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const int k = (c0 + j * 8) * 32 + t4 * 8;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const uint4 xv = (k < K && nt * 8 + g < rows) ? *reinterpret_cast<const uint4*>(xr[nt] + k) : zero;
        mma_bf16_16816(acc[nt], a[j].x, b[j].x, a[j].y, b[j].y, xv.x, xv.y);
        mma_bf16_16816(acc[nt], a[j].z, b[j].z, a[j].w, b[j].w, xv.z, xv.w);
      }
    }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int c = nt * 8 + t4 * 2;
    red[warp][g][c] = acc[nt][0];
    red[warp][g][c + 1] = acc[nt][1];
    red[warp][g + 8][c] = acc[nt][2];
    red[warp][g + 8][c + 1] = acc[nt][3];
  }
  __syncthreads();
  const DenseEpilogue epi = dense_epilogue_at<__nv_bfloat16>(p, at);
  const int width = dense_is_glu(epi.kind) ? 16 : 8, per = 16 / width;
  for (int i = threadIdx.x; i < rows * per; i += 256) {
    const int t = i / per, n = (i - t * per) * width;
    dense_store_item<__nv_bfloat16>(epi, at.t0 + t, n0 + n, [&](int row, float(&v)[8]) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        float s = 0.f;
#pragma unroll
        for (int z = 0; z < 8; ++z) s += red[z][row - n0 + j][t];
        v[j] = s;
      }
    });
  }
}

template <int NT>
static int launch_dense_gemv(const void* w, const void* x, int ldx, const DenseParams& p, int entries, cudaStream_t stream) {
  // The loads in flight live in L1.  On an SM that a kernel with much shared memory leaves behind, L1 would stay small and
  // the stream slow, so this kernel asks for a small shared-memory carve-out.
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(dense_gemv_kernel<NT>, cudaFuncAttributePreferredSharedMemoryCarveout, 15 * NT) != cudaSuccess) return -6;
    set = true;
  }
  launch_kernel(dense_gemv_kernel<NT>, dim3(p.N / 16 * p.groups, p.tiles ? entries : 1), dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(w),
                static_cast<const __nv_bfloat16*>(x), ldx, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// ---------------------------------------------------------------------------------------------
// fp32 operands: 64 tokens x 64 rows per CTA, 16-wide K steps, 4 x 4 outputs per thread.
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
dense_sgemm_kernel(const float* __restrict__ w, const float* __restrict__ x, int ldx, const DenseParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float sw[16][68], sx[16][68];
  __shared__ __align__(16) float tile[64][64];
  DenseAt at;
  if (!dense_locate(p, 64, 64, at)) return;
  const int n0 = at.n0, t0 = at.t0, tid = threadIdx.x;
  const int tn = (tid & 15) * 4, tt = (tid >> 4) * 4;
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
    const int k = k0 + lk;  // K is a multiple of 8: a group of 4 is inside or outside
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 a = (n0 + lr < p.N && k < p.K) ? *reinterpret_cast<const float4*>(w + size_t(at.w_row + lr) * p.K + k) : zero;
    const float4 b = (t0 + lr < at.t1 && k < p.K) ? *reinterpret_cast<const float4*>(x + size_t(t0 + lr) * ldx + at.x_col + k) : zero;
    sw[lk][lr] = a.x; sw[lk + 1][lr] = a.y; sw[lk + 2][lr] = a.z; sw[lk + 3][lr] = a.w;
    sx[lk][lr] = b.x; sx[lk + 1][lr] = b.y; sx[lk + 2][lr] = b.z; sx[lk + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float av[4], bv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { av[i] = sw[kk][tn + i]; bv[i] = sx[kk][tt + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(bv[i], av[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) tile[tt + i][tn + j] = acc[i][j];
  __syncthreads();
  const int tl = at.t1 - t0, nl = min(64, p.N - n0);
  const DenseEpilogue epi = dense_epilogue_at<float>(p, at);
  const int width = dense_is_glu(epi.kind) ? 16 : 8, per = nl / width;
  for (int i = tid; i < tl * per; i += 256) {
    const int t = i / per, n = (i - t * per) * width;
    dense_store_item<float>(epi, t0 + t, n0 + n, [&](int row, float(&v)[8]) { load8<float>(&tile[t][row - n0], v); });
  }
}

static int run_dense(const DenseParams& p, const void* w, const void* x, int ldx, int matrices, int entries, int token_tile, int splits,
                     int fp32, cudaStream_t stream) {
  const int kind = p.epi.kind;
  if (p.M <= 0 || p.N <= 0 || p.K <= 0 || p.N % 16 || p.K % 8 || ldx % 8 || ldx < (p.groups - 1) * p.x_step + p.K || p.epi.ldo % 8) return -1;
  if (kind < kDenseBias || kind > kDenseRelu2 || (kind == kDenseGelu && (!p.epi.table || !p.epi.ids))) return -1;
  if (kind == kDenseSoftcap && !(p.epi.limit > 0.f)) return -1;
  if (p.epi.ldo < (p.groups - 1) * p.out_step + (dense_is_glu(kind) ? p.N / 2 : p.N)) return -1;
  if (fp32) {
    launch_kernel(dense_sgemm_kernel, dim3((p.N + 63) / 64 * p.groups, p.tiles ? entries : (p.M + 63) / 64), dim3(256), 0, stream,
                  static_cast<const float*>(w), static_cast<const float*>(x), ldx, p);
    return cudaGetLastError() == cudaSuccess ? 0 : -7;
  }
  if (token_tile == 0) {
    if (!p.tiles && p.M > 16) return -1;
    return !p.tiles && p.M <= 8 ? launch_dense_gemv<1>(w, x, ldx, p, entries, stream) : launch_dense_gemv<2>(w, x, ldx, p, entries, stream);
  }
  switch (token_tile) {
    case 16: return launch_dense_gemm<16>(p, w, x, ldx, matrices, entries, splits, stream);
    case 32: return launch_dense_gemm<32>(p, w, x, ldx, matrices, entries, splits, stream);
    case 64: return launch_dense_gemm<64>(p, w, x, ldx, matrices, entries, splits, stream);
    case 128: return launch_dense_gemm<128>(p, w, x, ldx, matrices, entries, splits, stream);
    case 256: return launch_dense_gemm<256>(p, w, x, ldx, matrices, entries, splits, stream);
    default: return -1;
  }
}

}  // namespace mfq

// w [N, K] row-major, x [M, ldx], both bf16 (fp32 = 0) or fp32 (fp32 = 1).  N a multiple of 16, K and ldx of 8, M > 0; ldo of 8.
// token_tile 0: the weight-streaming kernel (M <= 16); 16 .. 256: the tcgen05 kernel with that tile and `splits` K splits.
// groups > 1: w [groups, N, K] (bias [groups, N]); matrix g reads x from column g * x_step on and writes out from g * out_step on
// (multiples of 8).
extern "C" int mfq_dense_linear(const void* w, const void* x, int ldx, void* out, int ldo, const float* bias, int M, int N, int K,
                                int groups, int x_step, int out_step, int epilogue, float alpha, float limit, const void* table,
                                const int* ids, int token_tile, int splits, int fp32, int* status, cudaStream_t stream) {
  using namespace mfq;
  if (groups < 1 || x_step % 8 || out_step % 8 || (groups > 1 && (epilogue == kDenseGelu || x_step < 0 || out_step < 0))) return -1;
  const DenseParams p{DenseEpilogue{epilogue, bias, alpha, limit, table, ids, out, ldo}, status, M, N, K, 0, groups, x_step, out_step,
                      nullptr, nullptr, nullptr};
  return run_dense(p, w, x, ldx, groups, 0, token_tile, splits, fp32, stream);
}

// Expert form: w [experts, N, K]; rows offsets[e] .. offsets[e + 1] - 1 of out (and of x, unless `gather` gives the row of x for each)
// belong to expert e.  tiles [entries]: (expert, token tile), tiles of `token_tile` rows, 16 for the streaming kernel (token_tile 0),
// 64 in fp32.  x has M rows.  `gather` is for the streaming kernel only.
extern "C" int mfq_dense_experts(const void* w, const void* x, int ldx, void* out, int ldo, int M, int N, int K, int experts,
                                 const int* tiles, int entries, const int* offsets, const int* gather, int epilogue, int token_tile,
                                 int fp32, int* status, cudaStream_t stream) {
  using namespace mfq;
  if (experts <= 0 || !tiles || entries <= 0 || entries > 65535 || !offsets || epilogue == kDenseGelu || epilogue == kDenseAdd) return -1;
  if (gather && (fp32 || token_tile)) return -1;
  const DenseParams p{DenseEpilogue{epilogue, nullptr, 0.f, 0.f, nullptr, nullptr, out, ldo}, status, M, N, K, 0, 1, 0, 0,
                      reinterpret_cast<const int2*>(tiles), offsets, gather};
  return run_dense(p, w, x, ldx, experts, entries, token_tile, 1, fp32, stream);
}
