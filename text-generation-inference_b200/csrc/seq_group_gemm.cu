// Groups of products on tcgen05 tensor cores: bfloat16 operands, fp32 accumulators in TMEM, one 128-feature x TN-row tile per block.
//   heads   (MODE 0): Y[t, z] = W[z] X[t, z] for every head z of every token; X and Y rows may be slices of wider rows (strides per token
//                     and per head): latent attention's absorbed query and its value up-projection.
//   experts (MODE 1): Y[row] = act(W[expert of row] X[row]) over the compact rows of a routing plan (seq_moe.cu): rows of one expert are
//                     contiguous, a block finds its (expert, row tile) from the plan's offsets, so nothing is read back to the host and
//                     the whole product is one launch for any distribution of the rows.
//
// The 128 features of a weight tile are the UMMA M dimension (K-major, 128-byte swizzle, by TMA), TN rows of X its N dimension.  A tile
// may reach into the next head's or expert's weight rows, or into the next expert's rows of X: those results are dropped in the
// epilogue.  Columns of X beyond K (another head's) meet zeros, which the tensor map of W supplies there.  Two blocks share an SM, so
// that one's epilogue (TMEM -> registers -> HBM) runs under the other's products.
// Warp roles: 0 = TMA producer, 1 = MMA issuer (one elected thread each), 2..5 = epilogue.
//
// Every wait is bounded: a block that gives up counts itself in `group_gemm_gave_up`, waits for its copies in flight, frees its TMEM and ends.
#include "seq_common.cuh"
#include "tmap.cuh"

namespace b200 {
namespace seq {

constexpr int kGgThreads = 192, kGgTileM = 128, kGgTileK = 64;

__device__ int group_gemm_gave_up;

template <int TN>
struct GgCfg {
  static constexpr int kABytes = kGgTileM * kGgTileK * 2, kBBytes = TN * kGgTileK * 2, kStageBytes = kABytes + kBBytes;
  static constexpr int kStages = TN == 256 ? 2 : TN == 128 ? 3 : 4;
  static constexpr int kTmemCols = TN < 32 ? 32 : TN;
  static constexpr int kSmemBytes = kStages * kStageBytes + (2 * kStages + 1) * 8 + 16 + 1024;
};

struct GgParams {
  void* y;
  int64_t ldy, head_y;    // heads: columns between two heads' results
  int64_t head_x;         // heads: columns between two heads' inputs
  const int32_t* offsets; // experts: first compact row of every expert [E + 1]
  int E, T, N, nkb, out_f32, act;
};

__device__ __forceinline__ bool mbar_wait_limited(uint64_t* bar, uint32_t parity) {
  for (uint32_t spins = 0; spins < (1u << 24); ++spins)
    if (mbar_try_wait(bar, parity)) return true;
  return false;
}

template <int TN, int MODE>
__global__ void __launch_bounds__(kGgThreads, 2) group_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x,
                                                                   const GgParams p) {
  using C = GgCfg<TN>;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + C::kStages * C::kStageBytes);
  uint64_t* empty_bar = full_bar + C::kStages;
  uint64_t* tmem_full = empty_bar + C::kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tmem_full + 1);
  __shared__ int s_expert, s_row0, s_row_end;

  pdl_launch_dependents();
  const int warp = warp_id(), lane = lane_id();
  int group = 0, row0 = 0, row_end = 0;
  if constexpr (MODE == 0) {
    group = blockIdx.z;
    row0 = blockIdx.y * TN;
    row_end = p.T;
  } else {
    pdl_wait();
    if (warp == 0) {   // which expert's which row tile is number blockIdx.y: a scan of the tile counts, 8 experts per lane
      int n[8], sum = 0;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int e = lane * 8 + i;
        n[i] = e < p.E ? (p.offsets[e + 1] - p.offsets[e] + TN - 1) / TN : 0;
        sum += n[i];
      }
      int before = sum;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += v;
      }
      before -= sum;
      if (lane == 0) s_expert = -1;
      __syncwarp();
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int tile = (int)blockIdx.y - before;
        if (tile >= 0 && tile < n[i]) {
          const int e = lane * 8 + i;
          s_expert = e;
          s_row0 = p.offsets[e] + tile * TN;
          s_row_end = p.offsets[e + 1];
        }
        before += n[i];
      }
    }
    __syncthreads();
    group = s_expert;
    if (group < 0) return;   // more blocks than tiles: block-uniform, nothing is held yet
    row0 = s_row0;
    row_end = s_row_end;
  }
  const int n0 = blockIdx.x * kGgTileM;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmap_w);
    tma_prefetch_desc(&tmap_x);
    for (int s = 0; s < C::kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    mbar_init(tmem_full, 1);
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc<C::kTmemCols>(tmem_slot);
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_d = *tmem_slot;
  bool ok = true;

  if (warp == 0) {
    if (elect_one()) {
      const int x_col = MODE == 0 ? (int)(group * p.head_x) : 0, w_row = group * p.N + n0;
      int issued = 0;
      // weights do not depend on the kernel before this one (heads): the ring is filled with them ahead of the wait for it
      const int npre = MODE == 0 ? min(p.nkb, C::kStages) : 0;
      for (; issued < npre; ++issued) {
        mbar_arrive_expect_tx(&full_bar[issued], C::kStageBytes);
        tma_load_2d(smem + issued * C::kStageBytes, &tmap_w, issued * kGgTileK, w_row, &full_bar[issued]);
      }
      if constexpr (MODE == 0) {
        pdl_wait();
        for (int i = 0; i < npre; ++i)
          tma_load_2d(smem + i * C::kStageBytes + C::kABytes, &tmap_x, x_col + i * kGgTileK, row0, &full_bar[i]);
      }
      for (; issued < p.nkb; ++issued) {
        const int s = issued % C::kStages;
        if (!mbar_wait_limited(&empty_bar[s], ((issued / C::kStages) & 1) ^ 1)) { ok = false; break; }
        mbar_arrive_expect_tx(&full_bar[s], C::kStageBytes);
        unsigned char* a = smem + s * C::kStageBytes;
        tma_load_2d(a, &tmap_w, issued * kGgTileK, w_row, &full_bar[s]);
        tma_load_2d(a + C::kABytes, &tmap_x, x_col + issued * kGgTileK, row0, &full_bar[s]);
      }
      // the copies of the last ring's worth have landed before the block may end, whatever the other warps met
      for (int i = max(0, issued - C::kStages); i < issued; ++i) ok = mbar_wait_limited(&full_bar[i % C::kStages], (i / C::kStages) & 1) && ok;
    }
    __syncwarp();
  } else if (warp == 1) {
    constexpr uint32_t idesc = umma_idesc_f16_f32acc(kGgTileM, TN) | (1u << 7) | (1u << 10);   // a / b format 1 = bf16
    for (int i = 0; i < p.nkb; ++i) {
      const int s = i % C::kStages;
      if (!mbar_wait_limited(&full_bar[s], (i / C::kStages) & 1)) { ok = false; break; }
      tcgen05_fence_after();
      if (elect_one()) {
        const uint32_t a_addr = smem_u32(smem + s * C::kStageBytes);
        const uint64_t adesc = umma_desc_kmajor_sw128(a_addr), bdesc = umma_desc_kmajor_sw128(a_addr + C::kABytes);
#pragma unroll
        for (int k = 0; k < kGgTileK / 16; ++k)
          umma_f16_ss(tmem_d, adesc + (uint64_t)(k * 2), bdesc + (uint64_t)(k * 2), idesc, (i > 0 || k > 0) ? 1u : 0u);
        umma_commit(&empty_bar[s]);
        if (i == p.nkb - 1) umma_commit(tmem_full);
      }
      __syncwarp();
    }
    // the accumulator is complete (or was given up) before this block may free it
    ok = mbar_wait_limited(tmem_full, 0) && ok;
  } else {
    const int m = (warp & 3) * 32 + lane, n = n0 + m;
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const bool n_ok = n < p.N;
    if constexpr (MODE == 0) pdl_wait();   // the output belongs to the stream order
    ok = mbar_wait_limited(tmem_full, 0);
    if (ok) {
      tcgen05_fence_after();
      const int rows = min(TN, row_end - row0);
      const int64_t base = (int64_t)row0 * p.ldy + (MODE == 0 ? group * p.head_y : 0) + n;
#pragma unroll 1
      for (int c = 0; c < rows; c += 16) {
        uint32_t d[16];
        tmem_ld_32x32b_x16(tmem_d + lane_base + c, d);
        tmem_ld_wait();
        if (n_ok) {
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            if (c + j >= rows) break;
            float v = __uint_as_float(d[j]);
            if (p.act) v = v < 0.f ? 0.f : v * v;
            const int64_t at = base + (int64_t)(c + j) * p.ldy;
            if (p.out_f32) reinterpret_cast<float*>(p.y)[at] = v;
            else reinterpret_cast<__nv_bfloat16*>(p.y)[at] = __float2bfloat16_rn(v);
          }
        }
      }
    }
  }
  if (!ok) atomicAdd(&group_gemm_gave_up, 1);
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc<C::kTmemCols>(tmem_d);
}

template <int TN, int MODE>
static int launch_group_gemm(const void* w, int64_t w_rows, int64_t K, const void* x, int64_t x_rows, int64_t x_cols, int64_t ldx, dim3 grid,
                             const GgParams& p, cudaStream_t st) {
  using C = GgCfg<TN>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(group_gemm_kernel<TN, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
    if (e != cudaSuccess) { b200_set_last_error(cudaGetErrorString(e)); return B200_ERR_CUDA; }
    configured = true;
  }
  const CUtensorMap* mw = get_tmap_2d(w, w_rows, K, K, kGgTileM, kGgTileK, TmapDtype::kF16, TmapSwizzle::k128B);
  const CUtensorMap* mx = get_tmap_2d(x, x_rows, x_cols, ldx, TN, kGgTileK, TmapDtype::kF16, TmapSwizzle::k128B);
  if (!mw || !mx) return B200_ERR_CUDA;
  B200_LAUNCH((group_gemm_kernel<TN, MODE>), grid, dim3(kGgThreads), (size_t)C::kSmemBytes, st, *mw, *mx, p);
  b200_count_launches(1);
  return B200_OK;
}

}  // namespace seq
}  // namespace b200

using namespace b200;
using namespace b200::seq;

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// blocks of this process's grouped products that gave up a wait (0 unless something is wrong); -1: the count could not be read
extern "C" int b200_seq_group_gemm_gave_up(void) {
  int n = 0;
  return cudaMemcpyFromSymbol(&n, group_gemm_gave_up, sizeof(int)) == cudaSuccess ? n : -1;
}

// Y[t, z, :N] = W[z] [N, K] X[t, z, :K] for z < Z, t < T: bfloat16 X (token stride ldx, head stride head_x) and dense W [Z, N, K]; Y of type
// y_dt (token stride ldy, head stride head_y).  K, ldx and head_x multiples of 8, X and W 16-byte aligned.
extern "C" int b200_seq_heads_gemm(const void* x, int64_t ldx, int64_t head_x, const void* w, void* y, int y_dt, int64_t ldy, int64_t head_y, int64_t T,
                                   int64_t Z, int64_t N, int64_t K, void* stream) {
  if (T == 0 || Z == 0 || N == 0) return B200_OK;
  if (K <= 0 || K % 8 || ldx % 8 || head_x % 8 || !aligned16(x) || !aligned16(w) || Z > 65535 || (y_dt != B200_DT_BF16 && y_dt != B200_DT_F32) ||
      ldx < (Z - 1) * head_x + K) {
    b200_set_last_error("seq_heads_gemm: need K, strides in multiples of 8, 16-byte aligned operands, heads inside a row");
    return B200_ERR_ARG;
  }
  GgParams p{y, ldy, head_y, head_x, nullptr, 0, (int)T, (int)N, (int)((K + kGgTileK - 1) / kGgTileK), y_dt == B200_DT_F32, 0};
  const int TN = T <= 16 ? 16 : T <= 32 ? 32 : T <= 64 ? 64 : T <= 128 ? 128 : 256;
  const int64_t tiles_t = (T + TN - 1) / TN;
  if (tiles_t > 65535) { b200_set_last_error("seq_heads_gemm: too many rows"); return B200_ERR_ARG; }
  const dim3 grid((unsigned)((N + kGgTileM - 1) / kGgTileM), (unsigned)tiles_t, (unsigned)Z);
  const int64_t x_cols = (Z - 1) * head_x + K;
  cudaStream_t st = (cudaStream_t)stream;
#define GG(TN_) launch_group_gemm<TN_, 0>(w, Z * N, K, x, T, x_cols, ldx, grid, p, st)
  switch (TN) {
    case 16: return GG(16);
    case 32: return GG(32);
    case 64: return GG(64);
    case 128: return GG(128);
    default: return GG(256);
  }
#undef GG
}

// Y[row, :N] = act(W[expert(row)] [N, K] X[row, :K]) for the compact rows of a routing plan: bfloat16 X [max_rows, K] (dense) and W [E, N, K]
// (dense), Y dense of type y_dt.  offsets int32 [E + 1]: the plan's first row of every expert (b200_seq_moe_offsets).  act 0: none, 1: relu squared.
extern "C" int b200_seq_experts_gemm(const void* x, const void* w, void* y, int y_dt, const int32_t* offsets, int64_t max_rows, int E, int64_t N,
                                     int64_t K, int act, void* stream) {
  if (max_rows == 0 || N == 0) return B200_OK;
  if (E < 1 || E > 256 || K <= 0 || K % 8 || !aligned16(x) || !aligned16(w) || (y_dt != B200_DT_BF16 && y_dt != B200_DT_F32)) {
    b200_set_last_error("seq_experts_gemm: need at most 256 experts, K a multiple of 8, 16-byte aligned operands");
    return B200_ERR_ARG;
  }
  GgParams p{y, N, 0, 0, offsets, E, (int)max_rows, (int)N, (int)((K + kGgTileK - 1) / kGgTileK), y_dt == B200_DT_F32, act};
  const int TN = max_rows / E >= 160 ? 256 : 128;   // rows per expert, were they dealt out evenly
  const int64_t tiles = (max_rows + TN - 1) / TN + E;
  if (tiles > 65535) { b200_set_last_error("seq_experts_gemm: too many rows"); return B200_ERR_ARG; }
  const dim3 grid((unsigned)((N + kGgTileM - 1) / kGgTileM), (unsigned)tiles, 1);
  cudaStream_t st = (cudaStream_t)stream;
  if (TN == 256) return launch_group_gemm<256, 1>(w, (int64_t)E * N, K, x, max_rows, K, K, grid, p, st);
  return launch_group_gemm<128, 1>(w, (int64_t)E * N, K, x, max_rows, K, K, grid, p, st);
}
