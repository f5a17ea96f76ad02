// Latent attention over a paged latent cache.
//
// A token caches ONE row of D = R + r elements per layer: its normalised latent c (R) and its rotated shared key part (r).
// Attention runs in the absorbed form: a head's query is carried into latent space once (q~ = Wuk_h^T q_plain, done by the
// per-head products of seq_group_gemm.cu / seq_linear.cu), so that score(i, j) = (q~_i . c_j + qrot_i . krot_j) * scale and the head's output is
// Wuv_h (sum_j p_ij c_j): every head reads the same cache row, nothing per head is ever stored.
//
//   latent_prepare_kernel : RMS-norms the latent slice of the down-projection, rotates the shared key part, writes both into the
//                           token's cache slot; rotates each head's query part into the absorbed-query buffer.
//   latent_attn_kernel    : one block per (query token, group of heads), one warp per head; streams the visible window
//                           [p - window + 1, p] of the sequence's pages in tiles of 32 keys through shared memory, fp32 online
//                           soft-max.  Serves prompts, portions of prompts that follow cached tokens and single decoded tokens
//                           alike: a query's keys are always read back from the cache, whatever step wrote them.
//   latent_attn_tile_kernel : bfloat16 caches, tensor-core products; see the note above the kernel.
// A sink logit per head may join the soft-max denominator (unscaled, no value).
//
// Rotation: interleaved pairs (2i, 2i+1) of the first `rot_dims` elements, angle tables [positions, rot_dims/2] (fp32, made
// by the host with any frequency scaling and amplitude factor folded in); elements past rot_dims pass unchanged.
#include "seq_common.cuh"

#include <cstdlib>

namespace b200 {
namespace seq {

constexpr int kPrepThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(
    const float* __restrict__ down, int64_t ld_down, int col_c, int col_kr,  // down-projection row: latent at col_c, key part at col_kr
    const T* __restrict__ q, int64_t ld_q, int q_head_stride, int q_rot_off,  // per head: rotated part at h*stride + off
    const T* __restrict__ cnorm_w, const float* __restrict__ cos_t, const float* __restrict__ sin_t, const int64_t* __restrict__ position_ids,
    const int64_t* __restrict__ slot_mapping, T* __restrict__ cache, T* __restrict__ q_abs, int H, int R, int r, int rot_dims, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int D = R + r, half = rot_dims / 2;
  const int64_t pos = position_ids[t];
  const int64_t slot = slot_mapping[t];
  const float* crow = down + t * ld_down + col_c;
  float s = 0.f;
  for (int i = threadIdx.x; i < R; i += kPrepThreads) s += crow[i] * crow[i];
  const float rstd = 1.f / sqrtf(block_sum(s, red) / R + eps);
  const float* cs = cos_t + pos * half;
  const float* sn = sin_t + pos * half;
  if (slot >= 0) {
    T* dst = cache + slot * D;
    for (int i = threadIdx.x; i < R; i += kPrepThreads) stf(dst + i, crow[i] * rstd * ldf(cnorm_w + i));
    const float* kr = down + t * ld_down + col_kr;
    for (int i = threadIdx.x; i < r; i += kPrepThreads) {
      float v;
      if (i < rot_dims) {
        const int p = i >> 1;
        const float a = kr[2 * p], b = kr[2 * p + 1];
        v = (i & 1) ? b * cs[p] + a * sn[p] : a * cs[p] - b * sn[p];
      } else {
        v = kr[i];
      }
      stf(dst + R + i, v);
    }
  }
  for (int idx = threadIdx.x; idx < H * r; idx += kPrepThreads) {
    const int h = idx / r, i = idx % r;
    const T* qr = q + t * ld_q + (int64_t)h * q_head_stride + q_rot_off;
    float v;
    if (i < rot_dims) {
      const int p = i >> 1;
      const float a = ldf(qr + 2 * p), b = ldf(qr + 2 * p + 1);
      v = (i & 1) ? b * cs[p] + a * sn[p] : a * cs[p] - b * sn[p];
    } else {
      v = ldf(qr + i);
    }
    stf(q_abs + (t * H + h) * D + R + i, v);
  }
}

constexpr int kHeadsPerBlock = 8, kKeyTile = 32;

template <typename T, int NR>
__global__ void __launch_bounds__(kHeadsPerBlock * 32) latent_attn_kernel(
    const T* __restrict__ q_abs, const T* __restrict__ cache, const int32_t* __restrict__ block_table, int64_t bt_stride,
    const int32_t* __restrict__ seq_of_token, const int64_t* __restrict__ position_ids, T* __restrict__ out, int H, int R, int D, int window,
    float scale, int page, const float* __restrict__ sink) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  float* qs = sm;                        // [kHeadsPerBlock][D]
  float* ks = sm + kHeadsPerBlock * D;   // [kKeyTile][D + 1]
  const int64_t t = blockIdx.x;
  const int h0 = blockIdx.y * kHeadsPerBlock;
  const int w = warp_id(), lane = lane_id();
  const int h = h0 + w;
  const int b = seq_of_token[t];
  const int p = (int)position_ids[t];
  const int j_lo = max(0, p - window + 1);
  const int nthreads = kHeadsPerBlock * 32;
  for (int idx = threadIdx.x; idx < kHeadsPerBlock * D; idx += nthreads) {
    const int hh = h0 + idx / D;
    qs[idx] = hh < H ? ldf(q_abs + (t * H + hh) * D + idx % D) : 0.f;
  }
  // a sink logit sits in the soft-max denominator like one more key (unscaled) whose value is zero
  float m = (sink && h < H) ? sink[h] : -INFINITY, l = (sink && h < H) ? 1.f : 0.f;
  float acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) acc[i] = 0.f;
  const int32_t* table = block_table + (int64_t)b * bt_stride;
  for (int j0 = j_lo; j0 <= p; j0 += kKeyTile) {
    __syncthreads();  // the previous tile is consumed (and qs is written, first time round)
    const int nk = min(kKeyTile, p - j0 + 1);
    for (int idx = threadIdx.x; idx < nk * D; idx += nthreads) {
      const int jj = idx / D, dd = idx % D;
      const int j = j0 + jj;
      const int64_t row = (int64_t)table[j / page] * page + j % page;
      ks[jj * (D + 1) + dd] = ldf(cache + row * D + dd);
    }
    __syncthreads();
    if (h < H) {
      float s = -INFINITY;
      if (lane < nk) {
        float a = 0.f;
        const float* kq = ks + lane * (D + 1);
        const float* qq = qs + w * D;
        for (int d = 0; d < D; ++d) a = fmaf(qq[d], kq[d], a);
        s = a * scale;
      }
      const float m_new = fmaxf(m, warp_max(s));
      const float pr = lane < nk ? expf(s - m_new) : 0.f;
      const float corr = expf(m - m_new);  // m = -inf on the first tile: 0
      l = l * corr + warp_sum(pr);
      m = m_new;
#pragma unroll
      for (int i = 0; i < NR; ++i) acc[i] *= corr;
      for (int jj = 0; jj < nk; ++jj) {
        const float pj = __shfl_sync(0xffffffffu, pr, jj);
        const float* kr = ks + jj * (D + 1);
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int d = lane + 32 * i;
          if (d < R) acc[i] = fmaf(pj, kr[d], acc[i]);
        }
      }
    }
  }
  if (h < H) {
    const float inv = 1.f / l;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = lane + 32 * i;
      if (d < R) stf(out + (t * H + h) * R + d, acc[i] * inv);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------------
// Tensor-core form for bfloat16 caches.  The rows of a sequence are its (token, head) pairs in order; one block has RG * 16 consecutive
// rows of one sequence, so a key tile that it fetches serves several tokens' heads at once: the cache row of a key is the B operand
// of S = Q K^T (all D columns) and, read transposed, of O += P V (its first R columns).  Key tiles of KT rows come in with 16-byte
// cp.async, kStages of them in flight.  S: warp (row group, 16 keys) with m16n8k16 products; the row maxima meet in shared memory (fp32
// online soft-max in powers of two, every warp of a row group keeps the same running maximum, each its own keys' sum), P goes to
// shared memory as bfloat16.  O: warp (PRT row groups, every PC-th 16 output columns), accumulators in registers.
// gridDim.z > 1 deals the block's key tiles out in runs whose partial (output, max, sum) latent_attn_merge_kernel joins.
// Needs R % 16 == 0, r % 16 == 0, R <= 512; other shapes and float32 caches take latent_attn_kernel above.
// ------------------------------------------------------------------------------------------------------------------------
constexpr int kTileThreads = 256, kTilePad = 8;

template <int RG>
struct LatentTile {
  static constexpr int kRows = RG * 16, KT = RG == 4 ? 32 : 64, KG = KT / 16, kStages = RG == 4 ? 3 : 2;
  static constexpr int PRT = RG == 4 ? 2 : RG, PC = 8 / (RG / PRT);   // row groups per warp and column groups of O
  static size_t smem(int D) {
    return ((size_t)(kRows + kStages * KT) * (D + kTilePad) + (size_t)kRows * (KT + kTilePad)) * 2 + (size_t)(2 * KG + 2) * kRows * 4;
  }
};

// which (sequence, tile of `rows` of its (token, head) rows) block `tile` has, a sequence's last tile first; b == B: none
__device__ __forceinline__ void latent_find_tile(const int32_t* cu_q, int B, int H, int rows, int tile, int& b, int& first, int& n_rows) {
  find_ragged_tile(cu_q, B, H, rows, b, tile);
  if (b >= B) return;
  const int n = (cu_q[b + 1] - cu_q[b]) * H, nt = (n + rows - 1) / rows;
  first = (nt - 1 - tile) * rows;   // the last rows see the most keys: they start first
  n_rows = min(rows, n - first);
}

template <typename T>
__device__ __forceinline__ void latent_store(void* out, int64_t i, float a, float b) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float2*>(reinterpret_cast<float*>(out) + i) = make_float2(a, b);
  else *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(out) + i) = __floats2bfloat162_rn(a, b);
}

template <int RG, int NP>  // NP: 16-column pieces of O per warp, at most
__global__ void __launch_bounds__(kTileThreads) latent_attn_tile_kernel(
    const __nv_bfloat16* __restrict__ q_abs, const __nv_bfloat16* __restrict__ cache, const int32_t* __restrict__ block_table, int64_t bt_stride,
    const int32_t* __restrict__ cu_q, int B, const int64_t* __restrict__ position_ids, __nv_bfloat16* __restrict__ out, int H, int R, int D, int window,
    float scale_log2, int page, float* __restrict__ partial, const float* __restrict__ sink) {
  using L = LatentTile<RG>;
  constexpr int ROWS = L::kRows, KT = L::KT, KG = L::KG, ST = L::kStages, PRT = L::PRT, PC = L::PC, PP = KT + kTilePad;
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int DP = D + kTilePad;                                       // padded row: rows 16 bytes apart modulo 128 -> conflict-free ldmatrix
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [ROWS][DP]
  __nv_bfloat16* Ks = Qs + ROWS * DP;                                // [ST][KT][DP]
  __nv_bfloat16* Ps = Ks + ST * KT * DP;                             // [ROWS][PP]
  float* red_max = reinterpret_cast<float*>(Ps + ROWS * PP);         // [KG][ROWS]
  float* red_sum = red_max + KG * ROWS;                              // [KG][ROWS]
  float* corr_s = red_sum + KG * ROWS;                               // [ROWS]
  float* max_s = corr_s + ROWS;                                      // [ROWS]
  int b, first = 0, n_rows = 0;
  latent_find_tile(cu_q, B, H, ROWS, blockIdx.x, b, first, n_rows);
  if (b >= B) return;  // block-uniform: no barrier has been met yet
  const int w = warp_id(), lane = lane_id();
  const int64_t row_base = (int64_t)cu_q[b] * H + first;             // this block's first row in q_abs and out
  const int p_seq = (int)position_ids[cu_q[b]];
  const int p_first = p_seq + first / H, p_last = p_seq + (first + n_rows - 1) / H;
  const int j_first = max(0, p_first - window + 1);
  const int n_ktiles = (p_last - j_first + KT) / KT;
  const int per_split = (n_ktiles + gridDim.z - 1) / gridDim.z;
  const int j_start = j_first + (int)blockIdx.z * per_split * KT;
  const int j_end = min(p_last, j_start + per_split * KT - 1);       // last key of this block's run
  const int n_tiles = j_start <= j_end ? (j_end - j_start + KT) / KT : 0;
  const int32_t* table = block_table + (int64_t)b * bt_stride;
  const int chunks = D / 8;  // 16-byte pieces of a row
  for (int row = threadIdx.x >> 3; row < ROWS; row += kTileThreads / 8)
    for (int ch = threadIdx.x & 7; ch < chunks; ch += 8)
      cp_async_16(Qs + row * DP + ch * 8, q_abs + (row < n_rows ? (row_base + row) * D + ch * 8 : 0), row < n_rows);   // rows beyond: zeros
  const int page_shift = (page & (page - 1)) == 0 ? 31 - __clz(page) : -1;
  auto load_tile = [&](int i) {   // one commit group per call, empty past the last tile
    if (i < n_tiles) {
      constexpr int kPer = kTileThreads / KT;   // threads per key row
      const int row = threadIdx.x / kPer, j = j_start + i * KT + row;
      __nv_bfloat16* dst = Ks + ((i % ST) * KT + row) * DP;
      const bool live = j <= j_end;
      const int64_t blk = live ? table[page_shift >= 0 ? j >> page_shift : j / page] : 0;
      const __nv_bfloat16* src = cache + (blk * page + (live ? (page_shift >= 0 ? j & (page - 1) : j % page) : 0)) * D;
      for (int ch = threadIdx.x % kPer; ch < chunks; ch += kPer) cp_async_16(dst + ch * 8, src + ch * 8, live);   // dead rows: zeros (they meet p = 0)
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < ST - 1; ++i) load_tile(i);

  // scores: warp (row group, key group); the thread's two accumulator rows
  const int rg = w % RG, kg = w / RG;
  const bool s_warp = kg < KG && rg * 16 < n_rows;
  const int cq = (lane & 3) * 2, lm = lane >> 3, lr = lane & 7;
  int p_row[2], lo_row[2];
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = min(rg * 16 + (lane >> 2) + i * 8, n_rows - 1);
    p_row[i] = p_seq + (first + r) / H;
    lo_row[i] = p_row[i] - window + 1;
    if (sink && blockIdx.z == 0) {   // the sink counts once: in the first run of the keys, by one lane of the row
      m_run[i] = sink[(first + r) % H] * 1.4426950408889634f;
      l_run[i] = kg == 0 && (lane & 3) == 0 ? 1.f : 0.f;
    }
  }
  const int lo_last = p_last - window + 1;
  // output: warp (PRT row groups from ro, 16-column pieces pc, pc + PC, ...)
  const int ro = (w / PC) * PRT, pc = w % PC, pieces = R / 16;
  const bool o_warp = ro * 16 < n_rows;
  float o[PRT][NP * 2][4];
#pragma unroll
  for (int t = 0; t < PRT; ++t)
#pragma unroll
    for (int i = 0; i < NP * 2; ++i) o[t][i][0] = o[t][i][1] = o[t][i][2] = o[t][i][3] = 0.f;
  const uint32_t ks_addr = smem_u32(Ks), ps_addr = smem_u32(Ps);
  const uint32_t a_lane = smem_u32(Qs) + (uint32_t)(((rg * 16 + (lm & 1) * 8 + lr) * DP + (lm >> 1) * 8) * 2);
  for (int it = 0; it < n_tiles; ++it) {
    cp_async_wait<ST - 2>();
    __syncthreads();   // tile `it` (first time round: Q as well) has landed for everyone; nobody reads the stage that is filled next
    load_tile(it + ST - 1);
    const uint32_t k_stage = ks_addr + (uint32_t)((it % ST) * KT * DP * 2);
    const int j0 = j_start + it * KT;
    float s[2][4] = {};
    if (s_warp) {
      const uint32_t b_lane = k_stage + (uint32_t)(((kg * 16 + (lm >> 1) * 8 + lr) * DP + (lm & 1) * 8) * 2);
      // two sets of accumulators and four k-steps of fragments at a time: the products of a warp must not wait for one another
      float s2[2][4] = {};
      uint32_t a[4][4], bb[4][4];
      int kk = 0;
      for (; kk + 64 <= D; kk += 64) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          ldmatrix_x4(a[u][0], a[u][1], a[u][2], a[u][3], a_lane + (kk + u * 16) * 2);
          ldmatrix_x4(bb[u][0], bb[u][1], bb[u][2], bb[u][3], b_lane + (kk + u * 16) * 2);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          mma_m16n8k16_bf16f32(u & 1 ? s2[0] : s[0], a[u], bb[u][0], bb[u][1]);
          mma_m16n8k16_bf16f32(u & 1 ? s2[1] : s[1], a[u], bb[u][2], bb[u][3]);
        }
      }
      for (; kk < D; kk += 16) {
        ldmatrix_x4(a[0][0], a[0][1], a[0][2], a[0][3], a_lane + kk * 2);
        ldmatrix_x4(bb[0][0], bb[0][1], bb[0][2], bb[0][3], b_lane + kk * 2);
        mma_m16n8k16_bf16f32(s[0], a[0], bb[0][0], bb[0][1]);
        mma_m16n8k16_bf16f32(s[1], a[0], bb[0][2], bb[0][3]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nt][e] += s2[nt][e];
      float mx[2] = {-INFINITY, -INFINITY};
      const bool interior = j0 + KT - 1 <= min(j_end, p_first) && j0 >= lo_last;   // every key is visible to every row
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = e >> 1, j = j0 + kg * 16 + nt * 8 + cq + (e & 1);
          s[nt][e] *= scale_log2;
          if (!interior && (j > p_row[i] || j < lo_row[i] || j > j_end)) s[nt][e] = -INFINITY;
          mx[i] = fmaxf(mx[i], s[nt][e]);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
        if ((lane & 3) == 0) red_max[kg * ROWS + rg * 16 + (lane >> 2) + i * 8] = mx[i];
      }
    }
    __syncthreads();   // the row maxima of the tile are complete
    if (s_warp) {
      float m_use[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int row = rg * 16 + (lane >> 2) + i * 8;
        float m_new = m_run[i];
#pragma unroll
        for (int g = 0; g < KG; ++g) m_new = fmaxf(m_new, red_max[g * ROWS + row]);
        m_use[i] = m_new == -INFINITY ? 0.f : m_new;   // a row that has met no visible key yet
        const float corr = exp2f(m_run[i] - m_use[i]);
        m_run[i] = m_new;
        l_run[i] *= corr;
        if (kg == 0 && (lane & 3) == 0) corr_s[row] = corr;
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(exp2f(s[nt][0] - m_use[0]), exp2f(s[nt][1] - m_use[0]));
        const __nv_bfloat162 hi = __floats2bfloat162_rn(exp2f(s[nt][2] - m_use[1]), exp2f(s[nt][3] - m_use[1]));
        // the sums use the rounded probabilities: numerator and denominator see the same weights
        l_run[0] += __low2float(lo) + __high2float(lo);
        l_run[1] += __low2float(hi) + __high2float(hi);
        const int row = rg * 16 + (lane >> 2), col = kg * 16 + nt * 8 + cq;
        *reinterpret_cast<__nv_bfloat162*>(Ps + row * PP + col) = lo;
        *reinterpret_cast<__nv_bfloat162*>(Ps + (row + 8) * PP + col) = hi;
      }
    }
    __syncthreads();   // P and the corrections are complete
    if (o_warp) {
#pragma unroll
      for (int t = 0; t < PRT; ++t) {
        const float c0 = corr_s[(ro + t) * 16 + (lane >> 2)], c1 = corr_s[(ro + t) * 16 + (lane >> 2) + 8];
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {   // (rows past the last may hold anything: they are never stored)
#pragma unroll
          for (int i = 0; i < NP * 2; ++i) {
            o[t][i][0] *= c0;
            o[t][i][1] *= c0;
            o[t][i][2] *= c1;
            o[t][i][3] *= c1;
          }
        }
      }
      const uint32_t p_lane = ps_addr + (uint32_t)(((ro * 16 + (lm & 1) * 8 + lr) * PP + (lm >> 1) * 8) * 2);
      const uint32_t v_lane = k_stage + (uint32_t)((((lm & 1) * 8 + lr) * DP + pc * 16 + (lm >> 1) * 8) * 2);
#pragma unroll
      for (int ks = 0; ks < KG; ++ks) {
        uint32_t a[PRT][4];
#pragma unroll
        for (int t = 0; t < PRT; ++t) ldmatrix_x4(a[t][0], a[t][1], a[t][2], a[t][3], p_lane + (uint32_t)((t * 16 * PP + ks * 16) * 2));
        constexpr int NF = NP < 4 ? NP : 4;   // pieces whose fragments are fetched together
#pragma unroll
        for (int i0 = 0; i0 < NP; i0 += NF) {
          uint32_t bb[NF][4];
#pragma unroll
          for (int i = 0; i < NF; ++i)
            if (pc + (i0 + i) * PC < pieces)
              ldmatrix_x4_trans(bb[i][0], bb[i][1], bb[i][2], bb[i][3], v_lane + (uint32_t)((ks * 16 * DP + (i0 + i) * PC * 16) * 2));
#pragma unroll
          for (int i = 0; i < NF; ++i)
            if (pc + (i0 + i) * PC < pieces)
#pragma unroll
              for (int t = 0; t < PRT; ++t) {
                mma_m16n8k16_bf16f32(o[t][2 * (i0 + i)], a[t], bb[i][0], bb[i][1]);
                mma_m16n8k16_bf16f32(o[t][2 * (i0 + i) + 1], a[t], bb[i][2], bb[i][3]);
              }
        }
      }
    }
  }
  cp_async_wait<0>();
  if (s_warp) {   // the sums of a row's lanes, then of its key groups
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
      l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
      const int row = rg * 16 + (lane >> 2) + i * 8;
      if ((lane & 3) == 0) {
        red_sum[kg * ROWS + row] = l_run[i];
        if (kg == 0) max_s[row] = m_run[i];
      }
    }
  }
  __syncthreads();
  if (!o_warp) return;
  float* base = gridDim.z > 1 ? partial + (((int64_t)blockIdx.x * gridDim.z + blockIdx.z) * ROWS) * (R + 2) : nullptr;
#pragma unroll
  for (int t = 0; t < PRT; ++t)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = (ro + t) * 16 + (lane >> 2) + i * 8;
      if (row >= n_rows) continue;
      float l = 0.f;
#pragma unroll
      for (int g = 0; g < KG; ++g) l += red_sum[g * ROWS + row];
      if (base) {   // [tile][run][row][R + 2]: unnormalised output, then the running maximum and the sum
        float* dst = base + (int64_t)row * (R + 2);
#pragma unroll
        for (int n = 0; n < NP * 2; ++n)
          if (pc + (n >> 1) * PC < pieces)
            *reinterpret_cast<float2*>(dst + (pc + (n >> 1) * PC) * 16 + (n & 1) * 8 + cq) = make_float2(o[t][n][i * 2], o[t][n][i * 2 + 1]);
        if (pc == 0 && (lane & 3) == 0) {
          dst[R] = max_s[row];
          dst[R + 1] = l;
        }
      } else {
        const float inv = 1.f / l;
#pragma unroll
        for (int n = 0; n < NP * 2; ++n)
          if (pc + (n >> 1) * PC < pieces)
            latent_store<__nv_bfloat16>(out, (row_base + row) * R + (pc + (n >> 1) * PC) * 16 + (n & 1) * 8 + cq, o[t][n][i * 2] * inv,
                                        o[t][n][i * 2 + 1] * inv);
      }
    }
}

// out[row] = sum_z 2^(m_z - M) O_z / sum_z 2^(m_z - M) l_z over the key runs of latent_attn_tile_kernel; a block per row, two columns per
// thread, the runs' loads in flight together (NS >= nsplit: runs past the last read the last again, with no weight)
constexpr int kLatentRuns = 16;

template <int NS>
__global__ void __launch_bounds__(256) latent_attn_merge_kernel(const float* __restrict__ partial, __nv_bfloat16* __restrict__ out,
                                                                const int32_t* __restrict__ cu_q, int B, int H, int R, int rows, int nsplit) {
  pdl_launch_dependents();
  pdl_wait();
  int b, first = 0, n_rows = 0;
  latent_find_tile(cu_q, B, H, rows, blockIdx.x, b, first, n_rows);
  const int row = blockIdx.y;
  if (b >= B || row >= n_rows) return;
  const float* base = partial + ((int64_t)blockIdx.x * nsplit * rows + row) * (R + 2);
  const int64_t zs = (int64_t)rows * (R + 2);
  float wz[NS], lz[NS], M = -INFINITY, den = 0.f;
#pragma unroll
  for (int z = 0; z < NS; ++z) {
    const float2 ml = *reinterpret_cast<const float2*>(base + min(z, nsplit - 1) * zs + R);
    wz[z] = z < nsplit ? ml.x : -INFINITY;
    lz[z] = ml.y;
    M = fmaxf(M, wz[z]);
  }
#pragma unroll
  for (int z = 0; z < NS; ++z) {
    wz[z] = wz[z] > -INFINITY ? exp2f(wz[z] - M) : 0.f;  // an empty run carries no weight
    den = fmaf(wz[z], lz[z], den);
  }
  const float inv = 1.f / den;
  const int64_t dst = ((int64_t)cu_q[b] * H + first + row) * R;
  for (int c = threadIdx.x * 2; c < R; c += blockDim.x * 2) {
    float2 v[NS], acc = make_float2(0.f, 0.f);
#pragma unroll
    for (int z = 0; z < NS; ++z) v[z] = *reinterpret_cast<const float2*>(base + min(z, nsplit - 1) * zs + c);
#pragma unroll
    for (int z = 0; z < NS; ++z) {
      acc.x = fmaf(wz[z], v[z].x, acc.x);
      acc.y = fmaf(wz[z], v[z].y, acc.y);
    }
    latent_store<__nv_bfloat16>(out, dst + c, acc.x * inv, acc.y * inv);
  }
}

}  // namespace seq
}  // namespace b200

using namespace b200::seq;

// down fp32; q, q_abs and cache of type dt
extern "C" int b200_seq_latent_prepare(const float* down, int64_t ld_down, int col_c, int col_kr, const void* q, int64_t ld_q, int q_head_stride,
                                       int q_rot_off, const void* cnorm_w, const float* cos_t, const float* sin_t, const int64_t* position_ids,
                                       const int64_t* slot_mapping, void* cache, int dt, void* q_abs, int64_t T, int H, int R, int r, int rot_dims,
                                       float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (rot_dims % 2 != 0 || rot_dims > r || rot_dims < 0) { b200_set_last_error("seq_latent_prepare: rot_dims must be even and <= r"); return B200_ERR_ARG; }
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((latent_prepare_kernel<E>), dim3((unsigned)T), dim3(kPrepThreads), 0, (cudaStream_t)stream, down, ld_down, col_c,
                                       col_kr, (const E*)q, ld_q, q_head_stride, q_rot_off, (const E*)cnorm_w, cos_t, sin_t, position_ids, slot_mapping,
                                       (E*)cache, (E*)q_abs, H, R, r, rot_dims, eps));
  b200_count_launches(1);
  return B200_OK;
}

template <typename T, int NR>
static int launch_latent_attn(const void* q_abs, const void* cache, const int32_t* block_table, int64_t bt_stride, const int32_t* seq_of_token,
                              const int64_t* position_ids, void* out, int64_t Tq, int H, int R, int D, int window, float scale, int page,
                              const float* sink, cudaStream_t st) {
  const size_t smem = ((size_t)kHeadsPerBlock * D + (size_t)kKeyTile * (D + 1)) * 4;
  if (smem > 200 * 1024) { b200_set_last_error("seq_latent_attn: cache row too wide"); return B200_ERR_ARG; }
  static bool cfg = false;
  if (!cfg) { cudaFuncSetAttribute(latent_attn_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); cfg = true; }
  dim3 grid((unsigned)Tq, (unsigned)((H + kHeadsPerBlock - 1) / kHeadsPerBlock));
  B200_LAUNCH((latent_attn_kernel<T, NR>), grid, dim3(kHeadsPerBlock * 32), smem, st, (const T*)q_abs, (const T*)cache, block_table, bt_stride,
              seq_of_token, position_ids, (T*)out, H, R, D, window, scale, page, sink);
  b200_count_launches(1);
  return B200_OK;
}

// Row groups of 16 (token, head) rows per block of the tensor-core kernel for this step; 0: the shape takes the plain kernel
static int latent_row_groups(int dt, int64_t Tq, int B, int H, int R, int r) {
  static const bool use_mma = []() { const char* e = getenv("B200_SEQ_ATTN_MMA"); return !(e && e[0] == '0'); }();
  const int D = R + r;
  if (!use_mma || dt != B200_DT_BF16 || R % 16 != 0 || r % 16 != 0 || R > 512 || R < 16 || B < 1) return 0;
  const int64_t rows = Tq * H / B;   // per sequence, on average
  const size_t limit = 227 * 1024;
  if (rows > 32 && LatentTile<4>::smem(D) <= limit) return 4;
  if (rows > 16 && LatentTile<2>::smem(D) <= limit) return 2;
  return LatentTile<1>::smem(D) <= limit ? 1 : 0;
}

// Over how many blocks the tensor-core kernel should split each row tile's keys (1 = no split), and the fp32 workspace that takes: few
// rows (decoding) leave most SMs idle otherwise.  0 when the shape takes the plain kernel.
extern "C" int b200_seq_latent_attn_splits(int dt, int64_t Tq, int B, int H, int R, int r, int64_t* workspace_floats) {
  if (workspace_floats) *workspace_floats = 0;
  const int rg = latent_row_groups(dt, Tq, B, H, R, r);
  if (rg == 0) return 0;
  const int64_t rows = rg * 16, tiles = (Tq * H + rows - 1) / rows;
  const int64_t busy = tiles > B ? tiles : B;
  const size_t smem = rg == 4 ? LatentTile<4>::smem(R + r) : rg == 2 ? LatentTile<2>::smem(R + r) : LatentTile<1>::smem(R + r);
  int64_t per_sm = (int64_t)(233472 / (smem + 1024));   // 228 KB per SM, 1 KB reserved per block
  per_sm = per_sm < 1 ? 1 : per_sm > 2 ? 2 : per_sm;
  int64_t n = 148 * per_sm / (busy > 0 ? busy : 1);
  n = n < 1 ? 1 : (n > kLatentRuns ? kLatentRuns : n);
  if (n > 1 && workspace_floats) *workspace_floats = (tiles + B) * n * rows * (R + 2);
  return (int)n;
}

// q_abs [Tq, H, D], cache [blocks, page, D] and out [Tq, H, R] of type dt.  window <= 0: every earlier token is visible.  `partial` / nsplit: from
// b200_seq_latent_attn_splits (NULL / <= 1: no split).  sink fp32 [H] or NULL: a logit per head that joins the soft-max denominator
// (unscaled) and carries no value.
extern "C" int b200_seq_latent_attn(const void* q_abs, const void* cache, int dt, const int32_t* block_table, int64_t bt_stride,
                                    const int32_t* seq_of_token, const int32_t* cu_q, int B, const int64_t* position_ids, void* out, int64_t Tq, int H,
                                    int R, int r, int window, float scale, int page, float* partial, int nsplit, const float* sink, void* stream) {
  if (Tq == 0) return B200_OK;
  const int D = R + r;
  if (window <= 0) window = 0x3fffffff;
  const int nr = (R + 31) / 32;
  cudaStream_t st = (cudaStream_t)stream;
  const int rg = latent_row_groups(dt, Tq, B, H, R, r);
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(q_abs) | reinterpret_cast<uintptr_t>(out);
  if (rg > 0 && (ptrs & 15) == 0) {
    const int64_t rows = rg * 16, tiles = (Tq * H + rows - 1) / rows + B;   // upper bound of sum_b ceil(n_b H / rows); surplus blocks return at once
    if (!partial || nsplit < 1) nsplit = 1;
    if (nsplit > kLatentRuns) nsplit = kLatentRuns;
    if (tiles > 0x7fffffff) { b200_set_last_error("seq_latent_attn: too many rows"); return B200_ERR_ARG; }
    const dim3 grid((unsigned)tiles, 1, (unsigned)nsplit);
    const float scale_log2 = scale * 1.4426950408889634f;
#define LAT(RG_, NP_)                                                                                                                             \
  do {                                                                                                                                            \
    static bool cfg = false;                                                                                                                      \
    if (!cfg) { cudaFuncSetAttribute(latent_attn_tile_kernel<RG_, NP_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024); cfg = true; }   \
    B200_LAUNCH((latent_attn_tile_kernel<RG_, NP_>), grid, dim3(kTileThreads), LatentTile<RG_>::smem(D), st, (const __nv_bfloat16*)q_abs,         \
                (const __nv_bfloat16*)cache, block_table, bt_stride, cu_q, B, position_ids, (__nv_bfloat16*)out, H, R, D, window, scale_log2, page, \
                partial, sink);                                                                                                                   \
  } while (0)
    const int pieces = R / 16;
    if (rg == 4) {
      if (pieces <= 4) LAT(4, 1);
      else if (pieces <= 8) LAT(4, 2);
      else if (pieces <= 16) LAT(4, 4);
      else LAT(4, 8);
    } else if (rg == 2) {
      if (pieces <= 8) LAT(2, 1);
      else if (pieces <= 16) LAT(2, 2);
      else LAT(2, 4);
    } else {
      if (pieces <= 8) LAT(1, 1);
      else if (pieces <= 16) LAT(1, 2);
      else LAT(1, 4);
    }
#undef LAT
#define MERGE(NS)                                                                                                                        \
  B200_LAUNCH(latent_attn_merge_kernel<NS>, dim3((unsigned)tiles, (unsigned)rows), dim3(R > 256 ? 256 : R > 128 ? 128 : 64), 0, st,       \
              (const float*)partial, (__nv_bfloat16*)out, cu_q, B, H, R, (int)rows, nsplit)
    if (nsplit > 8) MERGE(16);
    else if (nsplit > 4) MERGE(8);
    else if (nsplit > 2) MERGE(4);
    else if (nsplit > 1) MERGE(2);
#undef MERGE
    b200_count_launches(nsplit > 1 ? 2 : 1);
    return B200_OK;
  }
#define LA(NR)                                                                                                                         \
  B200_SEQ_DISPATCH(dt, E, return (launch_latent_attn<E, NR>(q_abs, cache, block_table, bt_stride, seq_of_token, position_ids, out, Tq, H, R, D, \
                                                            window, scale, page, sink, st)))
  if (nr <= 4) LA(4);
  else if (nr <= 8) LA(8);
  else if (nr <= 16) LA(16);
  else if (nr <= 32) LA(32);
#undef LA
  b200_set_last_error("seq_latent_attn: latent wider than 1024");
  return B200_ERR_UNSUPPORTED;
}
