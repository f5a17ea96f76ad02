// Gated delta rule over fp32 state slots: per head a [dk, dv] memory S; every token
//   S <- g_t S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   y_t = S^T q_t          (the read-out sees the token's own write)
// q_t, k_t unit vectors (x / sqrt(sum x^2 + 1e-6)), q_t times q_scale, shared by the heads of a group; beta_t = sigmoid(raw);
// g_t = exp(-exp(A_log) softplus(raw + dt_bias)), one number per head, or one per head and key channel (row n of S decays at rate n).
//
//   delta_prepare_kernel : everything of a token that does not depend on S, once per token: short depth-wise causal convolution + SiLU
//                          of the q / k / v columns (earlier inputs from the sequence's convolution state), unit vectors, decays,
//                          write strengths -> one row [q | k | v | g | beta] per token.  When every sequence brings one token it also
//                          advances the convolution state (otherwise delta_conv_state_kernel does, after it).
//   delta_chunk_kernel   : prompts and portions.  A block owns (sequence, head, up to 64 value columns) and takes four tokens at a
//                          time: their predictions and read-outs against the OLD memory are one pass over the state registers, the
//                          dependence among the four goes through 4 x 4 matrices of decayed inner products, and the memory is
//                          rewritten once.  With G_j = g_1 .. g_j and D_i = g_(i+1) .. g_4 (products per key channel, no division):
//                            P_j = (G_j k_j)^T S,  A_ji = k_j^T (g_(i+1) .. g_j) k_i,  u_j = beta_j (v_j - P_j - sum_(i<j) A_ji u_i)
//                            y_j = (G_j q_j)^T S + sum_(i<=j) B_ji u_i  (B as A with q_j),   S <- G_4 S + sum_i (D_i k_i) u_i^T
//                          Tokens that the last four lack are k = q = 0, g = 1, beta = 0: they change nothing.
//   delta_step_kernel    : steps of few rows per sequence (decoding): bound by reading and writing the state, which goes straight
//                          between global memory and registers in whole rows; tokens in order, one at a time.
//
// A sequence whose first token of the step is at position 0 starts from a zero state and never reads its (possibly reused) slot.
// All arithmetic is fp32; the two scan forms (and delta_scan_kernel of seq_recurrent.cu, which keeps one order of operations for any cut of
// a sequence and knows decays per head only) differ by rounding.
#include "seq_common.cuh"

namespace b200 {
namespace seq {

constexpr int kDeltaMaxTaps = 8, kPrepThreads = 256, kPrepSpan = 128, kPrepParts = 2;  // channels per warp task; blocks per token of a long step

// columns of a prepared row
struct DeltaRow {
  int k, v, g, b, width;  // q starts at 0
};
__host__ __device__ inline DeltaRow delta_row(int H, int G, int dk, int dv, bool channels) {
  DeltaRow r;
  r.k = G * dk;
  r.v = 2 * G * dk;
  r.g = r.v + H * dv;
  r.b = r.g + (channels ? H * dk : H);
  r.width = (r.b + H + 3) & ~3;
  return r;
}

// Where the inputs of one token's convolution lie: a row of this step, an entry of the sequence's state, or nowhere (before position 0).
// The rows serve every channel, so they are found once per token.
template <int TAPS>
struct ConvInputs {
  const float* src[TAPS];
};

// SiLU of channel c's convolution (w [taps, C]); a token alone in its step (`shift`) moves the state st [taps - 1, C] on by one input
template <typename TP, int TAPS>
__device__ __forceinline__ float conv_silu_at(const ConvInputs<TAPS>& in, const TP* __restrict__ w, float* st, int C, int taps, int c, bool shift) {
  float val[TAPS], acc = 0.f;
#pragma unroll
  for (int j = 0; j < TAPS; ++j) val[j] = (j < taps && in.src[j]) ? in.src[j][c] : 0.f;
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    if (j < taps) acc = fmaf(ldf(w + j * C + c), val[j], acc);
  if (shift) {
#pragma unroll
    for (int j = 1; j < TAPS; ++j)
      if (j < taps) st[(j - 1) * C + c] = val[j];
  }
  return silu_f(acc);
}

template <typename TP, int TAPS>  // taps <= TAPS
__global__ void __launch_bounds__(kPrepThreads, TAPS <= 4 ? 4 : 2) delta_prepare_kernel(
    const float* u, int64_t ld, int col0, int taps, const TP* __restrict__ w, float* conv_state, int shift, const int32_t* __restrict__ state_slots,
    const int32_t* __restrict__ seq_of_token, const int32_t* __restrict__ cu_q, const int64_t* __restrict__ position_ids, const float* __restrict__ raw,
    int64_t ldr, int col_b, const float* __restrict__ dec, int64_t ldd, int col_a, int channels, const TP* __restrict__ A_log,
    const TP* __restrict__ dt_bias, float q_scale, float* __restrict__ out, int H, int G, int dk, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int lane = lane_id();
  const int b = seq_of_token[t], row0 = cu_q[b];
  const int64_t s = position_ids[row0], p = position_ids[t];
  const int C = 2 * G * dk + H * dv;
  float* st = conv_state + (int64_t)state_slots[b] * (taps > 1 ? taps - 1 : 1) * C;
  ConvInputs<TAPS> in;
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const int64_t pp = p - (taps - 1) + j;
    in.src[j] = pp >= s ? u + (row0 + (pp - s)) * ld + col0 : (pp >= 0 ? st + (pp - s + taps - 1) * C : nullptr);
  }
  const DeltaRow lay = delta_row(H, G, dk, dv, channels != 0);
  float* row = out + t * lay.width;
  const int n_vec = 2 * G, n_v = (H * dv + kPrepSpan - 1) / kPrepSpan, n_dec = channels ? H * dk : H, n_g = (n_dec + kPrepSpan - 1) / kPrepSpan;
  const int tasks = n_vec + n_v + n_g + (H + kPrepSpan - 1) / kPrepSpan;
  for (int task = blockIdx.y * (kPrepThreads / 32) + warp_id(); task < tasks; task += gridDim.y * (kPrepThreads / 32)) {
    if (task < n_vec) {                      // a head's q or k: convolution, SiLU, unit length
      float x[8], sum = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int n = lane + 32 * i;
        x[i] = n < dk ? conv_silu_at<TP, TAPS>(in, w, st, C, taps, task * dk + n, shift != 0) : 0.f;
        sum = fmaf(x[i], x[i], sum);
      }
      const float r = (task < G ? q_scale : 1.f) / sqrtf(warp_sum(sum) + 1e-6f);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int n = lane + 32 * i;
        if (n < dk) row[task * dk + n] = x[i] * r;
      }
    } else if (task < n_vec + n_v) {
      const int first = (task - n_vec) * kPrepSpan + lane;
#pragma unroll
      for (int i = 0; i < kPrepSpan / 32; ++i) {
        const int c = first + 32 * i;
        if (c < H * dv) row[lay.v + c] = conv_silu_at<TP, TAPS>(in, w, st, C, taps, 2 * G * dk + c, shift != 0);
      }
    } else if (task < n_vec + n_v + n_g) {
      const int first = (task - n_vec - n_v) * kPrepSpan + lane;
      float z[kPrepSpan / 32];
#pragma unroll
      for (int i = 0; i < kPrepSpan / 32; ++i) {
        const int c = first + 32 * i;
        z[i] = c < n_dec ? dec[t * ldd + col_a + c] + ldf(dt_bias + c) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < kPrepSpan / 32; ++i) {
        const int c = first + 32 * i;
        if (c < n_dec) row[lay.g + c] = expf(-expf(ldf(A_log + (channels ? c / dk : c))) * softplus_f(z[i]));
      }
    } else {
      const int first = (task - n_vec - n_v - n_g) * kPrepSpan, c1 = min(H, first + kPrepSpan);
      for (int h = first + lane; h < c1; h += 32) row[lay.b + h] = sigmoid_f(raw[t * ldr + col_b + h]);
    }
  }
}

// the state becomes the last taps - 1 inputs of the sequence (older entries shift when the step brought fewer tokens than that)
__global__ void delta_conv_state_kernel(const float* __restrict__ u, int64_t ld_u, int col0, int C, int taps, float* __restrict__ conv_state,
                                        const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q,
                                        const int64_t* __restrict__ position_ids) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int row0 = cu_q[b], nq = cu_q[b + 1] - row0;
  if (nq <= 0) return;
  const int64_t s = position_ids[row0], e = s + nq;
  float* st = conv_state + (int64_t)state_slots[b] * (taps - 1) * C;
  for (int k = 0; k < taps - 1; ++k) {   // ascending: entry k is rewritten from an entry at or behind it
    const int64_t pp = e - (taps - 1) + k;
    float val = 0.f;
    if (pp >= s) val = u[(row0 + (pp - s)) * ld_u + col0 + c];
    else if (pp >= 0) val = st[(pp - s + taps - 1) * C + c];
    st[(int64_t)k * C + c] = val;
  }
}

__device__ __forceinline__ void cp_async_4(void* smem_dst, const void* gmem_src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(smem_dst)), "l"(gmem_src) : "memory");
}

constexpr int kTileTok = 16, kQuad = 4, kQuads = kTileTok / kQuad, kRowLanes = 16, kColsPerWarp = 8, kABPitch = 24;

// shared memory of delta_chunk_kernel in floats
__host__ __device__ inline int delta_raw_row(int dk, int NC, bool channels) { return (channels ? 3 : 2) * ((dk + 3) & ~3) + NC + 8; }
__host__ __device__ inline int delta_chunk_floats(int NR, int dk, int NC, bool channels) {
  return kQuads * NR * kRowLanes * 13 + kQuads * 2 * kABPitch + 2 * kTileTok * delta_raw_row(dk, NC, channels);
}

// values v[0 .. 2^k) summed over the lanes of a group of 2^k' lanes, each lane left with its share: one halving per lane bit
template <int N>
__device__ __forceinline__ void halve(float* v, int off, bool upper) {
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    const float send = upper ? v[i] : v[i + N / 2], keep = upper ? v[i + N / 2] : v[i];
    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
  }
}

// the same where every lane has put the values it keeps first
template <int N>
__device__ __forceinline__ void fold(float* v, int off) {
#pragma unroll
  for (int i = 0; i < N / 2; ++i) v[i] += __shfl_xor_sync(0xffffffffu, v[i + N / 2], off);
}

// o[x] = f[x ^ (lo + 2 hi)]; its own inverse
__device__ __forceinline__ void permute4(float4 f, bool lo, bool hi, float* o) {
  const float a = lo ? f.y : f.x, b = lo ? f.x : f.y, c = lo ? f.w : f.z, d = lo ? f.z : f.w;
  o[0] = hi ? c : a;
  o[1] = hi ? d : b;
  o[2] = hi ? a : c;
  o[3] = hi ? b : d;
}

template <int NR>  // state rows per lane: dk <= 16 NR
__global__ void __launch_bounds__(256, NR <= 8 ? 2 : 1) delta_chunk_kernel(
    const float* __restrict__ pre, float* __restrict__ S_state, const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q,
    const int64_t* __restrict__ position_ids, float* __restrict__ y, int64_t ld_y, int H, int G, int dk, int dv, int channels, int NC, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  constexpr int dkp = NR * kRowLanes;
  float4* KG = reinterpret_cast<float4*>(sm);       // [quad][dkp]: G_j k_j, j = 0 .. 3
  float4* QG = KG + kQuads * dkp;                   // G_j q_j
  float4* KD = QG + kQuads * dkp;                   // D_i k_i
  float* GA = reinterpret_cast<float*>(KD + kQuads * dkp);   // G_4
  float* AB = GA + kQuads * dkp;                    // [quad][half of the rows][A: 10 20 21 30 31 32 0 0 | B: 4 x 4, zero above the diagonal]
  float* raw = AB + kQuads * 2 * kABPitch;          // two tiles of [16 tokens][q | k | (g) | v | beta, g]
  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * NC, grp = h / (H / G);
  const int nthreads = blockDim.x, nw = nthreads >> 5, w = warp_id(), lane = lane_id();
  const int t_begin = cu_q[b], t_end = cu_q[b + 1];
  if (t_begin >= t_end) return;
  const bool fresh = position_ids[t_begin] == 0;
  const DeltaRow lay = delta_row(H, G, dk, dv, channels != 0);
  const int dk4 = (dk + 3) & ~3, rr = delta_raw_row(dk, NC, channels != 0);
  const int o_k = dk4, o_g = 2 * dk4, o_v = (channels ? 3 : 2) * dk4, o_b = o_v + NC;   // beta at o_b, a head's single decay at o_b + 4
  const int live_cols = min(NC, dv - v0);
  for (int i = threadIdx.x; i < kQuads * 2 * kABPitch; i += nthreads) AB[i] = 0.f;
  for (int i = threadIdx.x; i < 2 * kTileTok * NC; i += nthreads)   // value columns that the head lacks
    if (i % NC >= live_cols) raw[(i / NC) * rr + o_v + i % NC] = 0.f;

  auto load_tile = [&](int t0, int buf) {
    for (int tt = w; tt < kTileTok; tt += nw) {
      float* dst = raw + (buf * kTileTok + tt) * rr;
      if (t0 + tt < t_end) {
        const float* src = pre + (int64_t)(t0 + tt) * lay.width;
        if (vec) {
          for (int c = lane * 4; c < dk; c += 128) {
            cp_async_16(dst + c, src + grp * dk + c, true);
            cp_async_16(dst + o_k + c, src + lay.k + grp * dk + c, true);
            if (channels) cp_async_16(dst + o_g + c, src + lay.g + h * dk + c, true);
          }
          for (int c = lane * 4; c < live_cols; c += 128) cp_async_16(dst + o_v + c, src + lay.v + h * dv + v0 + c, true);
        } else {
          for (int c = lane; c < dk; c += 32) {
            cp_async_4(dst + c, src + grp * dk + c);
            cp_async_4(dst + o_k + c, src + lay.k + grp * dk + c);
            if (channels) cp_async_4(dst + o_g + c, src + lay.g + h * dk + c);
          }
          for (int c = lane; c < live_cols; c += 32) cp_async_4(dst + o_v + c, src + lay.v + h * dv + v0 + c);
        }
        if (lane == 0) {
          cp_async_4(dst + o_b, src + lay.b + h);
          if (!channels) cp_async_4(dst + o_b + 4, src + lay.g + h);
        }
      } else {   // a token that the step does not have changes nothing
        for (int c = lane; c < dk; c += 32) {
          dst[c] = dst[o_k + c] = 0.f;
          if (channels) dst[o_g + c] = 1.f;
        }
        for (int c = lane; c < NC; c += 32) dst[o_v + c] = 0.f;
        if (lane == 0) {
          dst[o_b] = 0.f;
          dst[o_b + 4] = 1.f;
        }
      }
    }
    cp_async_commit();
  };

  // this thread's part of the memory: rows rl + 16 i, columns c0 .. c0 + 3 of the block's.  Entry x of S[i] is column c0 + (x ^ perm): with
  // a lane's own column order a reduction over lanes always keeps the lower half of what it has and sends the upper half
  const int rl = lane & 15, c0 = w * kColsPerWarp + (lane >> 4) * 4;
  const bool b3 = lane & 8, b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const int perm = (lane >> 2) & 3, my_c = c0 + perm;    // my_c: the column whose reductions this lane ends up with
  float* Sp = S_state + ((int64_t)state_slots[b] * H + h) * dk * dv + v0;
  load_tile(t_begin, 0);
  float S[NR][4];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int n = rl + kRowLanes * i;
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (!fresh && n < dk) {
      if (vec) {
        if (c0 < live_cols) {
          const float4 f = *reinterpret_cast<const float4*>(Sp + (int64_t)n * dv + c0);
          permute4(f, b2, b3, S[i]);
        }
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (c0 + (x ^ perm) < live_cols) S[i][x] = Sp[(int64_t)n * dv + c0 + (x ^ perm)];
      }
    }
  }
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += kTileTok, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();   // this tile's rows are visible, the previous tile is used up
    if (t0 + kTileTok < t_end) load_tile(t0 + kTileTok, buf ^ 1);
    const float* tile = raw + buf * kTileTok * rr;
    const int quads = min(kQuads, (t_end - t0 + kQuad - 1) / kQuad);
    for (int item = w; item < 2 * quads; item += nw) {     // (four tokens, half of the key channels)
      const int qd = item >> 1, half = item & 1;
      const float* tr = tile + qd * kQuad * rr;
      float ab[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) ab[i] = 0.f;
      for (int n = half * (dkp / 2) + lane; n < (half + 1) * (dkp / 2); n += 32) {
        float k[4], q[4], g[4];
        const bool live = n < dk;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          k[j] = live ? tr[j * rr + o_k + n] : 0.f;
          q[j] = live ? tr[j * rr + n] : 0.f;
          g[j] = live ? (channels ? tr[j * rr + o_g + n] : tr[j * rr + o_b + 4]) : 1.f;
        }
        const float G1 = g[0] * g[1], G2 = G1 * g[2], G3 = G2 * g[3];
        const float g12 = g[1] * g[2], g23 = g[2] * g[3], g123 = g[1] * g23;
        KG[qd * dkp + n] = make_float4(k[0] * g[0], k[1] * G1, k[2] * G2, k[3] * G3);
        QG[qd * dkp + n] = make_float4(q[0] * g[0], q[1] * G1, q[2] * G2, q[3] * G3);
        KD[qd * dkp + n] = make_float4(k[0] * g123, k[1] * g23, k[2] * g[3], k[3]);
        GA[qd * dkp + n] = G3;
        const float k01 = k[0] * g[1], k02 = k[0] * g12, k03 = k[0] * g123, k12 = k[1] * g[2], k13 = k[1] * g23, k23 = k[2] * g[3];
        ab[0] = fmaf(k[1], k01, ab[0]);
        ab[1] = fmaf(k[2], k02, ab[1]);
        ab[2] = fmaf(k[2], k12, ab[2]);
        ab[3] = fmaf(k[3], k03, ab[3]);
        ab[4] = fmaf(k[3], k13, ab[4]);
        ab[5] = fmaf(k[3], k23, ab[5]);
        ab[6] = fmaf(q[0], k[0], ab[6]);
        ab[7] = fmaf(q[1], k01, ab[7]);
        ab[8] = fmaf(q[1], k[1], ab[8]);
        ab[9] = fmaf(q[2], k02, ab[9]);
        ab[10] = fmaf(q[2], k12, ab[10]);
        ab[11] = fmaf(q[2], k[2], ab[11]);
        ab[12] = fmaf(q[3], k03, ab[12]);
        ab[13] = fmaf(q[3], k13, ab[13]);
        ab[14] = fmaf(q[3], k23, ab[14]);
        ab[15] = fmaf(q[3], k[3], ab[15]);
      }
      halve<16>(ab, 16, lane & 16);
      halve<8>(ab, 8, b3);
      halve<4>(ab, 4, b2);
      halve<2>(ab, 2, b1);
      ab[0] += __shfl_xor_sync(0xffffffffu, ab[0], 1);
      if (!b0) {
        const int idx = lane >> 1, e = idx - 6, j = e < 1 ? 0 : (e < 3 ? 1 : (e < 6 ? 2 : 3));   // e: the lower triangle row by row
        AB[(qd * 2 + half) * kABPitch + (idx < 6 ? idx : 8 + j * 4 + e - j * (j + 1) / 2)] = ab[0];
      }
    }
    __syncthreads();
    for (int qd = 0; qd < quads; ++qd) {
      float P[16], O[16];   // [column][token]
#pragma unroll
      for (int i = 0; i < 16; ++i) P[i] = O[i] = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const float4 kg = KG[qd * dkp + rl + kRowLanes * i], qg = QG[qd * dkp + rl + kRowLanes * i];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float s = S[i][c];
          P[c * 4 + 0] = fmaf(kg.x, s, P[c * 4 + 0]);
          P[c * 4 + 1] = fmaf(kg.y, s, P[c * 4 + 1]);
          P[c * 4 + 2] = fmaf(kg.z, s, P[c * 4 + 2]);
          P[c * 4 + 3] = fmaf(kg.w, s, P[c * 4 + 3]);
          O[c * 4 + 0] = fmaf(qg.x, s, O[c * 4 + 0]);
          O[c * 4 + 1] = fmaf(qg.y, s, O[c * 4 + 1]);
          O[c * 4 + 2] = fmaf(qg.z, s, O[c * 4 + 2]);
          O[c * 4 + 3] = fmaf(qg.w, s, O[c * 4 + 3]);
        }
      }
      // predictions: every group of four lanes ends with the four tokens of one column
      fold<16>(P, 8);
      fold<8>(P, 4);
#pragma unroll
      for (int j = 0; j < 4; ++j) P[j] += __shfl_xor_sync(0xffffffffu, P[j], 2);
#pragma unroll
      for (int j = 0; j < 4; ++j) P[j] += __shfl_xor_sync(0xffffffffu, P[j], 1);
      const float* tr = tile + qd * kQuad * rr;
      const float4* ab0 = reinterpret_cast<const float4*>(AB + qd * 2 * kABPitch);
      const float4* ab1 = ab0 + kABPitch / 4;
      float4 a0 = ab0[0], a1 = ab0[1];
      {
        const float4 x0 = ab1[0], x1 = ab1[1];
        a0.x += x0.x; a0.y += x0.y; a0.z += x0.z; a0.w += x0.w;
        a1.x += x1.x; a1.y += x1.y;
      }
      float um[4];
      um[0] = tr[o_b] * (tr[o_v + my_c] - P[0]);
      um[1] = tr[rr + o_b] * (tr[rr + o_v + my_c] - P[1] - a0.x * um[0]);
      um[2] = tr[2 * rr + o_b] * (tr[2 * rr + o_v + my_c] - P[2] - a0.y * um[0] - a0.z * um[1]);
      um[3] = tr[3 * rr + o_b] * (tr[3 * rr + o_v + my_c] - P[3] - a0.w * um[0] - a1.x * um[1] - a1.y * um[2]);
      float U[4][4];   // [token][column]
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        U[j][0] = um[j];
        U[j][1] = __shfl_xor_sync(0xffffffffu, um[j], 4);
        U[j][2] = __shfl_xor_sync(0xffffffffu, U[j][0], 8);
        U[j][3] = __shfl_xor_sync(0xffffffffu, U[j][1], 8);
      }
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const float4 kd = KD[qd * dkp + rl + kRowLanes * i];
        const float ga = GA[qd * dkp + rl + kRowLanes * i];
#pragma unroll
        for (int c = 0; c < 4; ++c)
          S[i][c] = fmaf(kd.w, U[3][c], fmaf(kd.z, U[2][c], fmaf(kd.y, U[1][c], fmaf(kd.x, U[0][c], ga * S[i][c]))));
      }
      // read-outs: every lane ends with one (token, column)
      fold<16>(O, 8);
      fold<8>(O, 4);
      halve<4>(O, 2, b1);
      halve<2>(O, 1, b0);
      const int j = lane & 3, t = t0 + qd * kQuad + j;
      const float4 bj = ab0[2 + j], bx = ab1[2 + j];
      const float o = O[0] + (bj.x + bx.x) * um[0] + (bj.y + bx.y) * um[1] + (bj.z + bx.z) * um[2] + (bj.w + bx.w) * um[3];
      if (t < t_end && my_c < live_cols) y[(int64_t)t * ld_y + h * dv + v0 + my_c] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int n = rl + kRowLanes * i;
    if (n < dk) {
      if (vec) {
        float o[4];
        permute4(make_float4(S[i][0], S[i][1], S[i][2], S[i][3]), b2, b3, o);
        if (c0 < live_cols) *reinterpret_cast<float4*>(Sp + (int64_t)n * dv + c0) = make_float4(o[0], o[1], o[2], o[3]);
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (c0 + (x ^ perm) < live_cols) Sp[(int64_t)n * dv + c0 + (x ^ perm)] = S[i][x];
      }
    }
  }
}

constexpr int kStepThreads = 256, kStepWarps = kStepThreads / 32;

// CL lanes side by side hold VEC columns each, the 256 / CL groups of them take every so many-th state row: NR rows per thread
template <int NR, int VEC>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(
    const float* __restrict__ pre, float* __restrict__ S_state, const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q,
    const int64_t* __restrict__ position_ids, float* __restrict__ y, int64_t ld_y, int H, int G, int dk, int dv, int channels, int CL) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float qs[256], ks[256], gs[256];
  __shared__ float red_p[kStepWarps][32 * VEC], red_o[kStepWarps][32 * VEC];
  const int b = blockIdx.x, h = blockIdx.y, grp = h / (H / G);
  const int t_begin = cu_q[b], t_end = cu_q[b + 1];
  if (t_begin >= t_end) return;
  const bool fresh = position_ids[t_begin] == 0;
  const int cl = threadIdx.x & (CL - 1), rg = threadIdx.x / CL, RG = kStepThreads / CL, cols = CL * VEC;
  const int w = warp_id(), lane = lane_id();
  const int col = blockIdx.z * cols + cl * VEC;      // VEC 4: dv is a multiple of 4, a lane's columns all exist or none does
  const DeltaRow lay = delta_row(H, G, dk, dv, channels != 0);
  float* Sp = S_state + ((int64_t)state_slots[b] * H + h) * dk * dv + col;
  float S[NR][VEC];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int n = rg + RG * i;
#pragma unroll
    for (int c = 0; c < VEC; ++c) S[i][c] = 0.f;
    if (!fresh && n < dk && col < dv) {
      if constexpr (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4*>(Sp + (int64_t)n * dv);
        S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
      } else {
        S[i][0] = Sp[(int64_t)n * dv];
      }
    }
  }
  for (int t = t_begin; t < t_end; ++t) {
    const float* row = pre + (int64_t)t * lay.width;
    if (t > t_begin) __syncthreads();   // the previous token's vectors and sums are used up
    for (int n = threadIdx.x; n < dk; n += kStepThreads) {
      qs[n] = row[grp * dk + n];
      ks[n] = row[lay.k + grp * dk + n];
      gs[n] = row[lay.g + (channels ? h * dk + n : h)];
    }
    const float beta = row[lay.b + h];
    float v[VEC], part[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      v[c] = col < dv ? row[lay.v + h * dv + col + c] : 0.f;
      part[c] = 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int n = rg + RG * i;
      if (n < dk) {
        const float g = gs[n], k = ks[n];
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
          S[i][c] *= g;
          part[c] = fmaf(S[i][c], k, part[c]);
        }
      }
    }
    for (int off = CL; off < 32; off <<= 1)
#pragma unroll
      for (int c = 0; c < VEC; ++c) part[c] += __shfl_xor_sync(0xffffffffu, part[c], off);
    if (lane < CL)
#pragma unroll
      for (int c = 0; c < VEC; ++c) red_p[w][cl * VEC + c] = part[c];
    __syncthreads();
    float uu[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      float pred = 0.f;
#pragma unroll
      for (int k = 0; k < kStepWarps; ++k) pred += red_p[k][cl * VEC + c];
      uu[c] = beta * (v[c] - pred);
      part[c] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int n = rg + RG * i;
      if (n < dk) {
        const float k = ks[n], q = qs[n];
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
          S[i][c] = fmaf(k, uu[c], S[i][c]);
          part[c] = fmaf(S[i][c], q, part[c]);
        }
      }
    }
    for (int off = CL; off < 32; off <<= 1)
#pragma unroll
      for (int c = 0; c < VEC; ++c) part[c] += __shfl_xor_sync(0xffffffffu, part[c], off);
    if (lane < CL)
#pragma unroll
      for (int c = 0; c < VEC; ++c) red_o[w][cl * VEC + c] = part[c];
    __syncthreads();
    const int oc = blockIdx.z * cols + threadIdx.x;
    if (threadIdx.x < cols && oc < dv) {
      float o = 0.f;
#pragma unroll
      for (int k = 0; k < kStepWarps; ++k) o += red_o[k][threadIdx.x];
      y[(int64_t)t * ld_y + h * dv + oc] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int n = rg + RG * i;
    if (n < dk && col < dv) {
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(Sp + (int64_t)n * dv) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      else Sp[(int64_t)n * dv] = S[i][0];
    }
  }
}

}  // namespace seq
}  // namespace b200

using namespace b200::seq;

// floats per prepared row
extern "C" int b200_seq_delta_row_width(int H, int kv_heads, int dk, int dv, int channels) { return delta_row(H, kv_heads, dk, dv, channels != 0).width; }

// u fp32 [T, ld]: projected q / k (kv_heads x dk each) and v (H x dv) columns from col0; w [taps, 2 kv_heads dk + H dv] their convolution;
// conv_state fp32 [slots, max(taps - 1, 1), channels of u] advanced in place; raw fp32: write-strength logits, one per head, at col_b; dec
// fp32: decay logits from col_a, one per head or (channels != 0) dk per head; A_log [H], dt_bias ([H] or [H * dk]), w of element type dt
// -> out fp32 [T, b200_seq_delta_row_width]
extern "C" int b200_seq_delta_prepare(const float* u, int64_t ld, int col0, int taps, const void* w, float* conv_state, const int32_t* state_slots,
                                      const int32_t* seq_of_token, const int32_t* cu_q, const int64_t* position_ids, const float* raw, int64_t ldr,
                                      int col_b, const float* dec, int64_t ldd, int col_a, int channels, const void* A_log, const void* dt_bias, int dt,
                                      float q_scale, float* out, int64_t T, int B, int H, int kv_heads, int dk, int dv, void* stream) {
  if (T == 0) return B200_OK;
  if (kv_heads <= 0 || H % kv_heads != 0 || dk <= 0 || dk > 256 || dv <= 0 || taps < 1 || taps > kDeltaMaxTaps) {
    b200_set_last_error("seq_delta_prepare: need heads % kv_heads == 0, 0 < key size <= 256 and 1 <= taps <= 8");
    return B200_ERR_ARG;
  }
  cudaStream_t st = (cudaStream_t)stream;
  const int shift = (T == B && taps > 1) ? 1 : 0, C = 2 * kv_heads * dk + H * dv;
  const int tasks = 2 * kv_heads + (H * dv + kPrepSpan - 1) / kPrepSpan + ((channels ? H * dk : H) + kPrepSpan - 1) / kPrepSpan +
                    (H + kPrepSpan - 1) / kPrepSpan;
  int parts = (tasks + kPrepThreads / 32 - 1) / (kPrepThreads / 32);   // few rows: a warp per task; many: blocks that loop
  if (T > 1024 && parts > kPrepParts) parts = kPrepParts;
#define DPR(N)                                                                                                                                      \
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((delta_prepare_kernel<E, N>), dim3((unsigned)T, (unsigned)parts), dim3(kPrepThreads), 0, st, u, ld, col0, taps, \
                                       (const E*)w, conv_state, shift, state_slots, seq_of_token, cu_q, position_ids, raw, ldr, col_b, dec, ldd, col_a, \
                                       channels, (const E*)A_log, (const E*)dt_bias, q_scale, out, H, kv_heads, dk, dv))
  if (taps <= 2) DPR(2);
  else if (taps <= 4) DPR(4);
  else DPR(8);
#undef DPR
  if (!shift && taps > 1)
    B200_LAUNCH(delta_conv_state_kernel, dim3((unsigned)B, (unsigned)((C + 255) / 256)), dim3(256), 0, st, u, ld, col0, C, taps, conv_state, state_slots,
                cu_q, position_ids);
  b200_count_launches(!shift && taps > 1 ? 2 : 1);
  return B200_OK;
}

template <int NR>
static int launch_delta_chunk(const float* pre, float* S_state, const int32_t* state_slots, const int32_t* cu_q, const int64_t* position_ids, float* y,
                              int64_t ld_y, int B, int H, int G, int dk, int dv, int channels, int NC, int vec, cudaStream_t st) {
  const size_t smem = (size_t)delta_chunk_floats(NR, dk, NC, channels != 0) * 4;
  static bool cfg = false;
  if (!cfg) { cudaFuncSetAttribute(delta_chunk_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); cfg = true; }
  dim3 grid((unsigned)B, (unsigned)H, (unsigned)((dv + NC - 1) / NC));
  B200_LAUNCH((delta_chunk_kernel<NR>), grid, dim3((unsigned)(NC / kColsPerWarp * 32)), smem, st, pre, S_state, state_slots, cu_q, position_ids, y, ld_y,
              H, G, dk, dv, channels, NC, vec);
  b200_count_launches(1);
  return B200_OK;
}

template <int NR, int VEC>
static int launch_delta_step(const float* pre, float* S_state, const int32_t* state_slots, const int32_t* cu_q, const int64_t* position_ids, float* y,
                             int64_t ld_y, int B, int H, int G, int dk, int dv, int channels, int CL, cudaStream_t st) {
  dim3 grid((unsigned)B, (unsigned)H, (unsigned)((dv + CL * VEC - 1) / (CL * VEC)));
  B200_LAUNCH((delta_step_kernel<NR, VEC>), grid, dim3(kStepThreads), 0, st, pre, S_state, state_slots, cu_q, position_ids, y, ld_y, H, G, dk, dv,
              channels, CL);
  b200_count_launches(1);
  return B200_OK;
}

// pre fp32 [T, b200_seq_delta_row_width]: rows as b200_seq_delta_prepare leaves them; S_state fp32 [slots, H, dk, dv] advanced in place
// -> y fp32 [T, H * dv].  T: token rows of the step (steps with few rows per sequence take the form that is bound by the state's traffic)
extern "C" int b200_seq_delta_rows_scan(const float* pre, int channels, float* S_state, const int32_t* state_slots, const int32_t* cu_q,
                                   const int64_t* position_ids, float* y, int64_t ld_y, int64_t T, int B, int H, int kv_heads, int dk, int dv,
                                   void* stream) {
  if (T == 0 || B == 0) return B200_OK;
  if (kv_heads <= 0 || H % kv_heads != 0 || dk <= 0 || dk > 256 || dv <= 0) {
    b200_set_last_error("seq_delta_rows_scan: need heads % kv_heads == 0 and 0 < key size <= 256");
    return B200_ERR_ARG;
  }
  cudaStream_t st = (cudaStream_t)stream;
  const bool aligned = ((reinterpret_cast<uintptr_t>(pre) | reinterpret_cast<uintptr_t>(S_state)) & 15) == 0;
  if (T <= 2 * (int64_t)B) {
    const bool vec = dv % 4 == 0 && aligned;
    const int lanes = vec ? dv / 4 : dv;
    int CL = 1;
    while (CL < lanes && CL < 32) CL *= 2;
    const int rows = (dk + kStepThreads / CL - 1) / (kStepThreads / CL);
#define DST(NR, VEC) return (launch_delta_step<NR, VEC>(pre, S_state, state_slots, cu_q, position_ids, y, ld_y, B, H, kv_heads, dk, dv, channels, CL, st))
    if (vec) {
      if (rows <= 4) DST(4, 4);
      if (rows <= 8) DST(8, 4);
      if (rows <= 16) DST(16, 4);
      DST(32, 4);
    }
    if (rows <= 4) DST(4, 1);
    if (rows <= 8) DST(8, 1);
    if (rows <= 16) DST(16, 1);
    DST(32, 1);
#undef DST
  }
  const int vec = (dk % 4 == 0 && dv % 4 == 0 && aligned) ? 1 : 0;
  // 64 columns per block share each staged vector among more of the memory; 32 spread a small grid over more SMs
  const int most = (int64_t)B * H * ((dv + 31) / 32) <= 148 ? 32 : 64;
  const int blocks = (dv + most - 1) / most;
  const int NC = ((dv + blocks - 1) / blocks + 7) / 8 * 8;
#define DCH(NR) return (launch_delta_chunk<NR>(pre, S_state, state_slots, cu_q, position_ids, y, ld_y, B, H, kv_heads, dk, dv, channels, NC, vec, st))
  if (dk <= 64) DCH(4);
  if (dk <= 128) DCH(8);
  DCH(16);
#undef DCH
}
