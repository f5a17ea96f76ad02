// Row kernels around an fp32 residual stream: embedding lookup (scaled, or plus a learned position row), layer norm in and out of
// the stream, RMS norm of the stream with an offset weight, RMS norm of a
// column slice, grouped RMS norm with a gate, the clamped gated feed-forward activation, the per-layer token side input, the step
// between two sublayers of a decoder with several residual streams (write all streams, read and norm the next input) and of one
// whose sublayers have one or two branches, each with a norm of its own, the step between two layers that add a mixer and a routed
// feed-forward side by side, the soft cap on logits, plain activations, and the turn-back + gate of attention heads whose values carry their position.
// One block per token row; all statistics and the residual sum in fp32.
#include "seq_common.cuh"

namespace b200 {
namespace seq {

constexpr int kRowThreads = 256;

// x[t, :] = table[id[t], :] * scale  (fp32 residual stream)
template <typename T>
__global__ void __launch_bounds__(kRowThreads) embed_scale_kernel(const T* __restrict__ table, const int64_t* __restrict__ ids, float scale,
                                                                  float* __restrict__ out, int W, int64_t V) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  int64_t id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  for (int i = threadIdx.x; i < W; i += kRowThreads) out[t * W + i] = ldf(table + id * W + i) * scale;
}

// x[t, :] = table[id[t], :] + pos_table[position[t], :]  (learned absolute positions; fp32 residual stream)
template <typename T>
__global__ void __launch_bounds__(kRowThreads) embed_add_pos_kernel(const T* __restrict__ table, const T* __restrict__ pos_table,
                                                                    const int64_t* __restrict__ ids, const int64_t* __restrict__ position_ids,
                                                                    float* __restrict__ out, int W, int64_t V, int64_t P) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  int64_t id = ids[t], p = position_ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  p = p < 0 ? 0 : (p >= P ? P - 1 : p);
  for (int i = threadIdx.x; i < W; i += kRowThreads) out[t * W + i] = ldf(table + id * W + i) + ldf(pos_table + p * W + i);
}

// out[t] = x[t] / sqrt(mean(x[t]^2) + eps) * (w + w_offset): RMS norm of the fp32 stream whose weight is stored around -w_offset
// (w_offset 1: "one plus weight"; 0: plain weight)
template <typename TP>
__global__ void __launch_bounds__(kRowThreads) rmsnorm_rows_kernel(const float* __restrict__ x, const TP* __restrict__ w, float w_offset,
                                                                   TP* __restrict__ out, int W, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float v = x[t * W + i];
    q += v * v;
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / W + eps);
  for (int i = threadIdx.x; i < W; i += kRowThreads) stf(out + t * W + i, x[t * W + i] * rstd * (ldf(w + i) + w_offset));
}

// mode 0: out[t] = LN(x[t]) * w + b  (x fp32 or T, out T)      mode 1: resid[t] += LN(x[t]) * w + b  (resid fp32)
// In mode 1 `out`, when given, also receives the updated residual row in the activation type (the next projection's input).
template <typename TX, typename TP, typename TO>
__global__ void __launch_bounds__(kRowThreads) layernorm_kernel(const TX* __restrict__ x, const TP* __restrict__ w, const TP* __restrict__ b,
                                                                TO* __restrict__ out, float* __restrict__ resid, int W, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float s = 0.f;
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float v = ldf(x + t * W + i);
    row[i] = v;
    s += v;
  }
  const float mean = block_sum(s, red) / W;
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float d = row[i] - mean;
    q += d * d;
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / W + eps);
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float y = (row[i] - mean) * rstd * ldf(w + i) + ldf(b + i);
    if (resid) {
      const float r = resid[t * W + i] + y;
      resid[t * W + i] = r;
      if (out) stf(out + t * W + i, r);
    } else {
      stf(out + t * W + i, y);
    }
  }
}

// out[t, g*n + i] = gate_after * w[g*n+i] * v / sqrt(mean_i(v^2) + eps), v = x[t, g*n + i] * gate_before, per group g of n
// columns.  gate kinds: 0 none, 1 SiLU(gate) multiplied in before the statistics, 2 sigmoid(gate) multiplied in after the
// weight, 3 SiLU(gate) multiplied in after the weight.  groups == 0: no normalisation (gate only).  x and gate are column slices (leading dimensions given) of fp32 buffers.
template <typename TP, typename TO>
__global__ void __launch_bounds__(kRowThreads) group_rmsnorm_gate_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ gate,
                                                                         int64_t ldg, int gate_kind, const TP* __restrict__ w, int groups, int n,
                                                                         int C, float eps, TO* __restrict__ out, int64_t ldo) {
  // grid (rows, parts): a part is one group of n columns (groups > 0) or a run of n columns of an un-normalised row (groups == 0)
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int c0 = blockIdx.y * n, c1 = min(C, c0 + n);
  float rstd = 1.f;
  if (groups > 0) {
    float q = 0.f;
    for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
      float v = x[t * ldx + c];
      if (gate_kind == 1) v *= silu_f(gate[t * ldg + c]);
      q += v * v;
    }
    rstd = 1.f / sqrtf(block_sum(q, red) / n + eps);
  }
  for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
    float v = x[t * ldx + c];
    if (gate_kind == 1) v *= silu_f(gate[t * ldg + c]);
    v *= rstd;
    if (w) v *= ldf(w + c);
    if (gate_kind == 2) v *= sigmoid_f(gate[t * ldg + c]);
    else if (gate_kind == 3) v *= silu_f(gate[t * ldg + c]);
    stf(out + t * ldo + c, v);
  }
}

// y = g' * sigmoid(alpha g') * (u' + 1), g' = min(g, limit), u' = clamp(u, -limit, limit); gu = [g | u] per row
template <typename T>
__global__ void ff_clamped_gate_kernel(const T* __restrict__ gu, T* __restrict__ out, int64_t rows, int F, float limit, float alpha) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t total = rows * F;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t r = i / F, c = i % F;
    const float g = fminf(ldf(gu + r * 2 * F + c), limit);
    const float u = fminf(fmaxf(ldf(gu + r * 2 * F + F + c), -limit), limit);
    stf(out + i, g * sigmoid_f(alpha * g) * (u + 1.f));
  }
}

// Per-layer token input, the two row kernels around its projections:  g = gelu_tanh(a) * table[id, col0 : col0 + dim]  (a = Wg x),
// and  resid += y / sqrt(mean(y^2) + eps) * w  (y = Wp g).
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ a, const int64_t* __restrict__ ids, const T* __restrict__ table, int64_t ld_table,
                                 int64_t col0, int dim, int64_t V, T* __restrict__ out, int64_t rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t total = rows * dim;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / dim, j = i % dim;
    int64_t id = ids[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    stf(out + i, gelu_tanh_f(a[i]) * ldf(table + id * ld_table + col0 + j));
  }
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads) rms_add_kernel(const float* __restrict__ y, const T* __restrict__ w, float* __restrict__ resid, int W,
                                                              float eps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float v = y[t * W + i];
    q += v * v;
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / W + eps);
  for (int i = threadIdx.x; i < W; i += kRowThreads) resid[t * W + i] += y[t * W + i] * rstd * ldf(w + i);
}

// resid[t] += v / sqrt(mean(v^2) + eps) * w with v = y[t] * sigmoid(gate[t]) (gate NULL: v = y[t]): a sublayer's result, gated per
// channel, normalised and added to the fp32 stream.  `typed`, when given, also receives the updated row in the projections' type.
template <typename T>
__global__ void __launch_bounds__(kRowThreads) gated_rms_add_kernel(const float* __restrict__ y, const float* __restrict__ gate,
                                                                    const T* __restrict__ w, float* __restrict__ resid, T* __restrict__ typed, int W,
                                                                    float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    float v = y[t * W + i];
    if (gate) v *= sigmoid_f(gate[t * W + i]);
    row[i] = v;
    q += v * v;
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / W + eps);
  for (int i = threadIdx.x; i < W; i += kRowThreads) {
    const float r = resid[t * W + i] + row[i] * rstd * ldf(w + i);
    resid[t * W + i] = r;
    if (typed) stf(typed + t * W + i, r);
  }
}

template <typename T>
__global__ void cast_rows_kernel(const float* __restrict__ x, T* __restrict__ out, int64_t n) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) stf(out + i, x[i]);
}

// out = act(g) * u over rows [g | u]; act 0: SiLU, 1: GELU (tanh form)
template <typename T, int ACT>
__global__ void ff_gate_kernel(const T* __restrict__ gu, T* __restrict__ out, int64_t rows, int F) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t total = rows * F;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t r = i / F, c = i % F;
    const float g = ldf(gu + r * 2 * F + c), u = ldf(gu + r * 2 * F + F + c);
    stf(out + i, (ACT == 1 ? gelu_tanh_f(g) : silu_f(g)) * u);
  }
}

// Several residual streams per token ("hyper-connections"): X [T, S, W] fp32.  One launch does what lies between two sublayers:
//   write   (y given)        every stream at once from the old ones, X_t <- sum_s mix[s, t] X_s + out_coef[t] * y
//   read    (in_coef given)  u = sum_s in_coef[s] X_s of the (new) streams; typed <- u / sqrt(mean(u^2) + eps) * w (w NULL: typed <- u)
// `init`, when given, is the row every stream starts from (the embedding output) and X is not read.  One block per token; the
// row of u waits in shared memory between the two passes; S <= kMaxStreams.
constexpr int kMaxStreams = 8;

// VEC consecutive fp32 values in one access (VEC 4: 16 bytes, the pointer 16-byte aligned)
template <int VEC>
__device__ __forceinline__ void ld_vec(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = p[k];
  }
}
template <int VEC>
__device__ __forceinline__ void ld_vec(const __nv_bfloat16* p, float (&v)[VEC]) {   // VEC 4: 8 bytes
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  } else {
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = ldf(p + k);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void st_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (VEC == 4 && sizeof(T) == 2) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
#pragma unroll
    for (int k = 0; k < VEC; ++k) stf(p + k, v[k]);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads) streams_step_kernel(float* __restrict__ X, int S, const float* __restrict__ init,
                                                                   const float* __restrict__ y, const float* __restrict__ mix,
                                                                   const float* __restrict__ out_coef, const float* __restrict__ in_coef,
                                                                   const T* __restrict__ w, T* __restrict__ typed, int W, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  __shared__ float cm[kMaxStreams * kMaxStreams], co[kMaxStreams], ci[kMaxStreams];
  if (threadIdx.x < S * S) cm[threadIdx.x] = mix ? mix[threadIdx.x] : 0.f;
  if (threadIdx.x < S) {
    co[threadIdx.x] = out_coef ? out_coef[threadIdx.x] : 0.f;
    ci[threadIdx.x] = in_coef ? in_coef[threadIdx.x] : 0.f;
  }
  __syncthreads();
  const int64_t t = blockIdx.x;
  float* xr = X + t * S * W;
  float q = 0.f;
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {
    float x[kMaxStreams][VEC];
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s)
      if (s < S) ld_vec<VEC>(init ? init + t * W + i : xr + (int64_t)s * W + i, x[s]);
    float u[VEC];   // the read of the new streams, gathered while they are written
#pragma unroll
    for (int k = 0; k < VEC; ++k) u[k] = 0.f;
    if (y) {
      float yv[VEC];
      ld_vec<VEC>(y + t * W + i, yv);
#pragma unroll
      for (int o = 0; o < kMaxStreams; ++o) {
        if (o >= S) break;
        float nx[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) nx[k] = co[o] * yv[k];
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s)
          if (s < S) {
            const float c = cm[s * S + o];
#pragma unroll
            for (int k = 0; k < VEC; ++k) nx[k] = fmaf(c, x[s][k], nx[k]);
          }
        st_vec<float, VEC>(xr + (int64_t)o * W + i, nx);   // every old stream of this column is in registers already
#pragma unroll
        for (int k = 0; k < VEC; ++k) u[k] = fmaf(ci[o], nx[k], u[k]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) {
          if (init) st_vec<float, VEC>(xr + (int64_t)s * W + i, x[s]);
#pragma unroll
          for (int k = 0; k < VEC; ++k) u[k] = fmaf(ci[s], x[s][k], u[k]);
        }
    }
    if (in_coef) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) q += u[k] * u[k];
      st_vec<float, VEC>(row + i, u);
    }
  }
  if (!in_coef) return;
  const float rstd = w ? 1.f / sqrtf(block_sum(q, red) / W + eps) : 1.f;
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {   // every thread reads back what it wrote itself
    float u[VEC];
    ld_vec<VEC>(row + i, u);
    if (w) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) u[k] = u[k] * rstd * ldf(w + i + k);
    }
    st_vec<T, VEC>(typed + t * W + i, u);
  }
}

// One stream between two sublayers (row t of x, fp32):
//   r = (init ? init[t] : x[t]) + y_scale * (n_1(y1[t]) + n_2(y2[t])) + add[t] + step_vec,   n_i(y) = y / sqrt(mean(y^2) + eps) * w_i
// (w_i NULL: the branch is added as it is; any term may be missing), x[t] <- r, typed[t] <- r / sqrt(mean(r^2) + eps) * norm_w.
// One block per token; the branches' rows and r wait in shared memory between the passes (every thread reads back what it wrote).
template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads) branches_step_kernel(float* __restrict__ x, const float* __restrict__ init, const float* __restrict__ y1,
                                                                    const T* __restrict__ w1, const float* __restrict__ y2, const T* __restrict__ w2,
                                                                    float y_scale, const float* __restrict__ add, const T* __restrict__ step_vec,
                                                                    const T* __restrict__ norm_w, T* __restrict__ typed, int W, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float rows[];
  __shared__ float red[3][32];
  const int64_t t = blockIdx.x;
  const int pitch = (W + 3) & ~3;
  float *row = rows, *r1 = rows + pitch, *r2 = r1 + pitch;
  float q1 = 0.f, q2 = 0.f;
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {
    float r[VEC], v[VEC];
    ld_vec<VEC>((init ? init : x) + t * W + i, r);
    if (add) {
      ld_vec<VEC>(add + t * W + i, v);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[k] += v[k];
    }
    if (step_vec) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[k] += ldf(step_vec + i + k);
    }
    st_vec<float, VEC>(row + i, r);
    if (y1) {
      ld_vec<VEC>(y1 + t * W + i, v);
#pragma unroll
      for (int k = 0; k < VEC; ++k) q1 += v[k] * v[k];
      st_vec<float, VEC>(r1 + i, v);
    }
    if (y2) {
      ld_vec<VEC>(y2 + t * W + i, v);
#pragma unroll
      for (int k = 0; k < VEC; ++k) q2 += v[k] * v[k];
      st_vec<float, VEC>(r2 + i, v);
    }
  }
  float s1 = y_scale, s2 = y_scale;
  if (w1 || w2) {   // both statistics behind one barrier
    q1 = warp_sum(q1);
    q2 = warp_sum(q2);
    if (lane_id() == 0) {
      red[0][warp_id()] = q1;
      red[1][warp_id()] = q2;
    }
    __syncthreads();
    constexpr int kWarps = kRowThreads / 32;
    q1 = warp_sum(lane_id() < kWarps ? red[0][lane_id()] : 0.f);
    q2 = warp_sum(lane_id() < kWarps ? red[1][lane_id()] : 0.f);
    if (w1) s1 *= 1.f / sqrtf(q1 / W + eps);
    if (w2) s2 *= 1.f / sqrtf(q2 / W + eps);
  }
  float q = 0.f;
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {
    float r[VEC], v[VEC];
    ld_vec<VEC>(row + i, r);
    if (y1) {
      ld_vec<VEC>(r1 + i, v);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[k] = fmaf(s1 * v[k], w1 ? ldf(w1 + i + k) : 1.f, r[k]);
    }
    if (y2) {
      ld_vec<VEC>(r2 + i, v);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[k] = fmaf(s2 * v[k], w2 ? ldf(w2 + i + k) : 1.f, r[k]);
    }
    st_vec<float, VEC>(x + t * W + i, r);
    if (norm_w) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) q += r[k] * r[k];
      st_vec<float, VEC>(row + i, r);
    }
  }
  if (!norm_w) return;
  const float rstd = 1.f / sqrtf(block_sum(q, red[2]) / W + eps);
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {
    float r[VEC];
    ld_vec<VEC>(row + i, r);
#pragma unroll
    for (int k = 0; k < VEC; ++k) r[k] *= rstd * ldf(norm_w + i + k);
    st_vec<T, VEC>(typed + t * W + i, r);
  }
}

// One stream whose layers read it once and add two halves side by side (row t of x, fp32): what lies between two layers in one launch,
//   r = (init ? init[t] : x[t]) + y1[t] + sigmoid(gate[t]) * y2[t] + sum_k weights[t, k] * (row_of[t, k] >= 0 ? rows[row_of[t, k]] : pass[t]),
//   x[t] <- r, typed_a[t] <- n(r) * norm_a, typed_b[t] <- n(r) * norm_b with n(r) = r / sqrt(mean(r^2) + eps)
// (any term may be missing, gate NULL: y2 as it is).  The sum is a routed feed-forward's: experts' rows, and for a pick of an identity
// output the row `pass` that the router read.  One block per token; r waits in shared memory between the passes.
constexpr int kPicks = 16;

template <typename T, int VEC, int TOP>   // TOP >= top: the loads of all terms are in flight together
__global__ void __launch_bounds__(kRowThreads) halves_step_kernel(float* __restrict__ x, const float* __restrict__ init, const float* __restrict__ y1,
                                                                  const float* __restrict__ y2, const float* __restrict__ gate, int64_t ld_gate,
                                                                  const float* __restrict__ rows, int64_t ld_rows, const float* __restrict__ weights,
                                                                  const int32_t* __restrict__ row_of, int top, const T* __restrict__ pass,
                                                                  const T* __restrict__ norm_a, const T* __restrict__ norm_b, T* __restrict__ typed_a,
                                                                  T* __restrict__ typed_b, int W, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const float* base = (init ? init : x) + t * W;
  const float s2 = y2 ? (gate ? sigmoid_f(gate[t * ld_gate]) : 1.f) : 0.f;
  // the identity picks share one weight: their row is read once
  float w_pass = 0.f, w_k[TOP > 0 ? TOP : 1];
  const float* src[TOP > 0 ? TOP : 1];
#pragma unroll
  for (int k = 0; k < TOP; ++k) {
    const int r = k < top ? row_of[t * top + k] : -1;
    const float w = k < top ? weights[t * top + k] : 0.f;
    src[k] = r >= 0 ? rows + (int64_t)r * ld_rows : nullptr;
    w_k[k] = r >= 0 ? w : 0.f;
    w_pass += r >= 0 ? 0.f : w;
  }
  float q = 0.f;
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {
    float r[VEC], a[VEC] = {}, b[VEC] = {}, h[VEC] = {}, v[TOP > 0 ? TOP : 1][VEC] = {};
    ld_vec<VEC>(base + i, r);
    if (y1) ld_vec<VEC>(y1 + t * W + i, a);
    if (y2) ld_vec<VEC>(y2 + t * W + i, b);
#pragma unroll
    for (int e = 0; e < TOP; ++e)
      if (src[e]) ld_vec<VEC>(src[e] + i, v[e]);
    if (TOP > 0 && w_pass != 0.f) ld_vec<VEC>(pass + t * W + i, h);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      r[k] = fmaf(w_pass, h[k], fmaf(s2, b[k], r[k] + a[k]));
#pragma unroll
      for (int e = 0; e < TOP; ++e) r[k] = fmaf(w_k[e], v[e][k], r[k]);
      q += r[k] * r[k];
    }
    st_vec<float, VEC>(x + t * W + i, r);
    if (norm_a || norm_b) st_vec<float, VEC>(row + i, r);
  }
  if (!norm_a && !norm_b) return;
  const float rstd = 1.f / sqrtf(block_sum(q, red) / W + eps);
  for (int i = threadIdx.x * VEC; i < W; i += kRowThreads * VEC) {   // every thread reads back what it wrote itself
    float r[VEC], wa[VEC] = {}, wb[VEC] = {};
    ld_vec<VEC>(row + i, r);
    if (norm_a) ld_vec<VEC>(norm_a + i, wa);
    if (norm_b) ld_vec<VEC>(norm_b + i, wb);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      r[k] *= rstd;
      wa[k] *= r[k];
      wb[k] *= r[k];
    }
    if (norm_a) st_vec<T, VEC>(typed_a + t * W + i, wa);
    if (norm_b) st_vec<T, VEC>(typed_b + t * W + i, wb);
  }
}

// z <- cap * tanh(z / cap) in place (logits)
__global__ void __launch_bounds__(256) soft_cap_kernel(float* __restrict__ z, int64_t n, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t stride = (int64_t)gridDim.x * 256;
  for (int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x; i < n; i += stride) z[i] = cap * tanhf(z[i] / cap);
}

// out = act(in) element by element over rows of F columns (in may be a column slice: leading dimension ld_in);
// act 0: SiLU, 1: GELU (tanh form), 2: tanh, 3: relu squared, 4: none (a copy or a change of type).  Evaluated in fp32.
template <int ACT>
__device__ __forceinline__ float plain_act_f(float z) {
  if constexpr (ACT == 0) return silu_f(z);
  else if constexpr (ACT == 1) return gelu_tanh_f(z);
  else if constexpr (ACT == 2) return tanhf(z);
  else if constexpr (ACT == 3) { const float p = fmaxf(z, 0.f); return p * p; }
  else return z;
}

template <typename TI, typename TO, int ACT>
__global__ void ff_act_kernel(const TI* __restrict__ in, int64_t ld_in, TO* __restrict__ out, int64_t rows, int F) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t total = rows * F;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t r = i / F, c = i % F;
    const float z = ldf(in + r * ld_in + c);
    stf(out + i, plain_act_f<ACT>(z));
  }
}

// eight consecutive elements as 16-byte accesses
template <typename T>
__device__ __forceinline__ void ld8(const T* p, float (&v)[8]) {
  if constexpr (sizeof(T) == 4) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
}
template <typename T>
__device__ __forceinline__ void st8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 4) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&b);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
}

// ff_act_kernel for rows of whole 8-element pieces on 16-byte boundaries
template <typename TI, typename TO, int ACT>
__global__ void __launch_bounds__(kRowThreads) ff_act_vec_kernel(const TI* __restrict__ in, int64_t ld_in, TO* __restrict__ out, int64_t rows, int F) {
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t per_row = (uint32_t)F / 8;
  for (int64_t r = blockIdx.x; r < rows; r += gridDim.x)
    for (uint32_t c = blockIdx.y * kRowThreads + threadIdx.x; c < per_row; c += gridDim.y * kRowThreads) {
      float v[8];
      ld8(in + r * ld_in + c * 8, v);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] = plain_act_f<ACT>(v[k]);
      st8(out + r * F + c * 8, v);
    }
}

// group_rmsnorm_gate_kernel for groups of n <= 512 columns: one warp per (row, group), VEC columns per access, the group held in
// registers between its statistic and its way out
template <typename TP, typename TO, int VEC, int PIECES>
__global__ void __launch_bounds__(kRowThreads) group_rmsnorm_warp_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ gate,
                                                                         int64_t ldg, int gate_kind, const TP* __restrict__ w, int groups, int n,
                                                                         float eps, TO* __restrict__ out, int64_t ldo, int64_t items) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t item = (int64_t)blockIdx.x * (kRowThreads / 32) + warp_id();
  if (item >= items) return;
  const int64_t t = item / groups;
  const int c0 = (int)(item % groups) * n;
  float v[PIECES][VEC], g[PIECES][VEC], q = 0.f;
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    const int c = (lane_id() + 32 * i) * VEC;
    if (c < n) {
      ld_vec<VEC>(x + t * ldx + c0 + c, v[i]);
      if (gate_kind) ld_vec<VEC>(gate + t * ldg + c0 + c, g[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        if (gate_kind == 1) v[i][k] *= silu_f(g[i][k]);
        q += v[i][k] * v[i][k];
      }
    }
  }
  const float rstd = 1.f / sqrtf(warp_sum(q) / n + eps);
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    const int c = (lane_id() + 32 * i) * VEC;
    if (c < n) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        float o = v[i][k] * rstd;
        if (w) o *= ldf(w + c0 + c + k);
        if (gate_kind == 2) o *= sigmoid_f(g[i][k]);
        else if (gate_kind == 3) o *= silu_f(g[i][k]);
        v[i][k] = o;
      }
      st_vec<TO, VEC>(out + t * ldo + c0 + c, v[i]);
    }
  }
}

// Attention heads on their way to the output projection: a [T, H, dv] fp32; every head's first `rot` columns are turned by
// -position (pairs: column i with column i + rot / 2 when `interleaved` is 0, columns 2i and 2i + 1 otherwise; cos / sin
// [positions, rot / 2]), then the head is multiplied by sigmoid(gate[t, h]) (gate NULL: by 1) and by out_scale -> out rows of
// H * dv columns of type T (leading dimension ld_out: the rows may be a column slice of a wider buffer).
template <typename T>
__global__ void __launch_bounds__(kRowThreads) heads_turn_gate_kernel(const float* __restrict__ a, const float* __restrict__ gate, int64_t ld_gate,
                                                                      const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                                                                      int interleaved, const int64_t* __restrict__ position_ids,
                                                                      T* __restrict__ out, int64_t ld_out, float out_scale, int H, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int half = rot / 2;
  const float* cs = rot ? cos_t + position_ids[t] * half : nullptr;
  const float* sn = rot ? sin_t + position_ids[t] * half : nullptr;
  const float* row = a + t * H * dv;
  for (int e = threadIdx.x; e < H * dv; e += kRowThreads) {
    const int h = e / dv, i = e % dv;
    float x = row[e];
    if (i < rot) {
      int f, partner;
      bool first;
      if (interleaved) { f = i >> 1; first = (i & 1) == 0; partner = first ? e + 1 : e - 1; }
      else { first = i < half; f = first ? i : i - half; partner = first ? e + half : e - half; }
      const float yv = row[partner];
      // the inverse turn: (u, v) -> (u cos + v sin, v cos - u sin)
      x = first ? x * cs[f] + yv * sn[f] : x * cs[f] - yv * sn[f];
    }
    if (gate) x *= sigmoid_f(gate[t * ld_gate + h]);
    stf(out + t * ld_out + e, x * out_scale);
  }
}

}  // namespace seq
}  // namespace b200

using namespace b200::seq;

extern "C" int b200_seq_embed_scale(const void* table, int dt, const int64_t* ids, float scale, float* out, int64_t T, int64_t W, int64_t V,
                                    void* stream) {
  if (T == 0) return B200_OK;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((embed_scale_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), 0, (cudaStream_t)stream, (const E*)table, ids,
                                       scale, out, (int)W, V));
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_embed_add_pos(const void* table, const void* pos_table, int dt, const int64_t* ids, const int64_t* position_ids,
                                      float* out, int64_t T, int64_t W, int64_t V, int64_t P, void* stream) {
  if (T == 0) return B200_OK;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((embed_add_pos_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), 0, (cudaStream_t)stream, (const E*)table,
                                       (const E*)pos_table, ids, position_ids, out, (int)W, V, P));
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_rmsnorm_rows(const float* x, const void* w, int dt, float w_offset, void* out, int64_t T, int64_t W, float eps,
                                     void* stream) {
  if (T == 0) return B200_OK;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((rmsnorm_rows_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), 0, (cudaStream_t)stream, x, (const E*)w,
                                       w_offset, (E*)out, (int)W, eps));
  b200_count_launches(1);
  return B200_OK;
}

// x_dt: element type of x (fp32 stream or an activation of type dt).  resid == nullptr: out (type dt) = LN(x); else resid += LN(x).
extern "C" int b200_seq_layernorm(const void* x, int x_dt, const void* w, const void* b, int dt, void* out, float* resid, int64_t T, int64_t W,
                                  float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (W * 4 > 160 * 1024) { b200_set_last_error("seq_layernorm: row too wide"); return B200_ERR_ARG; }
  cudaStream_t st = (cudaStream_t)stream;
  const size_t smem = (size_t)W * 4;
#define LN_LAUNCH(TX, TP)                                                                                                              \
  do {                                                                                                                                 \
    static bool cfg = false;                                                                                                           \
    if (!cfg) { cudaFuncSetAttribute(layernorm_kernel<TX, TP, TP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); cfg = true; } \
    B200_LAUNCH((layernorm_kernel<TX, TP, TP>), dim3((unsigned)T), dim3(kRowThreads), smem, st, (const TX*)x, (const TP*)w, (const TP*)b,   \
                (TP*)out, resid, (int)W, eps);                                                                                         \
  } while (0)
  if (dt == B200_DT_F32 && x_dt == B200_DT_F32) LN_LAUNCH(float, float);
  else if (dt == B200_DT_BF16 && x_dt == B200_DT_F32) LN_LAUNCH(float, __nv_bfloat16);
  else if (dt == B200_DT_BF16 && x_dt == B200_DT_BF16) LN_LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else { b200_set_last_error("seq_layernorm: unsupported element types"); return B200_ERR_UNSUPPORTED; }
#undef LN_LAUNCH
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_group_rmsnorm_gate(const float* x, int64_t ldx, const float* gate, int64_t ldg, int gate_kind, const void* w, int w_dt,
                                           int groups, int n, float eps, void* out, int out_dt, int64_t ldo, int64_t T, void* stream) {
  if (T == 0) return B200_OK;
  if (gate_kind != 0 && gate == nullptr) { b200_set_last_error("seq_group_rmsnorm_gate: gate missing"); return B200_ERR_ARG; }
  cudaStream_t st = (cudaStream_t)stream;
  const int C = groups > 0 ? groups * n : n;
  const int part = groups > 0 ? n : 2048;
  const dim3 grid((unsigned)T, (unsigned)((C + part - 1) / part));
  // 16-byte accesses when every group starts on a 16-byte boundary (the gate and the typed rows included)
  const bool vec = groups > 0 && n % 4 == 0 && ldx % 4 == 0 && (gate == nullptr || ldg % 4 == 0) && ldo % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  if (vec && n <= 512) {
    const int64_t items = T * groups;
#define GW_LAUNCH(TP, TO, P)                                                                                                            \
  B200_LAUNCH((group_rmsnorm_warp_kernel<TP, TO, 4, P>), dim3((unsigned)((items + 7) / 8)), dim3(kRowThreads), 0, st, x, ldx, gate, ldg, gate_kind, \
              (const TP*)w, groups, n, eps, (TO*)out, ldo, items)
#define GW(TP, TO)                            \
  do {                                        \
    if (n <= 128) GW_LAUNCH(TP, TO, 1);       \
    else if (n <= 256) GW_LAUNCH(TP, TO, 2);  \
    else GW_LAUNCH(TP, TO, 4);                \
  } while (0)
    if (w_dt == B200_DT_F32 && out_dt == B200_DT_F32) GW(float, float);
    else if (w_dt == B200_DT_BF16 && out_dt == B200_DT_BF16) GW(__nv_bfloat16, __nv_bfloat16);
    else if (w_dt == B200_DT_BF16 && out_dt == B200_DT_F32) GW(__nv_bfloat16, float);
    else { b200_set_last_error("seq_group_rmsnorm_gate: unsupported element types"); return B200_ERR_UNSUPPORTED; }
#undef GW
#undef GW_LAUNCH
    b200_count_launches(1);
    return B200_OK;
  }
#define GN_LAUNCH(TP, TO)                                                                                                                   \
  B200_LAUNCH((group_rmsnorm_gate_kernel<TP, TO>), grid, dim3(kRowThreads), 0, st, x, ldx, gate, ldg, gate_kind, (const TP*)w, groups, part, \
              C, eps, (TO*)out, ldo)
  if (w_dt == B200_DT_F32 && out_dt == B200_DT_F32) GN_LAUNCH(float, float);
  else if (w_dt == B200_DT_BF16 && out_dt == B200_DT_BF16) GN_LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (w_dt == B200_DT_BF16 && out_dt == B200_DT_F32) GN_LAUNCH(__nv_bfloat16, float);
  else { b200_set_last_error("seq_group_rmsnorm_gate: unsupported element types"); return B200_ERR_UNSUPPORTED; }
#undef GN_LAUNCH
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_ff_clamped_gate(const void* gu, void* out, int dt, int64_t rows, int64_t F, float limit, float alpha, void* stream) {
  if (rows == 0 || F == 0) return B200_OK;
  int64_t blocks = (rows * F + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((ff_clamped_gate_kernel<E>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const E*)gu, (E*)out,
                                       rows, (int)F, limit, alpha));
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_side_gate(const float* a, const int64_t* ids, const void* table, int64_t ld_table, int64_t col0, int dim, int64_t V,
                                  void* out, int dt, int64_t rows, void* stream) {
  if (rows == 0 || dim == 0) return B200_OK;
  int64_t blocks = (rows * dim + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((side_gate_kernel<E>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, a, ids, (const E*)table,
                                       ld_table, col0, dim, V, (E*)out, rows));
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_rms_add(const float* y, const void* w, int dt, float* resid, int64_t T, int64_t W, float eps, void* stream) {
  if (T == 0) return B200_OK;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((rms_add_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), 0, (cudaStream_t)stream, y, (const E*)w, resid,
                                       (int)W, eps));
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_gated_rms_add(const float* y, const float* gate, const void* w, int dt, float* resid, void* typed, int64_t T, int64_t W,
                                      float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (W * 4 > 160 * 1024) { b200_set_last_error("seq_gated_rms_add: row too wide"); return B200_ERR_ARG; }
#define GRA(E)                                                                                                                          \
  do {                                                                                                                                  \
    static bool cfg = false;                                                                                                            \
    if (!cfg) { cudaFuncSetAttribute(gated_rms_add_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); cfg = true; }   \
    B200_LAUNCH((gated_rms_add_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), (size_t)W * 4, (cudaStream_t)stream, y, gate, (const E*)w, \
                resid, (E*)typed, (int)W, eps);                                                                                         \
  } while (0)
  if (dt == B200_DT_F32) GRA(float);
  else if (dt == B200_DT_BF16) GRA(__nv_bfloat16);
  else { b200_set_last_error("unknown element type"); return B200_ERR_ARG; }
#undef GRA
  b200_count_launches(1);
  return B200_OK;
}

extern "C" int b200_seq_cast_rows(const float* x, void* out, int dt, int64_t n, void* stream) {
  if (n == 0) return B200_OK;
  int64_t blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((cast_rows_kernel<E>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, x, (E*)out, n));
  b200_count_launches(1);
  return B200_OK;
}

// act 0: SiLU(g) * u, 1: GELU_tanh(g) * u
extern "C" int b200_seq_ff_gate(const void* gu, void* out, int dt, int64_t rows, int64_t F, int act, void* stream) {
  if (rows == 0 || F == 0) return B200_OK;
  int64_t blocks = (rows * F + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (act == 1)
    B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((ff_gate_kernel<E, 1>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const E*)gu, (E*)out,
                                         rows, (int)F));
  else
    B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((ff_gate_kernel<E, 0>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const E*)gu, (E*)out,
                                         rows, (int)F));
  b200_count_launches(1);
  return B200_OK;
}

// X fp32 [T, S, W] in place (S <= 8).  init fp32 [T, W] or NULL; y fp32 [T, W] or NULL (with mix fp32 [S, S] indexed [from, to] and
// out_coef fp32 [S]); in_coef fp32 [S] or NULL (with typed [T, W] of type dt and, optionally, the norm weight w of type dt).
extern "C" int b200_seq_streams_step(float* X, int S, const float* init, const float* y, const float* mix, const float* out_coef,
                                     const float* in_coef, const void* w, int dt, void* typed, int64_t T, int64_t W, float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (S < 1 || S > kMaxStreams || (y && (!mix || !out_coef)) || (in_coef && !typed) || W > 40000) {
    b200_set_last_error("seq_streams_step: 1 <= streams <= 8; a write needs mix and out_coef, a read needs an output");
    return B200_ERR_ARG;
  }
#define SST(E, V)                                                                                                                        \
  do {                                                                                                                                   \
    static bool cfg = false;                                                                                                             \
    if (!cfg) { cudaFuncSetAttribute(streams_step_kernel<E, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); cfg = true; }  \
    B200_LAUNCH((streams_step_kernel<E, V>), dim3((unsigned)T), dim3(kRowThreads), (size_t)W * 4, (cudaStream_t)stream, X, S, init, y, mix, \
                out_coef, in_coef, (const E*)w, (E*)typed, (int)W, eps);                                                                 \
  } while (0)
  // 16-byte accesses when every row starts on a 16-byte boundary
  const bool vec = W % 4 == 0 && ((reinterpret_cast<uintptr_t>(X) | reinterpret_cast<uintptr_t>(init) | reinterpret_cast<uintptr_t>(y) |
                                   reinterpret_cast<uintptr_t>(typed)) & 15) == 0;
  if (dt == B200_DT_F32) { if (vec) SST(float, 4); else SST(float, 1); }
  else if (dt == B200_DT_BF16) { if (vec) SST(__nv_bfloat16, 4); else SST(__nv_bfloat16, 1); }
  else { b200_set_last_error("unknown element type"); return B200_ERR_ARG; }
#undef SST
  b200_count_launches(1);
  return B200_OK;
}

// x fp32 [T, W] in place, or from `init` [T, W]; y1 / y2 fp32 [T, W] with optional norm weights w1 / w2 [W]; add fp32 [T, W], step_vec [W]; norm_w
// [W] with typed [T, W]; every pointer but x may be NULL.  Weights, step_vec and typed of element type dt.
extern "C" int b200_seq_branches_step(float* x, const float* init, const float* y1, const void* w1, const float* y2, const void* w2, float y_scale,
                                      const float* add, const void* step_vec, const void* norm_w, int dt, void* typed, int64_t T, int64_t W,
                                      float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (W > 13000 || (norm_w && !typed) || (w1 && !y1) || (w2 && !y2)) {
    b200_set_last_error("seq_branches_step: width <= 13000; a norm needs its row");
    return B200_ERR_ARG;
  }
  const size_t smem = (size_t)((W + 3) & ~3) * 4 * 3;
#define BST(E, V)                                                                                                                         \
  do {                                                                                                                                    \
    static bool cfg = false;                                                                                                              \
    if (!cfg) { cudaFuncSetAttribute(branches_step_kernel<E, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); cfg = true; }  \
    B200_LAUNCH((branches_step_kernel<E, V>), dim3((unsigned)T), dim3(kRowThreads), smem, (cudaStream_t)stream, x, init, y1, (const E*)w1, y2, \
                (const E*)w2, y_scale, add, (const E*)step_vec, (const E*)norm_w, (E*)typed, (int)W, eps);                                \
  } while (0)
  const bool vec = W % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(init) | reinterpret_cast<uintptr_t>(y1) |
                                   reinterpret_cast<uintptr_t>(y2) | reinterpret_cast<uintptr_t>(add) | reinterpret_cast<uintptr_t>(typed)) & 15) == 0;
  if (dt == B200_DT_F32) { if (vec) BST(float, 4); else BST(float, 1); }
  else if (dt == B200_DT_BF16) { if (vec) BST(__nv_bfloat16, 4); else BST(__nv_bfloat16, 1); }
  else { b200_set_last_error("unknown element type"); return B200_ERR_ARG; }
#undef BST
  b200_count_launches(1);
  return B200_OK;
}

// x fp32 [T, W] in place, or from `init`; y1, y2 fp32 [T, W]; gate: one fp32 logit per token (stride ld_gate); rows fp32 (leading dimension
// ld_rows), weights fp32 [T, top], row_of int32 [T, top] (-1: the pick adds `pass`, [T, W] of type dt), top <= 16; norm_a / norm_b [W] with
// typed_a / typed_b [T, W] of type dt; every pointer but x may be NULL.
extern "C" int b200_seq_halves_step(float* x, const float* init, const float* y1, const float* y2, const float* gate, int64_t ld_gate, const float* rows,
                                    int64_t ld_rows, const float* weights, const int32_t* row_of, int top, const void* pass, const void* norm_a,
                                    const void* norm_b, int dt, void* typed_a, void* typed_b, int64_t T, int64_t W, float eps, void* stream) {
  if (T == 0) return B200_OK;
  if (!row_of) top = 0;
  if (W > 40000 || top > kPicks || (norm_a && !typed_a) || (norm_b && !typed_b) || (top > 0 && (!rows || !weights || !pass))) {
    b200_set_last_error("seq_halves_step: width <= 40000, at most 16 picks, a norm needs its row, picks need rows, weights and the router's input");
    return B200_ERR_ARG;
  }
  const size_t smem = (size_t)((W + 3) & ~3) * 4;
#define HST_TOP(E, V, N)                                                                                                                 \
  do {                                                                                                                                   \
    static bool cfg = false;                                                                                                             \
    if (!cfg) { cudaFuncSetAttribute(halves_step_kernel<E, V, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); cfg = true; } \
    B200_LAUNCH((halves_step_kernel<E, V, N>), dim3((unsigned)T), dim3(kRowThreads), smem, (cudaStream_t)stream, x, init, y1, y2, gate, ld_gate, rows, \
                ld_rows, weights, row_of, top, (const E*)pass, (const E*)norm_a, (const E*)norm_b, (E*)typed_a, (E*)typed_b, (int)W, eps); \
  } while (0)
#define HST(E)                          \
  do {                                  \
    if (!vec) HST_TOP(E, 1, kPicks);    \
    else if (top == 0) HST_TOP(E, 4, 0); \
    else if (top <= 2) HST_TOP(E, 4, 2); \
    else if (top <= 4) HST_TOP(E, 4, 4); \
    else if (top <= 8) HST_TOP(E, 4, 8); \
    else HST_TOP(E, 4, kPicks);         \
  } while (0)
  const bool vec = W % 4 == 0 && ld_rows % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(init) | reinterpret_cast<uintptr_t>(y1) | reinterpret_cast<uintptr_t>(y2) |
                     reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(typed_a) | reinterpret_cast<uintptr_t>(typed_b) |
                     reinterpret_cast<uintptr_t>(pass) | reinterpret_cast<uintptr_t>(norm_a) | reinterpret_cast<uintptr_t>(norm_b)) & 15) == 0;
  if (dt == B200_DT_F32) HST(float);
  else if (dt == B200_DT_BF16) HST(__nv_bfloat16);
  else { b200_set_last_error("unknown element type"); return B200_ERR_ARG; }
#undef HST
#undef HST_TOP
  b200_count_launches(1);
  return B200_OK;
}

// z fp32, n values in place: cap * tanh(z / cap)
extern "C" int b200_seq_soft_cap(float* z, int64_t n, float cap, void* stream) {
  if (n == 0) return B200_OK;
  if (!(cap > 0.f)) { b200_set_last_error("seq_soft_cap: the cap must be positive"); return B200_ERR_ARG; }
  const int64_t blocks = (n + 1023) / 1024;
  B200_LAUNCH(soft_cap_kernel, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), 0, (cudaStream_t)stream, z, n, cap);
  b200_count_launches(1);
  return B200_OK;
}

// in: rows of type in_dt (leading dimension ld_in), out: dense rows of type out_dt; act 0 SiLU, 1 GELU (tanh form), 2 tanh, 3 relu squared, 4 none
extern "C" int b200_seq_ff_act(const void* in, int in_dt, int64_t ld_in, void* out, int out_dt, int64_t rows, int64_t F, int act, void* stream) {
  if (rows == 0 || F == 0) return B200_OK;
  int64_t blocks = (rows * F + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (act < 0 || act > 4) { b200_set_last_error("seq_ff_act: unknown activation"); return B200_ERR_ARG; }
  const size_t in_sz = in_dt == B200_DT_F32 ? 4 : 2;
  const bool vec = F % 8 == 0 && (ld_in * in_sz) % 16 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int64_t per_row = (F / 8 + kRowThreads - 1) / kRowThreads, many = 148 * 64;
  const dim3 vgrid((unsigned)(rows < many ? rows : many), (unsigned)(per_row < 8 ? per_row : 8));
#define FA(TI, TO, A)                                                                                                                              \
  do {                                                                                                                                             \
    if (vec) B200_LAUNCH((ff_act_vec_kernel<TI, TO, A>), vgrid, dim3(kRowThreads), 0, (cudaStream_t)stream, (const TI*)in, ld_in, (TO*)out, rows, (int)F); \
    else FA_PLAIN(TI, TO, A);                                                                                                                      \
  } while (0)
#define FA_PLAIN(TI, TO, A) B200_LAUNCH((ff_act_kernel<TI, TO, A>), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const TI*)in, ld_in, (TO*)out, rows, (int)F)
#define FA_ACT(TI, TO)            \
  do {                            \
    if (act == 0) FA(TI, TO, 0);  \
    else if (act == 1) FA(TI, TO, 1); \
    else if (act == 2) FA(TI, TO, 2); \
    else if (act == 3) FA(TI, TO, 3); \
    else FA(TI, TO, 4);           \
  } while (0)
  if (in_dt == B200_DT_F32 && out_dt == B200_DT_F32) FA_ACT(float, float);
  else if (in_dt == B200_DT_F32 && out_dt == B200_DT_BF16) FA_ACT(float, __nv_bfloat16);
  else if (in_dt == B200_DT_BF16 && out_dt == B200_DT_BF16) FA_ACT(__nv_bfloat16, __nv_bfloat16);
  else { b200_set_last_error("seq_ff_act: element types must be fp32 -> any or bf16 -> bf16"); return B200_ERR_ARG; }
#undef FA_ACT
#undef FA
#undef FA_PLAIN
  b200_count_launches(1);
  return B200_OK;
}

// a fp32 [T, H, dv]; gate fp32 rows (leading dimension ld_gate, one logit per head) or NULL; cos / sin fp32 [positions, rot / 2]
// (rot 0: no turn) -> out [T, ld_out] of type dt, H * dv columns written, times out_scale
extern "C" int b200_seq_heads_turn_gate(const float* a, const float* gate, int64_t ld_gate, const float* cos_t, const float* sin_t, int rot,
                                        int interleaved, const int64_t* position_ids, void* out, int dt, int64_t ld_out, float out_scale,
                                        int64_t T, int H, int dv, void* stream) {
  if (T == 0) return B200_OK;
  if (rot < 0 || rot > dv || rot % 2 != 0 || (rot > 0 && (!cos_t || !sin_t || !position_ids))) {
    b200_set_last_error("seq_heads_turn_gate: turned columns must be even, at most the head size, with tables and positions");
    return B200_ERR_ARG;
  }
  B200_SEQ_DISPATCH(dt, E, B200_LAUNCH((heads_turn_gate_kernel<E>), dim3((unsigned)T), dim3(kRowThreads), 0, (cudaStream_t)stream, a, gate, ld_gate,
                                       cos_t, sin_t, rot, interleaved, position_ids, (E*)out, ld_out, out_scale, H, dv));
  b200_count_launches(1);
  return B200_OK;
}
