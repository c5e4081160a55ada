// One pass over the residual stream between two sublayers: what the sublayer in front left is gated or normed, added,
// and the sum is normed for the sublayer behind. Per row, in float32:
//
//   y = delta_scale * (sum over its partial sums of delta)            (delta absent: nothing is added)
//   y <- y * sigmoid(gate + gate_bias)                                (with a gate)
//   y <- y / sqrt(mean(y^2) + post_eps) * post_w                      (with post_w: a norm behind the sublayer)
//   x <- x + y                                                        written back unless rows are gathered
//   copy = x in the compute dtype                                     (optional: for a product that reads the stream itself)
//   out = norm(x): layer norm (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b, or x / sqrt(mean(x^2) + eps) * w
//
// A row stays in registers between the steps; the mean and the variance are taken in two passes over it.
#include "common.cuh"

namespace dl {

constexpr int RN_NORM_NONE = 0, RN_NORM_LAYER = 1, RN_NORM_RMS = 2;

template <typename T, int V> struct RnVec {
  static __device__ __forceinline__ void load(const T* p, float* out) {
#pragma unroll
    for (int i = 0; i < V; ++i) out[i] = to_float(p[i]);
  }
  static __device__ __forceinline__ void store(T* p, const float* v) {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = from_float<T>(v[i]);
  }
};
template <> struct RnVec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* out) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct RnVec<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float* out) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    out[0] = __uint_as_float(v.x << 16); out[1] = __uint_as_float(v.x & 0xffff0000u);
    out[2] = __uint_as_float(v.y << 16); out[3] = __uint_as_float(v.y & 0xffff0000u);
  }
  static __device__ __forceinline__ void store(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  }
};

struct ResidualNormParams {
  float* x;
  int W;
  const void* delta;
  int parts;
  size_t part_stride;
  float delta_scale;
  const void* gate;
  size_t gate_stride;
  const float* gate_bias;
  const float* post_w;
  float post_eps;
  void* copy;
  int norm;
  const float* w;
  const float* b;
  float eps;
  void* out;
  const int* rows_idx;
  int total_rows;
  const void* ahead;
  long long ahead_bytes;
};

template <typename TO, typename TD, typename TG, int V, int N>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(const ResidualNormParams p) {
  __shared__ float red[33];
  l2_prefetch_share(p.ahead, p.ahead_bytes);
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, W = p.W, step = blockDim.x * V;
  const int row = p.rows_idx != nullptr ? ck_row(p.rows_idx[blockIdx.x], p.total_rows) : static_cast<int>(blockIdx.x);
  float* xrow = p.x + static_cast<size_t>(row) * W;
  float x[N][V], y[N][V];
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int c = tid * V + n * step;
#pragma unroll
    for (int i = 0; i < V; ++i) x[n][i] = y[n][i] = 0.0f;
    if (c < W) RnVec<float, V>::load(xrow + c, x[n]);
  }
  if (p.delta != nullptr) {
    const TD* delta = static_cast<const TD*>(p.delta) + static_cast<size_t>(row) * W;
    const TG* gate = static_cast<const TG*>(p.gate);
    float ss = 0.0f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = tid * V + n * step;
      if (c < W) {
        for (int k = 0; k < p.parts; ++k) {
          float d[V];
          RnVec<TD, V>::load(delta + k * p.part_stride + c, d);
#pragma unroll
          for (int i = 0; i < V; ++i) y[n][i] += d[i];
        }
        if (gate != nullptr) {
          float g[V], gb[V];
          RnVec<TG, V>::load(gate + static_cast<size_t>(row) * p.gate_stride + c, g);
          if (p.gate_bias != nullptr) {
            RnVec<float, V>::load(p.gate_bias + c, gb);
#pragma unroll
            for (int i = 0; i < V; ++i) g[i] += gb[i];
          }
#pragma unroll
          for (int i = 0; i < V; ++i)            // (16-bit results: the fast exponential and division, relative error below 1e-5)
            y[n][i] *= sizeof(TO) == 2 ? __fdividef(p.delta_scale, 1.0f + __expf(-g[i])) : p.delta_scale / (1.0f + expf(-g[i]));
        } else {
#pragma unroll
          for (int i = 0; i < V; ++i) y[n][i] *= p.delta_scale;
        }
#pragma unroll
        for (int i = 0; i < V; ++i) ss = fmaf(y[n][i], y[n][i], ss);
      }
    }
    float r = 1.0f;
    if (p.post_w != nullptr) r = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + p.post_eps);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = tid * V + n * step;
      if (c < W) {
        if (p.post_w != nullptr) {
          float pw[V];
          RnVec<float, V>::load(p.post_w + c, pw);
#pragma unroll
          for (int i = 0; i < V; ++i) y[n][i] *= r * pw[i];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) x[n][i] += y[n][i];
        if (p.rows_idx == nullptr) RnVec<float, V>::store(xrow + c, x[n]);
      }
    }
  }
  if (p.copy != nullptr) {
    TO* dst = static_cast<TO*>(p.copy) + static_cast<size_t>(blockIdx.x) * W;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = tid * V + n * step;
      if (c < W) RnVec<TO, V>::store(dst + c, x[n]);
    }
  }
  if (p.norm == RN_NORM_NONE) return;
  float mean = 0.0f;
  if (p.norm == RN_NORM_LAYER) {
    float sum = 0.0f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int i = 0; i < V; ++i) sum += x[n][i];          // zeros past the row's end
    mean = block_sum(sum, red) / static_cast<float>(W);
  }
  float sq = 0.0f;
#pragma unroll
  for (int n = 0; n < N; ++n)
    if (tid * V + n * step < W) {
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const float dv = x[n][i] - mean;
        sq = fmaf(dv, dv, sq);
      }
    }
  const float rstd = 1.0f / sqrtf(block_sum(sq, red) / static_cast<float>(W) + p.eps);
  TO* orow = static_cast<TO*>(p.out) + static_cast<size_t>(blockIdx.x) * W;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int c = tid * V + n * step;
    if (c < W) {
      float wv[V], bv[V], v[V];
      RnVec<float, V>::load(p.w + c, wv);
#pragma unroll
      for (int i = 0; i < V; ++i) bv[i] = 0.0f;
      if (p.b != nullptr) RnVec<float, V>::load(p.b + c, bv);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = (x[n][i] - mean) * rstd * wv[i] + bv[i];
      RnVec<TO, V>::store(orow + c, v);
    }
  }
}

template <typename TO, typename TD, typename TG>
int launch_residual_norm(const ResidualNormParams& p, int n_out, bool wide, cudaStream_t stream) {
#define DL_RN(V_, N_, T_) return launch_streaming(residual_norm_kernel<TO, TD, TG, V_, N_>, dim3(n_out), dim3(T_), 0, stream, p)
  if (wide) {                       // pieces of 4 numbers, 1 to 4 of them a thread
    const int pieces = (p.W + 3) / 4;
    if (pieces <= 128) DL_RN(4, 1, 128);
    if (pieces <= 256) DL_RN(4, 2, 128);
    if (pieces <= 512 && n_out >= 512) DL_RN(4, 4, 128);      // many rows: more of a row in flight per thread
    if (pieces <= 512) DL_RN(4, 2, 256);
    if (pieces <= 1024) DL_RN(4, 4, 256);
    if (pieces <= 4096) DL_RN(4, 4, 1024);
    return DL_ERR_UNSUPPORTED;
  }
  if (p.W <= 2048) DL_RN(1, 8, 256);
  if (p.W <= 8192) DL_RN(1, 8, 1024);
#undef DL_RN
  return DL_ERR_UNSUPPORTED;
}

}  // namespace dl

// Types: 0 float32, 1 bfloat16 (a float32 result goes with float32 delta and gate). x: float32 [total_rows, W], updated in place unless rows_idx (n_out row numbers) gathers.
// delta: [parts][total_rows, W], part_stride elements apart, or null; gate: rows of gate_stride elements or null;
// gate_bias, post_w: float32 [W] or null; copy, out: [n_out, W] of out_dtype or null. norm: 0 none, 1 layer, 2 RMS (w, and
// b or null). ahead, ahead_bytes: weights the kernel after this one will stream, asked into L2 before the wait.
DL_EXPORT int dl_residual_norm(int out_dtype, int delta_dtype, int gate_dtype, float* x, int W, const void* delta, int parts,
                               long long part_stride, float delta_scale, const void* gate, long long gate_stride,
                               const float* gate_bias, const float* post_w, float post_eps, void* copy, int norm,
                               const float* w, const float* b, float eps, void* out, const int* rows_idx, int n_out,
                               int total_rows, const void* ahead, long long ahead_bytes, cudaStream_t stream) {
  if (n_out <= 0) return 0;
  if (W <= 0 || (delta != nullptr && parts <= 0) || norm < 0 || norm > 2 || (norm != 0 && (w == nullptr || out == nullptr)))
    return DL_ERR_UNSUPPORTED;
  const bool wide = W % 4 == 0 && part_stride % 4 == 0 && gate_stride % 4 == 0 &&
                    ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate_bias) | reinterpret_cast<uintptr_t>(post_w) |
                      reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(b)) & 15) == 0 &&
                    ((reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(copy) |
                      reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const dl::ResidualNormParams p = {x, W, delta, parts, static_cast<size_t>(part_stride), delta_scale, gate,
                                    static_cast<size_t>(gate_stride), gate_bias, post_w, post_eps, copy, norm, w, b, eps, out,
                                    rows_idx, total_rows, dl::pdl_mode() >= 1 ? ahead : nullptr, dl::pdl_mode() >= 1 ? ahead_bytes : 0ll};
  if (out_dtype == 0 && delta_dtype == 0 && gate_dtype == 0) return dl::launch_residual_norm<float, float, float>(p, n_out, wide, stream);
  if (out_dtype != 1) return DL_ERR_UNSUPPORTED;
  if (delta_dtype == 0 && gate_dtype == 0) return dl::launch_residual_norm<dl::bf16, float, float>(p, n_out, wide, stream);
  if (delta_dtype == 0 && gate_dtype == 1) return dl::launch_residual_norm<dl::bf16, float, dl::bf16>(p, n_out, wide, stream);
  if (delta_dtype == 1 && gate_dtype == 0) return dl::launch_residual_norm<dl::bf16, dl::bf16, float>(p, n_out, wide, stream);
  if (delta_dtype == 1 && gate_dtype == 1) return dl::launch_residual_norm<dl::bf16, dl::bf16, dl::bf16>(p, n_out, wide, stream);
  return DL_ERR_UNSUPPORTED;
}
