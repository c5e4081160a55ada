// The closing norm of a sublayer whose result is normed before it joins the stream, fused with the sum and with the
// opening norm of the sublayer that follows:
//
//   x   <- x + rmsnorm(delta) * w_post            rmsnorm(v) = v / sqrt(mean(v^2) + eps)
//   out  = rmsnorm(x) * w_pre                     (left out when w_pre is null)
//
// x is the float32 stream, updated in place; delta is the sublayer's result, [n, width] of either type or split-K
// partial sums [parts, n, width] that are added in order. One block per row; the row waits in shared memory between
// the two passes. Everything is float32.
//
// Also here: the normed sum of two results side by side (dl_normed_sum),
//
//   out = sa * rmsnorm(a) * wa + sb * rmsnorm(b) * wb
//
// one block per row, both rows in registers between the passes.
#include "common.cuh"

namespace dl {

template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
norm_add_norm_kernel(float* __restrict__ x, const TD* __restrict__ delta, int parts, size_t part_stride,
                     const float* __restrict__ w_post, float eps_post, const float* __restrict__ w_pre, float eps_pre,
                     TO* __restrict__ out, int width) {
  extern __shared__ float row_s[];
  __shared__ float red[33];
  const size_t base = static_cast<size_t>(blockIdx.x) * width;
  float ss = 0.0f;
  for (int j = threadIdx.x; j < width; j += blockDim.x) {
    float d = 0.0f;
    for (int p = 0; p < parts; ++p) d += to_float(delta[p * part_stride + base + j]);
    row_s[j] = d;
    ss = fmaf(d, d, ss);
  }
  const float rs = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(width) + eps_post);
  float ss2 = 0.0f;
  for (int j = threadIdx.x; j < width; j += blockDim.x) {
    const float v = x[base + j] + row_s[j] * rs * w_post[j];
    x[base + j] = v;
    row_s[j] = v;
    ss2 = fmaf(v, v, ss2);
  }
  if (w_pre == nullptr) return;
  const float rs2 = 1.0f / sqrtf(block_sum(ss2, red) / static_cast<float>(width) + eps_pre);
  for (int j = threadIdx.x; j < width; j += blockDim.x) out[base + j] = from_float<TO>(row_s[j] * rs2 * w_pre[j]);
}

// V numbers at a time (4 where rows and bases allow it), at most N pieces a thread.
template <typename T, int V>
__device__ __forceinline__ void ns_add(const T* __restrict__ p, float* acc) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    acc[0] += v.x; acc[1] += v.y; acc[2] += v.z; acc[3] += v.w;
  } else if constexpr (V == 4) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    acc[0] += __uint_as_float(v.x << 16); acc[1] += __uint_as_float(v.x & 0xffff0000u);
    acc[2] += __uint_as_float(v.y << 16); acc[3] += __uint_as_float(v.y & 0xffff0000u);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] += to_float(p[i]);
  }
}

template <typename TA, typename TB, int V, int N>
__global__ void __launch_bounds__(1024)
normed_sum_kernel(const TA* __restrict__ a, int parts_a, size_t stride_a, const float* __restrict__ wa, float sa,
                  const TB* __restrict__ b, int parts_b, size_t stride_b, const float* __restrict__ wb, float sb, float eps,
                  float* __restrict__ out, int width) {
  __shared__ float red[66];
  const size_t base = static_cast<size_t>(blockIdx.x) * width;
  const int step = blockDim.x * V;
  float x[N][V], y[N][V], ss = 0.0f, tt = 0.0f;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int c = threadIdx.x * V + n * step;
#pragma unroll
    for (int i = 0; i < V; ++i) x[n][i] = y[n][i] = 0.0f;
    if (c < width) {
      for (int p = 0; p < parts_a; ++p) ns_add<TA, V>(a + p * stride_a + base + c, x[n]);
      for (int p = 0; p < parts_b; ++p) ns_add<TB, V>(b + p * stride_b + base + c, y[n]);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        ss = fmaf(x[n][i], x[n][i], ss);
        tt = fmaf(y[n][i], y[n][i], tt);
      }
    }
  }
  // both sums in one round
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  ss = warp_sum(ss);
  tt = warp_sum(tt);
  if (lane == 0) { red[warp] = ss; red[33 + warp] = tt; }
  __syncthreads();
  ss = warp_sum(lane < warps ? red[lane] : 0.0f);
  tt = warp_sum(lane < warps ? red[33 + lane] : 0.0f);
  const float ra = sa / sqrtf(ss / static_cast<float>(width) + eps), rb = sb / sqrtf(tt / static_cast<float>(width) + eps);
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int c = threadIdx.x * V + n * step;
    if (c < width) {
      float va[V], vb[V];
#pragma unroll
      for (int i = 0; i < V; ++i) va[i] = vb[i] = 0.0f;
      ns_add<float, V>(wa + c, va);
      ns_add<float, V>(wb + c, vb);
#pragma unroll
      for (int i = 0; i < V; ++i) x[n][i] = x[n][i] * ra * va[i] + y[n][i] * rb * vb[i];
      if constexpr (V == 4) {
        *reinterpret_cast<float4*>(out + base + c) = make_float4(x[n][0], x[n][1], x[n][2], x[n][3]);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) out[base + c + i] = x[n][i];
      }
    }
  }
}

template <typename TA, typename TB>
int launch_normed_sum(const void* a, int parts_a, size_t stride_a, const float* wa, float sa, const void* b, int parts_b,
                      size_t stride_b, const float* wb, float sb, float eps, float* out, int rows, int width, bool wide,
                      cudaStream_t stream) {
#define DL_NS(V_, N_, T_)                                                                                               \
  do {                                                                                                                  \
    normed_sum_kernel<TA, TB, V_, N_><<<rows, T_, 0, stream>>>(static_cast<const TA*>(a), parts_a, stride_a, wa, sa,    \
                                                               static_cast<const TB*>(b), parts_b, stride_b, wb, sb,    \
                                                               eps, out, width);                                        \
    return launch_status();                                                                                             \
  } while (0)
  if (wide) {
    const int pieces = width / 4;
    if (pieces <= 128) DL_NS(4, 1, 128);
    if (pieces <= 256) DL_NS(4, 1, 256);
    if (pieces <= 512) DL_NS(4, 2, 256);
    if (pieces <= 1024) DL_NS(4, 4, 256);
    if (pieces <= 4096) DL_NS(4, 4, 1024);
    return DL_ERR_UNSUPPORTED;
  }
  if (width <= 2048) DL_NS(1, 8, 256);
  if (width <= 8192) DL_NS(1, 8, 1024);
#undef DL_NS
  return DL_ERR_UNSUPPORTED;
}

}  // namespace dl

// out_dtype / delta_dtype: 0 float32, 1 bfloat16. w_pre and out may be null (no opening norm behind the sum).
DL_EXPORT int dl_norm_add_norm(int out_dtype, int delta_dtype, float* x, const void* delta, int parts, long long part_stride,
                               const float* w_post, float eps_post, const float* w_pre, float eps_pre, void* out, int rows,
                               int width, cudaStream_t stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (parts < 1 || width > 12000 || (out_dtype != 0 && out_dtype != 1) || (delta_dtype != 0 && delta_dtype != 1))
    return DL_ERR_UNSUPPORTED;
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
#define DL_NAN(TD, TO)                                                                                                 \
  dl::norm_add_norm_kernel<TD, TO><<<rows, 256, smem, stream>>>(x, static_cast<const TD*>(delta), parts,               \
                                                                static_cast<size_t>(part_stride), w_post, eps_post,    \
                                                                w_pre, eps_pre, static_cast<TO*>(out), width)
  if (delta_dtype == 0 && out_dtype == 0) DL_NAN(float, float);
  else if (delta_dtype == 0) DL_NAN(float, dl::bf16);
  else if (out_dtype == 0) DL_NAN(dl::bf16, float);
  else DL_NAN(dl::bf16, dl::bf16);
#undef DL_NAN
  return dl::launch_status();
}

// a, b: [parts, rows, width] with `stride` elements between parts, each float32 (0) or bfloat16 (1); wa, wb: float32 [width];
// out: float32 [rows, width].
DL_EXPORT int dl_normed_sum(int dtype_a, const void* a, int parts_a, long long stride_a, const float* wa, float sa, int dtype_b,
                            const void* b, int parts_b, long long stride_b, const float* wb, float sb, float eps, float* out,
                            int rows, int width, cudaStream_t stream) {
  if (rows <= 0 || width <= 0) return 0;
  if ((dtype_a != 0 && dtype_a != 1) || (dtype_b != 0 && dtype_b != 1) || parts_a < 1 || parts_b < 1) return DL_ERR_UNSUPPORTED;
  const bool wide = width % 4 == 0 && stride_a % 4 == 0 && stride_b % 4 == 0 &&
                    ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(out) |
                      reinterpret_cast<uintptr_t>(wa) | reinterpret_cast<uintptr_t>(wb)) & 15) == 0;
  const size_t pa = static_cast<size_t>(stride_a), pb = static_cast<size_t>(stride_b);
#define DL_NS(TA, TB) return dl::launch_normed_sum<TA, TB>(a, parts_a, pa, wa, sa, b, parts_b, pb, wb, sb, eps, out, rows, width, wide, stream)
  if (dtype_a == 0 && dtype_b == 0) DL_NS(float, float);
  if (dtype_a == 0) DL_NS(float, dl::bf16);
  if (dtype_b == 0) DL_NS(dl::bf16, float);
  DL_NS(dl::bf16, dl::bf16);
#undef DL_NS
}
