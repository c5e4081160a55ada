// Gated activation: out[t, j] = silu(gu[t, j]) * gu[t, inner + j], gu = [gate | up] side by side.
// silu(x) = x * sigmoid(x) (dynacore/cpu/cpu_device.cpp:117-123; CpuDevice::act_mul :1912-1929).
// The math is fp32 whatever the storage type. Also here: the squared ReLU, the tanh form of GELU and xIELU of an
// ungated feed-forward, and a gated activation with clamped halves.
#include "common.cuh"

namespace dl {

template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gu, T* __restrict__ out, int rows, int inner) {
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  const size_t total = static_cast<size_t>(rows) * inner;
  if (idx >= total) return;
  const size_t t = idx / inner, j = idx % inner;
  const float g = to_float(gu[t * 2 * inner + j]);
  const float u = to_float(gu[t * 2 * inner + inner + j]);
  const float s = g / (1.0f + expf(-g));
  out[idx] = from_float<T>(s * u);
}

// 16 bytes per access; inner is a multiple of the vector length and rows of gu are 16-byte aligned.
template <typename T>
__global__ void silu_mul_vec_kernel(const T* __restrict__ gu, T* __restrict__ out, int rows, int inner) {
  constexpr int V = PerVec<T>::n;
  const int per_row = inner / V;
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= static_cast<size_t>(rows) * per_row) return;
  const size_t t = idx / per_row, c = (idx % per_row) * V;
  float g[V], u[V], o[V];
  unpack<T>(*reinterpret_cast<const Vec16*>(gu + t * 2 * inner + c), g);
  unpack<T>(*reinterpret_cast<const Vec16*>(gu + t * 2 * inner + inner + c), u);
#pragma unroll
  for (int j = 0; j < V; ++j) o[j] = g[j] / (1.0f + expf(-g[j])) * u[j];
  *reinterpret_cast<Vec16*>(out + t * inner + c) = pack<T>(o);
}

// Squared ReLU: out[i] = max(x[i], 0)^2, the activation of an ungated feed-forward.
template <typename T>
__global__ void relu2_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = fmaxf(to_float(x[i]), 0.0f);
  out[i] = from_float<T>(v * v);
}

// 16 bytes per access; n counts vectors.
template <typename T>
__global__ void relu2_vec_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n) {
  constexpr int V = PerVec<T>::n;
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float f[V];
  unpack<T>(reinterpret_cast<const Vec16*>(x)[i], f);
#pragma unroll
  for (int j = 0; j < V; ++j) {
    f[j] = fmaxf(f[j], 0.0f);
    f[j] *= f[j];
  }
  reinterpret_cast<Vec16*>(out)[i] = pack<T>(f);
}

// GELU in its tanh form: 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), the activation of an ungated feed-forward.
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void gelu_tanh_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  out[i] = from_float<T>(gelu_tanh_f(to_float(x[i])));
}

// 16 bytes per access; n counts vectors.
template <typename T>
__global__ void gelu_tanh_vec_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n) {
  constexpr int V = PerVec<T>::n;
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float f[V];
  unpack<T>(reinterpret_cast<const Vec16*>(x)[i], f);
#pragma unroll
  for (int j = 0; j < V; ++j) f[j] = gelu_tanh_f(f[j]);
  reinterpret_cast<Vec16*>(out)[i] = pack<T>(f);
}

// xIELU with coefficients c = (c0, c1) from memory: c0 z^2 + z / 2 above zero, c1 (e^z - 1 - z) + z / 2 at and below it.
template <typename T>
__global__ void xielu_kernel(const T* __restrict__ x, T* __restrict__ out, const float* __restrict__ c, size_t n) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  out[i] = from_float<T>(xielu_f(to_float(x[i]), c[0], c[1]));
}

// 16 bytes per access; n counts vectors.
template <typename T>
__global__ void xielu_vec_kernel(const T* __restrict__ x, T* __restrict__ out, const float* __restrict__ c, size_t n) {
  constexpr int V = PerVec<T>::n;
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float c0 = c[0], c1 = c[1];
  float f[V];
  unpack<T>(reinterpret_cast<const Vec16*>(x)[i], f);
#pragma unroll
  for (int j = 0; j < V; ++j) f[j] = xielu_f(f[j], c0, c1);
  reinterpret_cast<Vec16*>(out)[i] = pack<T>(f);
}

// A gated activation whose halves are clamped: with g = min(gate + bias, limit), u = clamp(up + bias, -limit, limit),
// g sigmoid(gate_scale g) (u + 1). coeffs: as common.cuh says at CLAMPED_HEADER.
template <typename T, int V>
__global__ void clamped_swiglu_kernel(const T* __restrict__ gu, const float* __restrict__ coeffs, T* __restrict__ out, int rows,
                                      int inner) {
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int per = inner / V;
  if (idx >= static_cast<size_t>(rows) * per) return;
  const size_t t = idx / per;
  const int j = static_cast<int>(idx % per) * V;
  const T* row = gu + t * 2 * inner + j;
  const float* bias = coeffs + CLAMPED_HEADER;
  float g[V], u[V];
  if constexpr (V > 1) {
    unpack<T>(*reinterpret_cast<const Vec16*>(row), g);
    unpack<T>(*reinterpret_cast<const Vec16*>(row + inner), u);
  } else {
    g[0] = to_float(row[0]);
    u[0] = to_float(row[inner]);
  }
#pragma unroll
  for (int k = 0; k < V; ++k) {
    g[k] = clamped_swiglu_f(g[k] + bias[j + k], u[k] + bias[inner + j + k], coeffs[0], coeffs[1]);
  }
  if constexpr (V > 1) *reinterpret_cast<Vec16*>(out + t * inner + j) = pack<T>(g);
  else out[t * inner + j] = from_float<T>(g[0]);
}

}  // namespace dl

// out[i] = xIELU(x[i]) over n contiguous elements (out may be x); coeffs: two float32 on the device.
DL_EXPORT int dl_xielu(int dtype, const void* x, void* out, const float* coeffs, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if ((dtype != 0 && dtype != 1) || coeffs == nullptr) return DL_ERR_UNSUPPORTED;
  const int vec = dtype == 0 ? 4 : 8;
  const bool wide = n % vec == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0;
  const size_t count = static_cast<size_t>(wide ? n / vec : n);
  const unsigned blocks = static_cast<unsigned>((count + 255) / 256);
#define DL_XI(K, T) dl::K<T><<<blocks, 256, 0, stream>>>(static_cast<const T*>(x), static_cast<T*>(out), coeffs, count)
  if (dtype == 0) { if (wide) DL_XI(xielu_vec_kernel, float); else DL_XI(xielu_kernel, float); }
  else { if (wide) DL_XI(xielu_vec_kernel, dl::bf16); else DL_XI(xielu_kernel, dl::bf16); }
#undef DL_XI
  return dl::launch_status();
}

// out[i] = gelu_tanh(x[i]) over n contiguous elements (out may be x).
DL_EXPORT int dl_gelu_tanh(int dtype, const void* x, void* out, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dtype != 0 && dtype != 1) return DL_ERR_UNSUPPORTED;
  const int threads = 256;
  const int vec = dtype == 0 ? 4 : 8;
  if (n % vec == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
    const size_t nv = static_cast<size_t>(n / vec);
    const unsigned blocks = static_cast<unsigned>((nv + threads - 1) / threads);
    if (dtype == 0) dl::gelu_tanh_vec_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(x), static_cast<float*>(out), nv);
    else dl::gelu_tanh_vec_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(x), static_cast<dl::bf16*>(out), nv);
    return dl::launch_status();
  }
  const unsigned blocks = static_cast<unsigned>((static_cast<size_t>(n) + threads - 1) / threads);
  if (dtype == 0) dl::gelu_tanh_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(x), static_cast<float*>(out), static_cast<size_t>(n));
  else dl::gelu_tanh_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(x), static_cast<dl::bf16*>(out), static_cast<size_t>(n));
  return dl::launch_status();
}

// out[i] = max(x[i], 0)^2 over n contiguous elements (out may be x).
DL_EXPORT int dl_relu2(int dtype, const void* x, void* out, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dtype != 0 && dtype != 1) return DL_ERR_UNSUPPORTED;
  const int threads = 256;
  const int vec = dtype == 0 ? 4 : 8;
  if (n % vec == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
    const size_t nv = static_cast<size_t>(n / vec);
    const unsigned blocks = static_cast<unsigned>((nv + threads - 1) / threads);
    if (dtype == 0) dl::relu2_vec_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(x), static_cast<float*>(out), nv);
    else dl::relu2_vec_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(x), static_cast<dl::bf16*>(out), nv);
    return dl::launch_status();
  }
  const unsigned blocks = static_cast<unsigned>((static_cast<size_t>(n) + threads - 1) / threads);
  if (dtype == 0) dl::relu2_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(x), static_cast<float*>(out), static_cast<size_t>(n));
  else dl::relu2_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(x), static_cast<dl::bf16*>(out), static_cast<size_t>(n));
  return dl::launch_status();
}

DL_EXPORT int dl_silu_mul(int dtype, const void* gu, void* out, int rows, int inner, cudaStream_t stream) {
  if (rows <= 0 || inner <= 0) return 0;
  const int threads = 256;
  const int vec = dtype == 0 ? 4 : 8;
  if ((dtype == 0 || dtype == 1) && inner % vec == 0 && (reinterpret_cast<uintptr_t>(gu) & 15) == 0 &&
      (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
    const size_t n = static_cast<size_t>(rows) * (inner / vec);
    const unsigned blocks = static_cast<unsigned>((n + threads - 1) / threads);
    if (dtype == 0) dl::silu_mul_vec_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(gu), static_cast<float*>(out), rows, inner);
    else dl::silu_mul_vec_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(gu), static_cast<dl::bf16*>(out), rows, inner);
    return dl::launch_status();
  }
  const size_t total = static_cast<size_t>(rows) * inner;
  const unsigned blocks = static_cast<unsigned>((total + threads - 1) / threads);
  if (dtype == 0) dl::silu_mul_kernel<float><<<blocks, threads, 0, stream>>>(static_cast<const float*>(gu), static_cast<float*>(out), rows, inner);
  else if (dtype == 1) dl::silu_mul_kernel<dl::bf16><<<blocks, threads, 0, stream>>>(static_cast<const dl::bf16*>(gu), static_cast<dl::bf16*>(out), rows, inner);
  else return DL_ERR_UNSUPPORTED;
  return dl::launch_status();
}

// gu: contiguous [rows, 2 * inner] = [gate | up]; coeffs: float32 [4 + 2 * inner]; out: contiguous [rows, inner].
DL_EXPORT int dl_clamped_swiglu(int dtype, const void* gu, const float* coeffs, void* out, int rows, int inner,
                                cudaStream_t stream) {
  if (rows <= 0 || inner <= 0) return 0;
  if ((dtype != 0 && dtype != 1) || coeffs == nullptr) return DL_ERR_UNSUPPORTED;
  const int vec = dtype == 0 ? 4 : 8;
  const bool wide = inner % vec == 0 && ((reinterpret_cast<uintptr_t>(gu) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const size_t n = static_cast<size_t>(rows) * (wide ? inner / vec : inner);
  const unsigned blocks = static_cast<unsigned>((n + 255) / 256);
#define DL_CS(T, V)                                                                                                     \
  dl::clamped_swiglu_kernel<T, V><<<blocks, 256, 0, stream>>>(static_cast<const T*>(gu), coeffs, static_cast<T*>(out), rows, inner)
  if (dtype == 0) { if (wide) DL_CS(float, 4); else DL_CS(float, 1); }
  else { if (wide) DL_CS(dl::bf16, 8); else DL_CS(dl::bf16, 1); }
#undef DL_CS
  return dl::launch_status();
}
