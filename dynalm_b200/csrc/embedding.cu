// Token embedding gather: out[i, :] = table[ids[i], :] * scale, written as the fp32 residual stream.
// Reference op: CpuDevice::embedding (dynacore/cpu/cpu_device.cpp:212-219), scale applied as in
// dynalm/src/model/transformer.cpp:576-577.
#include "common.cuh"

namespace dl {

template <typename T>
__global__ void embed_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                             int width, int vocab, float scale) {
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x;
  int id = ck_token(ids[row], vocab);
  // The step function has already refused ids outside [0, vocab); clamping keeps a stray id
  // from reading outside the table.
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + static_cast<size_t>(id) * width;
  float* dst = out + static_cast<size_t>(row) * width;
  constexpr int V = PerVec<T>::n;
  if (width % V == 0) {
    const Vec16* s = reinterpret_cast<const Vec16*>(src);
    for (int i = threadIdx.x; i < width / V; i += blockDim.x) {
      float f[V];
      unpack<T>(s[i], f);
#pragma unroll
      for (int j = 0; j < V; j += 4) {
        float4 o = make_float4(f[j] * scale, f[j + 1] * scale, f[j + 2] * scale, f[j + 3] * scale);
        *reinterpret_cast<float4*>(dst + i * V + j) = o;
      }
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = to_float(src[i]) * scale;
  }
}

// The same with a row of a second table added, chosen by the token and the one in front of it:
//   out[i, :] = table[ids[i], :] * scale + pairs[r, :],  r = (mul_prev * previous + mul_cur * ids[i]) mod pair_rows,
// and r = pair_rows (the table's last row) for a sequence's first token. The token in front of a request's first row of
// the step is the request's last token of earlier steps, kept in state[slot]; the block of that row reads it and then
// leaves the request's newest token there. Block per row.
template <typename T>
__global__ void embed_pairs_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ ids,
                                   const int* __restrict__ positions, const int* __restrict__ row_request,
                                   const int* __restrict__ row_slot, const int* __restrict__ q_start,
                                   int* __restrict__ state, long long state_stride, float* __restrict__ out, int width,
                                   int vocab, float scale, int pair_rows, long long mul_prev, long long mul_cur) {
  const int row = blockIdx.x;
  int id = ck_token(ids[row], vocab);
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const int req = row_request[row];
  const bool first = row == q_start[req];
  int* last = state + static_cast<size_t>(ck_request(row_slot[row])) * state_stride;
  long long r = pair_rows;
  if (positions[row] > 0) {
    int prev = first ? *last : ids[row - 1];
    prev = prev < 0 ? 0 : (prev >= vocab ? vocab - 1 : prev);
    r = (mul_prev * prev + mul_cur * id) % pair_rows;
  }
  __syncthreads();                                        // every thread of the block has read the kept token
  if (first && threadIdx.x == 0) *last = ids[q_start[req + 1] - 1];
  const T* a = table + static_cast<size_t>(id) * width;
  const T* b = pairs + static_cast<size_t>(r) * width;
  float* dst = out + static_cast<size_t>(row) * width;
  constexpr int V = PerVec<T>::n;
  if (width % V == 0) {
    for (int i = threadIdx.x; i < width / V; i += blockDim.x) {
      float f[V], g[V];
      unpack<T>(reinterpret_cast<const Vec16*>(a)[i], f);
      unpack<T>(reinterpret_cast<const Vec16*>(b)[i], g);
#pragma unroll
      for (int j = 0; j < V; j += 4)
        *reinterpret_cast<float4*>(dst + i * V + j) = make_float4(fmaf(f[j], scale, g[j]), fmaf(f[j + 1], scale, g[j + 1]),
                                                                  fmaf(f[j + 2], scale, g[j + 2]), fmaf(f[j + 3], scale, g[j + 3]));
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = fmaf(to_float(a[i]), scale, to_float(b[i]));
  }
}

}  // namespace dl

// dtype: 0 = float32 table, 1 = bfloat16 table.
DL_EXPORT int dl_embed(int dtype, const void* table, const int* ids, float* out, int rows, int width, int vocab,
                       float scale, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int threads = width >= 1024 ? 256 : 128;
  if (dtype == 0) {
    return dl::launch(dl::embed_kernel<float>, dim3(rows), dim3(threads), 0, stream, static_cast<const float*>(table), ids, out, width, vocab, scale);
  } else if (dtype == 1) {
    return dl::launch(dl::embed_kernel<dl::bf16>, dim3(rows), dim3(threads), 0, stream, static_cast<const dl::bf16*>(table), ids, out, width, vocab, scale);
  } else {
    return DL_ERR_UNSUPPORTED;
  }
  return dl::launch_status();
}

// table [vocab, width], pairs [pair_rows + 1, width] of one dtype; state: int32, one word per request slot, state_stride
// apart; the other arrays are the step's.
DL_EXPORT int dl_embed_pairs(int dtype, const void* table, const void* pairs, const int* ids, const int* positions,
                             const int* row_request, const int* row_slot, const int* q_start, int* state,
                             long long state_stride, float* out, int rows, int width, int vocab, float scale, int pair_rows,
                             long long mul_prev, long long mul_cur, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (pair_rows <= 0) return DL_ERR_UNSUPPORTED;
  const int threads = width >= 1024 ? 256 : 128;
#define DL_EP(T)                                                                                                        \
  dl::embed_pairs_kernel<T><<<rows, threads, 0, stream>>>(static_cast<const T*>(table), static_cast<const T*>(pairs), ids, \
                                                          positions, row_request, row_slot, q_start, state, state_stride, \
                                                          out, width, vocab, scale, pair_rows, mul_prev, mul_cur)
  if (dtype == 0) DL_EP(float);
  else if (dtype == 1) DL_EP(dl::bf16);
  else return DL_ERR_UNSUPPORTED;
#undef DL_EP
  return dl::launch_status();
}
