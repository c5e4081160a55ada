// Paged causal attention, one thread block per (query row, head): the plain kernel.
//
// It serves the true 32-bit path and every shape the faster kernels refuse. A row at position
// `pos` of request r reads keys t in [lo, pos], lo = window > 0 ? max(0, pos - window + 1) : 0, and the keys
// t < keep_first behind them (or, in chunks, the keys from pos / chunk * chunk on), through block_table[r]; with `sink` the softmax's denominator holds one more term exp(0); query head h reads KV head h / (heads / kv_heads).
// With (rate, step) per head a distance bias comes off the scores: s_t = scale * q.k_t - rate_h ln(1 + step_h (pos - t)).
//   s_t = scale * q.k_t;  out = sum_t exp(s_t - max) v_t / sum_t exp(s_t - max)
// (dynacore/cpu/cpu_device.cpp:1309-1412,1717-1776). Keys are visited in chunks whose boundaries
// are multiples of CHUNK in absolute position, merged by the running (max, sum, acc) rule of the
// reference's split-K variant (:1782-1845). What a row computes therefore depends only on its own
// query, position and keys: not on the other rows of the batch nor on how the prompt was cut.
// Scores, softmax and the weighted sum are fp32.
#include "common.cuh"

namespace dl {

constexpr int ATT_THREADS = 256;
constexpr int ATT_CHUNK = 512;

template <typename T>
__global__ void __launch_bounds__(ATT_THREADS)
paged_attention_generic_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k_cache,
                               const T* __restrict__ v_cache, const int* __restrict__ block_table,
                               int max_blocks, const int* __restrict__ positions,
                               const int* __restrict__ row_request, T* __restrict__ out, int out_stride,
                               int n_heads, int n_kv_heads, int head_dim, int page_size, float scale,
                               int window, int vdim, size_t k_row, size_t v_row, int wide, int keep_first,
                               int sink, const float* __restrict__ rate, const float* __restrict__ dstep, int chunk) {
  __shared__ float red[33];
  __shared__ float sq[256];                 // the query, fp32
  __shared__ float sp[ATT_CHUNK];           // scores, then probabilities, of one chunk
  __shared__ float part[ATT_THREADS];       // partial weighted sums, [group][dim]
  const int row = blockIdx.x, head = blockIdx.y;
  const int kvh = head / (n_heads / n_kv_heads);
  const int pos = positions[row];
  const int lo = chunk > 0 ? pos / chunk * chunk : (window > 0 ? max(0, pos - window + 1) : 0);
  const int* table = block_table + static_cast<size_t>(ck_request(row_request[row])) * max_blocks;
  const int tid = threadIdx.x;

  const T* qrow = q + static_cast<size_t>(row) * q_stride + static_cast<size_t>(head) * head_dim;
  for (int d = tid; d < head_dim; d += ATT_THREADS) sq[d] = to_float(qrow[d]);
  __syncthreads();

  constexpr int V = PerVec<T>::n;
  const int groups = ATT_THREADS / vdim;              // >= 1 since vdim <= 256
  const int g = tid / vdim, d = tid % vdim;           // valid when g < groups

  float m_run = -INFINITY, l_run = 0.0f, acc = 0.0f;  // acc: dim `tid` of the output, threads < head_dim
  // keys below `keep_first` stay visible behind the window; chunks that hold no visible key are passed over
  const int kept = lo > 0 ? min(keep_first, lo) : 0;
  for (int c0 = kept > 0 ? 0 : (lo / ATT_CHUNK) * ATT_CHUNK; c0 <= pos; c0 += ATT_CHUNK) {
    if (c0 + ATT_CHUNK <= lo && c0 >= kept) continue;
    const int c1 = min(c0 + ATT_CHUNK, pos + 1);
    float m_loc = -INFINITY;
    for (int t = c0 + tid; t < c1; t += ATT_THREADS) {
      float s = -INFINITY;
      if (t >= lo || t < kept) {
        const size_t slot = static_cast<size_t>(ck_page(table, t / page_size, max_blocks)) * page_size + t % page_size;
        const T* kp = k_cache + slot * k_row + static_cast<size_t>(kvh) * head_dim;
        float dot = 0.0f;
        if (wide) {                                     // every key starts on a 16-byte boundary
          const Vec16* kr = reinterpret_cast<const Vec16*>(kp);
          for (int i = 0; i < head_dim / V; ++i) {
            float f[V];
            unpack<T>(kr[i], f);
#pragma unroll
            for (int j = 0; j < V; ++j) dot = fmaf(sq[i * V + j], f[j], dot);
          }
        } else {                                        // the same sum in the same order, number by number
          for (int i = 0; i < head_dim; ++i) dot = fmaf(sq[i], to_float(kp[i]), dot);
        }
        s = dot * scale;
        if (rate != nullptr) s -= rate[head] * logf(1.0f + dstep[head] * static_cast<float>(pos - t));
      }
      sp[t - c0] = s;
      m_loc = fmaxf(m_loc, s);
    }
    const float m_chunk = block_max(m_loc, red);
    const float m_new = fmaxf(m_run, m_chunk);          // finite: the chunk holds at least key max(lo, c0)
    float l_loc = 0.0f;
    for (int t = c0 + tid; t < c1; t += ATT_THREADS) {
      const float p = expf(sp[t - c0] - m_new);         // exp(-inf) = 0 for keys before lo
      sp[t - c0] = p;
      l_loc += p;
    }
    const float l_chunk = block_sum(l_loc, red);        // also orders the writes of sp before the reads below
    const float corr = expf(m_run - m_new);             // 0 on the first chunk
    l_run = l_run * corr + l_chunk;
    m_run = m_new;

    float pv = 0.0f;
    if (g < groups) {
      for (int t = c0 + g; t < c1; t += groups) {
        if (t < lo && t >= kept) continue;
        const size_t slot = static_cast<size_t>(ck_page(table, t / page_size, max_blocks)) * page_size + t % page_size;
        pv = fmaf(sp[t - c0], to_float(v_cache[slot * v_row + static_cast<size_t>(kvh) * vdim + d]), pv);
      }
    }
    part[tid] = pv;
    __syncthreads();
    if (tid < vdim) {
      float sum = 0.0f;
      for (int gg = 0; gg < groups; ++gg) sum += part[gg * vdim + tid];
      acc = acc * corr + sum;
    }
    __syncthreads();
  }
  if (sink) {                                            // one more term of score 0 in the denominator; it carries no value
    const float m_fin = fmaxf(m_run, 0.0f);
    const float corr = expf(m_run - m_fin);
    l_run = l_run * corr + expf(-m_fin);
    acc *= corr;
  }
  if (tid < vdim) {
    T* orow = out + static_cast<size_t>(row) * out_stride + static_cast<size_t>(head) * vdim;
    orow[tid] = from_float<T>(acc / l_run);
  }
}

}  // namespace dl

// q: rows of `q_stride` elements with head h at column h * head_dim; out: rows of out_stride elements with head h at
// column h * vdim. Keys of a token lie k_row elements apart from the next token's in k_cache (KV head j at j * head_dim),
// values v_row elements apart in v_cache (KV head j at j * vdim): two arrays [pages, page_size, n_kv_heads, size], or
// one array of records [k | v] given twice with two offsets. head_dim and vdim: 1 to 256; keys that all start on a
// 16-byte boundary are read 16 bytes at a time. chunk > 0 (without a window): a position sees its own chunk alone. rate, dstep: float32 [n_heads] of the distance bias, or both null.
DL_EXPORT int dl_paged_attention_generic_masked(int dtype, const void* q, int q_stride, const void* k_cache, long long k_row,
                                                const void* v_cache, long long v_row, const int* block_table, int max_blocks,
                                                const int* positions, const int* row_request, void* out, int out_stride,
                                                int rows, int n_heads, int n_kv_heads, int head_dim, int vdim, int page_size,
                                                float scale, int window, int keep_first, int sink, const float* rate,
                                                const float* dstep, int chunk, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (head_dim > 256 || head_dim <= 0 || vdim <= 0 || vdim > 256 || n_kv_heads <= 0 || n_heads % n_kv_heads != 0 ||
      page_size <= 0 || n_heads > 65535 || (dtype != 0 && dtype != 1) || keep_first < 0 || (rate != nullptr) != (dstep != nullptr) ||
      chunk < 0 || (chunk > 0 && (window > 0 || keep_first > 0)))
    return DL_ERR_UNSUPPORTED;
  const int per = dtype == 0 ? 4 : 8;           // numbers in 16 bytes
  const int wide = head_dim % per == 0 && k_row % per == 0 && (reinterpret_cast<uintptr_t>(k_cache) & 15) == 0;
  dim3 grid(rows, n_heads);
#define DL_LAUNCH(T)                                                                                          \
  dl::paged_attention_generic_kernel<T><<<grid, dl::ATT_THREADS, 0, stream>>>(                                 \
      static_cast<const T*>(q), q_stride, static_cast<const T*>(k_cache), static_cast<const T*>(v_cache),     \
      block_table, max_blocks, positions, row_request, static_cast<T*>(out), out_stride, n_heads, n_kv_heads, \
      head_dim, page_size, scale, window, vdim, static_cast<size_t>(k_row), static_cast<size_t>(v_row), wide,    \
      keep_first, sink, rate, dstep, chunk)
  if (dtype == 0) DL_LAUNCH(float);
  else if (dtype == 1) DL_LAUNCH(dl::bf16);
  else return DL_ERR_UNSUPPORTED;
#undef DL_LAUNCH
  return dl::launch_status();
}

// The same with a plain window and an ordinary softmax.
DL_EXPORT int dl_paged_attention_generic_kv(int dtype, const void* q, int q_stride, const void* k_cache, long long k_row,
                                            const void* v_cache, long long v_row, const int* block_table, int max_blocks,
                                            const int* positions, const int* row_request, void* out, int out_stride,
                                            int rows, int n_heads, int n_kv_heads, int head_dim, int vdim, int page_size,
                                            float scale, int window, cudaStream_t stream) {
  return dl_paged_attention_generic_masked(dtype, q, q_stride, k_cache, k_row, v_cache, v_row, block_table, max_blocks,
                                           positions, row_request, out, out_stride, rows, n_heads, n_kv_heads, head_dim, vdim,
                                           page_size, scale, window, 0, 0, nullptr, nullptr, 0, stream);
}

// The same for keys and values of one size in two arrays [pages, page_size, n_kv_heads, head_dim].
DL_EXPORT int dl_paged_attention_generic(int dtype, const void* q, int q_stride, const void* k_cache,
                                         const void* v_cache, const int* block_table, int max_blocks,
                                         const int* positions, const int* row_request, void* out,
                                         int out_stride, int rows, int n_heads, int n_kv_heads, int head_dim,
                                         int page_size, float scale, int window, cudaStream_t stream) {
  const long long kv_row = static_cast<long long>(n_kv_heads) * head_dim;
  return dl_paged_attention_generic_kv(dtype, q, q_stride, k_cache, kv_row, v_cache, kv_row, block_table, max_blocks,
                                       positions, row_request, out, out_stride, rows, n_heads, n_kv_heads, head_dim,
                                       head_dim, page_size, scale, window, stream);
}
