// Short causal convolutions over a projection's queries, keys and values, keys and values straight into the cache.
//
// A row of the projection holds [q: C_q | k: C_k | v: C_v | ...] (C_k = C_v = 0 for a layer that makes queries only). Per
// channel, with K taps (the last one the current token's) and an optional bias that every input inside the sequence
// carries:  y_t = sum_j taps[j] (u_(t - K + 1 + j) + bias), zeros before the sequence's start. Without taps y = u + bias.
// q goes to an array of its own, k and v to the token's place in the request's pages.
//
// The K - 1 inputs in front of a request's first row of the step come from its kept inputs (float32, without the bias,
// oldest first, one row of a state array per request). A request that brings ONE token has its kept inputs shifted by the
// thread that has just read them; the others are brought up to date by a second kernel (dl_conv_keep_many), since their
// first and last rows belong to different threads.
#include "common.cuh"

namespace dl {

struct ConvCacheParams {
  const void* proj;
  size_t proj_stride;
  int Cq, Ck, Cv, K;
  const float* taps;        // [K][Cq + Ck + Cv] or null
  const float* bias;        // [Cq + Ck + Cv] or null
  float* kept;              // [slots] rows of kept_stride, (K - 1) x (Cq + Ck + Cv)
  size_t kept_stride;
  const int* positions;
  const int* row_request;
  const int* row_slot;
  const int* q_start;
  const int* block_table;
  int max_blocks, page_size;
  void* q_out;
  size_t q_stride;
  void* k_cache;
  size_t k_row;
  void* v_cache;
  size_t v_row;
  int rows;
};

template <typename T, int V>
__device__ __forceinline__ void cc_load(const T* p, float* v) {
  if constexpr (V == 1) {
    v[0] = to_float(p[0]);
  } else if constexpr (V * sizeof(T) == 8) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(w.x << 16); v[1] = __uint_as_float(w.x & 0xffff0000u);
    v[2] = __uint_as_float(w.y << 16); v[3] = __uint_as_float(w.y & 0xffff0000u);
  } else unpack<T>(*reinterpret_cast<const Vec16*>(p), v);
}
template <typename T, int V>
__device__ __forceinline__ void cc_store(T* p, const float* v) {
  if constexpr (V == 1) {
    p[0] = from_float<T>(v[0]);
  } else if constexpr (V * sizeof(T) == 8) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  } else *reinterpret_cast<Vec16*>(p) = pack<T>(v);
}

// A thread takes V neighbouring channels of R consecutive rows.
template <typename T, int V, int R>
__global__ void __launch_bounds__(256)
conv_cache_kernel(const ConvCacheParams p) {
  const int C = p.Cq + p.Ck + p.Cv, per_row = C / V, K = p.K;
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int row0 = static_cast<int>(idx / per_row) * R, ch = static_cast<int>(idx % per_row) * V;
  if (row0 >= p.rows) return;
  const T* col = static_cast<const T*>(p.proj) + ch;
  float ib[V];
#pragma unroll
  for (int i = 0; i < V; ++i) ib[i] = p.bias != nullptr ? p.bias[ch + i] : 0.0f;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int row = row0 + r;
    if (row >= p.rows) return;
    const int pos = p.positions[row];
    const int slot = ck_request(p.row_slot[row]);
    float acc[V];
    if (p.taps == nullptr) {
      cc_load<T, V>(col + static_cast<size_t>(row) * p.proj_stride, acc);
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] += ib[i];
    } else {
      const int req = p.row_request[row];
      const int first_row = p.q_start[req];
      float* kept = p.kept + static_cast<size_t>(slot) * p.kept_stride + ch;
      const bool single = p.q_start[req + 1] - first_row == 1;
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = 0.0f;
      for (int k = K - 1; k >= 0; --k) {                             // oldest input first
        if (pos - k < 0) {                                           // in front of the sequence's start
          if (single && k < K - 1) {                                 // (kept entries there stay zero)
#pragma unroll
            for (int i = 0; i < V; ++i) kept[static_cast<size_t>(K - 2 - k) * C + i] = 0.0f;
          }
          continue;
        }
        float u[V];
        const int back = row - k;
        if (back >= first_row) {
          cc_load<T, V>(col + static_cast<size_t>(back) * p.proj_stride, u);
        } else {
          const float* kr = kept + static_cast<size_t>(K - 1 - (first_row - back)) * C;
#pragma unroll
          for (int i = 0; i < V; ++i) u[i] = kr[i];
        }
        // a single token's kept inputs move up by one: entry j (k = K - 1 - j) becomes entry j - 1, the token the last
        if (single && k < K - 1) {
#pragma unroll
          for (int i = 0; i < V; ++i) kept[static_cast<size_t>(K - 2 - k) * C + i] = u[i];
        }
        const float* tk = p.taps + static_cast<size_t>(K - 1 - k) * C + ch;
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(tk[i], u[i] + ib[i], acc[i]);
      }
    }
    if (ch < p.Cq) {
      cc_store<T, V>(static_cast<T*>(p.q_out) + static_cast<size_t>(row) * p.q_stride + ch, acc);
    } else {
      const int* table = p.block_table + static_cast<size_t>(slot) * p.max_blocks;
      const int page = ck_page_store(table, pos / p.page_size, p.max_blocks);
      if (page >= 0) {
        const size_t place = static_cast<size_t>(page) * p.page_size + pos % p.page_size;
        if (ch < p.Cq + p.Ck) cc_store<T, V>(static_cast<T*>(p.k_cache) + place * p.k_row + (ch - p.Cq), acc);
        else cc_store<T, V>(static_cast<T*>(p.v_cache) + place * p.v_row + (ch - p.Cq - p.Ck), acc);
      }
    }
  }
}

// The same for steps of many rows, bfloat16: a thread walks R consecutive rows of V = 4 channels with its taps and the last K - 1 inputs
// (bias included, zeros in front of a start) in registers, so that a row is read once; where a request begins among the
// rows the inputs come from what it kept. Rows of requests of one token shift their kept inputs as above.
template <typename T, int V, int R, int K>
__global__ void __launch_bounds__(256)
conv_cache_rows_kernel(const ConvCacheParams p) {
  static_assert(V == 4 && sizeof(T) == 2, "8 bytes a row and thread");
  const int C = p.Cq + p.Ck + p.Cv, per_row = C / V;
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int row0 = static_cast<int>(idx / per_row) * R, ch = static_cast<int>(idx % per_row) * V;
  if (row0 >= p.rows) return;
  const T* col = static_cast<const T*>(p.proj) + ch;
  float ib[V], tk[K][V], win[K][V];            // win[j]: the input j - (K - 1) tokens from the current one
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    const float4 b4 = p.bias != nullptr ? *reinterpret_cast<const float4*>(p.bias + ch + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    ib[i] = b4.x; ib[i + 1] = b4.y; ib[i + 2] = b4.z; ib[i + 3] = b4.w;
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const float4 t4 = *reinterpret_cast<const float4*>(p.taps + static_cast<size_t>(j) * C + ch + i);
      tk[j][i] = t4.x; tk[j][i + 1] = t4.y; tk[j][i + 2] = t4.z; tk[j][i + 3] = t4.w;
    }
  }
  uint2 raw[R];                                // all rows' numbers are asked for before any is used
#pragma unroll
  for (int r = 0; r < R; ++r)
    raw[r] = row0 + r < p.rows ? *reinterpret_cast<const uint2*>(col + static_cast<size_t>(row0 + r) * p.proj_stride) : make_uint2(0u, 0u);
  int first_row = 0, next_first = 0, slot = 0;
  const int* table = nullptr;
  float* kept = nullptr;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int row = row0 + r;
    if (row >= p.rows) return;
    const int pos = p.positions[row];
    bool fill = r == 0;
    if (r == 0 || row >= next_first) {           // another request begins
      const int req = p.row_request[row];
      first_row = p.q_start[req];
      next_first = p.q_start[req + 1];
      slot = ck_request(p.row_slot[row]);
      table = p.block_table + static_cast<size_t>(slot) * p.max_blocks;
      kept = p.kept + static_cast<size_t>(slot) * p.kept_stride + ch;
      fill = true;
    }
    if (fill) {
      const bool single = next_first - first_row == 1;
#pragma unroll
      for (int j = 0; j < K - 1; ++j) {
        const int k = K - 1 - j;                 // tokens back
        float u[V];
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] = 0.0f;
        if (pos - k >= 0) {
          const int back = row - k;
          if (back >= first_row) {
            cc_load<T, V>(col + static_cast<size_t>(back) * p.proj_stride, u);
          } else {
            const float* kr = kept + static_cast<size_t>(K - 1 - (first_row - back)) * C;
#pragma unroll
            for (int i = 0; i < V; ++i) u[i] = kr[i];
          }
          if (single && j > 0) {
#pragma unroll
            for (int i = 0; i < V; ++i) kept[static_cast<size_t>(j - 1) * C + i] = u[i];
          }
#pragma unroll
          for (int i = 0; i < V; ++i) u[i] += ib[i];
        } else if (single && j > 0) {
#pragma unroll
          for (int i = 0; i < V; ++i) kept[static_cast<size_t>(j - 1) * C + i] = 0.0f;
        }
#pragma unroll
        for (int i = 0; i < V; ++i) win[j][i] = u[i];
      }
    }
    float u[V], acc[V];
    u[0] = __uint_as_float(raw[r].x << 16); u[1] = __uint_as_float(raw[r].x & 0xffff0000u);
    u[2] = __uint_as_float(raw[r].y << 16); u[3] = __uint_as_float(raw[r].y & 0xffff0000u);
    if (next_first - first_row == 1) {
#pragma unroll
      for (int i = 0; i < V; ++i) kept[static_cast<size_t>(K - 2) * C + i] = u[i];
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      win[K - 1][i] = u[i] + ib[i];
      acc[i] = 0.0f;
#pragma unroll
      for (int j = 0; j < K; ++j) acc[i] = fmaf(tk[j][i], win[j][i], acc[i]);      // oldest input first
#pragma unroll
      for (int j = 0; j < K - 1; ++j) win[j][i] = win[j + 1][i];
    }
    if (ch < p.Cq) {
      cc_store<T, V>(static_cast<T*>(p.q_out) + static_cast<size_t>(row) * p.q_stride + ch, acc);
    } else {
      const int page = ck_page_store(table, pos / p.page_size, p.max_blocks);
      if (page >= 0) {
        const size_t place = static_cast<size_t>(page) * p.page_size + pos % p.page_size;
        if (ch < p.Cq + p.Ck) cc_store<T, V>(static_cast<T*>(p.k_cache) + place * p.k_row + (ch - p.Cq), acc);
        else cc_store<T, V>(static_cast<T*>(p.v_cache) + place * p.v_row + (ch - p.Cq - p.Ck), acc);
      }
    }
  }
}

// The last K - 1 inputs of every request that brought more than one token, oldest first. One thread per (request,
// channel); entries are written in ascending order, and entry j only ever needs an older entry at a higher index.
template <typename T>
__global__ void conv_keep_many_kernel(const T* __restrict__ proj, size_t proj_stride, int C, int K, float* __restrict__ kept_all,
                                      size_t kept_stride, const int* __restrict__ q_start, const int* __restrict__ state_slots,
                                      int requests) {
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= static_cast<size_t>(requests) * C) return;
  const int r = static_cast<int>(idx / C), ch = static_cast<int>(idx % C);
  const int r0 = q_start[r], n = q_start[r + 1] - r0;
  if (n <= 1) return;
  float* kept = kept_all + static_cast<size_t>(ck_request(state_slots[r])) * kept_stride;
  for (int j = 0; j < K - 1; ++j) {
    const int rel = n - (K - 1) + j;                               // which of the step's rows entry j is, if any
    kept[static_cast<size_t>(j) * C + ch] = rel >= 0 ? to_float(proj[static_cast<size_t>(r0 + rel) * proj_stride + ch])
                                                     : kept[static_cast<size_t>(j + n) * C + ch];
  }
}

}  // namespace dl

DL_EXPORT int dl_conv_cache(int dtype, const void* proj, long long proj_stride, int Cq, int Ck, int Cv, int K, const float* taps,
                            const float* bias, float* kept, long long kept_stride, const int* positions,
                            const int* row_request, const int* row_slot, const int* q_start, const int* block_table,
                            int max_blocks, int page_size, void* q_out, long long q_stride, void* k_cache, long long k_row,
                            void* v_cache, long long v_row, int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (Cq <= 0 || Ck < 0 || Cv < 0 || (Ck > 0) != (Cv > 0) || page_size <= 0 || (taps != nullptr && K < 1) ||
      (taps != nullptr && K > 1 && kept == nullptr) || (Ck > 0 && (k_cache == nullptr || v_cache == nullptr)))
    return DL_ERR_UNSUPPORTED;
  const dl::ConvCacheParams p = {proj, static_cast<size_t>(proj_stride), Cq, Ck, Cv, K, taps, bias, kept,
                                 static_cast<size_t>(kept_stride), positions, row_request, row_slot, q_start, block_table,
                                 max_blocks, page_size, q_out, static_cast<size_t>(q_stride), k_cache,
                                 static_cast<size_t>(k_row), v_cache, static_cast<size_t>(v_row), rows};
  const int vec = dtype == 0 ? 4 : 8;
  const bool wide = Cq % vec == 0 && Ck % vec == 0 && Cv % vec == 0 && proj_stride % vec == 0 && q_stride % vec == 0 &&
                    k_row % vec == 0 && v_row % vec == 0 &&
                    ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_cache) |
                      reinterpret_cast<uintptr_t>(v_cache)) & 15) == 0;
#define DL_CC(T, V, R)                                                                                          \
  do {                                                                                                          \
    const size_t n = static_cast<size_t>((rows + R - 1) / R) * ((Cq + Ck + Cv) / V);                            \
    dl::conv_cache_kernel<T, V, R><<<static_cast<unsigned>((n + 255) / 256), 256, 0, stream>>>(p);              \
  } while (0)
  // many rows: a thread walks eight of them (bfloat16, 2 to 4 taps)
  const bool walk = dtype == 1 && wide && rows >= 256 && taps != nullptr && K >= 2 && K <= 4 &&
                    ((reinterpret_cast<uintptr_t>(taps) | reinterpret_cast<uintptr_t>(bias)) & 15) == 0;
  if (walk) {
    constexpr int R = 8;
    const size_t n = static_cast<size_t>((rows + R - 1) / R) * ((Cq + Ck + Cv) / 4);
    const unsigned blocks = static_cast<unsigned>((n + 255) / 256);
    if (K == 2) dl::conv_cache_rows_kernel<dl::bf16, 4, R, 2><<<blocks, 256, 0, stream>>>(p);
    else if (K == 3) dl::conv_cache_rows_kernel<dl::bf16, 4, R, 3><<<blocks, 256, 0, stream>>>(p);
    else dl::conv_cache_rows_kernel<dl::bf16, 4, R, 4><<<blocks, 256, 0, stream>>>(p);
    return dl::launch_status();
  }
  if (dtype == 0) { if (wide) DL_CC(float, 4, 1); else DL_CC(float, 1, 1); }
  else if (dtype == 1) { if (wide) DL_CC(dl::bf16, 8, 1); else DL_CC(dl::bf16, 1, 1); }
  else return DL_ERR_UNSUPPORTED;
#undef DL_CC
  return dl::launch_status();
}

// After dl_conv_cache: the kept inputs of the requests that brought more than one token (C = Cq + Ck + Cv channels).
DL_EXPORT int dl_conv_keep_many(int dtype, const void* proj, long long proj_stride, int C, int K, float* kept,
                                long long kept_stride, const int* q_start, const int* state_slots, int requests,
                                cudaStream_t stream) {
  if (requests <= 0 || K <= 1) return 0;
  const size_t n = static_cast<size_t>(requests) * C;
  const unsigned blocks = static_cast<unsigned>((n + 255) / 256);
  if (dtype == 0)
    dl::conv_keep_many_kernel<float><<<blocks, 256, 0, stream>>>(static_cast<const float*>(proj), static_cast<size_t>(proj_stride), C,
                                                                 K, kept, static_cast<size_t>(kept_stride), q_start, state_slots, requests);
  else if (dtype == 1)
    dl::conv_keep_many_kernel<dl::bf16><<<blocks, 256, 0, stream>>>(static_cast<const dl::bf16*>(proj), static_cast<size_t>(proj_stride), C,
                                                                    K, kept, static_cast<size_t>(kept_stride), q_start, state_slots, requests);
  else return DL_ERR_UNSUPPORTED;
  return dl::launch_status();
}
