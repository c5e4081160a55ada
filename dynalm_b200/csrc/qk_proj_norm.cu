// Queries and keys normed over their whole projection, turned by position, keys and values written into the cache.
//
// A row of the projection holds [q: H * d | k: G * d | v: G * e | ...]. Per row, in float32:
//
//   q <- q / sqrt(mean over all H * d numbers of q^2 + eps) * wq        (one statistic for the whole projection,
//   k <- k / sqrt(mean over all G * d numbers of k^2 + eps) * wk         not one per head; either weight may be absent)
//   the first `rot` numbers of every head of q and k: number i pairs with number i + rot / 2 and the pair (u, v) turns
//   to (u cos a - v sin a, v cos a + u sin a), a = position * pos_scale * inv_freq[i]
//
// q is written back in place; k and v go to the token's place in the request's pages. The two arrays of the cache may
// be one (a record [k | v] per token) or two: each is given by its base and the elements between two tokens.
#include "common.cuh"

namespace dl {

template <typename T>
__global__ void __launch_bounds__(256)
qk_proj_norm_kernel(T* __restrict__ proj, int stride, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                    int do_norm, const float* __restrict__ inv_freq, int rot, float pos_scale,
                    const int* __restrict__ positions, const int* __restrict__ row_slot,
                    const int* __restrict__ block_table, int max_blocks, T* __restrict__ k_cache, size_t k_row,
                    T* __restrict__ v_cache, size_t v_row, int H, int G, int d, int e, int page_size) {
  __shared__ float red[33];
  const int row = blockIdx.x, tid = threadIdx.x;
  T* q = proj + static_cast<size_t>(row) * stride;
  T* k = q + H * d;
  const T* v = k + G * d;
  const int nq = H * d, nk = G * d, nv = G * e;
  float rq = 1.0f, rk = 1.0f;
  if (do_norm) {
    float sq = 0.0f, sk = 0.0f;
    for (int i = tid; i < nq; i += blockDim.x) { const float x = to_float(q[i]); sq = fmaf(x, x, sq); }
    for (int i = tid; i < nk; i += blockDim.x) { const float x = to_float(k[i]); sk = fmaf(x, x, sk); }
    rq = 1.0f / sqrtf(block_sum(sq, red) / static_cast<float>(nq) + eps);
    rk = 1.0f / sqrtf(block_sum(sk, red) / static_cast<float>(nk) + eps);
  }
  const int pos = positions[row];
  const int* table = block_table + static_cast<size_t>(ck_request(row_slot[row])) * max_blocks;
  const int page = ck_page_store(table, pos / page_size, max_blocks);
  const size_t slot = static_cast<size_t>(page < 0 ? 0 : page) * page_size + pos % page_size;
  const int half = rot / 2;
  const float fpos = static_cast<float>(pos) * pos_scale;
  // queries and keys together: index n < nq is a query number, the rest are key numbers
  for (int n = tid; n < nq + nk; n += blockDim.x) {
    const bool is_q = n < nq;
    const int idx = is_q ? n : n - nq;
    const int i = idx % d;
    if (i >= half && i < rot) continue;                      // the second number of a pair: its first number's thread writes it
    T* src = is_q ? q : k;
    const float* w = is_q ? wq : wk;
    const float r = is_q ? rq : rk;
    float a = to_float(src[idx]) * r * (w ? w[idx] : 1.0f);
    float b = 0.0f;
    const bool pair = i < half;
    if (pair) {
      b = to_float(src[idx + half]) * r * (w ? w[idx + half] : 1.0f);
      float s, c;
      sincosf(fpos * inv_freq[i], &s, &c);
      const float a2 = a * c - b * s, b2 = b * c + a * s;
      a = a2;
      b = b2;
    }
    if (is_q) {
      q[idx] = from_float<T>(a);
      if (pair) q[idx + half] = from_float<T>(b);
    } else if (page >= 0) {
      T* dst = k_cache + slot * k_row;
      dst[idx] = from_float<T>(a);
      if (pair) dst[idx + half] = from_float<T>(b);
    }
  }
  if (page >= 0) {
    T* dst = v_cache + slot * v_row;
    for (int i = tid; i < nv; i += blockDim.x) dst[i] = v[i];
  }
}


// The other order: turn first, then make every head of q and k a unit-RMS vector by itself (no weight), or leave it
// as it is. One warp per unit, a unit being a query head, a key head or the values of a KV head. The pairs of the
// rotation are (i, i + rot / 2) or, interleaved, (2i, 2i + 1); a pair (u, v) turns to (u cos a - v sin a, v cos a + u
// sin a), a = position * inv_freq[i], in float32. A bias of the projection (q | k | v) may be added on the way in.
template <typename T>
__global__ void __launch_bounds__(256)
qk_rot_head_norm_kernel(T* __restrict__ proj, int stride, const float* __restrict__ bias, const float* __restrict__ inv_freq, int rot, int interleaved,
                        int unit_norm, float eps, const int* __restrict__ positions, const int* __restrict__ row_slot,
                        const int* __restrict__ block_table, int max_blocks, T* __restrict__ k_cache, size_t k_row,
                        T* __restrict__ v_cache, size_t v_row, int rows, int H, int G, int d, int e, int page_size) {
  constexpr int PER = 8;                                   // numbers a lane holds: heads of up to 256
  const int units = H + 2 * G;
  const long long unit = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(rows) * units) return;
  const int row = static_cast<int>(unit / units), u = static_cast<int>(unit % units);
  const int pos = positions[row];
  const int* table = block_table + static_cast<size_t>(ck_request(row_slot[row])) * max_blocks;
  T* base = proj + static_cast<size_t>(row) * stride;
  size_t slot = 0;
  int page = 0;
  if (u >= H) {
    page = ck_page_store(table, pos / page_size, max_blocks);
    slot = static_cast<size_t>(page < 0 ? 0 : page) * page_size + pos % page_size;
  }
  if (u >= H + G) {                                         // values: a copy into the token's place
    if (page < 0) return;
    const int off = H * d + G * d + (u - H - G) * e;
    const T* v = base + off;
    T* dst = v_cache + slot * v_row + static_cast<size_t>(u - H - G) * e;
    if (bias != nullptr) {
      for (int i = lane; i < e; i += 32) dst[i] = from_float<T>(to_float(v[i]) + bias[off + i]);
    } else {
      for (int i = lane; i < e; i += 32) dst[i] = v[i];
    }
    return;
  }
  const int src_off = u < H ? u * d : H * d + (u - H) * d;
  T* src = base + src_off;
  const float* bsrc = bias != nullptr ? bias + src_off : nullptr;
  const int half = rot / 2;
  float x[PER], xp[PER];
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int i = lane + 32 * j;
    x[j] = i < d ? to_float(src[i]) + (bsrc != nullptr ? bsrc[i] : 0.0f) : 0.0f;
    xp[j] = 0.0f;
    if (i < rot) {
      const int partner = interleaved ? (i ^ 1) : (i < half ? i + half : i - half);
      xp[j] = to_float(src[partner]) + (bsrc != nullptr ? bsrc[partner] : 0.0f);
    }
  }
  __syncwarp();                                             // every lane has read before any lane writes in place
  const float fpos = static_cast<float>(pos);
  float ss = 0.0f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int i = lane + 32 * j;
    if (i < rot) {
      const bool first = interleaved ? !(i & 1) : i < half;
      const int f = interleaved ? (i >> 1) : (first ? i : i - half);
      float sn, cs;
      sincosf(fpos * inv_freq[f], &sn, &cs);
      x[j] = first ? x[j] * cs - xp[j] * sn : x[j] * cs + xp[j] * sn;
    }
    ss = fmaf(x[j], x[j], ss);
  }
  float r = 1.0f;
  if (unit_norm) r = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(d) + eps);
  T* dst = src;
  if (u >= H) {
    if (page < 0) return;
    dst = k_cache + slot * k_row + static_cast<size_t>(u - H) * d;
  }
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int i = lane + 32 * j;
    if (i < d) dst[i] = from_float<T>(x[j] * r);
  }
}

// The third order: every head of q and k normed by itself with a weight that all heads share, x / sqrt(mean(x^2) + eps) *
// w[i], then turned: numbers i and i + rot / 2 of its first `rot` numbers by position * freq[i], cos and sin times mag. The
// angle is formed and brought into half a turn around zero in double precision, so it is exact to float32 at any position.
// The values are columns of their own behind k, or (values_are_keys) the keys as they were projected.
__device__ __forceinline__ void qk_angle(int pos, double freq, float mag, float& cs, float& sn) {
  constexpr double TURN = 6.283185307179586476925286766559, INV_TURN = 0.15915494309189533576888376337251;
  const double a = static_cast<double>(pos) * freq;
  float s, c;
  sincosf(static_cast<float>(fma(-rint(a * INV_TURN), TURN, a)), &s, &c);
  cs = c * mag;
  sn = s * mag;
}

// One block per row; the row's angles are worked out once, in shared memory. A head is TG neighbouring lanes with 16 bytes
// each (the lanes past its end idle), TG a power of two up to 32, and half of `rot` a multiple of a lane's numbers.
template <typename T>
__global__ void __launch_bounds__(512)
qk_norm_turn_vec_kernel(T* __restrict__ proj, int stride, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                        const double* __restrict__ freq, int rot, float mag, const int* __restrict__ positions,
                        const int* __restrict__ row_slot, const int* __restrict__ block_table, int max_blocks,
                        T* __restrict__ k_cache, size_t k_row, T* __restrict__ v_cache, size_t v_row, int H, int G, int d, int e,
                        int page_size, int values_are_keys, int tg_shift) {
  constexpr int V = PerVec<T>::n;
  constexpr int MAX_PAIRS = 128;
  __shared__ __align__(16) float cos_s[MAX_PAIRS], sin_s[MAX_PAIRS];
  const int row = blockIdx.x, tid = threadIdx.x;
  T* base = proj + static_cast<size_t>(row) * stride;
  const int TG = 1 << tg_shift, tg_mask = TG - 1, per_head = d / V, half = rot / 2, half_lanes = half / V, own_values = values_are_keys ? 0 : G * e / V;
  const int turned = (H + G) * TG, total = turned + own_values;
  // where the 16 bytes of place i begin in the row (heads, then values), -1: an idle lane
  auto source = [&](int i) {
    if (i < turned) return (i & tg_mask) < per_head ? (i >> tg_shift) * d + (i & tg_mask) * V : -1;
    return i < total ? (H + G) * d + (i - turned) * V : -1;
  };
  Vec16 raw;
  raw.raw = make_uint4(0u, 0u, 0u, 0u);
  int at = source(tid);
  if (at >= 0) raw = *reinterpret_cast<const Vec16*>(base + at);      // asked for before the angles are worked out
  const int pos = positions[row];
  const int* table = block_table + static_cast<size_t>(ck_request(row_slot[row])) * max_blocks;
  const int page = ck_page_store(table, pos / page_size, max_blocks);
  const size_t slot = static_cast<size_t>(page < 0 ? 0 : page) * page_size + pos % page_size;
  for (int i = tid; i < half; i += blockDim.x) qk_angle(pos, freq[i], mag, cos_s[i], sin_s[i]);
  __syncthreads();
  // whole warps walk the heads, so that the shuffles below find their lanes
  for (int i = tid; i < (total + 31) / 32 * 32; i += blockDim.x) {
    if (i != tid) {
      at = source(i);
      raw.raw = make_uint4(0u, 0u, 0u, 0u);
      if (at >= 0) raw = *reinterpret_cast<const Vec16*>(base + at);
    }
    const int head = i >> tg_shift, l = i & tg_mask;
    const bool is_head = i < turned, live = is_head && at >= 0;
    float x[V];
    unpack<T>(raw, x);
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(x[j], x[j], ss);
    for (int o = TG >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = 1.0f / sqrtf(ss / static_cast<float>(d) + eps);
    if (live) {
      const float4* w = reinterpret_cast<const float4*>((head < H ? wq : wk) + l * V);
#pragma unroll
      for (int j = 0; j < V; j += 4) {
        const float4 f = w[j / 4];
        x[j] *= r * f.x;
        x[j + 1] *= r * f.y;
        x[j + 2] *= r * f.z;
        x[j + 3] *= r * f.w;
      }
    }
    const bool first = l < half_lanes, pair = l < 2 * half_lanes;
    const int lane = tid & 31, partner = pair ? (first ? lane + half_lanes : lane - half_lanes) : lane;
    const int a0 = pair ? (first ? l : l - half_lanes) * V : 0;
#pragma unroll
    for (int j = 0; j < V; j += 4) {
      float y[4];
#pragma unroll
      for (int n = 0; n < 4; ++n) y[n] = __shfl_sync(0xffffffffu, x[j + n], partner);
      if (pair && live) {
        const float4 c = *reinterpret_cast<const float4*>(cos_s + a0 + j), s = *reinterpret_cast<const float4*>(sin_s + a0 + j);
        const float f = first ? -1.0f : 1.0f;           // (u cos - v sin, v cos + u sin)
        x[j] = fmaf(x[j], c.x, f * y[0] * s.x);
        x[j + 1] = fmaf(x[j + 1], c.y, f * y[1] * s.y);
        x[j + 2] = fmaf(x[j + 2], c.z, f * y[2] * s.z);
        x[j + 3] = fmaf(x[j + 3], c.w, f * y[3] * s.w);
      }
    }
    if (live && head < H) {
      *reinterpret_cast<Vec16*>(base + at) = pack<T>(x);
    } else if (live && page >= 0) {
      const size_t to = static_cast<size_t>(head - H) * d + l * V;
      *reinterpret_cast<Vec16*>(k_cache + slot * k_row + to) = pack<T>(x);
      if (values_are_keys) *reinterpret_cast<Vec16*>(v_cache + slot * v_row + to) = raw;
    } else if (!is_head && at >= 0 && page >= 0) {
      *reinterpret_cast<Vec16*>(v_cache + slot * v_row + static_cast<size_t>(i - turned) * V) = raw;
    }
  }
}

// Any size up to 256: one warp per unit, a unit being a query head, a key head or the values of a KV head.
template <typename T>
__global__ void __launch_bounds__(256)
qk_norm_turn_kernel(T* __restrict__ proj, int stride, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                    const double* __restrict__ freq, int rot, float mag, const int* __restrict__ positions,
                    const int* __restrict__ row_slot, const int* __restrict__ block_table, int max_blocks,
                    T* __restrict__ k_cache, size_t k_row, T* __restrict__ v_cache, size_t v_row, int rows, int H, int G, int d,
                    int e, int page_size, int values_are_keys) {
  constexpr int PER = 8;
  const int units = H + 2 * G;
  const long long unit = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(rows) * units) return;
  const int row = static_cast<int>(unit / units), u = static_cast<int>(unit % units);
  const int pos = positions[row];
  const int* table = block_table + static_cast<size_t>(ck_request(row_slot[row])) * max_blocks;
  T* base = proj + static_cast<size_t>(row) * stride;
  size_t slot = 0;
  int page = 0;
  if (u >= H) {
    page = ck_page_store(table, pos / page_size, max_blocks);
    if (page < 0) return;
    slot = static_cast<size_t>(page) * page_size + pos % page_size;
  }
  if (u >= H + G) {                                         // values: a copy into the token's place
    const int j = u - H - G;
    const T* v = base + (values_are_keys ? (H + j) * d : (H + G) * d + j * e);
    T* dst = v_cache + slot * v_row + static_cast<size_t>(j) * e;
    for (int i = lane; i < e; i += 32) dst[i] = v[i];
    return;
  }
  T* src = base + static_cast<size_t>(u) * d;
  const float* w = u < H ? wq : wk;
  const int half = rot / 2;
  float x[PER], xp[PER], ss = 0.0f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int i = lane + 32 * j;
    x[j] = i < d ? to_float(src[i]) : 0.0f;
    xp[j] = i < rot ? to_float(src[i < half ? i + half : i - half]) : 0.0f;
    ss = fmaf(x[j], x[j], ss);
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(d) + eps);      // (the shuffles also order reads before writes)
  T* dst = u < H ? src : k_cache + slot * k_row + static_cast<size_t>(u - H) * d;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int i = lane + 32 * j;
    if (i >= d) continue;
    float v = x[j] * r * w[i];
    if (i < rot) {
      const bool first = i < half;
      const float y = xp[j] * r * w[first ? i + half : i - half];
      float c, s;
      qk_angle(pos, freq[first ? i : i - half], mag, c, s);
      v = first ? v * c - y * s : v * c + y * s;
    }
    dst[i] = from_float<T>(v);
  }
}

}  // namespace dl

DL_EXPORT int dl_qk_proj_norm_cache(int dtype, void* proj, int stride, const float* wq, const float* wk, float eps, int do_norm,
                                    const float* inv_freq, int rot, float pos_scale, const int* positions,
                                    const int* row_slot, const int* block_table, int max_blocks, void* k_cache,
                                    long long k_row, void* v_cache, long long v_row, int rows, int H, int G, int d, int e,
                                    int page_size, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || d <= 0 || e <= 0 || rot < 0 || rot > d || (rot & 1) || page_size <= 0 || (rot > 0 && inv_freq == nullptr))
    return DL_ERR_UNSUPPORTED;
#define DL_QK(T)                                                                                                          \
  dl::qk_proj_norm_kernel<T><<<rows, 256, 0, stream>>>(static_cast<T*>(proj), stride, wq, wk, eps, do_norm, inv_freq, rot, \
                                                       pos_scale, positions, row_slot, block_table, max_blocks,          \
                                                       static_cast<T*>(k_cache), static_cast<size_t>(k_row),              \
                                                       static_cast<T*>(v_cache), static_cast<size_t>(v_row), H, G, d, e,  \
                                                       page_size)
  if (dtype == 0) DL_QK(float);
  else if (dtype == 1) DL_QK(dl::bf16);
  else return DL_ERR_UNSUPPORTED;
#undef DL_QK
  return dl::launch_status();
}

// Rows [q: H*d | k: G*d | v: G*e | ...]: rotation first (rot numbers of every head, pairs by halves or interleaved),
// then every head of q and k divided by its own root mean square (unit_norm) or left; q in place, k and v into the
// pages. bias: float32 [H*d + G*d + G*e] added to q | k | v first, or null. d at most 256.
DL_EXPORT int dl_qk_rot_head_norm_cache(int dtype, void* proj, int stride, const float* bias, const float* inv_freq, int rot, int interleaved,
                                        int unit_norm, float eps, const int* positions, const int* row_slot,
                                        const int* block_table, int max_blocks, void* k_cache, long long k_row,
                                        void* v_cache, long long v_row, int rows, int H, int G, int d, int e, int page_size,
                                        cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || d <= 0 || d > 256 || e <= 0 || rot < 0 || rot > d || (rot & 1) || page_size <= 0 ||
      (rot > 0 && inv_freq == nullptr))
    return DL_ERR_UNSUPPORTED;
  const long long units = static_cast<long long>(rows) * (H + 2 * G);
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
#define DL_QK(T)                                                                                                          \
  dl::qk_rot_head_norm_kernel<T><<<blocks, 256, 0, stream>>>(static_cast<T*>(proj), stride, bias, inv_freq, rot, interleaved, \
                                                             unit_norm, eps, positions, row_slot, block_table, max_blocks, \
                                                             static_cast<T*>(k_cache), static_cast<size_t>(k_row),         \
                                                             static_cast<T*>(v_cache), static_cast<size_t>(v_row), rows, H, \
                                                             G, d, e, page_size)
  if (dtype == 0) DL_QK(float);
  else if (dtype == 1) DL_QK(dl::bf16);
  else return DL_ERR_UNSUPPORTED;
#undef DL_QK
  return dl::launch_status();
}

// Rows [q: H*d | k: G*d | v: G*e | ...] (without the values when they are the keys): every head of q and k normed by itself
// (wq, wk: float32 [d]), then turned (rot numbers, pairs i and i + rot / 2, freq: float64 [rot / 2]); q in
// place, k and v into the pages. d and e at most 256.
DL_EXPORT int dl_qk_norm_turn_cache(int dtype, void* proj, int stride, const float* wq, const float* wk, float eps,
                                    const double* freq, int rot, float mag, const int* positions, const int* row_slot,
                                    const int* block_table, int max_blocks, void* k_cache, long long k_row, void* v_cache,
                                    long long v_row, int rows, int H, int G, int d, int e, int page_size, int values_are_keys,
                                    cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || d <= 0 || d > 256 || e <= 0 || e > 256 || rot < 0 || rot > d || (rot & 1) || page_size <= 0 ||
      wq == nullptr || wk == nullptr || (rot > 0 && freq == nullptr) || (values_are_keys && d != e) || (dtype != 0 && dtype != 1))
    return DL_ERR_UNSUPPORTED;
  const int V = dtype == 0 ? 4 : 8;
  int TG = 1, tg_shift = 0;
  while (TG * V < d) {
    TG *= 2;
    ++tg_shift;
  }
  const uintptr_t bases = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
                          reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wk);
  if (d % V == 0 && e % V == 0 && TG <= 32 && (rot / 2) % V == 0 && stride % V == 0 && k_row % V == 0 && v_row % V == 0 && (bases & 15) == 0) {
    const int lanes = (H + G) * TG + (values_are_keys ? 0 : G * e / V);
    const int threads = lanes <= 64 ? 64 : lanes <= 128 ? 128 : rows >= 256 || lanes <= 256 ? 256 : 512;   // many rows: more blocks an SM
#define DL_QK(T)                                                                                                            \
  dl::qk_norm_turn_vec_kernel<T><<<rows, threads, 0, stream>>>(static_cast<T*>(proj), stride, wq, wk, eps, freq, rot, mag,  \
                                                               positions, row_slot, block_table, max_blocks,                \
                                                               static_cast<T*>(k_cache), static_cast<size_t>(k_row),        \
                                                               static_cast<T*>(v_cache), static_cast<size_t>(v_row), H, G,  \
                                                               d, e, page_size, values_are_keys, tg_shift)
    if (dtype == 0) DL_QK(float);
    else DL_QK(dl::bf16);
#undef DL_QK
    return dl::launch_status();
  }
  const long long units = static_cast<long long>(rows) * (H + 2 * G);
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
#define DL_QK(T)                                                                                                            \
  dl::qk_norm_turn_kernel<T><<<blocks, 256, 0, stream>>>(static_cast<T*>(proj), stride, wq, wk, eps, freq, rot, mag,        \
                                                         positions, row_slot, block_table, max_blocks,                      \
                                                         static_cast<T*>(k_cache), static_cast<size_t>(k_row),              \
                                                         static_cast<T*>(v_cache), static_cast<size_t>(v_row), rows, H, G,  \
                                                         d, e, page_size, values_are_keys)
  if (dtype == 0) DL_QK(float);
  else DL_QK(dl::bf16);
#undef DL_QK
  return dl::launch_status();
}
