// Mixture of experts: routing, the grouping of (token, expert) pairs by expert, the experts' products over those
// groups, and the weighted sum of a token's experts.
//
//   dl_moe_route     scores = softmax(router logits, + a bias per expert where there is one) over all experts, or sigmoid of each, float32; choice scores = scores
//                    (+ a correction per expert). Experts form `groups` equal groups of neighbours; a group's score is
//                    its largest choice score, or the sum of its two largest, and only experts of the `keep` best groups
//                    can be chosen. The `top` allowed experts with the largest choice scores are chosen (equal ones: the
//                    lower index), their weights are their scores, divided by their sum (+ 1e-20) or not, times `scale`.
//   dl_moe_group     a counting sort of the tokens' pairs by expert: where every pair stands in that order, which pair
//                    stands at every place, and the list of row tiles (expert, first place, places) for the products.
//   dl_moe_linear    C[place] = act(A[row of place] W_e^T) for every place of every tile, W_e the matrix of the tile's
//                    expert: a plain tiled product with float32 accumulation in a fixed order of k (any dtype), and one on
//                    the tensor cores for bfloat16 (mma.sync m16n8k16, float32 accumulation), with tiles of 32 places for
//                    steps that bring an expert few and of 128 for steps that bring it many.
//                    act "pairs": rows 2j and 2j + 1 of a matrix are the gate and up rows of feature j, and the result is
//                    silu(gate) * up, half as many columns.
//   dl_moe_combine   y[t] = sum_k weight[t, k] * C[place of pair (t, k)], float32, in the order of k; then, with a shared
//                    expert's output and its gate logit, + sigmoid(z[t]) * S[t].
#include "common.cuh"

namespace dl {

constexpr int MOE_MAX_EXPERTS = 256;
constexpr int MOE_TM = 32;          // places a tile of the kernels for few places an expert
constexpr int MOE_TM_WIDE = 128;    // places a tile of the kernel for many

// One warp per token. Lane l holds the scores of experts l, l + 32, ...; every choice is a warp-wide maximum (equal scores:
// the lower index).
constexpr int MOE_PER_LANE = MOE_MAX_EXPERTS / 32;
constexpr int MOE_ROUTE_WARPS = 4;

__device__ __forceinline__ int moe_warp_best(float v, int index) {      // the index of the largest v, -1 when none is a number
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, index, o);
    if (oi >= 0 && (index < 0 || ov > v || (ov == v && oi < index))) { v = ov; index = oi; }
  }
  return index;
}

__global__ void __launch_bounds__(MOE_ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, int stride, int tokens, int E, int top, int groups, int keep,
                 const float* __restrict__ bias, const float* __restrict__ correction, int sigmoid_scores, int group_top2, int renormalize, float scale,
                 int* __restrict__ ids, float* __restrict__ weights) {
  __shared__ float choice_s[MOE_ROUTE_WARPS][MOE_MAX_EXPERTS];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * MOE_ROUTE_WARPS + warp;
  if (t >= tokens) return;                                     // (no block barrier below: warps work alone)
  const float* z = logits + static_cast<size_t>(t) * stride;
  float s[MOE_PER_LANE], c[MOE_PER_LANE];                      // scores, choice scores
  float m = -INFINITY;
#pragma unroll
  for (int k = 0; k < MOE_PER_LANE; ++k) {
    const int i = lane + 32 * k;
    s[k] = i < E ? z[i] + (bias != nullptr ? bias[i] : 0.0f) : -INFINITY;
    m = fmaxf(m, s[k]);
  }
  if (sigmoid_scores) {
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k) s[k] = 1.0f / (1.0f + expf(-s[k]));
  } else {
    m = warp_max(m);
    float sum = 0.0f;
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k) {
      s[k] = expf(s[k] - m);                                   // 0 past the last expert
      sum += s[k];
    }
    const float inv = 1.0f / warp_sum(sum);
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k) s[k] *= inv;
  }
#pragma unroll
  for (int k = 0; k < MOE_PER_LANE; ++k) {
    const int i = lane + 32 * k;
    c[k] = i < E ? s[k] + (correction != nullptr ? correction[i] : 0.0f) : -INFINITY;
  }
  const int per = E / groups;
  if (keep < groups) {
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k)
      if (lane + 32 * k < E) choice_s[warp][lane + 32 * k] = c[k];
    __syncwarp();
    float gs[MOE_PER_LANE];                                    // scores of groups lane, lane + 32, ...
    bool kept[MOE_PER_LANE];
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k) {
      const int g = lane + 32 * k;
      gs[k] = -INFINITY;
      kept[k] = false;
      if (g < groups) {
        float a = -INFINITY, b = -INFINITY;                    // the two largest
        for (int i = g * per; i < (g + 1) * per; ++i) {
          const float v = choice_s[warp][i];
          if (v > a) { b = a; a = v; }
          else if (v > b) b = v;
        }
        gs[k] = group_top2 && per > 1 ? a + b : a;
      }
    }
    for (int r = 0; r < keep; ++r) {
      float v = -INFINITY;
      int who = -1;
#pragma unroll
      for (int k = 0; k < MOE_PER_LANE; ++k) {
        const int g = lane + 32 * k;
        if (g < groups && !kept[k] && (who < 0 || gs[k] > v)) { v = gs[k]; who = g; }
      }
      who = moe_warp_best(v, who);
#pragma unroll
      for (int k = 0; k < MOE_PER_LANE; ++k)
        if (who == lane + 32 * k) kept[k] = true;
    }
    __syncwarp();                                              // the choice scores have been read: group marks take their place
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k)
      if (lane + 32 * k < groups) choice_s[warp][lane + 32 * k] = kept[k] ? 1.0f : 0.0f;
    __syncwarp();
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k) {
      const int i = lane + 32 * k;
      if (i < E && choice_s[warp][i / per] == 0.0f) c[k] = -INFINITY;
    }
  }
  float wsum = 0.0f;
  int* my_ids = ids + static_cast<size_t>(t) * top;
  float* my_w = weights + static_cast<size_t>(t) * top;
  unsigned taken = 0;                                          // bit k: this lane's k-th expert has been chosen
  for (int r = 0; r < top; ++r) {
    float v = -INFINITY;
    int who = -1;
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k)
      if (!(taken >> k & 1u) && c[k] > v) { v = c[k]; who = lane + 32 * k; }
    who = moe_warp_best(v, who);
    if (who < 0) who = 0;                                      // (scores that are not numbers: some expert all the same)
    float w = 0.0f;
#pragma unroll
    for (int k = 0; k < MOE_PER_LANE; ++k)
      if (who == lane + 32 * k) { taken |= 1u << k; w = s[k]; }
    w = __shfl_sync(0xffffffffu, w, who & 31);
    wsum += w;
    if (lane == 0) {
      my_ids[r] = who;
      my_w[r] = renormalize ? w : w * scale;
    }
  }
  if (renormalize) {
    __syncwarp();
    const float f = scale / (wsum + 1e-20f);
    for (int r = lane; r < top; r += 32) my_w[r] *= f;
  }
}

// One block. pairs = tokens * top. Outputs: place_of[pair], pair_at[place], tiles[3 * i] = (expert, first place,
// places) for i < n_tiles[0].
__global__ void __launch_bounds__(1024)
moe_group_kernel(const int* __restrict__ ids, int pairs, int E, int* __restrict__ place_of, int* __restrict__ pair_at,
                 int* __restrict__ tiles, int* __restrict__ n_tiles, int TM) {
  __shared__ int count[MOE_MAX_EXPERTS], first[MOE_MAX_EXPERTS + 1], cursor[MOE_MAX_EXPERTS], tile0[MOE_MAX_EXPERTS + 1];
  const int tid = threadIdx.x;
  for (int i = tid; i < E; i += blockDim.x) { count[i] = 0; cursor[i] = 0; }
  __syncthreads();
  for (int p = tid; p < pairs; p += blockDim.x) atomicAdd(&count[min(max(ids[p], 0), E - 1)], 1);
  __syncthreads();
  if (tid == 0) {
    int at = 0, tl = 0;
    for (int i = 0; i < E; ++i) {
      first[i] = at;
      tile0[i] = tl;
      at += count[i];
      tl += (count[i] + TM - 1) / TM;
    }
    first[E] = at;
    tile0[E] = tl;
    n_tiles[0] = tl;
  }
  __syncthreads();
  // Places inside an expert's run are dealt in the order in which the threads arrive: a run's order changes no
  // result (every place is a product of its own), only which places share a tile.
  for (int p = tid; p < pairs; p += blockDim.x) {
    const int ex = min(max(ids[p], 0), E - 1);
    const int place = first[ex] + atomicAdd(&cursor[ex], 1);
    place_of[p] = place;
    pair_at[place] = p;
  }
  for (int i = tid; i < E; i += blockDim.x) {
    const int nt = (count[i] + TM - 1) / TM;
    for (int j = 0; j < nt; ++j) {
      int* tl = tiles + 3 * (tile0[i] + j);
      tl[0] = i;
      tl[1] = first[i] + j * TM;
      tl[2] = min(TM, count[i] - j * TM);
    }
  }
}

template <typename T>
__device__ __forceinline__ float apply_act(float v, int act) {
  if (act == 1) { v = fmaxf(v, 0.0f); v = v * v; }
  return v;
}
constexpr int MOE_ACT_PAIRS = 2;
__device__ __forceinline__ float silu_times(float g, float u) { return g / (1.0f + expf(-g)) * u; }

// Plain tiled product: tile = 32 places x 64 features, 256 threads, 2 x 4 results a thread, k in steps of 16.
// A row of place p: a[(rows_of ? rows_of[pair_at[p]] / div : p) * lda]; W of expert x: w + x * N * K, [N, K].
template <typename T, typename TO>
__global__ void __launch_bounds__(256)
moe_linear_simt_kernel(const T* __restrict__ a, int lda, const int* __restrict__ pair_at, int top_div,
                       const T* __restrict__ w, int N, int K, TO* __restrict__ c, int ldc, const int* __restrict__ tiles,
                       const int* __restrict__ n_tiles, int act) {
  constexpr int TN = 64, TK = 16;
  __shared__ float As[TK][MOE_TM + 1], Bs[TK][TN + 1];
  __shared__ int src[MOE_TM];
  if (static_cast<int>(blockIdx.y) >= n_tiles[0]) return;
  const int* tl = tiles + 3 * blockIdx.y;
  const int ex = tl[0], p0 = tl[1], np = tl[2];
  const int n0 = blockIdx.x * TN;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  if (tid < MOE_TM) src[tid] = tid < np ? (pair_at != nullptr ? pair_at[p0 + tid] / top_div : p0 + tid) : -1;
  __syncthreads();
  const T* wx = w + static_cast<size_t>(ex) * N * K;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < K; k0 += TK) {
    for (int x = tid; x < MOE_TM * TK; x += 256) {
      const int r = x / TK, k = x % TK;
      As[k][r] = (src[r] >= 0 && k0 + k < K) ? to_float(a[static_cast<size_t>(src[r]) * lda + k0 + k]) : 0.0f;
    }
    for (int x = tid; x < TN * TK; x += 256) {
      const int n = x / TK, k = x % TK;
      Bs[k][n] = (n0 + n < N && k0 + k < K) ? to_float(wx[static_cast<size_t>(n0 + n) * K + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float a0 = As[k][ty * 2], a1 = As[k][ty * 2 + 1];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = Bs[k][tx * 4 + j];
        acc[0][j] = fmaf(a0, b, acc[0][j]);
        acc[1][j] = fmaf(a1, b, acc[1][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = ty * 2 + i;
    if (r >= np) continue;
    if (act == MOE_ACT_PAIRS) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = n0 + tx * 4 + j;
        if (n + 1 < N) c[static_cast<size_t>(p0 + r) * ldc + n / 2] = from_float<TO>(silu_times(acc[i][j], acc[i][j + 1]));
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) c[static_cast<size_t>(p0 + r) * ldc + n] = from_float<TO>(apply_act<T>(acc[i][j], act));
    }
  }
}

__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

// bfloat16 on the tensor cores: tile = TM places x 128 features, 8 warps as WM x (8 / WM), k in steps of BK through a
// ring of STAGES cp.async buffers (the next steps' A and W are on their way while this one is multiplied, one block
// barrier a step), fragments by ldmatrix, rows padded by 16 bytes so that a fragment's rows fall on different banks.
//   TM = 128, WM = 2: a warp takes 64 places x 32 features; for steps that bring an expert many places, whose
//   matrix is then read once per 128 places.
//   TM = 32, WM = 1: a warp takes all 32 places x 16 features; for steps that bring an expert a few places (a
//   decode batch), which stream every touched expert's matrix once and are bound by that stream.
__device__ __forceinline__ void moe_cp16(void* smem, const void* gmem, bool valid) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  const int bytes = valid ? 16 : 0;   // 0 source bytes: the 16 destination bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void moe_ldmatrix_x4(uint32_t (&r)[4], const void* smem) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}

template <int TM, int WM, int BK, int STAGES, typename TO>
__global__ void __launch_bounds__(256)
moe_linear_tc_kernel(const bf16* __restrict__ a, int lda, const int* __restrict__ pair_at, int top_div,
                     const bf16* __restrict__ w, int N, int K, TO* __restrict__ c, int ldc, const int* __restrict__ tiles,
                     const int* __restrict__ n_tiles, int act) {
  constexpr int TN = 128, LD = BK + 8, WN = 8 / WM;
  constexpr int MI = TM / WM / 16;          // m16 fragments a warp
  constexpr int NI = TN / WN / 8;           // n8 fragments a warp (two per ldmatrix.x4)
  constexpr int CH = BK / 8;                // 16-byte pieces a row of a stage
  extern __shared__ __align__(16) unsigned char moe_smem[];
  bf16 (*As)[TM][LD] = reinterpret_cast<bf16 (*)[TM][LD]>(moe_smem);                                  // [STAGES][TM][LD]
  bf16 (*Bs)[TN][LD] = reinterpret_cast<bf16 (*)[TN][LD]>(moe_smem + sizeof(bf16) * STAGES * TM * LD);  // [STAGES][TN][LD]
  __shared__ int src[TM];
  if (static_cast<int>(blockIdx.y) >= n_tiles[0]) return;
  const int* tl = tiles + 3 * blockIdx.y;
  const int ex = tl[0], p0 = tl[1], np = tl[2];
  const int n0 = blockIdx.x * TN;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp / WN, wn = warp % WN;
  if (tid < TM) src[tid] = tid < np ? (pair_at != nullptr ? pair_at[p0 + tid] / top_div : p0 + tid) : -1;
  __syncthreads();
  const bf16* wx = w + static_cast<size_t>(ex) * N * K;
  auto load = [&](int stage, int k0) {
    for (int x = tid; x < TM * CH; x += 256) {
      const int r = x / CH, piece = x % CH;
      const bool ok = src[r] >= 0;
      moe_cp16(&As[stage][r][piece * 8], a + static_cast<size_t>(ok ? src[r] : 0) * lda + k0 + piece * 8, ok);
    }
    for (int x = tid; x < TN * CH; x += 256) {
      const int r = x / CH, piece = x % CH;
      const bool ok = n0 + r < N;
      moe_cp16(&Bs[stage][r][piece * 8], wx + static_cast<size_t>(ok ? n0 + r : 0) * K + k0 + piece * 8, ok);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  float acc[MI][NI][4] = {};
  const int steps = K / BK;
  // STAGES - 1 steps are on their way at any time; a group is committed every round (an empty one past the end), so that
  // "all but the newest STAGES - 2 groups have landed" always names the step about to be multiplied
  for (int i = 0; i < STAGES - 1; ++i) {
    if (i < steps) load(i, i * BK);
    else asm volatile("cp.async.commit_group;\n" ::);
  }
  for (int s = 0; s < steps; ++s) {
    const int st = s % STAGES;
    asm volatile("cp.async.wait_group %0;\n" ::"n"(STAGES - 2));
    __syncthreads();                         // step s is in shared memory, and every warp is done with step s - 1
    if (s + STAGES - 1 < steps) load((s + STAGES - 1) % STAGES, (s + STAGES - 1) * BK);
    else asm volatile("cp.async.commit_group;\n" ::);
#pragma unroll
    for (int kk = 0; kk < BK; kk += 16) {
      uint32_t af[MI][4], bfr[NI / 2][4];
#pragma unroll
      for (int mi = 0; mi < MI; ++mi)
        moe_ldmatrix_x4(af[mi], &As[st][wm * (TM / WM) + mi * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][kk + (lane >> 4) * 8]);
#pragma unroll
      for (int nj = 0; nj < NI / 2; ++nj)       // two n8 fragments per ldmatrix.x4
        moe_ldmatrix_x4(bfr[nj], &Bs[st][wn * (TN / WN) + nj * 16 + (lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]);
#pragma unroll
      for (int mi = 0; mi < MI; ++mi)
#pragma unroll
        for (int ni = 0; ni < NI; ++ni) {
          const uint32_t b2[2] = {bfr[ni >> 1][(ni & 1) * 2], bfr[ni >> 1][(ni & 1) * 2 + 1]};
          mma_bf16_16816(acc[mi][ni], af[mi], b2);
        }
    }
  }
  const int g = lane >> 2, q = lane & 3;
#pragma unroll
  for (int mi = 0; mi < MI; ++mi)
#pragma unroll
    for (int ni = 0; ni < NI; ++ni)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = wm * (TM / WM) + mi * 16 + g + 8 * h;
        const int n = n0 + wn * (TN / WN) + ni * 8 + q * 2;
        if (r >= np) continue;
        if (act == MOE_ACT_PAIRS) {
          if (n + 1 < N)
            c[static_cast<size_t>(p0 + r) * ldc + n / 2] = from_float<TO>(silu_times(acc[mi][ni][2 * h], acc[mi][ni][2 * h + 1]));
          continue;
        }
        TO* dst = c + static_cast<size_t>(p0 + r) * ldc + n;
        if (n < N) dst[0] = from_float<TO>(apply_act<bf16>(acc[mi][ni][2 * h], act));
        if (n + 1 < N) dst[1] = from_float<TO>(apply_act<bf16>(acc[mi][ni][2 * h + 1], act));
      }
}

// out[place] = a[pair_at[place] / top_div]: the rows of a step in the order of their experts, 16 bytes a thread.
__global__ void moe_gather_kernel(const uint4* __restrict__ a, int lda16, const int* __restrict__ pair_at, int top_div,
                                  uint4* __restrict__ out, int row16, size_t total) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const size_t place = i / row16;
  const int c = static_cast<int>(i % row16);
  out[i] = a[static_cast<size_t>(pair_at[place] / top_div) * lda16 + c];
}

// V columns a thread (4 where every row starts on a 16-byte boundary).
template <typename TO, typename TS, int V>
__global__ void moe_combine_kernel(const float* __restrict__ c, int width, const int* __restrict__ place_of,
                                   const float* __restrict__ weights, int top, const TS* __restrict__ shared, int parts,
                                   size_t part_stride, const float* __restrict__ shared_z, int z_stride, TO* __restrict__ y,
                                   size_t total) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int per_row = width / V;
  const size_t t = i / per_row;
  const int col = static_cast<int>(i % per_row) * V;
  float sum[V];
#pragma unroll
  for (int j = 0; j < V; ++j) sum[j] = 0.0f;
  for (int k = 0; k < top; ++k) {
    const float w = weights[t * top + k];
    const float* row = c + static_cast<size_t>(place_of[t * top + k]) * width + col;
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(row);
      sum[0] = fmaf(w, v.x, sum[0]); sum[1] = fmaf(w, v.y, sum[1]); sum[2] = fmaf(w, v.z, sum[2]); sum[3] = fmaf(w, v.w, sum[3]);
    } else {
      sum[0] = fmaf(w, row[0], sum[0]);
    }
  }
  if (shared != nullptr) {
    const float g = 1.0f / (1.0f + expf(-shared_z[t * z_stride]));
    float v[V];
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = 0.0f;
    for (int p = 0; p < parts; ++p) {
      const TS* src = shared + p * part_stride + t * width + col;
      float s[V];
      if constexpr (V == 4 && sizeof(TS) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(src);
        s[0] = __uint_as_float(raw.x << 16); s[1] = __uint_as_float(raw.x & 0xffff0000u);
        s[2] = __uint_as_float(raw.y << 16); s[3] = __uint_as_float(raw.y & 0xffff0000u);
      } else if constexpr (V == 4) {
        const float4 raw = *reinterpret_cast<const float4*>(src);
        s[0] = raw.x; s[1] = raw.y; s[2] = raw.z; s[3] = raw.w;
      } else {
        s[0] = to_float(src[0]);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += s[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) sum[j] = fmaf(g, v[j], sum[j]);
  }
  TO* dst = y + t * width + col;
  if constexpr (V == 4 && sizeof(TO) == 2) {
    __nv_bfloat162 a = __floats2bfloat162_rn(sum[0], sum[1]), b = __floats2bfloat162_rn(sum[2], sum[3]);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) dst[j] = from_float<TO>(sum[j]);
  }
}

}  // namespace dl

// bias (joins the logits), correction (joins the scores for the choice alone): float32 [E] or null; sigmoid_scores 0: softmax over all experts; group_top2 0: a group's largest choice score.
DL_EXPORT int dl_moe_route(const float* logits, int stride, int tokens, int E, int top, int groups, int keep,
                           const float* bias, const float* correction, int sigmoid_scores, int group_top2, int renormalize, float scale, int* ids,
                           float* weights, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (E <= 0 || E > dl::MOE_MAX_EXPERTS || top <= 0 || top > E || groups <= 0 || E % groups || keep <= 0 || keep > groups ||
      top > keep * (E / groups))
    return DL_ERR_UNSUPPORTED;
  constexpr int WARPS = dl::MOE_ROUTE_WARPS;
  dl::moe_route_kernel<<<(tokens + WARPS - 1) / WARPS, WARPS * 32, 0, stream>>>(logits, stride, tokens, E, top, groups, keep, bias, correction,
                                                                               sigmoid_scores, group_top2, renormalize, scale, ids, weights);
  return dl::launch_status();
}

DL_EXPORT int dl_moe_group(const int* ids, int pairs, int E, int* place_of, int* pair_at, int* tiles, int* n_tiles,
                           int tile_rows, cudaStream_t stream) {
  if (pairs <= 0) return 0;
  if (E <= 0 || E > dl::MOE_MAX_EXPERTS || (tile_rows != dl::MOE_TM && tile_rows != dl::MOE_TM_WIDE)) return DL_ERR_UNSUPPORTED;
  dl::moe_group_kernel<<<1, 1024, 0, stream>>>(ids, pairs, E, place_of, pair_at, tiles, n_tiles, tile_rows);
  return dl::launch_status();
}

// dtype of a and w: 0 float32, 1 bfloat16; out_dtype of c likewise. pair_at null: the rows of a are the places
// themselves; else the row of a place is pair_at[place] / top_div. act: 0 none, 1 squared ReLU, 2 pairs (N even; c has N / 2
// columns). tensor_cores: use the
// mma.sync kernels where they apply (bfloat16, K a multiple of 64, rows of a and w on 16-byte boundaries).
// tile_rows: the places a tile as dl_moe_group was told: 32, or 128 for the wide tensor-core kernel (bfloat16 only).
DL_EXPORT int dl_moe_linear(int dtype, int out_dtype, const void* a, int lda, const int* pair_at, int top_div, const void* w,
                            int N, int K, void* c, int ldc, const int* tiles, const int* n_tiles, int max_tiles, int act,
                            int tensor_cores, int tile_rows, cudaStream_t stream) {
  if (max_tiles <= 0) return 0;
  if (N <= 0 || K <= 0 || top_div <= 0 || max_tiles > 65535 || act < 0 || act > 2 || (act == 2 && (N & 1))) return DL_ERR_UNSUPPORTED;
  const bool wide = tile_rows == dl::MOE_TM_WIDE;
  if (!wide && tile_rows != dl::MOE_TM) return DL_ERR_UNSUPPORTED;
  const bool tc_ok = dtype == 1 && tensor_cores && K % 64 == 0 && lda % 8 == 0 && (reinterpret_cast<uintptr_t>(a) & 15) == 0 &&
                     (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  if (wide && !tc_ok) return DL_ERR_UNSUPPORTED;
  if (tc_ok) {
    dim3 grid((N + 127) / 128, max_tiles);
#define DL_MOE_TC_ONE(TM_, WM_, BK_, TO)                                                                                  \
  do {                                                                                                                    \
    constexpr int ST = 3;                                                                                                 \
    constexpr int smem = ST * (TM_ + 128) * (BK_ + 8) * 2;                                                                \
    static bool configured = false;                                                                                       \
    if (!configured) {                                                                                                    \
      cudaError_t e = cudaFuncSetAttribute(dl::moe_linear_tc_kernel<TM_, WM_, BK_, ST, TO>,                               \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, smem);                            \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                   \
      configured = true;                                                                                                  \
    }                                                                                                                     \
    dl::moe_linear_tc_kernel<TM_, WM_, BK_, ST, TO><<<grid, 256, smem, stream>>>(                                         \
        static_cast<const dl::bf16*>(a), lda, pair_at, top_div, static_cast<const dl::bf16*>(w), N, K, static_cast<TO*>(c), \
        ldc, tiles, n_tiles, act);                                                                                        \
  } while (0)
#define DL_MOE_TC(TO)                                         \
  do {                                                        \
    if (wide) DL_MOE_TC_ONE(dl::MOE_TM_WIDE, 2, 64, TO);      \
    else DL_MOE_TC_ONE(dl::MOE_TM, 1, 64, TO);                \
  } while (0)
    if (out_dtype == 1) DL_MOE_TC(dl::bf16);
    else if (out_dtype == 0) DL_MOE_TC(float);
    else return DL_ERR_UNSUPPORTED;
#undef DL_MOE_TC
#undef DL_MOE_TC_ONE
    return dl::launch_status();
  }
  dim3 grid((N + 63) / 64, max_tiles);
#define DL_MOE(T, TO)                                                                                                      \
  dl::moe_linear_simt_kernel<T, TO><<<grid, 256, 0, stream>>>(static_cast<const T*>(a), lda, pair_at, top_div,              \
                                                              static_cast<const T*>(w), N, K, static_cast<TO*>(c), ldc, tiles, \
                                                              n_tiles, act)
  if (dtype == 0 && out_dtype == 0) DL_MOE(float, float);
  else if (dtype == 1 && out_dtype == 1) DL_MOE(dl::bf16, dl::bf16);
  else if (dtype == 1 && out_dtype == 0) DL_MOE(dl::bf16, float);
  else return DL_ERR_UNSUPPORTED;
#undef DL_MOE
  return dl::launch_status();
}

// out [pairs, K] = the rows of a (bf16, K a multiple of 8, lda a multiple of 8, both 16-byte aligned) in place order.
DL_EXPORT int dl_moe_gather(const void* a, int lda, const int* pair_at, int top_div, void* out, int pairs, int K,
                            cudaStream_t stream) {
  if (pairs <= 0) return 0;
  if (K <= 0 || (K & 7) || (lda & 7) || top_div <= 0 || (reinterpret_cast<uintptr_t>(a) & 15) || (reinterpret_cast<uintptr_t>(out) & 15))
    return DL_ERR_UNSUPPORTED;
  const size_t total = static_cast<size_t>(pairs) * (K / 8);
  dl::moe_gather_kernel<<<static_cast<unsigned>((total + 255) / 256), 256, 0, stream>>>(
      static_cast<const uint4*>(a), lda / 8, pair_at, top_div, static_cast<uint4*>(out), K / 8, total);
  return dl::launch_status();
}

// shared: the shared expert's output [parts][tokens, width] (part_stride elements apart; shared_dtype) with its gate's logits
// at shared_z[t * z_stride] (float32), or null.
DL_EXPORT int dl_moe_combine(int out_dtype, const float* c, int width, const int* place_of, const float* weights, int top,
                             int shared_dtype, const void* shared, int parts, long long part_stride, const float* shared_z,
                             int z_stride, void* y, int tokens, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (shared != nullptr && (parts <= 0 || shared_z == nullptr)) return DL_ERR_UNSUPPORTED;
  const bool wide = width % 4 == 0 && part_stride % 4 == 0 &&
                    ((reinterpret_cast<uintptr_t>(c) | reinterpret_cast<uintptr_t>(shared) | reinterpret_cast<uintptr_t>(y)) & 15) == 0;
  const size_t total = static_cast<size_t>(tokens) * (wide ? width / 4 : width);
  const unsigned blocks = static_cast<unsigned>((total + 255) / 256);
#define DL_MC(TO, TS, V)                                                                                              \
  dl::moe_combine_kernel<TO, TS, V><<<blocks, 256, 0, stream>>>(c, width, place_of, weights, top, static_cast<const TS*>(shared), \
                                                                parts, static_cast<size_t>(part_stride), shared_z, z_stride,     \
                                                                static_cast<TO*>(y), total)
#define DL_MCV(TO, TS)            \
  do {                            \
    if (wide) DL_MC(TO, TS, 4);   \
    else DL_MC(TO, TS, 1);        \
  } while (0)
  if (out_dtype == 0 && shared_dtype == 0) DL_MCV(float, float);
  else if (out_dtype == 1 && shared_dtype == 0) DL_MCV(dl::bf16, float);
  else if (out_dtype == 1 && shared_dtype == 1) DL_MCV(dl::bf16, dl::bf16);
  else return DL_ERR_UNSUPPORTED;
#undef DL_MCV
#undef DL_MC
  return dl::launch_status();
}
