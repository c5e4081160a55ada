// The gated delta rule: a matrix state per head that forgets, corrects and then is read, token by token.
//
// Per token and head h (query/key head j = h / (H / G), key size d, value size e), all in float32:
//
//   q = q_j / sqrt(sum(q_j^2) + 1e-6) * d^(-1/2),   k = k_j / sqrt(sum(k_j^2) + 1e-6)
//   beta = sigmoid(b_h),   g = exp(-exp(A_h) * softplus(a_h + dt_h))
//   S <- g S;   u = beta (v_h - S^T k);   S <- S + k u^T;   o_h = S^T q            (S is d x e, it starts at zero)
//
// or with a decay per key channel, g_i = exp(-exp(A_h) * softplus(z_i + dt_i)) for row i of S, i < d (the raw numbers z of
// every head and channel are float32 rows of their own; dl_delta_decay forms g in place once per token for portions of
// prompts, the kernel of single tokens forms it itself).
//
// q, k and v come from the short convolution's output (columns q | k | v of a row), b, a and the output gate from the
// projection's row. What a request keeps is S of every head, float32 [H][d][e], at the head of its state row.
//
// Tokens are taken in runs of four. With S the state in front of a run, G_t the product of the run's decays up to token t
// and D_st that from behind token s up to t,
//
//   u_t = beta_t (v_t - S^T (G_t k_t) - sum_{s<t} u_s (D_st k_s . k_t)),   o_t = S^T (G_t q_t) + sum_{s<=t} u_s (D_st k_s . q_t)
//   S <- G_4 S + sum_s (D_s4 k_s) u_s^T
//
// so all dot products of a run over S are independent of one another, and what one token does to the next is a triangle of
// four numbers a column; the sixteen dot products in brackets are the same for every column.
//
// Block = (slice of the e columns, head, request), 256 threads: four warps that compute and four that fetch.
// A computing lane holds R rows of FOUR columns of S in registers, so that a number read from shared memory serves four
// multiply-adds (what a lane reads, not what banks deliver, limits shared memory here); P neighbouring lanes hold a column's
// rows. A run's 8 x 4 dot products are finished by shuffles: two rounds hand every lane one of the four columns (its slot s
// holds column s xor lane % 4 of the four, so that nothing has to be selected), the rest finish the sums; after the triangle
// the lanes swap what they write into their columns. A request's tokens are walked in tiles
// of 16 (of 8 for heads of more than 256) held twice in shared memory: while the computing warps run a tile's runs over
// their registers, each fetching warp writes a run of the next tile (queries and keys made unit vectors and multiplied by
// their decays; the run's dot products; write strengths; the values of the block's columns) and asks for the one after it,
// whose numbers then have a whole tile's time to arrive in its registers: no token waits for global memory. Tokens past a
// tile's end are zeros with a decay of 1 and change nothing.
//
// dl_head_norm_gate: out[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * w * act(gate[t, h, :]), act silu or sigmoid.
#include "common.cuh"

namespace dl {

constexpr int DR_RUN = 4;                               // tokens of a run
constexpr int DR_COLS = 4;                              // columns of a lane
constexpr int DR_COMPUTE = 128;
constexpr int DR_THREADS = 256;

__device__ __forceinline__ float dr_softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }

template <int R, int P>
struct DrTile {
  static constexpr int TT = R > 8 ? 8 : 16;             // tokens of a tile
  static constexpr int RUNS = TT / DR_RUN;
  static constexpr int RS = R % 8 == 0 ? R + 4 : R;     // floats between two lanes' rows: 16-byte loads in different banks
  static constexpr int TS = P * RS;                     // floats of one token's query (or key)
  static constexpr int COLS = DR_COMPUTE / P * DR_COLS;
  // G_t k_t | G_t q_t | D_t4 k_t of every token, G_4 of every run, the triangles of every run (t-th row: against the keys
  // s < t, against the query s <= t), write strengths, values
  static constexpr int Q = TT * TS, KD = 2 * TT * TS, G = 3 * TT * TS;
  static constexpr int TRI = G + RUNS * TS, BETA = TRI + RUNS * 2 * DR_RUN * DR_RUN, V = BETA + TT;
  static constexpr int FLOATS = V + TT * COLS;
};

// What a fetching thread holds of one tile between asking for it and writing it to shared memory: of its warp's run the
// numbers lane, lane + 32, ... of every query, key and row of decays, and lane t < 4 the write strength (and step size) of
// token t; as they lie in memory, so that nothing waits for a load before the tile is written.
template <typename T, int R, int P, bool CH>
struct DrRaw {
  static constexpr int NL = (R * P + 31) / 32;
  static constexpr int NV = (DrTile<R, P>::TT * DrTile<R, P>::COLS + DR_COMPUTE - 1) / DR_COMPUTE;
  float g[CH ? DR_RUN : 1][CH ? NL : 1];
  T q[DR_RUN][NL], k[DR_RUN][NL], v[NV], b, a;
};

// A lane's R rows of a vector in shared memory.
template <int R>
__device__ __forceinline__ void dr_rows(const float* p, float* x) {
  if constexpr (R % 4 == 0) {
#pragma unroll
    for (int i = 0; i < R; i += 4) {
      const float4 v = *reinterpret_cast<const float4*>(p + i);
      x[i] = v.x;
      x[i + 1] = v.y;
      x[i + 2] = v.z;
      x[i + 3] = v.w;
    }
  } else {
    const float2 v = *reinterpret_cast<const float2*>(p);
    x[0] = v.x;
    x[1] = v.y;
  }
}

// The fetching warps ask for tile [first_row, first_row + tn) of the request's rows: every load is issued, none is
// waited for. The tile is asked for one tile's time before it is written, so its numbers are there by then.
template <typename T, int R, int P, bool CH>
__device__ __forceinline__ void dr_ask(DrRaw<T, R, P, CH>& raw, const T* __restrict__ u, int u_stride, int q_at, int k_at,
                                       int v_at, const T* __restrict__ proj, int proj_stride, int b_at, int a_at,
                                       const float* __restrict__ decay, int decay_stride, int first_row, int tn, int d, int e,
                                       int col0, int lt) {
  using L = DrTile<R, P>;
  using W = DrRaw<T, R, P, CH>;
  const int lane = lt & 31, run0 = (lt >> 5) * DR_RUN;
  const T zero = from_float<T>(0.0f);
  raw.b = zero;
  raw.a = zero;
  if (run0 < L::TT) {
#pragma unroll
    for (int t = 0; t < DR_RUN; ++t) {
      const int tt = run0 + t;
      const size_t row = static_cast<size_t>(first_row + max(min(tt, tn - 1), 0));
      const T* urow = u + row * u_stride;
#pragma unroll
      for (int c = 0; c < W::NL; ++c) {
        const int i = lane + 32 * c;
        const bool ok = tt < tn && i < d;
        raw.q[t][c] = ok ? urow[q_at + i] : zero;
        raw.k[t][c] = ok ? urow[k_at + i] : zero;
        if constexpr (CH) raw.g[t][c] = ok ? decay[row * decay_stride + i] : 1.0f;
      }
    }
    if (lane < DR_RUN && run0 + lane < tn) {
      const T* prow = proj + static_cast<size_t>(first_row + run0 + lane) * proj_stride;
      raw.b = prow[b_at];
      if constexpr (!CH) raw.a = prow[a_at];
    }
  }
#pragma unroll
  for (int c = 0; c < W::NV; ++c) {
    const int idx = lt + DR_COMPUTE * c;
    const int tt = idx / L::COLS, col = col0 + idx % L::COLS;
    raw.v[c] = (tt < tn && col < e) ? u[static_cast<size_t>(first_row + tt) * u_stride + v_at + col] : zero;
  }
}

// ... and write it into one of the two buffers.
template <typename T, int R, int P, bool CH>
__device__ __forceinline__ void dr_put(const DrRaw<T, R, P, CH>& raw, float* buf, int tn, int d, float q_scale, float decay_rate,
                                       float bias, int lt) {
  using L = DrTile<R, P>;
  using W = DrRaw<T, R, P, CH>;
  const int lane = lt & 31, run = lt >> 5, run0 = run * DR_RUN;
#pragma unroll
  for (int c = 0; c < W::NV; ++c) {
    const int idx = lt + DR_COMPUTE * c;
    if (idx < L::TT * L::COLS) buf[L::V + idx] = to_float(raw.v[c]);
  }
  if (run0 >= L::TT) return;                            // (a whole warp)
  float gs[DR_RUN];                                     // one decay a token
  if constexpr (!CH) {
    const float mine = lane < DR_RUN && run0 + lane < tn ? expf(-decay_rate * dr_softplus(to_float(raw.a) + bias)) : 1.0f;
#pragma unroll
    for (int t = 0; t < DR_RUN; ++t) gs[t] = __shfl_sync(0xffffffffu, mine, t);
  }
  auto g_of = [&](int t, int c) {
    if constexpr (CH) return raw.g[t][c];
    else return gs[t];
  };
  // sums over the channels: 0..3 q.q, 4..7 k.k, 8..13 (D_st k_s).k_t for s < t, 14..23 (D_st k_s).q_t for s <= t
  float sum[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) sum[i] = 0.0f;
#pragma unroll
  for (int c = 0; c < W::NL; ++c) {
    float q[DR_RUN], k[DR_RUN];
#pragma unroll
    for (int t = 0; t < DR_RUN; ++t) {
      q[t] = to_float(raw.q[t][c]);
      k[t] = to_float(raw.k[t][c]);
      sum[t] = fmaf(q[t], q[t], sum[t]);
      sum[4 + t] = fmaf(k[t], k[t], sum[4 + t]);
    }
    int a = 8, b = 14;
#pragma unroll
    for (int s = 0; s < DR_RUN; ++s) {
      float w = k[s];
#pragma unroll
      for (int t = s; t < DR_RUN; ++t) {
        if (t > s) {
          w *= g_of(t, c);
          sum[a] = fmaf(w, k[t], sum[a]);
          ++a;
        }
        sum[b] = fmaf(w, q[t], sum[b]);
        ++b;
      }
    }
  }
  // every round halves the sums a lane is in charge of: in the end lane i holds sum i over all lanes
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? sum[i] : sum[i + o], keep = up ? sum[i + o] : sum[i];
      sum[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  const float f = lane < 8 ? (lane < 4 ? q_scale : 1.0f) / sqrtf(sum[0] + 1e-6f) : 0.0f;      // to unit length
  {
    const bool keys = lane < 14;
    int s = 0, t = 0;
    if (lane >= 8 && lane < 24) {                       // which pair of tokens this lane's sum is of
      int n = keys ? lane - 8 : lane - 14, len = keys ? DR_RUN - 1 : DR_RUN;
      while (n >= len) { n -= len; --len; ++s; }
      t = s + n + (keys ? 1 : 0);
    }
    const float fs = __shfl_sync(0xffffffffu, f, 4 + s), ft = __shfl_sync(0xffffffffu, f, keys ? 4 + t : t);
    if (lane >= 8 && lane < 24) buf[L::TRI + (run * 2 + (keys ? 0 : 1)) * DR_RUN * DR_RUN + t * DR_RUN + s] = sum[0] * fs * ft;
  }
  float fq[DR_RUN], fk[DR_RUN];
#pragma unroll
  for (int t = 0; t < DR_RUN; ++t) {
    fq[t] = __shfl_sync(0xffffffffu, f, t);
    fk[t] = __shfl_sync(0xffffffffu, f, 4 + t);
  }
#pragma unroll
  for (int c = 0; c < W::NL; ++c) {
    const int i = lane + 32 * c;
    if (i < d) {
      const int at = (i / R) * L::RS + i % R;
      float G = 1.0f;
#pragma unroll
      for (int t = 0; t < DR_RUN; ++t) {
        G *= g_of(t, c);
        buf[(run0 + t) * L::TS + at] = to_float(raw.k[t][c]) * fk[t] * G;
        buf[L::Q + (run0 + t) * L::TS + at] = to_float(raw.q[t][c]) * fq[t] * G;
      }
      buf[L::G + run * L::TS + at] = G;
      float D = 1.0f;
#pragma unroll
      for (int t = DR_RUN - 1; t >= 0; --t) {
        buf[L::KD + (run0 + t) * L::TS + at] = to_float(raw.k[t][c]) * fk[t] * D;
        D *= g_of(t, c);
      }
    }
  }
  if (lane < DR_RUN) buf[L::BETA + run0 + lane] = run0 + lane < tn ? 1.0f / (1.0f + expf(-to_float(raw.b))) : 0.0f;
}

template <typename T, int R, int P, bool CH>
__global__ void __launch_bounds__(DR_THREADS)
delta_rule_kernel(const T* __restrict__ u, int u_stride, int q_col, int k_col, int v_col,
                  const T* __restrict__ proj, int proj_stride, int b_col, int a_col,
                  const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ decays,
                  int decay_stride, float* __restrict__ state, size_t state_stride, const int* __restrict__ q_start,
                  const int* __restrict__ state_slots, float* __restrict__ out, int H, int G, int d, int e) {
  using L = DrTile<R, P>;
  extern __shared__ __align__(16) float sm[];   // two tiles
  const int h = blockIdx.y, r = blockIdx.z;
  const int j = h / (H / G);
  const int tid = threadIdx.x;
  const int col0 = blockIdx.x * L::COLS;
  const int row0 = q_start[r], n = q_start[r + 1] - row0;
  if (n <= 0) return;
  const float q_scale = rsqrtf(static_cast<float>(d));
  const float decay_rate = CH ? 0.0f : expf(a_log[h]), bias = CH ? 0.0f : dt_bias[h];
  const float* decay = CH ? decays + static_cast<size_t>(h) * d : nullptr;
  const int q_at = q_col + j * d, k_at = k_col + j * d, v_at = v_col + h * e, b_at = b_col + h, a_at = a_col + h;

  // rows past d (a lane's share rounded up) and the empty halves of the triangles stay zero in both tiles
  for (int idx = tid; idx < 2 * L::FLOATS; idx += DR_THREADS) sm[idx] = 0.0f;
  __syncthreads();

  const bool computes = tid < DR_COMPUTE;
  const int part = tid % P, four = tid / P * DR_COLS, mine = part & 3;
  const int cl = four + mine, col = col0 + cl;          // the lane's own column of its four
  const bool live = computes && col < e;
  float* S_g = state + static_cast<size_t>(ck_request(state_slots[r])) * state_stride + static_cast<size_t>(h) * d * e;
  float S[DR_COLS][R];
  DrRaw<T, R, P, CH> raw;
  const int lt = tid - DR_COMPUTE;
  if (computes) {
#pragma unroll
    for (int c = 0; c < DR_COLS; ++c) {
      const int cc = col0 + four + (c ^ mine);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int row = part * R + i;
        S[c][i] = (cc < e && row < d) ? S_g[static_cast<size_t>(row) * e + cc] : 0.0f;
      }
    }
  } else {
    dr_ask<T, R, P, CH>(raw, u, u_stride, q_at, k_at, v_at, proj, proj_stride, b_at, a_at, decay, decay_stride, row0,
                        min(L::TT, n), d, e, col0, lt);
    dr_put<T, R, P, CH>(raw, sm, min(L::TT, n), d, q_scale, decay_rate, bias, lt);
    if (n > L::TT)
      dr_ask<T, R, P, CH>(raw, u, u_stride, q_at, k_at, v_at, proj, proj_stride, b_at, a_at, decay, decay_stride,
                          row0 + L::TT, min(L::TT, n - L::TT), d, e, col0, lt);
  }
  __syncthreads();

  int which = 0;
  for (int t0 = 0; t0 < n; t0 += L::TT, which ^= 1) {
    const int tn = min(L::TT, n - t0);
    if (!computes) {
      // the tile after this one was asked for a tile ago: write it, then ask for the one after it
      if (t0 + L::TT < n) {
        dr_put<T, R, P, CH>(raw, sm + (which ^ 1) * L::FLOATS, min(L::TT, n - t0 - L::TT), d, q_scale, decay_rate, bias, lt);
        if (t0 + 2 * L::TT < n)
          dr_ask<T, R, P, CH>(raw, u, u_stride, q_at, k_at, v_at, proj, proj_stride, b_at, a_at, decay, decay_stride,
                              row0 + t0 + 2 * L::TT, min(L::TT, n - t0 - 2 * L::TT), d, e, col0, lt);
      }
    } else {
      const float* buf = sm + which * L::FLOATS;
      for (int run = 0; run * DR_RUN < tn; ++run) {
        const float* kg = buf + run * DR_RUN * L::TS + part * L::RS;
        float a[DR_RUN][DR_COLS], o[DR_RUN][DR_COLS];
#pragma unroll
        for (int t = 0; t < DR_RUN; ++t) {
          float kv[R], qv[R];
          dr_rows<R>(kg + t * L::TS, kv);
          dr_rows<R>(kg + L::Q + t * L::TS, qv);
#pragma unroll
          for (int c = 0; c < DR_COLS; ++c) {
            a[t][c] = S[c][0] * kv[0];
            o[t][c] = S[c][0] * qv[0];
          }
#pragma unroll
          for (int i = 1; i < R; ++i) {
#pragma unroll
            for (int c = 0; c < DR_COLS; ++c) {
              a[t][c] = fmaf(S[c][i], kv[i], a[t][c]);
              o[t][c] = fmaf(S[c][i], qv[i], o[t][c]);
            }
          }
        }
        // every lane its own column: slots 1 and 3, then slot 2 go to the lanes whose own columns they are
#pragma unroll
        for (int t = 0; t < DR_RUN; ++t) {
#pragma unroll
          for (int c = 0; c < DR_COLS; c += 2) {
            a[t][c] += __shfl_xor_sync(0xffffffffu, a[t][c + 1], 1);
            o[t][c] += __shfl_xor_sync(0xffffffffu, o[t][c + 1], 1);
          }
        }
        float as[DR_RUN], os[DR_RUN];
#pragma unroll
        for (int t = 0; t < DR_RUN; ++t) {
          as[t] = a[t][0] + __shfl_xor_sync(0xffffffffu, a[t][2], 2);
          os[t] = o[t][0] + __shfl_xor_sync(0xffffffffu, o[t][2], 2);
        }
#pragma unroll
        for (int x = P >> 1; x > 2; x >>= 1) {
#pragma unroll
          for (int t = 0; t < DR_RUN; ++t) as[t] += __shfl_xor_sync(0xffffffffu, as[t], x);
        }
        const float* tri = buf + L::TRI + run * 2 * DR_RUN * DR_RUN;
        const float4 beta = *reinterpret_cast<const float4*>(buf + L::BETA + run * DR_RUN);
        const float* v = buf + L::V + run * DR_RUN * L::COLS + cl;
        const float4 t2 = *reinterpret_cast<const float4*>(tri + 2 * DR_RUN), t3 = *reinterpret_cast<const float4*>(tri + 3 * DR_RUN);
        float w[DR_RUN][DR_COLS];                       // what every token writes into the lane's columns; slot 0: its own
        w[0][0] = beta.x * (v[0] - as[0]);
        w[1][0] = beta.y * (v[L::COLS] - as[1] - tri[DR_RUN] * w[0][0]);
        w[2][0] = beta.z * (v[2 * L::COLS] - as[2] - t2.x * w[0][0] - t2.y * w[1][0]);
        w[3][0] = beta.w * (v[3 * L::COLS] - as[3] - t3.x * w[0][0] - t3.y * w[1][0] - t3.z * w[2][0]);
#pragma unroll
        for (int t = 0; t < DR_RUN; ++t) {
#pragma unroll
          for (int c = 1; c < DR_COLS; ++c) w[t][c] = __shfl_xor_sync(0xffffffffu, w[t][0], c);
        }
        {
          float gv[R], kv[DR_RUN][R];
          dr_rows<R>(buf + L::G + run * L::TS + part * L::RS, gv);
#pragma unroll
          for (int t = 0; t < DR_RUN; ++t) dr_rows<R>(kg + L::KD + t * L::TS, kv[t]);
#pragma unroll
          for (int i = 0; i < R; ++i) {
#pragma unroll
            for (int c = 0; c < DR_COLS; ++c) S[c][i] *= gv[i];
#pragma unroll
            for (int t = 0; t < DR_RUN; ++t) {
#pragma unroll
              for (int c = 0; c < DR_COLS; ++c) S[c][i] = fmaf(kv[t][i], w[t][c], S[c][i]);
            }
          }
        }
        // the four read-outs of the lane's column: up to two rounds share them out among its lanes, the rest finish the sums
        const float* tq = tri + DR_RUN * DR_RUN;
        float* orow = out + static_cast<size_t>(row0 + t0 + run * DR_RUN) * (H * e) + h * e + col;
        auto write = [&](int t, float sum) {
          if (run * DR_RUN + t < tn) {
            const float4 f = *reinterpret_cast<const float4*>(tq + t * DR_RUN);
            orow[static_cast<size_t>(t) * (H * e)] = fmaf(f.w, w[3][0], fmaf(f.z, w[2][0], fmaf(f.y, w[1][0], fmaf(f.x, w[0][0], sum))));
          }
        };
        if constexpr (P >= 8) {
          const bool hi = part & (P >> 1);
          float x0 = (hi ? os[2] : os[0]) + __shfl_xor_sync(0xffffffffu, hi ? os[0] : os[2], P >> 1);
          float x1 = (hi ? os[3] : os[1]) + __shfl_xor_sync(0xffffffffu, hi ? os[1] : os[3], P >> 1);
          if constexpr (P >= 16) {
            const bool lo = part & (P >> 2);
            float y = (lo ? x1 : x0) + __shfl_xor_sync(0xffffffffu, lo ? x0 : x1, P >> 2);
#pragma unroll
            for (int x = P >> 3; x > 2; x >>= 1) y += __shfl_xor_sync(0xffffffffu, y, x);
            if (live && (part & ((P >> 2) - 1)) < 4) write((hi ? 2 : 0) + (lo ? 1 : 0), y);
          } else if (live) {
            write(hi ? 2 : 0, x0);
            write(hi ? 3 : 1, x1);
          }
        } else if (live) {
#pragma unroll
          for (int t = 0; t < DR_RUN; ++t) write(t, os[t]);
        }
      }
    }
    __syncthreads();                            // the tile has been read, the next one is whole
  }
  if (computes) {
#pragma unroll
    for (int c = 0; c < DR_COLS; ++c) {
      const int cc = col0 + four + (c ^ mine);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int row = part * R + i;
        if (cc < e && row < d) S_g[static_cast<size_t>(row) * e + cc] = S[c][i];
      }
    }
  }
}

// Steps of single tokens (decoding): what counts is the state's trip through memory, H d e floats read and written a
// request. Block = (32 columns, head, request), 128 threads as 32 columns x 4 runs of rows, so that a warp reads 128
// bytes of a state row at once and many light blocks share an SM. The block's slice of S waits in shared memory
// between the two dot products and the update. A request that brought several tokens is walked token by token
// (correct, not fast: the host sends such steps to the tiled kernel above); one that brought none is left alone.
constexpr int DS_COLS = 32;
constexpr int DS_RUNS = 4;

template <typename T, bool CH>
__global__ void __launch_bounds__(DS_COLS * DS_RUNS)
delta_rule_step_kernel(const T* __restrict__ u, int u_stride, int q_col, int k_col, int v_col,
                       const T* __restrict__ proj, int proj_stride, int b_col, int a_col,
                       const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ decays,
                       int decay_stride, float* __restrict__ state, size_t state_stride, const int* __restrict__ q_start,
                       const int* __restrict__ state_slots, float* __restrict__ out, int H, int G, int d, int e) {
  extern __shared__ __align__(16) float sm[];
  float* sS = sm;                               // [d][DS_COLS]
  float* sk = sS + static_cast<size_t>(d) * DS_COLS;      // [d]
  float* sq = sk + d;                           // [d]
  float* part = sq + d;                         // [2][DS_RUNS][DS_COLS]
  float* sgd = part + 2 * DS_RUNS * DS_COLS;    // [d], with a decay per channel
  __shared__ float red[33];
  const int h = blockIdx.y, r = blockIdx.z;
  const int j = h / (H / G);
  const int tid = threadIdx.x, c = tid % DS_COLS, run = tid / DS_COLS;
  const int col = blockIdx.x * DS_COLS + c;
  const bool live = col < e;
  const int row0 = q_start[r], row1 = q_start[r + 1];
  if (row1 <= row0) return;
  float* S_g = state + static_cast<size_t>(ck_request(state_slots[r])) * state_stride + static_cast<size_t>(h) * d * e;
  const float q_scale = rsqrtf(static_cast<float>(d));
  const float decay_rate = expf(a_log[h]), bias = CH ? 0.0f : dt_bias[h];
  for (int row = row0; row < row1; ++row) {
    const T* urow = u + static_cast<size_t>(row) * u_stride;
    float qq = 0.0f, kk = 0.0f, kq = 0.0f;
    for (int i = tid; i < d; i += DS_COLS * DS_RUNS) {
      const float a = to_float(urow[q_col + j * d + i]), b = to_float(urow[k_col + j * d + i]);
      sq[i] = a;
      sk[i] = b;
      qq = fmaf(a, a, qq);
      kk = fmaf(b, b, kk);
      kq = fmaf(a, b, kq);
      if constexpr (CH)
        sgd[i] = expf(-decay_rate * dr_softplus(decays[static_cast<size_t>(row) * decay_stride + h * d + i] + dt_bias[h * d + i]));
    }
    float dot = 0.0f, rd = 0.0f;
    if (row == row0) {                          // the state comes in under the three sums
#pragma unroll 8
      for (int i = run; i < d; i += DS_RUNS) sS[i * DS_COLS + c] = live ? S_g[static_cast<size_t>(i) * e + col] : 0.0f;
    }
    qq = block_sum(qq, red);
    kk = block_sum(kk, red);
    kq = block_sum(kq, red);
    const float fq = q_scale / sqrtf(qq + 1e-6f), fk = 1.0f / sqrtf(kk + 1e-6f);
    const T* prow = proj + static_cast<size_t>(row) * proj_stride;
    const float beta = 1.0f / (1.0f + expf(-to_float(prow[b_col + h])));
    const float g = CH ? 1.0f : expf(-decay_rate * dr_softplus(to_float(prow[a_col + h]) + bias));
    const float v = live ? to_float(urow[v_col + h * e + col]) : 0.0f;
#pragma unroll 8
    for (int i = run; i < d; i += DS_RUNS) {
      const float s = CH ? sgd[i] * sS[i * DS_COLS + c] : sS[i * DS_COLS + c];
      dot = fmaf(s, sk[i], dot);
      rd = fmaf(s, sq[i], rd);
    }
    part[run * DS_COLS + c] = dot;
    part[(DS_RUNS + run) * DS_COLS + c] = rd;
    __syncthreads();
    dot = 0.0f;
    rd = 0.0f;
#pragma unroll
    for (int w = 0; w < DS_RUNS; ++w) {
      dot += part[w * DS_COLS + c];
      rd += part[(DS_RUNS + w) * DS_COLS + c];
    }
    // with S' = g S + k u^T:  S'^T q = g S^T q + u (k . q)
    const float uval = beta * (v - g * fk * dot);
    if (live && run == 0) out[static_cast<size_t>(row) * (H * e) + h * e + col] = fmaf(uval, kq * fq * fk, g * fq * rd);
    const float ku = uval * fk;
    const bool last = row + 1 == row1;
#pragma unroll 8
    for (int i = run; i < d; i += DS_RUNS) {
      const float s = fmaf(sk[i], ku, (CH ? sgd[i] : g) * sS[i * DS_COLS + c]);
      if (last) {
        if (live) S_g[static_cast<size_t>(i) * e + col] = s;
      } else {
        sS[i * DS_COLS + c] = s;
      }
    }
    __syncthreads();                            // sk, sq and the partial sums are free again
  }
}

// z (raw numbers of H heads of d channels, float32) -> exp(-exp(A_h) softplus(z + dt)), in place.
__global__ void delta_decay_kernel(float* __restrict__ z, int stride, const float* __restrict__ a_log,
                                   const float* __restrict__ dt_bias, int H, int d, size_t total) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int c = static_cast<int>(i % (H * d));
  float* p = z + (i / (H * d)) * stride + c;
  *p = expf(-expf(a_log[c / d]) * dr_softplus(*p + dt_bias[c]));
}

// The same for channels in fours (d a multiple of 4, 16-byte rows).
__global__ void delta_decay_vec_kernel(float* __restrict__ z, int stride, const float* __restrict__ a_log,
                                       const float* __restrict__ dt_bias, int H, int d, size_t total) {
  const size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int per = H * d / 4, c = static_cast<int>(i % per) * 4;
  float4* p = reinterpret_cast<float4*>(z + (i / per) * stride + c);
  const float4 b = *reinterpret_cast<const float4*>(dt_bias + c);
  const float rate = -expf(a_log[c / d]);
  float4 v = *p;
  v.x = expf(rate * dr_softplus(v.x + b.x));
  v.y = expf(rate * dr_softplus(v.y + b.y));
  v.z = expf(rate * dr_softplus(v.z + b.z));
  v.w = expf(rate * dr_softplus(v.w + b.w));
  *p = v;
}

// One warp per (row, head); TG: the gate's type.
template <typename T, typename TG>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, const TG* __restrict__ gate, int gate_stride, int gate_col,
                                      const float* __restrict__ w, float eps, int sigmoid_gate, T* __restrict__ out, int rows, int H,
                                      int e) {
  const int unit = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= rows * H) return;
  const int row = unit / H, h = unit % H;
  const float* orow = o + static_cast<size_t>(row) * H * e + h * e;
  float ss = 0.0f;
  for (int i = lane; i < e; i += 32) ss = fmaf(orow[i], orow[i], ss);
  const float rs = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(e) + eps);
  const TG* grow = gate + static_cast<size_t>(row) * gate_stride + gate_col + h * e;
  T* dst = out + static_cast<size_t>(row) * H * e + h * e;
  for (int i = lane; i < e; i += 32) {
    const float z = to_float(grow[i]);
    dst[i] = from_float<T>(orow[i] * rs * w[i] * ((sigmoid_gate ? 1.0f : z) / (1.0f + expf(-z))));
  }
}

template <typename T, int R, int P, bool CH>
int delta_rule_launch(const void* u, int u_stride, int q_col, int k_col, int v_col, const void* proj, int proj_stride,
                      int b_col, int a_col, const float* a_log, const float* dt_bias, const float* decays, int decay_stride,
                      float* state, long long state_stride,
                      const int* q_start, const int* state_slots, float* out, int requests, int H, int G, int d, int e,
                      cudaStream_t stream) {
  using L = DrTile<R, P>;
  const size_t smem = static_cast<size_t>(2 * L::FLOATS) * sizeof(float);
  auto kernel = delta_rule_kernel<T, R, P, CH>;
  if (smem > 48 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (err != cudaSuccess) return static_cast<int>(err);
  }
  dim3 grid((e + L::COLS - 1) / L::COLS, H, requests);
  kernel<<<grid, DR_THREADS, smem, stream>>>(static_cast<const T*>(u), u_stride, q_col, k_col, v_col,
                                             static_cast<const T*>(proj), proj_stride, b_col, a_col, a_log, dt_bias, decays,
                                             decay_stride, state, static_cast<size_t>(state_stride), q_start, state_slots, out, H, G, d, e);
  return launch_status();
}

}  // namespace dl

// u: rows of u_stride elements with q of all G heads at q_col, k at k_col (G * d each) and v of all H heads at v_col
// (H * e); proj: rows of proj_stride elements with b at b_col and a at a_col (H each); state: float32 rows of
// state_stride floats, S of head h at h * d * e; out: float32 contiguous [rows, H * e]. d up to 512.
// decays: null, or float32 rows of decay_stride numbers with H * d decays per channel (formed by dl_delta_decay; a_col and
// dt_bias are then not read).
DL_EXPORT int dl_delta_rule(int dtype, const void* u, int u_stride, int q_col, int k_col, int v_col, const void* proj,
                            int proj_stride, int b_col, int a_col, const float* a_log, const float* dt_bias,
                            const float* decays, int decay_stride, float* state, long long state_stride, const int* q_start,
                            const int* state_slots, float* out, int requests, int H, int G, int d, int e, int sm_count,
                            cudaStream_t stream) {
  if (requests <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || d <= 0 || e <= 0 || d > 512 || H > 65535 || requests > 65535 ||
      (dtype != 0 && dtype != 1))
    return DL_ERR_UNSUPPORTED;
  // four rows a lane up to d = 128 (on 4 to 32 lanes), more on 32 lanes beyond; two rows on 32 lanes where four would leave
  // SMs without a block
  int P = 4, R = 4;
  while (P < 32 && P * R < d) P *= 2;
  while (P * R < d) R += 4;
  const int cols = dl::DR_COMPUTE / P * dl::DR_COLS;
  if (P == 16 && 3ll * ((e + cols - 1) / cols) * H * requests < 2ll * sm_count) {
    P = 32;
    R = 2;
  }
#define DL_DR_T(T, RR, PP, CH)                                                                                             \
  return dl::delta_rule_launch<T, RR, PP, CH>(u, u_stride, q_col, k_col, v_col, proj, proj_stride, b_col, a_col, a_log,    \
                                              dt_bias, decays, decay_stride, state, state_stride, q_start, state_slots,    \
                                              out, requests, H, G, d, e, stream)
#define DL_DR(RR, PP)                                                                                                      \
  if (R == RR && P == PP) {                                                                                                \
    if (dtype == 0) {                                                                                                      \
      if (decays != nullptr) DL_DR_T(float, RR, PP, true);                                                                 \
      DL_DR_T(float, RR, PP, false);                                                                                       \
    }                                                                                                                      \
    if (decays != nullptr) DL_DR_T(dl::bf16, RR, PP, true);                                                                \
    DL_DR_T(dl::bf16, RR, PP, false);                                                                                      \
  }
  DL_DR(4, 4); DL_DR(4, 8); DL_DR(4, 16); DL_DR(4, 32); DL_DR(2, 32);      // d up to 16, 32, 64, 128; 33 .. 64
  DL_DR(8, 32); DL_DR(12, 32); DL_DR(16, 32);                              // d up to 256, 384, 512
#undef DL_DR
#undef DL_DR_T
  return DL_ERR_UNSUPPORTED;
}

// The same step for batches of single tokens: the same arguments, any d; `decays` holds the RAW numbers of every channel
// (dt_bias is then float32 [H * d]).
DL_EXPORT int dl_delta_rule_step(int dtype, const void* u, int u_stride, int q_col, int k_col, int v_col, const void* proj,
                                 int proj_stride, int b_col, int a_col, const float* a_log, const float* dt_bias,
                                 const float* decays, int decay_stride, float* state, long long state_stride,
                                 const int* q_start, const int* state_slots, float* out, int requests, int H, int G, int d,
                                 int e, cudaStream_t stream) {
  if (requests <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || d <= 0 || e <= 0 || H > 65535 || requests > 65535 || (dtype != 0 && dtype != 1))
    return DL_ERR_UNSUPPORTED;
  const size_t smem = (static_cast<size_t>(d) * dl::DS_COLS + (decays != nullptr ? 3 : 2) * d + 2 * dl::DS_RUNS * dl::DS_COLS) * sizeof(float);
  if (smem > 200 * 1024) return DL_ERR_UNSUPPORTED;
  dim3 grid((e + dl::DS_COLS - 1) / dl::DS_COLS, H, requests);
#define DL_DS(T, CH)                                                                                                    \
  do {                                                                                                                  \
    auto kernel = dl::delta_rule_step_kernel<T, CH>;                                                                    \
    if (smem > 48 * 1024) {                                                                                             \
      const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
      if (err != cudaSuccess) return static_cast<int>(err);                                                             \
    }                                                                                                                   \
    kernel<<<grid, dl::DS_COLS * dl::DS_RUNS, smem, stream>>>(static_cast<const T*>(u), u_stride, q_col, k_col, v_col,  \
                                                              static_cast<const T*>(proj), proj_stride, b_col, a_col,   \
                                                              a_log, dt_bias, decays, decay_stride, state,              \
                                                              static_cast<size_t>(state_stride), q_start, state_slots,  \
                                                              out, H, G, d, e);                                         \
  } while (0)
  if (dtype == 0) { if (decays != nullptr) DL_DS(float, true); else DL_DS(float, false); }
  else { if (decays != nullptr) DL_DS(dl::bf16, true); else DL_DS(dl::bf16, false); }
#undef DL_DS
  return dl::launch_status();
}

// z: float32 rows of `stride` numbers, the first H * d of each turned into decays in place; a_log: float32 [H], dt_bias:
// float32 [H * d].
DL_EXPORT int dl_delta_decay(float* z, int stride, const float* a_log, const float* dt_bias, int rows, int H, int d,
                             cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || d <= 0 || stride < H * d) return DL_ERR_UNSUPPORTED;
  const size_t total = static_cast<size_t>(rows) * H * d;
  if (d % 4 == 0 && stride % 4 == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(dt_bias)) & 15) == 0) {
    const size_t fours = total / 4;
    dl::delta_decay_vec_kernel<<<static_cast<unsigned>((fours + 255) / 256), 256, 0, stream>>>(z, stride, a_log, dt_bias, H, d, fours);
  } else {
    dl::delta_decay_kernel<<<static_cast<unsigned>((total + 255) / 256), 256, 0, stream>>>(z, stride, a_log, dt_bias, H, d, total);
  }
  return dl::launch_status();
}

// o: float32 contiguous [rows, H * e]; gate (of gate_dtype): rows of gate_stride elements, the gate of head h at gate_col +
// h * e; w: float32 [e]; out (of dtype): contiguous [rows, H * e]. sigmoid_gate 0: the gate's activation is silu.
DL_EXPORT int dl_head_norm_gate(int dtype, int gate_dtype, const float* o, const void* gate, int gate_stride, int gate_col,
                                const float* w, float eps, int sigmoid_gate, void* out, int rows, int H, int e,
                                cudaStream_t stream) {
  if (rows <= 0 || H <= 0 || e <= 0) return 0;
  const long long units = static_cast<long long>(rows) * H;
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
#define DL_HN(T, TG)                                                                                                     \
  dl::head_norm_gate_kernel<T, TG><<<blocks, 256, 0, stream>>>(o, static_cast<const TG*>(gate), gate_stride, gate_col, w, \
                                                               eps, sigmoid_gate, static_cast<T*>(out), rows, H, e)
  if (dtype == 0 && gate_dtype == 0) DL_HN(float, float);
  else if (dtype == 1 && gate_dtype == 1) DL_HN(dl::bf16, dl::bf16);
  else if (dtype == 1 && gate_dtype == 0) DL_HN(dl::bf16, float);
  else return DL_ERR_UNSUPPORTED;
#undef DL_HN
  return dl::launch_status();
}
