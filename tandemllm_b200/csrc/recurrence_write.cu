// Linear recurrences that form what they write from more than one projection, over a matrix state a head in 32-bit, carried in a
// request's slot as [values][keys]:
//
//   gated delta rule      S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                         g one decay a head (and token), or one a head and key channel:
//                         g = exp(-exp(a_log_h) softplus(z + dt_bias)); beta = sigmoid(b'); q, k, v each pass a short causal
//                         convolution over time and silu; q and k are brought to unit length, q times q_scale; q and k have
//                         `groups` heads, each shared by H / groups heads of the values
//   gated matrix memory   m_t = max(f + m, i);  S <- exp(f + m - m_t) S + exp(i - m_t) k v^T;  o = S^T q
//                         i = cap tanh((i' + b_i) / cap), f = log sigmoid(cap tanh((f' + b_f) / cap)); m starts at 0. The sum n of
//                         the keys is carried as one more column of S whose value is always 1: its output is n . q
//
// Steps of a few rows a request run one kernel whose blocks prepare up to eight tokens in shared memory and walk them. The
// convolution's inputs before the step come from the slot (its last taps - 1 inputs, oldest first); they are moved on by a
// kernel of their own behind the scan, because the heads that share a key read the same inputs. The running maximum m is a chain
// over a request's rows in a kernel of its own in front (a warp a request and head), which leaves the two factors of every row.
//
// Longer portions go through chunks of eight tokens, counted from the portion's first row. With S the state in front of a chunk,
// d_t a token's decay and G_t = d_1 .. d_t, what token t writes is k_t w_t^T with
//
//   w_t = beta_t v_t - beta_t (G_t k_t)^T S - sum over s < t of beta_t (k_t^T d_(s+1) .. d_t k_s) w_s
//   o_t = (G_t q_t)^T S + sum over s <= t of (q_t^T d_(s+1) .. d_t k_s) w_s
//   S  <- G_8 S + sum over s of (d_(s+1) .. d_8 k_s) w_s^T
//
// so a column of S is read for eight tokens at once and only the 8 x 8 triangle is a chain. A first kernel, a warp a (head, chunk),
// forms everything that does not depend on S side by side into scratch: convolutions, unit vectors, decay products (never a
// quotient: the products only shrink) and the two triangles. The scan then walks a request's chunks, a column of S held by the
// neighbouring lanes that share it; a producer warp keeps the chunks and the columns' values coming through a ring of cp.async
// stages. The memory is the same without the read of S (w_t = v_t). Everything is 32-bit on the CUDA cores. A row's result depends
// on its request's earlier rows only; how a prompt is cut changes the order of additions, nothing else.
#include "recurrence.cuh"

namespace tl {

// A rule's prepared token in the form for a few rows, and the update of a column s of the state with the column's value v:
//   WRITE_CHANNEL  q, k, d, w                s <- d s + k (v - w . s)         (w = beta d k, v already times beta)
//   WRITE_HEAD     q, k; numbers d, w        s <- d s + k (v - w (k . s))     (d and w = beta d one number a head)
//   MEMORY         q, k; number d            s <- d s + k v                   (k already times its input gate)
constexpr int WRITE_CHANNEL = 0, WRITE_HEAD = 1, MEMORY = 2;
constexpr int STEP_TOKENS = 8;                  // tokens staged at a time in that form: one a warp
__host__ __device__ constexpr int token_arrays(int rule) { return rule == WRITE_CHANNEL ? 4 : 2; }
// a token's arrays and, behind them, its numbers (filled up to 16 bytes)
__host__ __device__ constexpr int token_floats(int rule, int Dp) { return token_arrays(rule) * Dp + 4; }

struct TokenParams {
  const float* proj;             // [rows, ld]
  long long ld;
  int q_col, k_col, v_col;
  float q_scale;
  int H, groups, D, VD;          // VD: columns of the state (the memory's includes the column of ones)
  // gated delta rule
  int b_col, a_col;              // a_col < 0: the decays' logits come in wl
  const float* wl;               // [rows, ld_w]: H * D logits
  long long ld_w;
  const float* a_log;            // [H]
  const float* dt_bias;          // [H] or [H * D]
  float unit_eps;
  const float* taps;             // [columns of proj, K]
  int K;
  const float* conv_state;       // a slot's K - 1 inputs [K - 1, conv_cols] begin at conv_state + slot * slot_floats
  int conv_cols;
  // gated matrix memory
  const float* factors;          // [rows, H, 2]: what S keeps, what the key is multiplied by
  long long slot_floats;
  const int *state_slot, *row_start, *req_of_row;
};

// One column of the convolution with its activation at row r of a request whose rows begin at `first`.
template <int K>
__device__ __forceinline__ float conv_at(const TokenParams& p, long long r, int first, const float* __restrict__ past, int c, int taps) {
  const int n = K > 0 ? K : taps;
  const float* tap = p.taps + (long long)c * n;
  float acc = 0.f;
#pragma unroll
  for (int j = 0; j < n; ++j) {
    const long long src = r - (n - 1) + j;
    const float u = src >= first ? p.proj[src * p.ld + c] : past[(long long)(n - 1 + (src - first)) * p.conv_cols + c];
    acc = fmaf(tap[j], u, acc);
  }
  return acc;
}
__device__ __forceinline__ float conv_silu_at(const TokenParams& p, long long r, int first, const float* __restrict__ past, int c) {
  if (p.K == 4) return siluf_(conv_at<4>(p, r, first, past, c, 4));
  return siluf_(conv_at<0>(p, r, first, past, c, p.K));
}

// The form for a few rows prepares a token in two passes. First every number of it on its own, `e` from 0 on: the entries of q and k
// (convolved, not yet of unit length), the decays a key channel, the values of the block's columns from col0 on, and last the write
// strength and the decay of the whole head. All numbers of a block's tokens are spread over its threads, so that their loads are one
// round trip to memory.
template <int RULE>
__host__ __device__ constexpr int token_numbers(int Dp, int cols) { return (RULE == WRITE_CHANNEL ? 3 : 2) * Dp + cols + 2; }
template <int RULE>
__device__ __forceinline__ void token_number(const TokenParams& p, long long r, int h, int first, const float* __restrict__ past, int e,
                                             float* __restrict__ tok, float* __restrict__ vals, int Dp, int col0, int cols) {
  const int D = p.D;
  float* num = tok + token_arrays(RULE) * Dp;
  if (e < 2 * Dp) {
    const bool is_k = e >= Dp;
    const int i = is_k ? e - Dp : e;
    float x = 0.f;
    if (i < D) {
      if (RULE == MEMORY) {
        x = p.proj[r * p.ld + (is_k ? p.k_col : p.q_col) + (long long)h * D + i];
        x *= is_k ? p.factors[(r * p.H + h) * 2 + 1] : p.q_scale;
      } else {
        x = conv_silu_at(p, r, first, past, (is_k ? p.k_col : p.q_col) + h / (p.H / p.groups) * D + i);
      }
    }
    tok[e] = x;
    return;
  }
  e -= 2 * Dp;
  if (RULE == WRITE_CHANNEL) {
    if (e < Dp) {
      tok[2 * Dp + e] =
          e < D ? expf(-expf(p.a_log[h]) * softplusf_(p.wl[r * p.ld_w + (long long)h * D + e] + p.dt_bias[h * D + e])) : 0.f;
      return;
    }
    e -= Dp;
  }
  if (e < cols) {
    const int j = col0 + e;
    float x = 0.f;
    if (j < p.VD) {
      if (RULE == MEMORY) x = j == p.VD - 1 ? 1.f : p.proj[r * p.ld + p.v_col + (long long)h * (p.VD - 1) + j];
      else x = conv_silu_at(p, r, first, past, p.v_col + h * p.VD + j);
    }
    vals[e] = x;
    return;
  }
  e -= cols;
  if (RULE == MEMORY) {
    if (e == 0) num[0] = p.factors[(r * p.H + h) * 2];
  } else if (e == 1) {
    num[1] = sigmoidf_(p.proj[r * p.ld + p.b_col + h]);
  } else if (RULE == WRITE_HEAD) {
    num[0] = expf(-expf(p.a_log[h]) * softplusf_(p.proj[r * p.ld + p.a_col + h] + p.dt_bias[h]));
  }
}
// Then a warp a token: unit lengths, and what the update wants of them.
template <int RULE>
__device__ __forceinline__ void finish_token(const TokenParams& p, float* __restrict__ tok, float* __restrict__ vals, int Dp, int cols,
                                             int lane) {
  float* num = tok + token_arrays(RULE) * Dp;
  float qq = 0.f, kk = 0.f;
  for (int i = lane; i < Dp; i += 32) {
    qq = fmaf(tok[i], tok[i], qq);
    kk = fmaf(tok[Dp + i], tok[Dp + i], kk);
  }
  const float qs = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), ks = 1.f / sqrtf(warp_sum(kk) + p.unit_eps);
  const float beta = num[1];
  for (int i = lane; i < Dp; i += 32) {
    const float k = tok[Dp + i] * ks;
    tok[i] *= qs;
    tok[Dp + i] = k;
    if (RULE == WRITE_CHANNEL) tok[3 * Dp + i] = beta * (tok[2 * Dp + i] * k);
  }
  for (int c = lane; c < cols; c += 32) vals[c] *= beta;
  __syncwarp();
  if (RULE == WRITE_HEAD && lane == 0) num[1] = num[0] * beta;
}

// ---- chunks of eight tokens ----
constexpr int CH = 8;
// A prepared chunk: CH x 2 arrays of Dp (WRITE_CHANNEL: beta_t G_t k_t and G_t q_t; else k_t and q_t), for WRITE_CHANNEL CH arrays
// d_(t+1) .. d_8 k_t and G_8; then 32 numbers (not WRITE_CHANNEL: [0, 8) what k_t^T S is multiplied by, [8, 16) q_t^T S, [16, 24) the
// write of token t in the chunk's last state, [24] S itself); then the triangles [s][t] of w (t > s) and [t][s] of o (s <= t).
__host__ __device__ constexpr int chunk_floats(int rule, int Dp) {
  return (rule == WRITE_CHANNEL ? (3 * CH + 1) * Dp : 2 * CH * Dp) + 32 + 2 * CH * CH;
}
// Where a request's chunk lies: requests follow one another with a place to spare each, so no table is needed.
__device__ __forceinline__ long long chunk_place(int first_row, int request, int chunk) { return first_row / CH + request + chunk; }

// grid (chunks / 4, H), a warp a (head, chunk of a request): `places` chunks a head in prep [H][places][chunk_floats], the columns'
// values in vact [H][places][VD][CH] (times beta). A warp's q and k (and decays) of the chunk wait in shared memory, each lane with
// entries of its own, between the passes: unit lengths, triangles, what the scan reads.
template <int RULE>
__global__ void __launch_bounds__(128, 4) chunk_prepare_kernel(TokenParams p, float* __restrict__ prep, float* __restrict__ vact, int Dp,
                                                            long long places, int requests) {
  extern __shared__ __align__(16) float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long place = (long long)blockIdx.x * 4 + warp;
  const int h = blockIdx.y, D = p.D;
  if (place >= places) return;
  float* sq = sm + warp * (RULE == WRITE_CHANNEL ? 3 : 2) * CH * Dp;       // [Dp][CH]: an entry's eight tokens together
  float* sk = sq + CH * Dp;
  float* sd = sk + CH * Dp;
  // the request whose chunks hold this place: the last one whose first place is not behind it
  int lo = 0, hi = requests - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (chunk_place(p.row_start[mid], mid, 0) <= place) lo = mid;
    else hi = mid - 1;
  }
  const int b = lo, first = p.row_start[b], end = p.row_start[b + 1];
  const long long r0 = first + (place - chunk_place(first, b, 0)) * CH;
  if (r0 >= end) return;                                    // a place to spare
  const int n = (int)min((long long)CH, end - r0);
  const float* past = RULE == MEMORY ? nullptr : p.conv_state + (long long)p.state_slot[b] * p.slot_floats;
  float* out = prep + ((long long)h * places + place) * chunk_floats(RULE, Dp);
  float* num = out + (RULE == WRITE_CHANNEL ? (3 * CH + 1) * Dp : 2 * CH * Dp);
  float* tri_w = num + 32;
  float* tri_o = tri_w + CH * CH;
  float my_beta = 0.f, my_d = 1.f, my_add = 1.f;             // of token `lane` (lane < n): beta, the decay of the whole head, the input gate
  float my_qs = p.q_scale, my_ks = 1.f;                      // what its q and k are multiplied by
  // the convolved columns of eight tokens: every input of the chunk and the taps - 1 in front of it is read once
  auto conv_column = [&](int c, float (&v)[CH]) {
    const int K = p.K;
    const float* tap = p.taps + (long long)c * K;
    if (K == 4) {
      float u[CH + 3];
#pragma unroll
      for (int j = 0; j < CH + 3; ++j) {
        const long long src = r0 - 3 + j;
        u[j] = src >= end ? 0.f : (src >= first ? p.proj[src * p.ld + c] : past[(3 + (src - first)) * p.conv_cols + c]);
      }
      const float t0 = tap[0], t1 = tap[1], t2 = tap[2], t3 = tap[3];
#pragma unroll
      for (int t = 0; t < CH; ++t) v[t] = siluf_(fmaf(t3, u[t + 3], fmaf(t2, u[t + 2], fmaf(t1, u[t + 1], t0 * u[t]))));
      return;
    }
#pragma unroll
    for (int t = 0; t < CH; ++t) v[t] = 0.f;
    for (int j = 0; j < K; ++j) {
      const float tj = tap[j];
#pragma unroll
      for (int t = 0; t < CH; ++t) {
        const long long src = r0 + t - (K - 1) + j;
        const float u = src >= end ? 0.f : (src >= first ? p.proj[src * p.ld + c] : past[(K - 1 + (src - first)) * p.conv_cols + c]);
        v[t] = fmaf(tj, u, v[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < CH; ++t) v[t] = siluf_(v[t]);
  };
  auto put8 = [](float* to, const float (&v)[CH]) {
    reinterpret_cast<float4*>(to)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(to)[1] = make_float4(v[4], v[5], v[6], v[7]);
  };
  auto get8 = [](const float* from, float (&v)[CH]) {
    const float4 a = reinterpret_cast<const float4*>(from)[0], c = reinterpret_cast<const float4*>(from)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = c.x; v[5] = c.y; v[6] = c.z; v[7] = c.w;
  };

  // ---- q and k of the chunk (and the decays a key channel); their lengths ----
  float ss[2 * CH];
#pragma unroll
  for (int t = 0; t < 2 * CH; ++t) ss[t] = 0.f;
  const float rate = RULE == MEMORY ? 0.f : -expf(p.a_log[h]);
#pragma unroll 1
  for (int i = lane; i < Dp; i += 32) {
    float q[CH], k[CH];
    if (i < D) {
      if constexpr (RULE == MEMORY) {
        const float* at = p.proj + r0 * p.ld + (long long)h * D + i;
#pragma unroll
        for (int t = 0; t < CH; ++t) {
          q[t] = t < n ? at[t * p.ld + p.q_col] : 0.f;
          k[t] = t < n ? at[t * p.ld + p.k_col] : 0.f;
        }
      } else {
        const int g = h / (p.H / p.groups);
        conv_column(p.q_col + g * D + i, q);
        conv_column(p.k_col + g * D + i, k);
      }
    } else {
#pragma unroll
      for (int t = 0; t < CH; ++t) q[t] = k[t] = 0.f;
    }
    put8(sq + i * CH, q);
    put8(sk + i * CH, k);
#pragma unroll
    for (int t = 0; t < CH; ++t) {
      ss[t] = fmaf(q[t], q[t], ss[t]);
      ss[CH + t] = fmaf(k[t], k[t], ss[CH + t]);
    }
    if constexpr (RULE == WRITE_CHANNEL) {
      float d[CH];
      const float bias = i < D ? p.dt_bias[h * D + i] : 0.f;
#pragma unroll
      for (int t = 0; t < CH; ++t)
        d[t] = (i < D && t < n) ? expf(rate * softplusf_(p.wl[(r0 + t) * p.ld_w + (long long)h * D + i] + bias)) : 1.f;
      put8(sd + i * CH, d);
    }
  }
  if constexpr (RULE == MEMORY) {
    if (lane < n) {
      my_d = p.factors[((r0 + lane) * p.H + h) * 2];
      my_add = p.factors[((r0 + lane) * p.H + h) * 2 + 1];
    }
  } else {
    // lane 2 t holds q's sum of token t, lane 16 + 2 t k's; lane t takes both
    rec_reduce_scatter<2 * CH, 32>(ss, lane);
    const float inv = 1.f / sqrtf(ss[0] + p.unit_eps);
    const float iq = __shfl_sync(0xffffffffu, inv, 2 * (lane & 7)), ik = __shfl_sync(0xffffffffu, inv, 16 + 2 * (lane & 7));
    my_qs = lane < n ? p.q_scale * iq : 0.f;
    my_ks = lane < n ? ik : 0.f;
    if (lane < n) {
      my_beta = sigmoidf_(p.proj[(r0 + lane) * p.ld + p.b_col + h]);
      if (RULE == WRITE_HEAD) my_d = expf(rate * softplusf_(p.proj[(r0 + lane) * p.ld + p.a_col + h] + p.dt_bias[h]));
    }
  }
  float qs[CH], ks[CH];
#pragma unroll
  for (int t = 0; t < CH; ++t) {
    qs[t] = __shfl_sync(0xffffffffu, my_qs, t);
    ks[t] = __shfl_sync(0xffffffffu, my_ks, t);
  }

  // ---- the columns' values, a column's eight tokens together ----
  float times[CH];
#pragma unroll
  for (int t = 0; t < CH; ++t) times[t] = RULE == MEMORY ? 1.f : __shfl_sync(0xffffffffu, my_beta, t);
#pragma unroll 1
  for (int j = lane; j < p.VD; j += 32) {
    float v[CH];
    if constexpr (RULE == MEMORY) {
#pragma unroll
      for (int t = 0; t < CH; ++t)
        v[t] = t < n ? (j == p.VD - 1 ? 1.f : p.proj[(r0 + t) * p.ld + p.v_col + (long long)h * (p.VD - 1) + j]) : 0.f;
    } else {
      conv_column(p.v_col + h * p.VD + j, v);
#pragma unroll
      for (int t = 0; t < CH; ++t) v[t] *= times[t];
    }
    put8(vact + (((long long)h * places + place) * p.VD + j) * CH, v);
  }

  // ---- the two triangles: with one decay a head the inner products k_t . k_s and q_t . k_s, else with the decays between inside the
  // sums. 36 sums of the o triangle (s <= t) and 28 of the w triangle (s < t) fill two batches of 32, a lane each in the end ----
#pragma unroll
  for (int batch = 0; batch < 2; ++batch) {
    float v[32];
#pragma unroll
    for (int x = 0; x < 32; ++x) v[x] = 0.f;
#pragma unroll 1
    for (int i = lane; i < Dp; i += 32) {
      float q[CH], k[CH], d[CH];
      get8(sq + i * CH, q);
      get8(sk + i * CH, k);
      if (RULE == WRITE_CHANNEL) get8(sd + i * CH, d);
#pragma unroll
      for (int t = 0; t < CH; ++t) {
        q[t] *= qs[t];
        k[t] *= ks[t];
      }
      int at = 0;
#pragma unroll
      for (int s = 0; s < CH; ++s) {
        const bool o_here = (s < 4) == (batch == 0), w_here = !o_here;       // batch 0: o of s < 4 and w of s >= 4
        float x = k[s];
#pragma unroll
        for (int t = s; t < CH; ++t) {
          if (RULE == WRITE_CHANNEL && t > s) x *= d[t];
          if (o_here) {
            v[at] = fmaf(q[t], x, v[at]);
            ++at;
          }
          if (w_here && t > s) {
            v[at] = fmaf(k[t], x, v[at]);
            ++at;
          }
        }
      }
    }
    rec_reduce_scatter<32, 32>(v, lane);
    // which sum this lane holds: o's rows s = 0 .. 3 have 8, 7, 6, 5 sums and w's s = 4 .. 6 then 3, 2, 1; in the other batch w's
    // s = 0 .. 3 have 7, 6, 5, 4 and o's s = 4 .. 7 then 4, 3, 2, 1
    int my_s = 0, left = lane;
    while (true) {
      const bool o_row = (my_s < 4) == (batch == 0);
      const int len = o_row ? CH - my_s : CH - 1 - my_s;
      if (left < len) break;
      left -= len;
      ++my_s;
    }
    const bool is_o = (my_s < 4) == (batch == 0);
    const int my_t = my_s + left + (is_o ? 0 : 1);
    __syncwarp();
    float x = v[0];
    if constexpr (RULE != WRITE_CHANNEL) {
#pragma unroll
      for (int t = 1; t < CH; ++t) {
        const float dt = __shfl_sync(0xffffffffu, my_d, t);
        if (t > my_s && t <= my_t) x *= dt;
      }
    }
    if constexpr (RULE == MEMORY) {
      x *= __shfl_sync(0xffffffffu, my_add, my_s);
    } else {
      const float beta = __shfl_sync(0xffffffffu, my_beta, my_t);
      if (!is_o) x *= beta;
    }
    if (is_o) tri_o[my_t * CH + my_s] = x;
    else tri_w[my_s * CH + my_t] = x;
  }
  // the entries of the triangles nobody's sum fills
#pragma unroll
  for (int x = lane; x < CH * CH; x += 32) {
    if ((x & 7) <= (x >> 3)) tri_w[x] = 0.f;               // [s][t], t <= s
    if ((x & 7) > (x >> 3)) tri_o[x] = 0.f;                // [t][s], s > t
  }

  // ---- what the scan reads ----
#pragma unroll 1
  for (int i = lane; i < Dp; i += 32) {
    float q[CH], k[CH];
    get8(sq + i * CH, q);
    get8(sk + i * CH, k);
    if constexpr (RULE == WRITE_CHANNEL) {
      float d[CH];
      get8(sd + i * CH, d);
      float G = 1.f, R = 1.f;
#pragma unroll
      for (int t = 0; t < CH; ++t) {
        G *= d[t];
        out[t * Dp + i] = k[t] * ks[t] * G;
        out[(CH + t) * Dp + i] = q[t] * qs[t] * G;
      }
      out[3 * CH * Dp + i] = G;
#pragma unroll
      for (int t = CH - 1; t >= 0; --t) {
        out[(2 * CH + t) * Dp + i] = k[t] * ks[t] * R;
        R *= d[t];
      }
    } else {
#pragma unroll
      for (int t = 0; t < CH; ++t) {
        out[t * Dp + i] = k[t] * ks[t];
        out[(CH + t) * Dp + i] = q[t] * qs[t];
      }
    }
  }
  if constexpr (RULE == WRITE_CHANNEL) {
    if (lane < CH) num[lane] = my_beta;                    // (what k_t^T S is multiplied by, as in the other form)
  } else {
    float G = 1.f, upto = 1.f, behind = 1.f;
#pragma unroll
    for (int t = 0; t < CH; ++t) {
      const float dt = __shfl_sync(0xffffffffu, my_d, t);
      G *= dt;
      if (t <= lane) upto *= dt;
      else behind *= dt;
    }
    if (lane < CH) {
      num[lane] = my_beta * upto;
      num[CH + lane] = upto;
      num[2 * CH + lane] = RULE == MEMORY ? behind * my_add : behind;
    }
    if (lane == 0) num[3 * CH] = G;
  }
}

// A lane's KPL keys of its column go through a chunk. `base`: the prepared chunk in shared memory; `vals`: the column's eight values.
template <int RULE, int KPL, int DP>
__device__ __forceinline__ void chunk_step(float (&s)[KPL], const float* __restrict__ base, const float* __restrict__ vals,
                                           float* __restrict__ yg, long long ldy, int n, int part, bool owns) {
  constexpr int P = DP / KPL, M = KPL / 4, Q = DP / 4;
  constexpr bool CHANNEL = RULE == WRITE_CHANNEL;
  const float4* arr = reinterpret_cast<const float4*>(base) + part;
  const float* num = base + (CHANNEL ? (3 * CH + 1) * DP : 2 * CH * DP);
  const float* tri_w = num + 32;
  const float* tri_o = tri_w + CH * CH;
  float a[CH], o[CH], w[CH];
  {
    const float4 v0 = reinterpret_cast<const float4*>(vals)[0], v1 = reinterpret_cast<const float4*>(vals)[1];
    w[0] = v0.x; w[1] = v0.y; w[2] = v0.z; w[3] = v0.w; w[4] = v1.x; w[5] = v1.y; w[6] = v1.z; w[7] = v1.w;
  }
#pragma unroll
  for (int t = 0; t < CH; ++t) {
    float a0 = 0.f, a1 = 0.f, o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      if (RULE != MEMORY) {
        const float4 k = arr[t * Q + P * m];
        a0 = fmaf(k.x, s[4 * m], a0);
        a1 = fmaf(k.y, s[4 * m + 1], a1);
        a0 = fmaf(k.z, s[4 * m + 2], a0);
        a1 = fmaf(k.w, s[4 * m + 3], a1);
      }
      const float4 q = arr[(CH + t) * Q + P * m];
      o0 = fmaf(q.x, s[4 * m], o0);
      o1 = fmaf(q.y, s[4 * m + 1], o1);
      o0 = fmaf(q.z, s[4 * m + 2], o0);
      o1 = fmaf(q.w, s[4 * m + 3], o1);
    }
    a[t] = a0 + a1;
    o[t] = o0 + o1;
  }
  if constexpr (RULE != MEMORY) {
#pragma unroll
    for (int off = P >> 1; off > 0; off >>= 1)
#pragma unroll
      for (int t = 0; t < CH; ++t) a[t] += __shfl_xor_sync(0xffffffffu, a[t], off);
    const float4 b0 = reinterpret_cast<const float4*>(num)[0], b1 = reinterpret_cast<const float4*>(num)[1];
    w[0] = fmaf(-b0.x, a[0], w[0]); w[1] = fmaf(-b0.y, a[1], w[1]); w[2] = fmaf(-b0.z, a[2], w[2]); w[3] = fmaf(-b0.w, a[3], w[3]);
    w[4] = fmaf(-b1.x, a[4], w[4]); w[5] = fmaf(-b1.y, a[5], w[5]); w[6] = fmaf(-b1.z, a[6], w[6]); w[7] = fmaf(-b1.w, a[7], w[7]);
    // the triangle: a token's write goes into all later ones as soon as it is known
#pragma unroll
    for (int e = 0; e < CH - 1; ++e) {
      const float4 c0 = reinterpret_cast<const float4*>(tri_w + e * CH)[0], c1 = reinterpret_cast<const float4*>(tri_w + e * CH)[1];
      const float c[CH] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
#pragma unroll
      for (int t = e + 1; t < CH; ++t) w[t] = fmaf(-c[t], w[e], w[t]);
    }
  }
  // the outputs of the lane's tokens: its share of the sums over keys, then what the chunk itself wrote
  rec_reduce_scatter<CH, P>(o, part);
  constexpr int each = P <= CH ? CH / P : 1, share = P > CH ? P / CH : 1;
#pragma unroll
  for (int i = 0; i < each; ++i) {
    const int t = P <= CH ? part * each + i : part / share;
    const float4 c0 = reinterpret_cast<const float4*>(tri_o + t * CH)[0], c1 = reinterpret_cast<const float4*>(tri_o + t * CH)[1];
    float x = CHANNEL ? o[i] : num[CH + t] * o[i];
    x = fmaf(c0.x, w[0], x);
    x = fmaf(c0.y, w[1], x);
    x = fmaf(c0.z, w[2], x);
    x = fmaf(c0.w, w[3], x);
    x = fmaf(c1.x, w[4], x);
    x = fmaf(c1.y, w[5], x);
    x = fmaf(c1.z, w[6], x);
    x = fmaf(c1.w, w[7], x);
    if (owns && t < n && (P <= CH || part % share == 0)) yg[t * ldy] = x;
  }
  // the state behind the chunk (with 16 keys a lane the keys are read again, through a pointer the compiler cannot tell from another:
  // held from above they would not fit the registers)
  const float4* behind = arr + (CHANNEL ? 2 * CH * Q : 0);
  if (!CHANNEL && KPL == 16) asm volatile("" : "+l"(behind));
  if constexpr (!CHANNEL) {
    const float4 h0 = reinterpret_cast<const float4*>(num + 2 * CH)[0], h1 = reinterpret_cast<const float4*>(num + 2 * CH)[1];
    w[0] *= h0.x; w[1] *= h0.y; w[2] *= h0.z; w[3] *= h0.w; w[4] *= h1.x; w[5] *= h1.y; w[6] *= h1.z; w[7] *= h1.w;
  }
  const float G_h = CHANNEL ? 0.f : num[3 * CH];
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const float4 G = CHANNEL ? arr[3 * CH * Q + P * m] : make_float4(G_h, G_h, G_h, G_h);
    s[4 * m] *= G.x;
    s[4 * m + 1] *= G.y;
    s[4 * m + 2] *= G.z;
    s[4 * m + 3] *= G.w;
#pragma unroll
    for (int t = 0; t < CH; ++t) {
      const float4 k = behind[t * Q + P * m];
      s[4 * m] = fmaf(k.x, w[t], s[4 * m]);
      s[4 * m + 1] = fmaf(k.y, w[t], s[4 * m + 1]);
      s[4 * m + 2] = fmaf(k.z, w[t], s[4 * m + 2]);
      s[4 * m + 3] = fmaf(k.w, w[t], s[4 * m + 3]);
    }
  }
}

// Waits until all but the last `n` groups of this thread's copies have landed.
__device__ __forceinline__ void cp_wait_all_but(int n) {
  switch (n) {
    case 0: asm volatile("cp.async.wait_group 0;" ::: "memory"); break;
    case 1: asm volatile("cp.async.wait_group 1;" ::: "memory"); break;
    case 2: asm volatile("cp.async.wait_group 2;" ::: "memory"); break;
    case 3: asm volatile("cp.async.wait_group 3;" ::: "memory"); break;
    case 4: asm volatile("cp.async.wait_group 4;" ::: "memory"); break;
    case 5: asm volatile("cp.async.wait_group 5;" ::: "memory"); break;
    default: asm volatile("cp.async.wait_group 6;" ::: "memory"); break;
  }
}

// grid (requests, heads, tiles of value columns): cols_per_block * P computing threads (a multiple of 32) and the producer warp, which
// keeps stages - 1 chunks in flight and meets the others at one barrier a chunk. Lane (column, part) holds keys 4 (part + P m) + c.
constexpr int CHUNK_STAGES = 8;         // at most: a chunk takes less time than a copy from L2, so several are under way
template <int RULE, int KPL, int DP>
__global__ void __launch_bounds__(REC_THREADS + 32) chunk_scan_kernel(const float* __restrict__ prep, const float* __restrict__ vact,
                                                                      long long places, float* __restrict__ state, long long slot_floats,
                                                                      const int* __restrict__ state_slot,
                                                                      const int* __restrict__ row_start, float* __restrict__ y, int H,
                                                                      int D, int VD, int cols_per_block, int stages, int write_state) {
  constexpr int P = DP / KPL, M = KPL / 4, CF = chunk_floats(RULE, DP);
  extern __shared__ __align__(16) float sm[];
  const int stage_floats = CF + CH * cols_per_block;
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x, nth = blockDim.x - 32;
  const bool producer = tid >= nth;
  const int part = tid % P, jl = tid / P, j = col0 + jl;
  const bool owns = !producer && j < VD;
  const int r0 = row_start[b], r1 = row_start[b + 1];
  if (r1 <= r0) return;
  float* S = state + (long long)state_slot[b] * slot_floats + (long long)h * D * VD;
  const bool vec = (D & 3) == 0 && ((uintptr_t)S & 15) == 0;
  const int n_chunks = (r1 - r0 + CH - 1) / CH;
  const long long place0 = (long long)h * places + chunk_place(r0, b, 0);

  auto load = [&](int chunk, int stage) {        // (the producer's lanes only)
    const int lane = tid - nth;
    float* to = sm + stage * stage_floats;
    const float* src = prep + (place0 + chunk) * CF;
#pragma unroll 4
    for (int i = lane; i < CF / 4; i += 32) rec_cp16(to + 4 * i, src + 4 * i);
    const float* vs = vact + ((place0 + chunk) * VD + col0) * CH;
    const int pieces = 2 * min(cols_per_block, VD - col0);
    for (int i = lane; i < pieces; i += 32) rec_cp16(to + CF + 4 * i, vs + 4 * i);
  };
  float s[KPL];
  if (producer) {
    // (columns past VD in the last tile: their lanes read what is there and store nothing)
    for (int i = tid - nth; i < stages * CH * cols_per_block; i += 32)
      sm[(i / (CH * cols_per_block)) * stage_floats + CF + i % (CH * cols_per_block)] = 0.f;
    __syncwarp();
    for (int s0 = 0; s0 < stages - 1; ++s0) {
      if (s0 < n_chunks) load(s0, s0);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    cp_wait_all_but(stages - 2);
  } else {
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int i = 4 * (part + P * m);
      const float* at = S + (long long)j * D + i;
      if (vec) {
        const float4 v = (owns && i < D) ? *reinterpret_cast<const float4*>(at) : make_float4(0.f, 0.f, 0.f, 0.f);
        s[4 * m] = v.x; s[4 * m + 1] = v.y; s[4 * m + 2] = v.z; s[4 * m + 3] = v.w;
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c) s[4 * m + c] = (owns && i + c < D) ? at[c] : 0.f;
      }
    }
  }
  __syncthreads();
  const float* base = sm;                        // the chunk's stage; the one before it, which is free, is the last of the ring at first
  for (int chunk = 0, stage = 0, freed = stages - 1; chunk < n_chunks; ++chunk) {
    if (producer) {
      // the stage of chunk - 1 is free (everybody passed the barrier behind it): refill it, then wait for chunk + 1
      if (chunk + stages - 1 < n_chunks) load(chunk + stages - 1, freed);
      asm volatile("cp.async.commit_group;" ::: "memory");
      cp_wait_all_but(stages - 2);
    } else {
      const long long ldy = (long long)H * VD, t0 = r0 + (long long)chunk * CH;
      chunk_step<RULE, KPL, DP>(s, base, base + CF + jl * CH, y + t0 * ldy + (long long)h * VD + j, ldy,
                                (int)min((long long)CH, r1 - t0), part, owns);
    }
    freed = stage;
    stage = stage + 1 == stages ? 0 : stage + 1;
    base = sm + stage * stage_floats;
    __syncthreads();
  }
  if (write_state && owns) {
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int i = 4 * (part + P * m);
      float* at = S + (long long)j * D + i;
      if (vec) {
        if (i < D) *reinterpret_cast<float4*>(at) = make_float4(s[4 * m], s[4 * m + 1], s[4 * m + 2], s[4 * m + 3]);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (i + c < D) at[c] = s[4 * m + c];
      }
    }
  }
}

// Steps of a few rows a request: grid (requests, heads, tiles of value columns); thread (column, part) holds 16 keys of a column.
template <int RULE>
__global__ void __launch_bounds__(REC_THREADS) write_scan_kernel(TokenParams p, float* __restrict__ state, float* __restrict__ y, int P,
                                                                 int cols_per_block, int write_state) {
  extern __shared__ __align__(16) float sm[];
  const int Dp = 16 * P, tok_floats = token_floats(RULE, Dp), D = p.D, VD = p.VD;
  float* s_v = sm + STEP_TOKENS * tok_floats;            // [STEP_TOKENS][cols_per_block]
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = tid % P, jl = tid / P, j = col0 + jl;
  const bool owns = jl < cols_per_block && j < VD;
  const int r0 = p.row_start[b], r1 = p.row_start[b + 1];
  if (r1 <= r0) return;
  const long long slot = p.state_slot[b];
  float* S = state + slot * p.slot_floats + (long long)h * D * VD;
  const float* past = RULE == MEMORY ? nullptr : p.conv_state + slot * p.slot_floats;
  const bool vec = (D & 3) == 0 && ((uintptr_t)S & 15) == 0;

  float s[16];
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    const int i = 4 * (part + P * m);
    const float* at = S + (long long)j * D + i;
    if (vec) {
      const float4 v = (owns && i < D) ? *reinterpret_cast<const float4*>(at) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[4 * m] = v.x; s[4 * m + 1] = v.y; s[4 * m + 2] = v.z; s[4 * m + 3] = v.w;
    } else {
#pragma unroll
      for (int c = 0; c < 4; ++c) s[4 * m + c] = (owns && i + c < D) ? at[c] : 0.f;
    }
  }
  const int chunk_tokens = min(STEP_TOKENS, (int)(blockDim.x >> 5));      // a warp a token
  for (int t0 = r0; t0 < r1; t0 += chunk_tokens) {
    const int nt = min(chunk_tokens, r1 - t0);
    __syncthreads();                      // the chunk before has been read
    const int each = token_numbers<RULE>(Dp, cols_per_block);
    for (int x = tid; x < nt * each; x += blockDim.x) {
      const int t = x / each;
      token_number<RULE>(p, t0 + t, h, r0, past, x - t * each, sm + t * tok_floats, s_v + t * cols_per_block, Dp, col0, cols_per_block);
    }
    __syncthreads();
    if (RULE != MEMORY) {
      if (warp < nt) finish_token<RULE>(p, sm + warp * tok_floats, s_v + warp * cols_per_block, Dp, cols_per_block, lane);
      __syncthreads();
    }
    // (warps without columns of their own only help to prepare the tokens)
    for (int t = 0; t < nt && warp * 32 < cols_per_block * P; ++t) {
      const float4* a = reinterpret_cast<const float4*>(sm + t * tok_floats) + part;
      const float* num = sm + t * tok_floats + token_arrays(RULE) * Dp;
      const int Q = 4 * P;
      float w = jl < cols_per_block ? s_v[t * cols_per_block + jl] : 0.f;
      if constexpr (RULE != MEMORY) {
        const float4* u4 = a + (RULE == WRITE_CHANNEL ? 3 : 1) * Q;
        float us0 = 0.f, us1 = 0.f, us2 = 0.f, us3 = 0.f;
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          const float4 u = u4[P * m];
          us0 = fmaf(u.x, s[4 * m], us0);
          us1 = fmaf(u.y, s[4 * m + 1], us1);
          us2 = fmaf(u.z, s[4 * m + 2], us2);
          us3 = fmaf(u.w, s[4 * m + 3], us3);
        }
        float us = (us0 + us1) + (us2 + us3);
        for (int off = P >> 1; off > 0; off >>= 1) us += __shfl_xor_sync(0xffffffffu, us, off);
        w = RULE == WRITE_HEAD ? fmaf(-num[1], us, w) : w - us;
      }
      const float d_h = RULE == WRITE_CHANNEL ? 0.f : num[0];
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float4 q = a[P * m], k = a[Q + P * m];
        const float4 d = RULE == WRITE_CHANNEL ? a[2 * Q + P * m] : make_float4(d_h, d_h, d_h, d_h);
        s[4 * m] = fmaf(d.x, s[4 * m], k.x * w);
        s[4 * m + 1] = fmaf(d.y, s[4 * m + 1], k.y * w);
        s[4 * m + 2] = fmaf(d.z, s[4 * m + 2], k.z * w);
        s[4 * m + 3] = fmaf(d.w, s[4 * m + 3], k.w * w);
        o0 = fmaf(s[4 * m], q.x, o0);
        o1 = fmaf(s[4 * m + 1], q.y, o1);
        o2 = fmaf(s[4 * m + 2], q.z, o2);
        o3 = fmaf(s[4 * m + 3], q.w, o3);
      }
      float o = (o0 + o1) + (o2 + o3);
      for (int off = P >> 1; off > 0; off >>= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
      if (part == 0 && owns) y[((long long)(t0 + t) * p.H + h) * VD + j] = o;
    }
  }
  if (write_state && owns) {
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const int i = 4 * (part + P * m);
      float* at = S + (long long)j * D + i;
      if (vec) {
        if (i < D) *reinterpret_cast<float4*>(at) = make_float4(s[4 * m], s[4 * m + 1], s[4 * m + 2], s[4 * m + 3]);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (i + c < D) at[c] = s[4 * m + c];
      }
    }
  }
}

// A warp a (request, head): the two log gates of 32 rows at a time, then the chain of the running maximum through them.
__global__ void __launch_bounds__(128) memory_factors_kernel(const float* __restrict__ proj, long long ld, int i_col, int f_col,
                                                             const float* __restrict__ i_bias, const float* __restrict__ f_bias,
                                                             float cap, float* __restrict__ m_state, long long slot_floats,
                                                             const int* __restrict__ state_slot, const int* __restrict__ row_start,
                                                             float* __restrict__ factors, float* __restrict__ maxima, int requests,
                                                             int H, int write_state) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int idx = blockIdx.x * 4 + warp;
  if (idx >= requests * H) return;
  const int b = idx / H, h = idx - b * H;
  const int r0 = row_start[b], r1 = row_start[b + 1];
  if (r1 <= r0) return;
  float* slot = m_state + (long long)state_slot[b] * slot_floats + h;
  float m = *slot;
  const float bi = i_bias[h], bf = f_bias[h];
  float zi = 0.f, zf = 0.f;
  if (r0 + lane < r1) {
    zi = proj[(long long)(r0 + lane) * ld + i_col + h];
    zf = proj[(long long)(r0 + lane) * ld + f_col + h];
  }
  for (int t0 = r0; t0 < r1; t0 += 32) {
    const float i = cap * tanhf((zi + bi) / cap);
    const float f = -softplusf_(-cap * tanhf((zf + bf) / cap));
    const long long next = (long long)t0 + 32 + lane;         // the next rows are on their way while the chain runs
    if (next < r1) {
      zi = proj[next * ld + i_col + h];
      zf = proj[next * ld + f_col + h];
    }
    const int n = min(32, r1 - t0);
    float before = 0.f, mine = 0.f;
#pragma unroll
    for (int t = 0; t < 32; ++t) {
      const float ft = __shfl_sync(0xffffffffu, f, t), it = __shfl_sync(0xffffffffu, i, t);
      const float now = t < n ? fmaxf(ft + m, it) : m;
      if (lane == t) {
        before = m;
        mine = now;
      }
      m = now;
    }
    if (lane < n) {
      const long long at = (long long)(t0 + lane) * H + h;
      factors[2 * at] = expf(f + before - mine);
      factors[2 * at + 1] = expf(i - mine);
      maxima[at] = mine;
    }
  }
  if (write_state && lane == 0) *slot = m;
}

// A warp a (row, head): o = y / (max(|y_ones|, exp(-maximum)) + floor), the head's output of the column of ones behind its others, then
// o / rms(o), times the weight, times sigmoid(gate). HELD: entries a lane holds between the passes (VD <= 32 HELD).
template <typename T, int HELD>
__global__ void __launch_bounds__(128) memory_norm_gate_kernel(const float* __restrict__ y, const float* __restrict__ maxima,
                                                               const float* __restrict__ gate, long long ld_gate,
                                                               const float* __restrict__ weight, float eps, float floor_,
                                                               T* __restrict__ out, long long ld_out, int rows, int H, int VD) {
  const int lane = threadIdx.x & 31;
  const long long idx = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (idx >= (long long)rows * H) return;
  const long long r = idx / H;
  const int c0 = (int)(idx - r * H) * VD;
  const float* yr = y + idx * (VD + 1);
  float v[HELD], g[HELD], w[HELD];
  const float ones = yr[VD], maximum = maxima[idx];
#pragma unroll
  for (int e = 0; e < HELD; ++e) {
    const int i = lane + 32 * e;
    const bool ok = i < VD;
    v[e] = ok ? yr[i] : 0.f;
    g[e] = ok ? gate[r * ld_gate + c0 + i] : 0.f;
    w[e] = ok ? weight[c0 + i] : 0.f;
    if (32 * (e + 1) >= VD) break;
  }
  const float inv_den = 1.f / (fmaxf(fabsf(ones), expf(-maximum)) + floor_);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < HELD; ++e) {
    const float o = v[e] * inv_den;
    ss = fmaf(o, o, ss);
    if (32 * (e + 1) >= VD) break;
  }
  const float inv = inv_den / sqrtf(warp_sum(ss) / (float)VD + eps);
#pragma unroll
  for (int e = 0; e < HELD; ++e) {
    const int i = lane + 32 * e;
    if (i < VD) out[r * ld_out + c0 + i] = from_f32<T>(v[e] * inv * w[e] * sigmoidf_(g[e]));
    if (32 * (e + 1) >= VD) break;
  }
}

static long long chunk_places(long long rows, int requests) { return rows / CH + requests + 1; }

template <int RULE, int KPL, int DP>
static int launch_chunk_scan(const TokenParams& p, const float* prep, const float* vact, long long places, float* state, float* y,
                             int requests, int write_state, int sms, cudaStream_t stream) {
  constexpr int P = DP / KPL;
  int threads, cols_per_block;
  recurrence_block(requests, p.H, p.VD, P, (3LL * sms) / 4, &threads, &cols_per_block);
  const int tiles = ceil_div(p.VD, cols_per_block);
  TL_REQUIRE(tiles <= 65535, "recurrence: %d tiles of value columns exceed the grid limit", tiles);
  const size_t stage = (size_t)(chunk_floats(RULE, DP) + CH * cols_per_block) * sizeof(float);
  int stages = CHUNK_STAGES;
  while (stages > 3 && stages * stage > 100 * 1024) --stages;
  const size_t smem = stages * stage;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(chunk_scan_kernel<RULE, KPL, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  chunk_scan_kernel<RULE, KPL, DP><<<dim3(requests, p.H, tiles), threads + 32, smem, stream>>>(
      prep, vact, places, state, p.slot_floats, p.state_slot, p.row_start, y, p.H, p.D, p.VD, cols_per_block, stages,
      write_state);
  TL_LAUNCH_CHECK();
  return 0;
}

template <int RULE, int DP>
static int chunk_scan(const TokenParams& p, float* state, float* y, int requests, int write_state, float* scratch, long long rows,
                      int sms, cudaStream_t stream) {
  const long long places = chunk_places(rows, requests);
  float* prep = scratch;
  float* vact = scratch + places * p.H * chunk_floats(RULE, DP);
  const dim3 grid((unsigned)((places + 3) / 4), p.H);
  const size_t smem = (size_t)4 * (RULE == WRITE_CHANNEL ? 3 : 2) * CH * DP * sizeof(float);
  if (smem > 48 * 1024) cudaFuncSetAttribute(chunk_prepare_kernel<RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  chunk_prepare_kernel<RULE><<<grid, 128, smem, stream>>>(p, prep, vact, DP, places, requests);
  TL_LAUNCH_CHECK();
  // a column goes to four times as many lanes (4 keys a lane) until the GPU has two warps a scheduler
  if constexpr (DP <= 128) {
    if ((long long)requests * p.H * p.VD * (DP / 16) < 256LL * sms)
      return launch_chunk_scan<RULE, 4, DP>(p, prep, vact, places, state, y, requests, write_state, sms, stream);
  }
  return launch_chunk_scan<RULE, 16, DP>(p, prep, vact, places, state, y, requests, write_state, sms, stream);
}

template <int RULE>
static int write_scan(const TokenParams& p, float* state, float* y, int requests, int write_state, float* scratch, long long rows,
                      int sms, cudaStream_t stream) {
  int P = 1;
  while (16 * P < p.D) P <<= 1;
  const int Dp = 16 * P;
  if (sms <= 0) sms = 148;
  if (scratch) {
    switch (Dp) {
      case 16: return chunk_scan<RULE, 16>(p, state, y, requests, write_state, scratch, rows, sms, stream);
      case 32: return chunk_scan<RULE, 32>(p, state, y, requests, write_state, scratch, rows, sms, stream);
      case 64: return chunk_scan<RULE, 64>(p, state, y, requests, write_state, scratch, rows, sms, stream);
      case 128: return chunk_scan<RULE, 128>(p, state, y, requests, write_state, scratch, rows, sms, stream);
      case 256: return chunk_scan<RULE, 256>(p, state, y, requests, write_state, scratch, rows, sms, stream);
      default: return chunk_scan<RULE, 512>(p, state, y, requests, write_state, scratch, rows, sms, stream);
    }
  }
  int threads, cols_per_block;
  recurrence_block(requests, p.H, p.VD, P, 2LL * sms, &threads, &cols_per_block);
  const int tiles = ceil_div(p.VD, cols_per_block);
  TL_REQUIRE(tiles <= 65535, "recurrence: %d tiles of value columns exceed the grid limit", tiles);
  const size_t smem = (size_t)(STEP_TOKENS * token_floats(RULE, Dp) + STEP_TOKENS * cols_per_block) * sizeof(float);
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(write_scan_kernel<RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  // (enough threads for every number of a token to be asked for at once)
  const int numbers = ceil_div(token_numbers<RULE>(Dp, cols_per_block), 32) * 32;
  if (threads < numbers) threads = numbers < REC_THREADS ? numbers : REC_THREADS;
  write_scan_kernel<RULE><<<dim3(requests, p.H, tiles), threads, smem, stream>>>(p, state, y, P, cols_per_block, write_state);
  TL_LAUNCH_CHECK();
  return 0;
}

}  // namespace tl

using namespace tl;

// floats of scratch the form for long portions wants (rule: 0 a decay a key channel, 1 a decay a head, 2 the gated memory; VD: the
// columns of the state)
extern "C" long long tl_write_scan_scratch_floats(long long rows, int requests, int H, int D, int VD, int rule) {
  int P = 1;
  while (16 * P < D) P <<= 1;
  return chunk_places(rows, requests) * H * ((long long)chunk_floats(rule, 16 * P) + (long long)CH * VD);
}

// The gated delta rule. A slot holds the last K - 1 inputs of the first `conv_cols` columns of proj at its beginning and the state
// [H, VD, D] `state_offset` floats behind. a_col >= 0: one decay a head, its logit at that column; else wl holds H * D logits a row.
// scratch: null runs the one-kernel form. The slot's inputs are not moved on here (tl_conv_state).
extern "C" int tl_gated_delta_scan(const float* proj, long long ld, int q_col, int k_col, int v_col, int b_col, int a_col,
                                   const float* wl, long long ld_w, const float* a_log, const float* dt_bias, float unit_eps,
                                   float q_scale, const float* taps, int K, int conv_cols, float* slots, long long slot_floats,
                                   long long state_offset, const int* state_slot, const int* row_start, const int* req_of_row,
                                   int requests, float* y, int H, int groups, int D, int VD, int write_state, float* scratch,
                                   long long rows, int sms, cudaStream_t stream) {
  if (requests == 0 || rows == 0) return 0;
  TL_REQUIRE(H > 0 && groups > 0 && H % groups == 0 && D >= 1 && D <= 512 && VD >= 1 && H <= 65535,
             "gated delta rule: %d heads over %d key heads, %d keys (up to 512), %d values", H, groups, D, VD);
  TL_REQUIRE(K >= 1 && taps && slots && a_log && dt_bias && (a_col >= 0 || wl), "gated delta rule: taps, decays and slots are needed");
  TokenParams p = {};
  p.proj = proj; p.ld = ld; p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.q_scale = q_scale; p.H = H; p.groups = groups;
  p.D = D; p.VD = VD; p.b_col = b_col; p.a_col = a_col; p.wl = wl; p.ld_w = ld_w; p.a_log = a_log; p.dt_bias = dt_bias;
  p.unit_eps = unit_eps; p.taps = taps; p.K = K; p.conv_state = slots; p.conv_cols = conv_cols; p.slot_floats = slot_floats;
  p.state_slot = state_slot; p.row_start = row_start; p.req_of_row = req_of_row;
  if (a_col >= 0) return write_scan<WRITE_HEAD>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
  return write_scan<WRITE_CHANNEL>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
}

// The gated matrix memory. A slot holds the heads' running maxima [H] at its beginning and the state [H, VD + 1, D] `state_offset`
// floats behind. y [rows, H, VD + 1]; maxima [rows, H]; factors: scratch [rows, H, 2].
extern "C" int tl_matrix_memory_scan(const float* proj, long long ld, int q_col, int k_col, int v_col, int i_col, int f_col,
                                     const float* i_bias, const float* f_bias, float cap, float q_scale, float* slots,
                                     long long slot_floats, long long state_offset, const int* state_slot, const int* row_start,
                                     int requests, float* y, float* maxima, float* factors, int H, int D, int VD, int write_state,
                                     float* scratch, long long rows, int sms, cudaStream_t stream) {
  if (requests == 0 || rows == 0) return 0;
  TL_REQUIRE(H > 0 && D >= 1 && D <= 512 && VD >= 1 && H <= 65535 && cap > 0.f,
             "matrix memory: %d heads, %d keys (up to 512), %d values, gates capped at %f", H, D, VD, cap);
  memory_factors_kernel<<<ceil_div(requests * H, 4), 128, 0, stream>>>(proj, ld, i_col, f_col, i_bias, f_bias, cap, slots, slot_floats,
                                                                       state_slot, row_start, factors, maxima, requests, H, write_state);
  TL_LAUNCH_CHECK();
  TokenParams p = {};
  p.proj = proj; p.ld = ld; p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.q_scale = q_scale; p.H = H; p.groups = H;
  p.D = D; p.VD = VD + 1; p.factors = factors; p.slot_floats = slot_floats; p.state_slot = state_slot; p.row_start = row_start;
  return write_scan<MEMORY>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
}

extern "C" int tl_memory_norm_gate(const float* y, const float* maxima, const float* gate, long long ld_gate, const float* weight,
                                   float eps, float floor_, void* out, long long ld_out, int rows, int H, int VD, int dtype,
                                   cudaStream_t stream) {
  if (rows == 0) return 0;
  TL_REQUIRE(H > 0 && VD > 0 && VD <= 2048, "memory norm: %d heads of %d (up to 2048)", H, VD);
  const unsigned blocks = (unsigned)(((long long)rows * H + 3) / 4);
#define TL_MNG(T_, HELD_)                                                                                                   \
  memory_norm_gate_kernel<T_, HELD_><<<blocks, 128, 0, stream>>>(y, maxima, gate, ld_gate, weight, eps, floor_, (T_*)out, ld_out, \
                                                                 rows, H, VD)
  if (dtype == TL_FP32) {
    if (VD <= 256) TL_MNG(float, 8);
    else TL_MNG(float, 64);
  } else {
    if (VD <= 256) TL_MNG(bf16, 8);
    else TL_MNG(bf16, 64);
  }
#undef TL_MNG
  TL_LAUNCH_CHECK();
  return 0;
}
