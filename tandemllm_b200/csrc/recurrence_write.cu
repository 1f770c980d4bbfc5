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
// As in recurrence.cu there are two forms. Steps of a few rows a request: one kernel whose blocks prepare up to eight tokens in
// shared memory, a warp a token, and walk them. Longer portions: a warp a (row, head) prepares all rows side by side into scratch,
// convolutions included, and the scan of recurrence.cuh fetches them through its ring. Both prepare a token with the same code.
// The convolution's inputs before the step come from the slot (its last taps - 1 inputs, oldest first); they are moved on by a
// kernel of their own behind the scan, because the heads that share a key read the same inputs. The running maximum m is a chain
// over a request's rows in a kernel of its own in front (a warp a request and head), which leaves the two factors of every row.
#include "recurrence.cuh"

namespace tl {

__device__ __forceinline__ float softplusf_(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

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
__device__ __forceinline__ float conv_silu_at(const TokenParams& p, long long r, int first, const float* __restrict__ past, int c) {
  const float* tap = p.taps + (long long)c * p.K;
  float acc = 0.f;
  for (int j = 0; j < p.K; ++j) {
    const long long src = r - (p.K - 1) + j;
    const float u = src >= first ? p.proj[src * p.ld + c] : past[(long long)(p.K - 1 + (src - first)) * p.conv_cols + c];
    acc = fmaf(tap[j], u, acc);
  }
  return siluf_(acc);
}

// One warp prepares (row r, head h) into tok (rec_token_floats of it); returns what the head's values are multiplied by.
template <int RULE>
__device__ __forceinline__ float prepare_token(const TokenParams& p, long long r, int h, int first, const float* __restrict__ past,
                                               float* __restrict__ tok, int Dp, int lane) {
  const int D = p.D;
  float* tq = tok;
  float* tk = tok + Dp;
  float* num = tok + rec_arrays(RULE) * Dp;
  if constexpr (RULE == RULE_MEMORY) {
    const float* q = p.proj + r * p.ld + p.q_col + (long long)h * D;
    const float* k = p.proj + r * p.ld + p.k_col + (long long)h * D;
    const float keep = p.factors[(r * p.H + h) * 2], add = p.factors[(r * p.H + h) * 2 + 1];
    for (int i = lane; i < Dp; i += 32) {
      tq[i] = i < D ? q[i] * p.q_scale : 0.f;
      tk[i] = i < D ? k[i] * add : 0.f;
    }
    if (lane < 4) num[lane] = lane == 0 ? keep : 0.f;
    return 1.f;
  } else {
    const int g = h / (p.H / p.groups);
    constexpr int HELD = 512 / 32;              // entries a lane holds of a head of up to 512 keys
    float q[HELD], k[HELD];
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int t = 0; t < HELD; ++t) {
      const int i = lane + 32 * t;
      q[t] = k[t] = 0.f;
      if (i < D) {
        q[t] = conv_silu_at(p, r, first, past, p.q_col + g * D + i);
        k[t] = conv_silu_at(p, r, first, past, p.k_col + g * D + i);
        qq = fmaf(q[t], q[t], qq);
        kk = fmaf(k[t], k[t], kk);
      }
      if (32 * (t + 1) >= Dp) break;
    }
    const float qs = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), ks = 1.f / sqrtf(warp_sum(kk) + p.unit_eps);
    const float beta = sigmoidf_(p.proj[r * p.ld + p.b_col + h]);
    const float rate = -expf(p.a_log[h]);
    float d_h = 0.f;
    if constexpr (RULE == RULE_WRITE_HEAD) {
      d_h = expf(rate * softplusf_(p.proj[r * p.ld + p.a_col + h] + p.dt_bias[h]));
      if (lane < 4) num[lane] = lane == 0 ? d_h : (lane == 1 ? d_h * beta : 0.f);
    }
#pragma unroll
    for (int t = 0; t < HELD; ++t) {
      const int i = lane + 32 * t;
      if (i < Dp) {
        const float ki = k[t] * ks;
        tq[i] = q[t] * qs;
        tk[i] = ki;
        if constexpr (RULE == RULE_WRITE_CHANNEL) {
          const float d = i < D ? expf(rate * softplusf_(p.wl[r * p.ld_w + (long long)h * D + i] + p.dt_bias[h * D + i])) : 0.f;
          tok[2 * Dp + i] = d;
          tok[3 * Dp + i] = beta * (d * ki);
        }
      }
      if (32 * (t + 1) >= Dp) break;
    }
    return beta;
  }
}

// The value of column j of (row r, head h).
template <int RULE>
__device__ __forceinline__ float token_value(const TokenParams& p, long long r, int h, int first, const float* __restrict__ past,
                                             int j, float times) {
  if constexpr (RULE == RULE_MEMORY) return j == p.VD - 1 ? 1.f : p.proj[r * p.ld + p.v_col + (long long)h * (p.VD - 1) + j];
  else return times * conv_silu_at(p, r, first, past, p.v_col + h * p.VD + j);
}

// One warp a (row, head): the prepared token into prep [H][rows][rec_token_floats], its values into vact [rows][H * VD].
template <int RULE>
__global__ void __launch_bounds__(128) write_prepare_kernel(TokenParams p, float* __restrict__ prep, float* __restrict__ vact, int Dp,
                                                            long long rows) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long idx = (long long)blockIdx.x * 4 + warp;
  if (idx >= rows * p.H) return;
  const long long r = idx / p.H;
  const int h = (int)(idx - r * p.H);
  const int b = RULE == RULE_MEMORY ? 0 : p.req_of_row[r];
  const int first = RULE == RULE_MEMORY ? 0 : p.row_start[b];
  const float* past = RULE == RULE_MEMORY ? nullptr : p.conv_state + (long long)p.state_slot[b] * p.slot_floats;
  float* tok = prep + ((long long)h * rows + r) * rec_token_floats(RULE, Dp);
  const float times = prepare_token<RULE>(p, r, h, first, past, tok, Dp, lane);
  for (int j = lane; j < p.VD; j += 32) vact[idx * p.VD + j] = token_value<RULE>(p, r, h, first, past, j, times);
}

// Steps of a few rows a request: grid (requests, heads, tiles of value columns); thread (column, part) holds 16 keys of a column.
template <int RULE>
__global__ void __launch_bounds__(REC_THREADS) write_scan_kernel(TokenParams p, float* __restrict__ state, float* __restrict__ y, int P,
                                                                 int cols_per_block, int write_state) {
  extern __shared__ __align__(16) float sm[];
  const int Dp = 16 * P, tok_floats = rec_token_floats(RULE, Dp), D = p.D, VD = p.VD;
  float* s_v = sm + REC_TOKENS * tok_floats;            // [REC_TOKENS][cols_per_block]
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = tid % P, jl = tid / P, j = col0 + jl;
  const bool owns = jl < cols_per_block && j < VD;
  const int r0 = p.row_start[b], r1 = p.row_start[b + 1];
  if (r1 <= r0) return;
  const long long slot = p.state_slot[b];
  float* S = state + slot * p.slot_floats + (long long)h * D * VD;
  const float* past = RULE == RULE_MEMORY ? nullptr : p.conv_state + slot * p.slot_floats;
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
  const int chunk_tokens = min(REC_TOKENS, (int)(blockDim.x >> 5));      // a warp a token
  for (int t0 = r0; t0 < r1; t0 += chunk_tokens) {
    const int nt = min(chunk_tokens, r1 - t0);
    __syncthreads();                      // the chunk before has been read
    if (warp < nt) {
      const float times = prepare_token<RULE>(p, t0 + warp, h, r0, past, sm + warp * tok_floats, Dp, lane);
      for (int c = lane; c < cols_per_block; c += 32)
        s_v[warp * cols_per_block + c] = col0 + c < VD ? token_value<RULE>(p, t0 + warp, h, r0, past, col0 + c, times) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float4* a = reinterpret_cast<const float4*>(sm + t * tok_floats) + part;
      const float* num = sm + t * tok_floats + rec_arrays(RULE) * Dp;
      const int Q = 4 * P;
      float w = jl < cols_per_block ? s_v[t * cols_per_block + jl] : 0.f;
      if constexpr (RULE != RULE_MEMORY) {
        const float4* u4 = a + (RULE == RULE_WRITE_CHANNEL ? 3 : 1) * Q;
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
        w = RULE == RULE_WRITE_HEAD ? fmaf(-num[1], us, w) : w - us;
      }
      const float d_h = RULE == RULE_WRITE_CHANNEL ? 0.f : num[0];
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float4 q = a[P * m], k = a[Q + P * m];
        const float4 d = RULE == RULE_WRITE_CHANNEL ? a[2 * Q + P * m] : make_float4(d_h, d_h, d_h, d_h);
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

// grid (rows, heads): o = y / (max(|y_ones|, exp(-maximum)) + floor) with the head's output of the column of ones behind its others,
// then o / rms(o), times the weight, times sigmoid(gate)
template <typename T>
__global__ void memory_norm_gate_kernel(const float* __restrict__ y, const float* __restrict__ maxima, const float* __restrict__ gate,
                                        long long ld_gate, const float* __restrict__ weight, float eps, float floor_,
                                        T* __restrict__ out, long long ld_out, int H, int VD) {
  __shared__ float red[33];
  const int r = blockIdx.x, h = blockIdx.y;
  const float* yr = y + ((long long)r * H + h) * (VD + 1);
  const float inv_den = 1.f / (fmaxf(fabsf(yr[VD]), expf(-maxima[(long long)r * H + h])) + floor_);
  float ss = 0.f;
  for (int i = threadIdx.x; i < VD; i += blockDim.x) {
    const float o = yr[i] * inv_den;
    ss = fmaf(o, o, ss);
  }
  ss = block_sum(ss, red);
  const float inv = inv_den / sqrtf(ss / (float)VD + eps);
  for (int i = threadIdx.x; i < VD; i += blockDim.x) {
    const int c = h * VD + i;
    out[(long long)r * ld_out + c] = from_f32<T>(yr[i] * inv * weight[c] * sigmoidf_(gate[(long long)r * ld_gate + c]));
  }
}

template <int RULE>
static int write_scan(const TokenParams& p, float* state, float* y, int requests, int write_state, float* scratch, long long rows,
                      int sms, cudaStream_t stream) {
  int P = 1;
  while (16 * P < p.D) P <<= 1;
  const int Dp = 16 * P;
  if (scratch) {
    const long long pairs = rows * p.H;
    float* prep = scratch;
    float* vact = scratch + pairs * rec_token_floats(RULE, Dp);
    write_prepare_kernel<RULE><<<(unsigned)((pairs + 3) / 4), 128, 0, stream>>>(p, prep, vact, Dp, rows);
    TL_LAUNCH_CHECK();
    const StagedScan a{prep, vact, (long long)p.H * p.VD, 0, nullptr, state, p.slot_floats, p.state_slot, p.row_start, requests, y,
                       rows, p.H, p.D, p.VD, write_state, sms};
    return launch_staged_scan<RULE>(a, stream);
  }
  int threads, cols_per_block;
  recurrence_block(requests, p.H, p.VD, P, 2LL * (sms > 0 ? sms : 148), &threads, &cols_per_block);
  const int tiles = ceil_div(p.VD, cols_per_block);
  TL_REQUIRE(tiles <= 65535, "recurrence: %d tiles of value columns exceed the grid limit", tiles);
  const size_t smem = (size_t)(REC_TOKENS * rec_token_floats(RULE, Dp) + REC_TOKENS * cols_per_block) * sizeof(float);
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(write_scan_kernel<RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  write_scan_kernel<RULE><<<dim3(requests, p.H, tiles), threads, smem, stream>>>(p, state, y, P, cols_per_block, write_state);
  TL_LAUNCH_CHECK();
  return 0;
}

}  // namespace tl

using namespace tl;

// floats of scratch the form for long portions wants (rule: 3 a decay a key channel, 4 a decay a head, 5 the gated memory; VD: the
// columns of the state)
extern "C" long long tl_write_scan_scratch_floats(long long rows, int H, int D, int VD, int rule) {
  int P = 1;
  while (16 * P < D) P <<= 1;
  return rows * H * ((long long)rec_token_floats(rule, 16 * P) + VD);
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
  if (a_col >= 0) return write_scan<RULE_WRITE_HEAD>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
  return write_scan<RULE_WRITE_CHANNEL>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
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
  return write_scan<RULE_MEMORY>(p, slots + state_offset, y, requests, write_state, scratch, rows, sms, stream);
}

extern "C" int tl_memory_norm_gate(const float* y, const float* maxima, const float* gate, long long ld_gate, const float* weight,
                                   float eps, float floor_, void* out, long long ld_out, int rows, int H, int VD, int dtype,
                                   cudaStream_t stream) {
  if (rows == 0) return 0;
  TL_REQUIRE(H > 0 && H <= 65535 && VD > 0, "memory norm: %d heads of %d", H, VD);
  const int threads = VD > 128 ? 128 : (VD > 32 ? 64 : 32);
  if (dtype == TL_FP32)
    memory_norm_gate_kernel<float><<<dim3(rows, H), threads, 0, stream>>>(y, maxima, gate, ld_gate, weight, eps, floor_, (float*)out,
                                                                          ld_out, H, VD);
  else
    memory_norm_gate_kernel<bf16><<<dim3(rows, H), threads, 0, stream>>>(y, maxima, gate, ld_gate, weight, eps, floor_, (bf16*)out,
                                                                         ld_out, H, VD);
  TL_LAUNCH_CHECK();
  return 0;
}
