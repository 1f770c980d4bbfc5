// What the scans over a matrix state share: the rules, a token group's arithmetic, the scan over prepared tokens and its launcher
// (see recurrence.cu for how the scan is laid out; recurrence.cu and recurrence_write.cu instantiate it for their rules).
#pragma once

#include "common.cuh"

namespace tl {

constexpr int REC_TOKENS = 8;       // tokens staged at a time: one a warp
constexpr int REC_THREADS = 256;

__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float siluf_(float x) { return x / (1.f + expf(-x)); }
// sigmoid(z)^rate without forming the sigmoid: exp(-rate * log(1 + e^-z)), the logarithm split so that neither e^-z nor e^z overflows
__device__ __forceinline__ float sigmoid_powf_(float z, float rate) {
  return expf(-rate * (fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))));
}

// A rule's update of a column s of the state with the column's value v, from what a prepared token holds:
//   RULE_FIXED          q, k                      s <- c_h s + k v                     (c_h fixed for the head)
//   RULE_DELTA          q, k, d, u, au            s <- d s - au (u . s) + k v
//   RULE_GATED          q, k, d                   s <- d s + k v
//   RULE_WRITE_CHANNEL  q, k, d, w                s <- d s + k (v - w . s)             (w = beta d k, v already times beta)
//   RULE_WRITE_HEAD     q, k; numbers d, w        s <- d s + k (v - w (k . s))         (d and w = beta d one number a head)
//   RULE_MEMORY         q, k; number d            s <- d s + k v                       (k already times its input gate)
constexpr int RULE_FIXED = 0, RULE_DELTA = 1, RULE_GATED = 2, RULE_WRITE_CHANNEL = 3, RULE_WRITE_HEAD = 4, RULE_MEMORY = 5;
__host__ __device__ constexpr int rec_arrays(int rule) {
  return rule == RULE_DELTA ? 5 : (rule == RULE_WRITE_CHANNEL ? 4 : (rule == RULE_GATED ? 3 : 2));
}
// numbers of the whole token behind its arrays (filled up to 16 bytes)
__host__ __device__ constexpr int rec_numbers(int rule) { return rule >= RULE_WRITE_HEAD ? 4 : 0; }
__host__ __device__ constexpr int rec_token_floats(int rule, int Dp) { return rec_arrays(rule) * Dp + rec_numbers(rule); }
// the state in a slot: [keys][values], or [values][keys] (a lane's four neighbouring keys are 16 bytes of a column)
__host__ __device__ constexpr bool rec_value_major(int rule) { return rule >= RULE_WRITE_CHANNEL; }

__device__ __forceinline__ void rec_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void rec_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Sums v[0..T) over the P neighbouring lanes that share a column (`part` = the lane's place among them; P divides 32). Each
// crossing halves what a lane still holds: afterwards v[i], i < T / P, of lane `part` are the whole sums of tokens
// part * (T / P) + i; with more lanes than tokens, v[0] of the P / T lanes from part = token * (P / T) on is that token's sum.
constexpr int REC_GROUP = 8;
constexpr int REC_CHUNK = 16;     // the most tokens a stage holds; a column's values of a stage lie this far apart
template <int T, int P>
__device__ __forceinline__ void rec_reduce_scatter(float (&v)[T], int part) {
#pragma unroll
  for (int step = 0; (P >> 1 >> step) > 0; ++step) {
    const int off = P >> 1 >> step;
    const int cnt = (T >> step) > 1 ? (T >> step) : 1;
    if (cnt > 1) {
      const int half = cnt / 2;
      const bool up = (part & off) != 0;
#pragma unroll
      for (int i = 0; i < half; ++i) {
        const float send = up ? v[i] : v[i + half];
        const float keep = up ? v[i + half] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
    }
  }
}

// REC_GROUP tokens (FULL) or the first n of them for one lane: the lane's KPL keys of its column go through the tokens, the
// outputs wait in registers and cross the lanes together. Everything a token needs lies at offsets the compiler knows
// (`tok`: the lane's first four floats of the group's first prepared token; `vcol`: the column's values, a token a float),
// so the group is straight-line code whose loads the compiler moves ahead of the chain.
template <int RULE, int KPL, int DP, bool FULL>
__device__ __forceinline__ void rec_group(float (&s)[KPL], const float* __restrict__ tok, const float* __restrict__ vcol,
                                          float* __restrict__ yg, long long ldy, int n, int part, bool owns, float c_h) {
  constexpr bool DELTA = RULE == RULE_DELTA, GATED = RULE == RULE_GATED;
  constexpr bool WRITE = RULE == RULE_WRITE_CHANNEL || RULE == RULE_WRITE_HEAD;
  constexpr int P = DP / KPL, M = KPL / 4, tok_floats = rec_token_floats(RULE, DP), Q = DP / 4;
  float o[REC_GROUP];
#pragma unroll
  for (int tt = 0; tt < REC_GROUP; ++tt) {
    o[tt] = 0.f;
    if (FULL || tt < n) {
      const float4* a = reinterpret_cast<const float4*>(tok + tt * tok_floats);
      const float vj = vcol[tt];
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
      if (DELTA) {
        float us0 = 0.f, us1 = 0.f, us2 = 0.f, us3 = 0.f;      // four short chains of additions instead of one long one
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const float4 u = a[3 * Q + P * m];
          us0 = fmaf(u.x, s[4 * m], us0);
          us1 = fmaf(u.y, s[4 * m + 1], us1);
          us2 = fmaf(u.z, s[4 * m + 2], us2);
          us3 = fmaf(u.w, s[4 * m + 3], us3);
        }
        float us = (us0 + us1) + (us2 + us3);
#pragma unroll
        for (int off = P >> 1; off > 0; off >>= 1) us += __shfl_xor_sync(0xffffffffu, us, off);
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const float4 q = a[P * m], k = a[Q + P * m], d = a[2 * Q + P * m], au = a[4 * Q + P * m];
          s[4 * m] = fmaf(d.x, s[4 * m], fmaf(-au.x, us, k.x * vj));
          s[4 * m + 1] = fmaf(d.y, s[4 * m + 1], fmaf(-au.y, us, k.y * vj));
          s[4 * m + 2] = fmaf(d.z, s[4 * m + 2], fmaf(-au.z, us, k.z * vj));
          s[4 * m + 3] = fmaf(d.w, s[4 * m + 3], fmaf(-au.w, us, k.w * vj));
          o0 = fmaf(s[4 * m], q.x, o0);
          o1 = fmaf(s[4 * m + 1], q.y, o1);
          o2 = fmaf(s[4 * m + 2], q.z, o2);
          o3 = fmaf(s[4 * m + 3], q.w, o3);
        }
      } else if (GATED) {
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const float4 q = a[P * m], k = a[Q + P * m], d = a[2 * Q + P * m];
          s[4 * m] = fmaf(d.x, s[4 * m], k.x * vj);
          s[4 * m + 1] = fmaf(d.y, s[4 * m + 1], k.y * vj);
          s[4 * m + 2] = fmaf(d.z, s[4 * m + 2], k.z * vj);
          s[4 * m + 3] = fmaf(d.w, s[4 * m + 3], k.w * vj);
          o0 = fmaf(s[4 * m], q.x, o0);
          o1 = fmaf(s[4 * m + 1], q.y, o1);
          o2 = fmaf(s[4 * m + 2], q.z, o2);
          o3 = fmaf(s[4 * m + 3], q.w, o3);
        }
      } else if (WRITE) {
        // what the decayed state already holds for this key, taken off the value before it is written
        const float* num = tok - 4 * part + tt * tok_floats + rec_arrays(RULE) * DP;
        float us0 = 0.f, us1 = 0.f, us2 = 0.f, us3 = 0.f;
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const float4 u = a[(RULE == RULE_WRITE_CHANNEL ? 3 : 1) * Q + P * m];
          us0 = fmaf(u.x, s[4 * m], us0);
          us1 = fmaf(u.y, s[4 * m + 1], us1);
          us2 = fmaf(u.z, s[4 * m + 2], us2);
          us3 = fmaf(u.w, s[4 * m + 3], us3);
        }
        float us = (us0 + us1) + (us2 + us3);
#pragma unroll
        for (int off = P >> 1; off > 0; off >>= 1) us += __shfl_xor_sync(0xffffffffu, us, off);
        const float d_h = RULE == RULE_WRITE_HEAD ? num[0] : 0.f;
        const float w = RULE == RULE_WRITE_HEAD ? fmaf(-num[1], us, vj) : vj - us;
#pragma unroll
        for (int m = 0; m < M; ++m) {
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
      } else {
        const float c_t = RULE == RULE_MEMORY ? (tok - 4 * part)[tt * tok_floats + rec_arrays(RULE) * DP] : c_h;
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const float4 q = a[P * m], k = a[Q + P * m];
          s[4 * m] = fmaf(c_t, s[4 * m], k.x * vj);
          s[4 * m + 1] = fmaf(c_t, s[4 * m + 1], k.y * vj);
          s[4 * m + 2] = fmaf(c_t, s[4 * m + 2], k.z * vj);
          s[4 * m + 3] = fmaf(c_t, s[4 * m + 3], k.w * vj);
          o0 = fmaf(s[4 * m], q.x, o0);
          o1 = fmaf(s[4 * m + 1], q.y, o1);
          o2 = fmaf(s[4 * m + 2], q.z, o2);
          o3 = fmaf(s[4 * m + 3], q.w, o3);
        }
      }
      o[tt] = (o0 + o1) + (o2 + o3);
    }
  }
  rec_reduce_scatter<REC_GROUP, P>(o, part);
  if (!owns) return;
  if (P <= REC_GROUP) {
    constexpr int each = P <= REC_GROUP ? REC_GROUP / P : 1;
#pragma unroll
    for (int i = 0; i < each; ++i) {
      const int t = part * each + i;
      if (FULL || t < n) yg[t * ldy] = o[i];
    }
  } else {
    constexpr int share = P > REC_GROUP ? P / REC_GROUP : 1;
    const int t = part / share;
    if (part % share == 0 && (FULL || t < n)) yg[t * ldy] = o[0];
  }
}

// A lane's KPL keys of column j of a head's state: keys 4 (part + P m) + c.
template <int KPL, int P, bool VALUE_MAJOR>
__device__ __forceinline__ void rec_load_state(float (&s)[KPL], const float* __restrict__ S, int part, int j, int D, int VD,
                                               bool owns) {
  if (VALUE_MAJOR && (D & 3) == 0 && ((uintptr_t)S & 15) == 0) {
#pragma unroll
    for (int m = 0; m < KPL / 4; ++m) {
      const int i = 4 * (part + P * m);
      const float4 v = (owns && i < D) ? *reinterpret_cast<const float4*>(S + (long long)j * D + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[4 * m] = v.x; s[4 * m + 1] = v.y; s[4 * m + 2] = v.z; s[4 * m + 3] = v.w;
    }
    return;
  }
#pragma unroll
  for (int m = 0; m < KPL / 4; ++m)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int i = 4 * (part + P * m) + c;
      s[4 * m + c] = (owns && i < D) ? S[VALUE_MAJOR ? (long long)j * D + i : (long long)i * VD + j] : 0.f;
    }
}
template <int KPL, int P, bool VALUE_MAJOR>
__device__ __forceinline__ void rec_store_state(const float (&s)[KPL], float* __restrict__ S, int part, int j, int D, int VD) {
  if (VALUE_MAJOR && (D & 3) == 0 && ((uintptr_t)S & 15) == 0) {
#pragma unroll
    for (int m = 0; m < KPL / 4; ++m) {
      const int i = 4 * (part + P * m);
      if (i < D) *reinterpret_cast<float4*>(S + (long long)j * D + i) = make_float4(s[4 * m], s[4 * m + 1], s[4 * m + 2], s[4 * m + 3]);
    }
    return;
  }
#pragma unroll
  for (int m = 0; m < KPL / 4; ++m)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int i = 4 * (part + P * m) + c;
      if (i < D) S[VALUE_MAJOR ? (long long)j * D + i : (long long)i * VD + j] = s[4 * m + c];
    }
}

// The scan over prepared tokens. Block: cols_per_block * P computing threads (a multiple of 32) and one more warp, the
// producer, which does nothing but fetch: it keeps STAGES - 1 chunks of TC tokens in flight (each token's NARR * Dp prepared
// floats, then the chunk's values, a column's REC_CHUNK apart) and meets the computing warps at one barrier a chunk, when the next
// chunk has landed and the last one has been read.
// KPL keys of a column a lane (16 or 4): with 4, four times as many lanes share a column and a token takes a warp a
// third of the instructions, at the price of two more lane crossings a sum; the launcher takes 4 where the GPU would
// otherwise stand idle. DP: the keys a head, filled up to a power of two (16 at least); sizes known to the compiler keep
// the loop free of address arithmetic.
constexpr int REC_STAGES = 3;
template <int RULE, int KPL, int DP>
__global__ void __launch_bounds__(REC_THREADS + 32) recurrence_scan_staged_kernel(
    const float* __restrict__ prep, const float* __restrict__ vsrc, long long ld_v, int v_col, const float* __restrict__ head_decay,
    float* __restrict__ state, long long slot_floats, const int* __restrict__ state_slot, const int* __restrict__ row_start,
    float* __restrict__ y, long long rows, int H, int D, int VD, int cols_per_block, int TC, int write_state) {
  constexpr int STAGES = REC_STAGES, P = DP / KPL, Dp = DP;
  extern __shared__ __align__(16) float sm[];
  constexpr int tok_floats = rec_token_floats(RULE, Dp);
  const int stage_floats = TC * tok_floats + REC_CHUNK * cols_per_block;
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x, nth = blockDim.x - 32;
  const bool producer = tid >= nth;
  const int part = tid % P, jl = tid / P, j = col0 + jl;
  const bool owns = !producer && j < VD;
  const int r0 = row_start[b], r1 = row_start[b + 1];
  if (r1 <= r0) return;
  float* S = state + (long long)state_slot[b] * slot_floats + (long long)h * D * VD;
  const float c_h = RULE == RULE_FIXED ? head_decay[h] : 0.f;
  const int n_chunks = (r1 - r0 + TC - 1) / TC;

  // (the producer's lanes only)
  auto load = [&](int chunk) {
    const int lane = tid - nth;
    const int t0 = r0 + chunk * TC, nt = min(TC, r1 - t0);
    float* base = sm + (chunk % STAGES) * stage_floats;
    const float* src = prep + ((long long)h * rows + t0) * tok_floats;
    const int pieces = nt * (tok_floats / 4);
#pragma unroll 4
    for (int i = lane; i < pieces; i += 32) rec_cp16(base + 4 * i, src + 4 * i);
    float* vb = base + TC * tok_floats;
    const float* vs = vsrc + (long long)t0 * ld_v + v_col + (long long)h * VD + col0;
    for (int e = lane; e < nt * cols_per_block; e += 32) {
      const int t = e / cols_per_block, c = e - t * cols_per_block;
      if (col0 + c < VD) rec_cp4(vb + c * REC_CHUNK + t, vs + (long long)t * ld_v + c);
      else vb[c * REC_CHUNK + t] = 0.f;
    }
  };
  float s[KPL];
  if (producer) {
#pragma unroll
    for (int s0 = 0; s0 < STAGES - 1; ++s0) {
      if (s0 < n_chunks) load(s0);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");       // chunk 0 has landed
  } else {
    rec_load_state<KPL, P, rec_value_major(RULE)>(s, S, part, j, D, VD, owns);
  }
  __syncthreads();

  for (int chunk = 0; chunk < n_chunks; ++chunk) {
    if (producer) {
      // the stage of chunk - 1 is free (everybody passed the barrier behind it): refill it, then wait for chunk + 1
      if (chunk + STAGES - 1 < n_chunks) load(chunk + STAGES - 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    } else {
      const int t0 = r0 + chunk * TC, nt = min(TC, r1 - t0);
      const float* base = sm + (chunk % STAGES) * stage_floats;
      const float* tok = base + 4 * part;
      const float* vcol = base + TC * tok_floats + jl * REC_CHUNK;
      const long long ldy = (long long)H * VD;
      float* yg = y + (long long)t0 * ldy + (long long)h * VD + j;
      int g = 0;
      for (; g + REC_GROUP <= nt; g += REC_GROUP)
        rec_group<RULE, KPL, DP, true>(s, tok + g * tok_floats, vcol + g, yg + g * ldy, ldy, REC_GROUP, part, owns, c_h);
      if (g < nt) rec_group<RULE, KPL, DP, false>(s, tok + g * tok_floats, vcol + g, yg + g * ldy, ldy, nt - g, part, owns, c_h);
    }
    __syncthreads();
  }
  if (write_state && owns) rec_store_state<KPL, P, rec_value_major(RULE)>(s, S, part, j, D, VD);
}

// Threads a block (a multiple of 32, at least P) and the value columns it takes: the largest block that still gives the GPU
// `want_blocks` blocks, else a single warp; never more columns than there are. (Steps of a few rows want many blocks in
// flight for the states they read and write; the staged form's blocks each fetch every prepared token of their head, so
// they stay as large as fills three SMs in four.)
static void recurrence_block(int requests, int H, int VD, int P, long long want_blocks, int* threads, int* cols) {
  const int needed = ((VD * P + 31) / 32) * 32;
  int th = REC_THREADS;
  while (th > 32 && th / 2 >= P && (long long)requests * H * ceil_div(VD, th / P) < want_blocks) th >>= 1;
  if (th > needed) th = needed;
  if (th < P) th = P;
  *threads = th;
  *cols = th / P;
}

struct StagedScan {
  const float* prep;           // [H][rows][rec_token_floats]
  const float* vsrc;           // the columns' values: entry v_col + h VD + j of rows ld_v apart
  long long ld_v;
  int v_col;
  const float* head_decay;
  float* state;
  long long slot_floats;
  const int *state_slot, *row_start;
  int requests;
  float* y;
  long long rows;
  int H, D, VD, write_state, sm_count;
};

// Sizes the blocks and stages and launches the scan over prepared tokens.
template <int RULE>
static int launch_staged_scan(const StagedScan& a, cudaStream_t stream) {
  const int D = a.D, VD = a.VD, H = a.H;
  int P = 1;
  while (16 * P < D) P <<= 1;
  const int Dp = 16 * P;
  const int sms = a.sm_count > 0 ? a.sm_count : 148;
  // a column goes to four times as many lanes (4 keys a lane) until the GPU has two warps a scheduler
  int kpl = 16;
  if (4 * P <= 32 && (long long)a.requests * H * VD * P < 256LL * sms) {
    kpl = 4;
    P *= 4;
  }
  int threads, cols_per_block;
  recurrence_block(a.requests, H, VD, P, (3LL * sms) / 4, &threads, &cols_per_block);
  const int tiles = ceil_div(VD, cols_per_block);
  TL_REQUIRE(tiles <= 65535, "recurrence_scan: %d tiles of value columns exceed the grid limit", tiles);
  dim3 grid(a.requests, H, tiles);
  // tokens a stage: as many (16 at most) as 96 KB hold in three stages
  int TC = REC_CHUNK;
  auto bytes = [&](int tc) { return (size_t)REC_STAGES * (tc * rec_token_floats(RULE, Dp) + REC_CHUNK * cols_per_block) * sizeof(float); };
  while (TC > 1 && bytes(TC) > 96 * 1024) TC >>= 1;
  const size_t smem = bytes(TC);
#define TL_RSS(KPL_, DP_)                                                                                                       \
  do {                                                                                                                          \
    if (smem > 48 * 1024)                                                                                                       \
      cudaFuncSetAttribute(recurrence_scan_staged_kernel<RULE, KPL_, DP_>, cudaFuncAttributeMaxDynamicSharedMemorySize,         \
                           96 * 1024);                                                                                          \
    recurrence_scan_staged_kernel<RULE, KPL_, DP_><<<grid, threads + 32, smem, stream>>>(                                       \
        a.prep, a.vsrc, a.ld_v, a.v_col, a.head_decay, a.state, a.slot_floats, a.state_slot, a.row_start, a.y, a.rows, H, D, VD, \
        cols_per_block, TC, a.write_state);                                                                                     \
  } while (0)
#define TL_RSS_D(DP_)                                          \
  do {                                                         \
    if (kpl == 16) TL_RSS(16, DP_);                            \
    else if (DP_ <= 128) TL_RSS(4, (DP_ <= 128 ? DP_ : 128));  \
  } while (0)
  switch (Dp) {
    case 16: TL_RSS_D(16); break;
    case 32: TL_RSS_D(32); break;
    case 64: TL_RSS_D(64); break;
    case 128: TL_RSS_D(128); break;
    case 256: TL_RSS_D(256); break;
    default: TL_RSS_D(512); break;
  }
#undef TL_RSS_D
#undef TL_RSS
  TL_LAUNCH_CHECK();
  return 0;
}

}  // namespace tl
