// Row-wise kernels: embedding gather (with a second table over pairs of tokens), residual add fused with RMS norm (and, for the rows of an expert layer, with
// the router), SwiGLU gating, and the last error message of the library.
//
// The residual stream is 32-bit in both precisions; norms compute mean(x^2), rsqrt and the scale in
// 32-bit and round once to the compute type. Formulas: engine/models/lfm2_moe/ref.py:105-109 (norm),
// :230 (embedding), :180-183 (SwiGLU), :185-197 (router) of the reference, which fuses the add and the norm too
// (`add_rms`, engine/models/lfm2_moe/kernels.py:90-107).
#include "add_rmsnorm.cuh"

extern "C" const char* tl_last_error() { return tl_error_text; }

// The constants that the gated launches of this thread pass beside their activation code from now on.
extern "C" int tl_set_gate_constants(float a0, float a1) {
  tl_gate_constants[0] = a0;
  tl_gate_constants[1] = a1;
  return 0;
}

extern "C" const char* tl_cuda_error_string(int code) { return cudaGetErrorString((cudaError_t)code); }

namespace tl {

// residual[r, :] = float(table[token[r], :]) * scale, written `copies` times, copy_stride floats apart (a model that carries
// several streams starts them all from the embedded row)
template <typename T>
__global__ void embed_rows_kernel(const T* __restrict__ table, const int* __restrict__ tokens,
                                  float* __restrict__ residual, int hidden, int vocab, int* __restrict__ status, float scale,
                                  int copies, long long copy_stride) {
  chain_next();
  chain_wait();
  const int r = blockIdx.x;
  int tok = tokens[r];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0) atomicExch(status, 1);   // recorded, and the row reads token 0 instead of faulting
    tok = 0;
  }
  const T* src = table + (size_t)tok * hidden;
  float* dst = residual + (size_t)r * hidden;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    const float v = to_f32(src[c]) * scale;
    for (int s = 0; s < copies; ++s) dst[(long long)s * copy_stride + c] = v;
  }
}

// residual[r, :] = float(table[t, :]) * scale + float(pairs[row, :]), t the row's token and row = (before * mul_prev + t * mul_cur)
// mod buckets, `before` the token in front of it in its sequence; a sequence's first token reads row `buckets`. Inside a portion the
// token in front is the row before; a portion's first row finds it in the request's slot (last_token; negative: there is none), and
// leaves the portion's last token there once it has read it. No other block touches the slot.
template <typename T>
__global__ void embed_token_pairs_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ tokens,
                                         const int* __restrict__ req_of_row, const int* __restrict__ row_start,
                                         const int* __restrict__ state_slot, int* __restrict__ last_token,
                                         float* __restrict__ residual, int hidden, int vocab, long long buckets, long long mul_prev,
                                         long long mul_cur, int* __restrict__ status, float scale) {
  __shared__ long long s_row;
  chain_next();
  chain_wait();
  const int r = blockIdx.x;
  int tok = tokens[r];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0) atomicExch(status, 1);   // recorded, and the row reads token 0 instead of faulting
    tok = 0;
  }
  if (threadIdx.x == 0) {
    const int b = req_of_row[r], first = row_start[b];
    int before;
    if (r == first) {
      int* slot = last_token + state_slot[b];
      before = *slot;
      *slot = tokens[row_start[b + 1] - 1];
    } else {
      before = tokens[r - 1];
    }
    long long at = buckets;
    if (before >= 0) {
      at = ((long long)before * mul_prev + (long long)tok * mul_cur) % buckets;
      if (at < 0) at += buckets;
    }
    s_row = at;
  }
  __syncthreads();
  const T* src = table + (size_t)tok * hidden;
  const T* pair = pairs + (size_t)s_row * hidden;
  float* dst = residual + (size_t)r * hidden;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) dst[c] = to_f32(src[c]) * scale + to_f32(pair[c]);
}

// out[r, i] = act(gate_up[r, i]) * gate_up[r, inter + i]
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gate_up, T* __restrict__ out, long long rows, int inter, int act,
                                float ga0, float ga1) {
  chain_next();
  chain_wait();
  const long long n = rows * inter;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / inter;
    const int c = (int)(i - r * inter);
    const float g = to_f32(gate_up[r * 2 * inter + c]);
    const float u = to_f32(gate_up[r * 2 * inter + inter + c]);
    out[i] = from_f32<T>(gated(g, u, act, ga0, ga1));
  }
}

}  // namespace tl

using namespace tl;

extern "C" int tl_embed_rows_copies(const void* table, const int* tokens, float* residual, int rows, int hidden, int vocab,
                                    int dtype, int* status, float scale, int copies, long long copy_stride, cudaStream_t stream) {
  if (rows == 0) return 0;
  TL_REQUIRE(rows > 0 && hidden > 0 && vocab > 0 && copies >= 1, "embed_rows: rows %d hidden %d vocab %d copies %d", rows, hidden,
             vocab, copies);
  const int threads = hidden >= 1024 ? 256 : 128;
  cudaError_t e;
  if (dtype == TL_FP32)
    e = launch_chained(embed_rows_kernel<float>, dim3(rows), dim3(threads), 0, stream, (const float*)table, tokens, residual,
                       hidden, vocab, status, scale, copies, copy_stride);
  else
    e = launch_chained(embed_rows_kernel<bf16>, dim3(rows), dim3(threads), 0, stream, (const bf16*)table, tokens, residual,
                       hidden, vocab, status, scale, copies, copy_stride);
  return (int)e;
}

extern "C" int tl_embed_rows(const void* table, const int* tokens, float* residual, int rows, int hidden, int vocab,
                             int dtype, int* status, float scale, cudaStream_t stream) {
  return tl_embed_rows_copies(table, tokens, residual, rows, hidden, vocab, dtype, status, scale, 1, 0, stream);
}

// pairs [buckets + 1, hidden] of the table's type; last_token [slots]. See embed_token_pairs_kernel.
extern "C" int tl_embed_token_pairs(const void* table, const void* pairs, const int* tokens, const int* req_of_row,
                                    const int* row_start, const int* state_slot, int* last_token, float* residual, int rows,
                                    int hidden, int vocab, long long buckets, long long mul_prev, long long mul_cur, int dtype,
                                    int* status, float scale, cudaStream_t stream) {
  if (rows == 0) return 0;
  TL_REQUIRE(rows > 0 && hidden > 0 && vocab > 0 && buckets > 0, "embed_token_pairs: rows %d hidden %d vocab %d buckets %lld", rows,
             hidden, vocab, buckets);
  TL_REQUIRE(table && pairs && req_of_row && row_start && state_slot && last_token, "embed_token_pairs: two tables, the rows' requests "
             "and a slot a request are needed (%d rows)", rows);
  const int threads = hidden >= 1024 ? 256 : 128;
#define TL_PAIRS(T_)                                                                                                            \
  return (int)launch_chained(embed_token_pairs_kernel<T_>, dim3(rows), dim3(threads), 0, stream, (const T_*)table,              \
                             (const T_*)pairs, tokens, req_of_row, row_start, state_slot, last_token, residual, hidden, vocab,  \
                             buckets, mul_prev, mul_cur, status, scale)
  if (dtype == TL_FP32) TL_PAIRS(float);
  TL_PAIRS(bf16);
#undef TL_PAIRS
}

extern "C" void tl_set_chained_launches(int enabled) { chained_launches() = enabled; }

// See NormParams for the forms of what is added. Null pointers switch a form or the router off. `streams` residual streams; 0 is
// the plain residual add.
extern "C" int tl_add_rmsnorm_streams(float* residual, const float* delta, int parts, long long part_stride,
                              const float* expert_rows, int expert_parts, long long expert_part_stride,
                              const int* pos_of_pair, const int* ids, const float* wts, int top_k,
                              const float* weight, void* normed, float* normed32, const int* gather, int out_rows,
                              int hidden, float eps, int dtype, const float* router_w, const float* router_bias, int E,
                              int route_k, int normalize, float floor_, float scale, int* route_ids, float* route_wts,
                              int streams, long long stream_stride, const float* hc_mix, const float* hc_out, const float* hc_in,
                              cudaStream_t stream);

extern "C" int tl_add_rmsnorm(float* residual, const float* delta, int parts, long long part_stride,
                              const float* expert_rows, int expert_parts, long long expert_part_stride,
                              const int* pos_of_pair, const int* ids, const float* wts, int top_k,
                              const float* weight, void* normed, float* normed32, const int* gather, int out_rows,
                              int hidden, float eps, int dtype, const float* router_w, const float* router_bias, int E,
                              int route_k, int normalize, float floor_, float scale, int* route_ids, float* route_wts,
                              cudaStream_t stream) {
  return tl_add_rmsnorm_streams(residual, delta, parts, part_stride, expert_rows, expert_parts, expert_part_stride, pos_of_pair,
                                ids, wts, top_k, weight, normed, normed32, gather, out_rows, hidden, eps, dtype, router_w,
                                router_bias, E, route_k, normalize, floor_, scale, route_ids, route_wts, 0, 0, nullptr, nullptr,
                                nullptr, stream);
}

extern "C" int tl_add_rmsnorm_streams(float* residual, const float* delta, int parts, long long part_stride,
                              const float* expert_rows, int expert_parts, long long expert_part_stride,
                              const int* pos_of_pair, const int* ids, const float* wts, int top_k,
                              const float* weight, void* normed, float* normed32, const int* gather, int out_rows,
                              int hidden, float eps, int dtype, const float* router_w, const float* router_bias, int E,
                              int route_k, int normalize, float floor_, float scale, int* route_ids, float* route_wts,
                              int streams, long long stream_stride, const float* hc_mix, const float* hc_out, const float* hc_in,
                              cudaStream_t stream) {
  if (out_rows == 0) return 0;
  TL_REQUIRE(streams >= 0 && streams <= MAX_STREAMS, "add_rmsnorm: %d residual streams; up to %d are implemented", streams,
             MAX_STREAMS);
  TL_REQUIRE(streams == 0 || ((hc_mix != nullptr) == (hc_out != nullptr) && (hc_mix || (!delta && !expert_rows))),
             "add_rmsnorm: what is added to %d streams needs their mixing matrix and their output weights", streams);
  NormParams p = {};
  p.residual = residual; p.delta = delta; p.parts = parts; p.part_stride = part_stride; p.expert_rows = expert_rows;
  p.expert_parts = expert_parts < 1 ? 1 : expert_parts; p.expert_part_stride = expert_part_stride;
  p.pos_of_pair = pos_of_pair; p.ids = ids; p.wts = wts; p.top_k = top_k; p.weight = weight; p.eps = eps;
  p.normed = normed; p.normed32 = normed32; p.gather = gather; p.hidden = hidden; p.router_w = router_w;
  p.router_bias = router_bias; p.E = E; p.route_k = route_k; p.normalize = normalize; p.floor_ = floor_; p.scale = scale;
  p.route_ids = route_ids; p.route_wts = route_wts;
  p.out_rows = out_rows;
  p.streams = streams; p.stream_stride = stream_stride; p.hc_mix = hc_mix; p.hc_out = hc_out; p.hc_in = hc_in;
  if (streams > 0) return launch_add_rmsnorm<NORM_STREAMS>(p, dtype, stream);
  return launch_add_rmsnorm<NORM_PLAIN>(p, dtype, stream);
}

// out [rows, inter] = act(gate_up[:, :inter]) * gate_up[:, inter:], act a gate's code (tl_is_gate)
extern "C" int tl_gated_mul(const void* gate_up, void* out, int rows, int inter, int act, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  TL_REQUIRE(rows > 0 && inter > 0, "gated_mul: rows %d width %d", rows, inter);
  TL_REQUIRE(tl_is_gate(act), "gated_mul: gate activation %d is none", act);
  const long long n = (long long)rows * inter;
  const long long most = (long long)sm_count() * 16;
  const int blocks = (int)(ceil_div64(n, 256) < most ? ceil_div64(n, 256) : most);
  cudaError_t e;
  if (dtype == TL_FP32)
    e = launch_chained(silu_mul_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)gate_up, (float*)out,
                       (long long)rows, inter, act, tl_gate_constants[0], tl_gate_constants[1]);
  else
    e = launch_chained(silu_mul_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)gate_up, (bf16*)out,
                       (long long)rows, inter, act, tl_gate_constants[0], tl_gate_constants[1]);
  return (int)e;
}
