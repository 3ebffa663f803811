// The delta rule behind a decay per key channel (channel_delta): what stands in front of the recurrence, and the
// recurrence of a step of single tokens with all that follows it.
//
//   delta_conv   queries, keys and values through a short causal convolution per channel and SiLU; queries and keys
//                made unit vectors per head (queries also scaled); the step sizes' sigmoids; the convolution's last
//                inputs per sequence kept for the next step.
//
// Everything is 32-bit; the projections come as 32-bit rows.
#include "common.cuh"

namespace {

struct DeltaConvArgs {
  float* out;                  // [tokens][G dk queries | G dk keys | H dv values | H step sizes], rows out_ld apart
  long long out_ld;
  const float* proj;           // packed projection rows
  long long ld;
  int off[3], off_b;           // where the sections q, k, v and the step sizes' logits begin
  const float* taps_w;         // [taps][C], the last tap on the token itself; C = 2 G dk + H dv
  float* history;              // [slots][taps - 1][C]
  const int *positions, *seq_of_token, *slots, *seq_starts;
  int taps, G, H, dk, dv;
  float key_eps, query_scale;
};

// Where channel c (of q | k | v) lies in a projection row.
__device__ __forceinline__ int dc_col(const DeltaConvArgs& a, int c) {
  const int n = a.G * a.dk;
  return c < n ? a.off[0] + c : c < 2 * n ? a.off[1] + c - n : a.off[2] + c - 2 * n;
}

// silu of the convolution of channel c at token t, `back` tokens of whose sequence lie in the step before it.
__device__ __forceinline__ float dc_value(const DeltaConvArgs& a, int t, int c, int pos, int back, int slot, int C) {
  const int keep = a.taps - 1;
  const float* src = a.proj + (size_t)t * a.ld + dc_col(a, c);
  float v = 0.f;
  for (int j = 0; j < a.taps; ++j) {
    const int d = keep - j;                                  // how far back this tap looks
    if (d > pos) continue;                                   // (before the sequence's first token)
    float u = 0.f;
    if (d <= back) u = src[-(long long)d * a.ld];
    else if (slot >= 0) u = a.history[((size_t)slot * keep + keep - (d - back)) * C + c];
    v = fmaf(a.taps_w[(size_t)j * C + c], u, v);
  }
  return v / (1.f + expf(-v));
}

// A warp takes a head's query or key of a token, or 32 NE of its values; NE: channels a lane holds.  SINGLE: every
// sequence brings one token, and the warp moves its channels' history on as well (nobody else reads it).
template <int NE, bool SINGLE>
__global__ void __launch_bounds__(128)
delta_conv_kernel(DeltaConvArgs a) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x, job = blockIdx.y * 4 + (threadIdx.x >> 5);
  const int nq = a.G * a.dk, C = 2 * nq + a.H * a.dv;
  const int pos = a.positions[t], seq = a.seq_of_token[t], slot = a.slots[seq], back = t - a.seq_starts[seq];
  const int head_jobs = 2 * a.G, value_jobs = (a.H * a.dv + 32 * NE - 1) / (32 * NE);
  pdl_wait();
  a.proj = pdl_fresh(a.proj);
  if (job > head_jobs + value_jobs) return;
  float* row = a.out + (size_t)t * a.out_ld;
  if (job == head_jobs + value_jobs) {                       // the step sizes
    for (int h = lane; h < a.H; h += 32) row[C + h] = 1.f / (1.f + expf(-a.proj[(size_t)t * a.ld + a.off_b + h]));
    return;
  }
  const bool is_head = job < head_jobs;
  const int c0 = is_head ? job * a.dk : 2 * nq + (job - head_jobs) * 32 * NE;
  const int n = is_head ? a.dk : min(32 * NE, C - c0);
  float v[NE], ss = 0.f;
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int i = lane + 32 * e;
    v[e] = i < n ? dc_value(a, t, c0 + i, pos, back, slot, C) : 0.f;
    ss += v[e] * v[e];
  }
  float f = 1.f;
  if (is_head) f = (job < a.G ? a.query_scale : 1.f) / sqrtf(warp_sum(ss) + a.key_eps);
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int i = lane + 32 * e;
    if (i < n) row[c0 + i] = v[e] * f;
  }
  if (SINGLE && slot >= 0) {
    const int keep = a.taps - 1;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int i = lane + 32 * e;
      if (i >= n) continue;
      float* h = a.history + (size_t)slot * keep * C + c0 + i;
      for (int s = 0; s + 1 < keep; ++s) h[(size_t)s * C] = h[(size_t)(s + 1) * C];
      if (keep > 0) h[(size_t)(keep - 1) * C] = a.proj[(size_t)t * a.ld + dc_col(a, c0 + i)];
    }
  }
}

// One thread a (sequence, channel): the history after a step of prompts = the last taps - 1 of (history, the step's inputs).
__global__ void __launch_bounds__(256)
delta_history_kernel(DeltaConvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int C = 2 * a.G * a.dk + a.H * a.dv, keep = a.taps - 1;
  const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int slot = a.slots[seq];
  if (c >= C || slot < 0) return;
  const int first = a.seq_starts[seq], n = a.seq_starts[seq + 1] - first, old = max(0, keep - n);
  float* h = a.history + (size_t)slot * keep * C + c;
  const float* src = a.proj + dc_col(a, c);
  for (int i = 0; i < old; ++i) h[(size_t)i * C] = h[(size_t)(i + n) * C];      // (ascending: read before it is overwritten)
  for (int i = old; i < keep; ++i) h[(size_t)i * C] = src[(size_t)(first + n - keep + i) * a.ld];
}

template <int NE>
void dc_launch(const DeltaConvArgs& a, int n_tokens, bool single, cudaStream_t stream) {
  const int jobs = 2 * a.G + (a.H * a.dv + 32 * NE - 1) / (32 * NE) + 1;
  const dim3 grid(n_tokens, (jobs + 3) / 4);
  if (single) af_launch(delta_conv_kernel<NE, true>, grid, dim3(128), 0, stream, a);
  else af_launch(delta_conv_kernel<NE, false>, grid, dim3(128), 0, stream, a);
}

}  // namespace

// out [n_tokens][2 G dk + H dv + H] float, see above; history [slots][taps - 1][2 G dk + H dv] is left with the sequences'
// last taps - 1 inputs.
AF_EXPORT int af_delta_conv(float* out, long long out_ld, const float* proj, long long ld, int off_q, int off_k, int off_v,
                            int off_b, const float* taps_w, float* history, const int* positions, const int* seq_of_token,
                            const int* slots, const int* seq_starts, int n_tokens, int n_seqs, int taps, int G, int H,
                            int dk, int dv, float key_eps, float query_scale, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  AF_REQUIRE(n_tokens > 0 && n_seqs > 0 && G > 0 && H % G == 0 && dk > 0 && dk <= 1024 && dv > 0 && taps >= 1,
             "af_delta_conv: bad sizes (keys up to 1024)");
  AF_REQUIRE(taps_w != nullptr && (taps == 1 || history != nullptr), "af_delta_conv: a convolution needs its taps and a history");
  AF_REQUIRE(2 * G + (long long)H * dv / 32 < 4 * 65535 && n_seqs < 65536, "af_delta_conv: too many heads or sequences for one grid");
  DeltaConvArgs a{out, out_ld, proj, ld, {off_q, off_k, off_v}, off_b, taps_w, history, positions, seq_of_token, slots,
                  seq_starts, taps, G, H, dk, dv, key_eps, query_scale};
  const bool single = n_tokens == n_seqs;
  if (dk <= 32) dc_launch<1>(a, n_tokens, single, stream);
  else if (dk <= 64) dc_launch<2>(a, n_tokens, single, stream);
  else if (dk <= 128) dc_launch<4>(a, n_tokens, single, stream);
  else if (dk <= 256) dc_launch<8>(a, n_tokens, single, stream);
  else dc_launch<32>(a, n_tokens, single, stream);
  AF_COUNT_LAUNCH("af_delta_conv");
  if (single || taps == 1) return 0;
  const int C = 2 * G * dk + H * dv;
  af_launch(delta_history_kernel, dim3((C + 255) / 256, n_seqs), dim3(256), 0, stream, a);
  AF_CHECK_LAUNCH("af_delta_conv (history)");
}
