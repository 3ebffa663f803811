// The delta rule behind a decay per key channel (channel_delta): what stands in front of the recurrence, and the
// recurrence of a step of single tokens with all that follows it.
//
//   delta_conv   queries, keys and values through a short causal convolution per channel and SiLU; queries and keys
//                made unit vectors per head (queries also scaled); the step sizes' sigmoids; the convolution's last
//                inputs per sequence kept for the next step;
//   delta_prompt a prompt's recurrence in chunks on the tensor cores, two kernels.
//
// Everything is 32-bit; the projections come as 32-bit rows.  The tensor cores' operands are pairs (mma_pairs.cuh).
//
// The chunks.  With P_t = g_1 ... g_t the decays' running product within a chunk (per key channel), S the state that
// enters it and u_t = beta_t (v_t - (diag(g_t) S_(t-1))^T k_t) what token t writes along k_t:
//   S_t = diag(P_t) S + sum over s <= t of diag(P_t / P_s) k_s u_s^T
//   (I + A) U = diag(beta) (V - (K . P) S),    A_ts = beta_t sum_c k_t k_s P_t / P_s  (s < t)
//   o_t = S^T (q_t . P_t) + sum over s <= t of B_ts u_s,    B_ts = sum_c q_t k_s P_t / P_s
//   S_out = diag(P_end) S + sum over s of diag(P_end / P_s) k_s u_s^T
// so with W = (I + A)^-1 diag(beta) (K . P) and U0 = (I + A)^-1 diag(beta) V, which need no state, a chunk is four products:
// U = U0 - W S, O = (Q . P) S + B U, S_out = P_end S + (K . P_end / P)^T U.  The first kernel makes W, U0, B and the scaled
// queries and keys of all chunks side by side, the second walks a sequence's chunks.  Nothing is divided by a decay: P_t / P_s
// is the product g_(s+1) ... g_t itself, taken along a chain within 16 tokens, and across two groups of 16 tokens as the
// product from s to its group's end times the product from the next group's start to t.
#include "mma_pairs.cuh"
#include "tma.cuh"

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
  // the low-rank factors of decays and gates in bfloat16, for products on the tensor cores (low null: none)
  __nv_bfloat16* low;          // [tokens][low_ld]: `rank[0]` values from column 0, `rank[1]` from `low_at`
  int off_low[2], rank[2], low_at, low_ld;
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
  if (job == head_jobs + value_jobs) {                       // the step sizes, the low-rank factors
    if (a.low != nullptr) {
#pragma unroll
      for (int f = 0; f < 2; ++f)
        for (int i = lane; i < a.rank[f]; i += 32)
          a.low[(size_t)t * a.low_ld + (f ? a.low_at : 0) + i] = __float2bfloat16_rn(a.proj[(size_t)t * a.ld + a.off_low[f] + i]);
    }
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

// The same where everything comes in 16-byte pieces, heads are 4 .. 128 channels (a power of two) and the convolution has up
// to TAPS = 4 taps: a lane takes four channels of R tokens in a row, so that a row is read once for all taps, and a head's sum
// of squares is joined over its dk / 4 lanes.  All loads of a warp are in flight at once; single tokens (R 1) ask for taps
// and history before the wait.
template <int R, bool SINGLE>
__global__ void __launch_bounds__(128)
delta_conv_row_kernel(DeltaConvArgs a, int n_tokens) {
  pdl_launch_dependents();
  constexpr int TAPS = 4;
  const int lane = threadIdx.x & 31, t0 = blockIdx.x * R, slice = blockIdx.y * 4 + (threadIdx.x >> 5);
  const int nq = a.G * a.dk, C = 2 * nq + a.H * a.dv, slices = (C + 127) / 128, keep = a.taps - 1;
  if (slice > slices) return;
  if (slice == slices) {                                     // step sizes, low-rank factors
    pdl_wait();
    a.proj = pdl_fresh(a.proj);
    for (int r = 0; r < R && t0 + r < n_tokens; ++r) {
      const size_t t = (size_t)t0 + r;
      if (a.low != nullptr) {
#pragma unroll
        for (int f = 0; f < 2; ++f)
          for (int i = lane; i < a.rank[f]; i += 32)
            a.low[t * a.low_ld + (f ? a.low_at : 0) + i] = __float2bfloat16_rn(a.proj[t * a.ld + a.off_low[f] + i]);
      }
      for (int h = lane; h < a.H; h += 32) a.out[t * a.out_ld + C + h] = 1.f / (1.f + expf(-a.proj[t * a.ld + a.off_b + h]));
    }
    return;
  }
  const int c = slice * 128 + lane * 4;
  const bool on = c < C;
  const int cc = on ? c : 0, col = dc_col(a, cc), L = a.dk / 4;
  // lane r knows token t0 + r: how many tokens of its sequence lie in the step before it, its slot, its position
  int my_back = 0, my_slot = -1, my_pos = 0;
  if (lane < R && t0 + lane < n_tokens) {
    const int seq = a.seq_of_token[t0 + lane];
    my_pos = a.positions[t0 + lane], my_slot = a.slots[seq], my_back = t0 + lane - a.seq_starts[seq];
  }
  float4 w[TAPS];                                            // w[d]: the tap that looks d tokens back
#pragma unroll
  for (int d = 0; d < TAPS; ++d)
    w[d] = d <= keep ? *reinterpret_cast<const float4*>(a.taps_w + (size_t)(keep - d) * C + cc) : make_float4(0.f, 0.f, 0.f, 0.f);
  float4 old[TAPS - 1];                                      // single tokens: the history, newest last
  float* hist = nullptr;
  if (SINGLE) {
    const int slot = __shfl_sync(0xffffffffu, my_slot, 0);
    if (slot >= 0 && keep > 0) hist = a.history + (size_t)slot * keep * C + cc;
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i)
      old[i] = hist != nullptr && i < keep ? *reinterpret_cast<const float4*>(hist + (size_t)i * C) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  a.proj = pdl_fresh(a.proj);
  float4 u[R + TAPS - 1];
#pragma unroll
  for (int i = 0; i < R + TAPS - 1; ++i) {
    const int t = t0 + i - (TAPS - 1);
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t >= 0 && t < n_tokens && (!SINGLE || i == TAPS - 1)) u[i] = *reinterpret_cast<const float4*>(a.proj + (size_t)t * a.ld + col);
  }
  if (SINGLE) {
#pragma unroll
    for (int d = 1; d < TAPS; ++d) {                         // (history row keep - d holds the input d tokens back)
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i)
        if (i == keep - d) x = old[i];
      u[TAPS - 1 - d] = x;
    }
  }
  const bool heads = slice * 128 < 2 * nq;                   // (the whole warp: some of its channels are queries or keys)
  const float scale = c < nq ? a.query_scale : 1.f;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int t = t0 + r;
    if (t >= n_tokens) break;
    const int back = SINGLE ? TAPS : __shfl_sync(0xffffffffu, my_back, r);
    float4 x[TAPS];
#pragma unroll
    for (int d = 0; d < TAPS; ++d) x[d] = u[r + TAPS - 1 - d];
    if (!SINGLE && back < keep) {                            // taps that look before the step: the history, or nothing before the sequence
      const int slot = __shfl_sync(0xffffffffu, my_slot, r), pos = __shfl_sync(0xffffffffu, my_pos, r);
#pragma unroll
      for (int d = 1; d < TAPS; ++d) {
        if (d <= back) continue;
        x[d] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d <= pos && d <= keep && slot >= 0)
          x[d] = *reinterpret_cast<const float4*>(a.history + ((size_t)slot * keep + keep - (d - back)) * C + cc);
      }
    }
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int d = TAPS - 1; d >= 0; --d)
      v.x = fmaf(w[d].x, x[d].x, v.x), v.y = fmaf(w[d].y, x[d].y, v.y), v.z = fmaf(w[d].z, x[d].z, v.z), v.w = fmaf(w[d].w, x[d].w, v.w);
    v.x = __fdividef(v.x, 1.f + __expf(-v.x)), v.y = __fdividef(v.y, 1.f + __expf(-v.y));
    v.z = __fdividef(v.z, 1.f + __expf(-v.z)), v.w = __fdividef(v.w, 1.f + __expf(-v.w));
    if (heads) {
      float ss = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      for (int o = 1; o < L; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (c < 2 * nq) {
        const float f = scale * rsqrtf(ss + a.key_eps);
        v.x *= f, v.y *= f, v.z *= f, v.w *= f;
      }
    }
    if (on) *reinterpret_cast<float4*>(a.out + (size_t)t * a.out_ld + c) = v;
  }
  if (SINGLE && on && hist != nullptr) {
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i)
      if (i < keep) *reinterpret_cast<float4*>(hist + (size_t)i * C) = i + 1 < keep ? old[i + 1 < TAPS - 1 ? i + 1 : i] : u[TAPS - 1];
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
// last taps - 1 inputs.  low (or null): bfloat16 copies of two more sections of the projection rows.
AF_EXPORT int af_delta_conv(float* out, long long out_ld, const float* proj, long long ld, int off_q, int off_k, int off_v,
                            int off_b, const float* taps_w, float* history, const int* positions, const int* seq_of_token,
                            const int* slots, const int* seq_starts, int n_tokens, int n_seqs, int taps, int G, int H,
                            int dk, int dv, float key_eps, float query_scale, void* low, int off_low0, int off_low1,
                            int rank0, int rank1, int low_at, int low_ld, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  AF_REQUIRE(low == nullptr || (rank0 > 0 && rank1 > 0 && low_at >= rank0 && low_ld >= low_at + rank1), "af_delta_conv: low-rank rows");
  AF_REQUIRE(n_tokens > 0 && n_seqs > 0 && G > 0 && H % G == 0 && dk > 0 && dk <= 1024 && dv > 0 && taps >= 1,
             "af_delta_conv: bad sizes (keys up to 1024)");
  AF_REQUIRE(taps_w != nullptr && (taps == 1 || history != nullptr), "af_delta_conv: a convolution needs its taps and a history");
  AF_REQUIRE(2 * G + (long long)H * dv / 32 < 4 * 65535 && n_seqs < 65536, "af_delta_conv: too many heads or sequences for one grid");
  DeltaConvArgs a{out, out_ld, proj, ld, {off_q, off_k, off_v}, off_b, taps_w, history, positions, seq_of_token, slots,
                  seq_starts, taps, G, H, dk, dv, key_eps, query_scale, (__nv_bfloat16*)low, {off_low0, off_low1},
                  {rank0, rank1}, low_at, low_ld};
  const bool single = n_tokens == n_seqs;
  const bool rows = taps <= 4 && dk >= 4 && dk <= 128 && (dk & (dk - 1)) == 0 && (H * dv) % 4 == 0 &&
                    ((ld | out_ld | off_q | off_k | off_v) & 3) == 0 &&
                    (((uintptr_t)out | (uintptr_t)proj | (uintptr_t)taps_w | (uintptr_t)history) & 15) == 0;
  if (rows) {
    const int slices = (2 * G * dk + H * dv + 127) / 128 + 1;
    if (single) af_launch(delta_conv_row_kernel<1, true>, dim3(n_tokens, (slices + 3) / 4), dim3(128), 0, stream, a, n_tokens);
    else af_launch(delta_conv_row_kernel<8, false>, dim3((n_tokens + 7) / 8, (slices + 3) / 4), dim3(128), 0, stream, a, n_tokens);
  } else if (dk <= 32) dc_launch<1>(a, n_tokens, single, stream);
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

// ---------------------------------------------------------------- prompts in chunks

namespace {

constexpr int DP_C = 32;           // tokens of a chunk: two groups of 16

struct DeltaPromptArgs {
  const float *q, *k, *v, *beta, *z;   // rows of the step: unit queries and keys (G heads), values, step sizes, decays' logits
  long long qkv_ts, beta_ts, z_ts;
  const float *dt_bias, *rate;         // [H * dk]: decay = exp(-rate softplus(z + dt_bias))
  __nv_bfloat16* blob;                 // [chunks * H][dp_blob(dk).size]: what the second kernel needs of a chunk and head
  float* u0;                           // [chunks * H][tiles of `tile` value columns][DP_C][tile + 4]
  int tile;
  float* state;                        // [slots][H][dv][dk]
  float* out;                          // [tokens][H * dv]
  const int *chunk_starts, *seq_first_chunk, *slots;
  int G, H, dk, dv;
  int* err;                            // set to 1 when a bounded wait ran out
};

__device__ __forceinline__ void dp_put(__nv_bfloat16* hi, __nv_bfloat16* lo, float y) {
  const __nv_bfloat16 h = __float2bfloat16_rn(y);
  *hi = h;
  *lo = __float2bfloat16_rn(y - __bfloat162float(h));
}

// Where the pieces of a chunk lie, in global memory as in the walking kernel's shared memory (elements of bfloat16; rows of
// dk + 8): W, Q . P, K . P_end / P (each hi then lo), B (hi, lo; rows of 40), P_end (floats).  A tile of U0 (floats, rows of
// N + 4) follows in a stage.
constexpr int DP_PB = DP_C + 8;
struct DpBlob {
  int pk, b, p_end, size;
};
__host__ __device__ inline DpBlob dp_blob(int dk) {
  DpBlob s;
  s.pk = dk + 8;
  s.b = 6 * DP_C * s.pk;
  s.p_end = s.b + 2 * DP_C * DP_PB;
  s.size = s.p_end + 2 * dk;
  return s;
}

size_t dp_prep_smem(int dk) { return ((size_t)3 * DP_C * (dk + 4) + 2 * DP_C * 36 + DP_C) * sizeof(float); }

// 32 sums over the warp's lanes at once: lane l ends with the sum of everybody's v[l].
__device__ __forceinline__ float dp_sum32(float* v) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = up ? v[i + o] : v[i], give = up ? v[i] : v[i + o];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

// Block (chunk, head), 256 threads; NE = channels a lane holds (dk / 32 rounded up).
template <int NE>
__global__ void __launch_bounds__(256, NE <= 4 ? 3 : 1)
delta_chunk_kernel(DeltaPromptArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  const int dk = a.dk, dv = a.dv, DP = dk + 4, quads = dk / 4;
  float *k_s = sm, *q_s = k_s + DP_C * DP, *g_s = q_s + DP_C * DP;
  float *A_s = g_s + DP_C * DP, *B_s = A_s + DP_C * 36, *beta_s = B_s + DP_C * 36;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ch = blockIdx.x, h = blockIdx.y, hk = h / (a.H / a.G);
  const int first = a.chunk_starts[ch], rows = a.chunk_starts[ch + 1] - first;
  const size_t unit = (size_t)ch * a.H + h;
  const DpBlob L = dp_blob(dk);
  __nv_bfloat16* blob = a.blob + unit * L.size;
  pdl_wait();
  a.q = pdl_fresh(a.q), a.k = pdl_fresh(a.k), a.v = pdl_fresh(a.v), a.beta = pdl_fresh(a.beta), a.z = pdl_fresh(a.z);
#pragma unroll 2
  for (int i = tid; i < DP_C * quads; i += 256) {
    const int r = i / quads, c = (i - r * quads) * 4;
    float4 kq = make_float4(0.f, 0.f, 0.f, 0.f), qq = kq, gq = make_float4(1.f, 1.f, 1.f, 1.f);
    if (r < rows) {
      const size_t at = (size_t)(first + r) * a.qkv_ts + (size_t)hk * dk + c;
      kq = *reinterpret_cast<const float4*>(a.k + at);
      qq = *reinterpret_cast<const float4*>(a.q + at);
      const float4 z = *reinterpret_cast<const float4*>(a.z + (size_t)(first + r) * a.z_ts + (size_t)h * dk + c);
      const float4 bi = *reinterpret_cast<const float4*>(a.dt_bias + (size_t)h * dk + c);
      const float4 ra = *reinterpret_cast<const float4*>(a.rate + (size_t)h * dk + c);
      auto decay = [](float x, float f) { return expf(-f * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))))); };
      gq = make_float4(decay(z.x + bi.x, ra.x), decay(z.y + bi.y, ra.y), decay(z.z + bi.z, ra.z), decay(z.w + bi.w, ra.w));
    }
    *reinterpret_cast<float4*>(k_s + r * DP + c) = kq;
    *reinterpret_cast<float4*>(q_s + r * DP + c) = qq;
    *reinterpret_cast<float4*>(g_s + r * DP + c) = gq;
  }
  if (tid < DP_C) beta_s[tid] = tid < rows ? a.beta[(size_t)(first + tid) * a.beta_ts + h] : 0.f;
  for (int i = tid; i < 2 * DP_C * 36; i += 256) A_s[i] = 0.f;       // (what lies above the diagonals stays zero)
  __syncthreads();

  // ---- the two groups by themselves: a warp takes a source token and walks the tokens behind it in its group
#pragma unroll 1
  for (int job = 0; job < 4; ++job) {
    const int base = (job >> 1) * 16, s = base + ((job & 1) ? 15 - warp : warp);
    float p[NE], v[32];
#pragma unroll
    for (int e = 0; e < NE; ++e) p[e] = lane + 32 * e < dk ? k_s[s * DP + lane + 32 * e] : 0.f;
#pragma unroll
    for (int d = 0; d < 16; ++d) {
      float ak = 0.f, aq = 0.f;
      if (s + d < base + 16) {
        const int at = (s + d) * DP + lane;
#pragma unroll
        for (int e = 0; e < NE; ++e) {
          if (lane + 32 * e >= dk) continue;
          if (d > 0) p[e] *= g_s[at + 32 * e];
          ak = fmaf(k_s[at + 32 * e], p[e], ak);
          aq = fmaf(q_s[at + 32 * e], p[e], aq);
        }
      }
      v[2 * d] = ak, v[2 * d + 1] = aq;
    }
    const float sum = dp_sum32(v);
    const int t = s + (lane >> 1);
    if (t < base + 16) {
      if (lane & 1) B_s[t * 36 + s] = sum;
      else if (t > s) A_s[t * 36 + s] = sum * beta_s[t];
    }
  }
  __syncthreads();
  // ---- a thread a channel: running products from the front (half the threads) and from the back; the scaled queries and
  // keys go out.  Left in place behind it: k times P from its group's start; q of the second group likewise; in the first
  // group's place of q the keys times what follows them in their group; in g's first row the first group's whole product.
  for (int c0 = 0; c0 < dk; c0 += 128) {
    const int c = c0 + (tid & 127);
    const bool on = c < dk, front = tid < 128;
    float r[DP_C], half = 1.f;
    if (on && front) {
      __nv_bfloat16* o = blob + 2 * DP_C * L.pk + c;
      float P = 1.f;
#pragma unroll
      for (int t = 0; t < DP_C; ++t) {
        if (t == 16) half = P, P = 1.f;
        P *= g_s[t * DP + c];
        r[t] = k_s[t * DP + c] * P;
        float q = q_s[t * DP + c] * P;
        if (t >= 16) {
          q_s[t * DP + c] = q;
          q *= half;
        }
        dp_put(o, o + DP_C * L.pk, q);
        o += L.pk;
      }
      reinterpret_cast<float*>(blob + L.p_end)[c] = half * P;
    } else if (on) {
      __nv_bfloat16* o = blob + (4 * DP_C + DP_C - 1) * L.pk + c;
      float x = 1.f, second = 1.f;
#pragma unroll
      for (int s = DP_C - 1; s >= 0; --s) {
        if (s == 15) second = x, x = 1.f;
        r[s] = k_s[s * DP + c] * x;
        dp_put(o, o + DP_C * L.pk, s < 16 ? r[s] * second : r[s]);
        o -= L.pk;
        x *= g_s[s * DP + c];
      }
    }
    __syncthreads();
    if (on && front) {
#pragma unroll
      for (int t = 0; t < DP_C; ++t) k_s[t * DP + c] = r[t];
      g_s[c] = half;
    } else if (on) {
#pragma unroll
      for (int s = 0; s < 16; ++s) q_s[s * DP + c] = r[s];
    }
  }
  __syncthreads();
  // ---- the second group's tokens against the first group's: a thread a pair
  {
    const int t = 16 + (tid >> 4), s = tid & 15;
    const float *kr = k_s + t * DP, *qr = q_s + t * DP, *xr = q_s + s * DP;
    float ak = 0.f, aq = 0.f, ak2 = 0.f, aq2 = 0.f;
    for (int c = 0; c < dk; c += 4) {
      const float4 x = *reinterpret_cast<const float4*>(xr + c), kk = *reinterpret_cast<const float4*>(kr + c),
                   qq = *reinterpret_cast<const float4*>(qr + c);
      ak = fmaf(kk.x, x.x, fmaf(kk.y, x.y, ak)), ak2 = fmaf(kk.z, x.z, fmaf(kk.w, x.w, ak2));
      aq = fmaf(qq.x, x.x, fmaf(qq.y, x.y, aq)), aq2 = fmaf(qq.z, x.z, fmaf(qq.w, x.w, aq2));
    }
    A_s[t * 36 + s] = (ak + ak2) * beta_s[t];
    B_s[t * 36 + s] = aq + aq2;
  }
  __syncthreads();
  for (int i = tid; i < DP_C * DP_C; i += 256) {
    __nv_bfloat16* o = blob + L.b + (i >> 5) * DP_PB + (i & 31);
    dp_put(o, o + DP_C * DP_PB, B_s[(i >> 5) * 36 + (i & 31)]);
  }
  // ---- (I + A) X = diag(beta) [K . P | V]: a thread a column, from the first row down
  for (int col = tid; col < dk + dv; col += 256) {
    const bool is_w = col < dk;
    float x[DP_C];
    if (is_w) {
      const float half = g_s[col];
#pragma unroll
      for (int t = 0; t < DP_C; ++t) x[t] = k_s[t * DP + col] * (t < 16 ? 1.f : half);
    } else {
      const float* src = a.v + (size_t)first * a.qkv_ts + (size_t)h * dv + col - dk;
#pragma unroll
      for (int t = 0; t < DP_C; ++t) {
        x[t] = t < rows ? *src : 0.f;
        src += a.qkv_ts;
      }
    }
    __nv_bfloat16* w = blob + col;
    const int j = is_w ? 0 : col - dk, n = a.tile;
    float* u = a.u0 + ((unit * ((dv + n - 1) / n) + j / n) * DP_C) * (n + 4) + j % n;
#pragma unroll
    for (int t = 0; t < DP_C; ++t) {
      float acc = x[t] * beta_s[t], acc2 = 0.f;
#pragma unroll
      for (int s = 0; s < t; s += 4) {
        const float4 q = *reinterpret_cast<const float4*>(A_s + t * 36 + s);      // (zero from the diagonal on)
        acc = fmaf(-q.x, x[s], acc);
        if (s + 1 < t) acc2 = fmaf(-q.y, x[s + 1], acc2);
        if (s + 2 < t) acc = fmaf(-q.z, x[s + 2], acc);
        if (s + 3 < t) acc2 = fmaf(-q.w, x[s + 3], acc2);
      }
      x[t] = acc + acc2;
      if (is_w) {
        dp_put(w, w + DP_C * L.pk, x[t]);
        w += L.pk;
      } else {
        *u = x[t];
        u += n + 4;
      }
      // (the factors are read when it is their rows' turn: all at once they would fill the registers)
      if ((t & 3) == 3) asm volatile("" ::: "memory");
    }
  }
}

size_t dp_stage_bytes(int dk, int n) { return (size_t)dp_blob(dk).size * 2 + (size_t)DP_C * (n + 4) * 4; }
size_t dp_walk_smem(int dk, int n, int stages) {
  return stages * dp_stage_bytes(dk, n) + (2 * (size_t)dk * (n + 8) + 2 * (size_t)DP_C * (n + 8)) * sizeof(__nv_bfloat16);
}

// A contiguous piece from global to shared memory, counted by an mbarrier (16-byte aligned, a multiple of 16 bytes).
__device__ __forceinline__ void dp_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// Block (N value columns, head, sequence), eight warps, walks the sequence's chunks with its columns of the state in registers
// (a warp holds MT tiles of 16 key channels) and, in two parts, in shared memory.  Warps 0 .. 3 make U = U0 - W S, warps 4 .. 7
// O = (Q . P) S + B U (a warp: 16 tokens by 16 columns), all of them the new state; the next chunk's pieces are on their
// way meanwhile if there is room for two.  In the narrow form the two warps of 16 tokens take all columns and halves of the
// key channels, joined through shared memory: every piece of an operand is then loaded by one warp.
template <int N, int MT>
__global__ void __launch_bounds__(256)
delta_walk_kernel(DeltaPromptArgs a, int stages) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ uint64_t full[2];
  __shared__ int give_up_s;
  volatile int* give_up = &give_up_s;
  constexpr int PN = N + 8, NT = 2;                // NT: n8 tiles of a U or O warp
  constexpr bool SPLIT = N == 16;
  __shared__ float2 join_s[SPLIT ? 4 : 1][NT][2][32];
  const int dk = a.dk, dv = a.dv;
  const DpBlob L = dp_blob(dk);
  const uint32_t blob_bytes = (uint32_t)L.size * 2, u0_bytes = DP_C * (N + 4) * 4;
  __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(raw + (size_t)stages * (blob_bytes + u0_bytes));
  __nv_bfloat16* s_lo = s_hi + dk * PN;
  __nv_bfloat16* u_hi = s_lo + dk * PN;
  __nv_bfloat16* u_lo = u_hi + DP_C * PN;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, b = blockIdx.z, j0 = blockIdx.x * N, tiles = gridDim.x;
  const int slot = a.slots[b], ch0 = a.seq_first_chunk[b], ch1 = a.seq_first_chunk[b + 1];
  if (slot < 0 || ch0 >= ch1) return;
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    give_up_s = 0;
    mbar_fence_init();
  }
  float* st = a.state + ((size_t)slot * a.H + h) * dv * dk;
  float S[MT][N / 8][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < N / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = (warp + 8 * m) * 16 + g + 8 * (e >> 1), col = j0 + n * 8 + 2 * t4 + (e & 1);
        S[m][n][e] = (key < dk && col < dv) ? st[(size_t)col * dk + key] : 0.f;
      }
  auto put_state = [&]() {
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int key = (warp + 8 * m) * 16 + g;
      if (key >= dk) continue;                     // (dk is a multiple of 16: whole tiles)
#pragma unroll
      for (int n = 0; n < N / 8; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          mp_split2(S[m][n][2 * r], S[m][n][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(s_hi + (key + 8 * r) * PN + n * 8 + 2 * t4) = hi;
          *reinterpret_cast<uint32_t*>(s_lo + (key + 8 * r) * PN + n * 8 + 2 * t4) = lo;
        }
    }
  };
  put_state();
  __syncthreads();                                 // (the barriers are set up)
  pdl_wait();
  auto load = [&](int ch, int which) {             // (one thread)
    unsigned char* sg = raw + (size_t)which * (blob_bytes + u0_bytes);
    const size_t unit = (size_t)ch * a.H + h;
    mbar_expect_tx(&full[which], blob_bytes + u0_bytes);
    dp_bulk(sg, a.blob + unit * L.size, blob_bytes, &full[which]);
    dp_bulk(sg + blob_bytes, a.u0 + (unit * tiles + blockIdx.x) * (DP_C * (N + 4)), u0_bytes, &full[which]);
  };
  if (tid == 0) load(ch0, 0);
  const int kind = warp >> 2, mt = (warp >> 1) & 1, half = warp & 1, n0 = SPLIT ? 0 : half * 16;
  bool ok = true;
  for (int ch = ch0; ch < ch1; ++ch) {
    const int i = ch - ch0, which = stages == 2 ? i & 1 : 0;
    mbar_wait(&full[which], (stages == 2 ? i >> 1 : i) & 1, give_up);
    __syncthreads();                               // (the chunk's pieces and the state are there; the other stage is free)
    if (*give_up) {
      ok = false;
      break;
    }
    if (stages == 2 && ch + 1 < ch1 && tid == 0) load(ch + 1, which ^ 1);
    const __nv_bfloat16* sg = reinterpret_cast<const __nv_bfloat16*>(raw + (size_t)which * (blob_bytes + u0_bytes));
    const int first = a.chunk_starts[ch], rows = a.chunk_starts[ch + 1] - first;
    // ---- W S, or (Q . P) S: the three products of a pair in chains of their own
    float part[3][NT][4];
#pragma unroll
    for (int p = 0; p < 3; ++p)
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) part[p][n][e] = 0.f;
    const __nv_bfloat16* left = sg + (size_t)kind * 2 * DP_C * L.pk + (mt * 16 + (lane & 15)) * L.pk + (lane >> 4) * 8;
#pragma unroll 4
    for (int kk = SPLIT ? half * 16 : 0; kk < dk; kk += SPLIT ? 32 : 16) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      mp_ldm4(ah, left + kk);
      mp_ldm4(al, left + DP_C * L.pk + kk);
      const int sa = (kk + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n0 + (lane >> 4) * 8;
      mp_ldm4t(bh, s_hi + sa);
      mp_ldm4t(bl, s_lo + sa);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        mp_mma(part[0][n], ah, bh[2 * n], bh[2 * n + 1]);
        mp_mma(part[1][n], ah, bl[2 * n], bl[2 * n + 1]);
        mp_mma(part[2][n], al, bh[2 * n], bh[2 * n + 1]);
      }
    }
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = part[0][n][e] + (part[1][n][e] + part[2][n][e]);
    if constexpr (SPLIT) {                         // the second half of the key channels joins the first
      float2(*mine)[2][32] = join_s[warp >> 1];
      if (half == 1) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int r = 0; r < 2; ++r) mine[n][r][lane] = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
      }
      asm volatile("bar.sync %0, 64;" ::"r"(1 + (warp >> 1)) : "memory");
      if (half == 0) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float2 v = mine[n][r][lane];
            acc[n][2 * r] += v.x, acc[n][2 * r + 1] += v.y;
          }
      }
    }
    const bool owner = !SPLIT || half == 0;        // (of this warp pair's U or O)
    if (kind == 0 && owner) {                               // U = U0 - W S, in two parts
      const float* us = reinterpret_cast<const float*>(sg + L.size);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int row = mt * 16 + g + 8 * r, c = n0 + n * 8 + 2 * t4;
          const float2 u = *reinterpret_cast<const float2*>(us + row * (N + 4) + c);
          uint32_t hi, lo;
          mp_split2(u.x - acc[n][2 * r], u.y - acc[n][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(u_hi + row * PN + c) = hi;
          *reinterpret_cast<uint32_t*>(u_lo + row * PN + c) = lo;
        }
    }
    __syncthreads();                               // (U is there, and nobody reads the old state any more)
    // ---- S = P_end S + (K . P_end / P)^T U
    const __nv_bfloat16* d_hi = sg + (size_t)4 * DP_C * L.pk;
    const float* pe = reinterpret_cast<const float*>(sg + L.p_end);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int key0 = (warp + 8 * m) * 16;
      if (key0 >= dk) continue;
      const float w0 = pe[key0 + g], w1 = pe[key0 + g + 8];
#pragma unroll
      for (int n = 0; n < N / 8; ++n) S[m][n][0] *= w0, S[m][n][1] *= w0, S[m][n][2] *= w1, S[m][n][3] *= w1;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        uint32_t ah[4], al[4];                     // (rows are key channels, stored [token][channel]: transposed loads)
        const int da = (ks * 16 + (lane & 7) + (lane >> 4) * 8) * L.pk + key0 + ((lane >> 3) & 1) * 8;
        mp_ldm4t(ah, d_hi + da);
        mp_ldm4t(al, d_hi + DP_C * L.pk + da);
#pragma unroll
        for (int n2 = 0; n2 < N / 16; ++n2) {
          uint32_t bh[4], bl[4];
          const int ua = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n2 * 16 + (lane >> 4) * 8;
          mp_ldm4t(bh, u_hi + ua);
          mp_ldm4t(bl, u_lo + ua);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mp_mma(S[m][2 * n2 + n], ah, bh[2 * n], bh[2 * n + 1]);
            mp_mma(S[m][2 * n2 + n], ah, bl[2 * n], bl[2 * n + 1]);
            mp_mma(S[m][2 * n2 + n], al, bh[2 * n], bh[2 * n + 1]);
          }
        }
      }
    }
    if (ch + 1 < ch1) put_state();
    if (kind == 1 && owner) {                      // O += B U: the tokens up to this warp's
      const __nv_bfloat16* bs = sg + L.b + (mt * 16 + (lane & 15)) * DP_PB + (lane >> 4) * 8;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        if (ks > mt) continue;
        uint32_t ah[4], al[4], bh[4], bl[4];
        mp_ldm4(ah, bs + ks * 16);
        mp_ldm4(al, bs + DP_C * DP_PB + ks * 16);
        const int ua = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n0 + (lane >> 4) * 8;
        mp_ldm4t(bh, u_hi + ua);
        mp_ldm4t(bl, u_lo + ua);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          mp_mma(acc[n], ah, bh[2 * n], bh[2 * n + 1]);
          mp_mma(acc[n], ah, bl[2 * n], bl[2 * n + 1]);
          mp_mma(acc[n], al, bh[2 * n], bh[2 * n + 1]);
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int row = mt * 16 + g + 8 * r, c = j0 + n0 + n * 8 + 2 * t4;
          if (row < rows && c < dv)                // (dv is even: a pair lies inside or outside)
            *reinterpret_cast<float2*>(a.out + ((size_t)(first + row) * a.H + h) * dv + c) = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
        }
    }
    if (stages == 1 && ch + 1 < ch1) {
      __syncthreads();                             // (the only stage is read)
      if (tid == 0) load(ch + 1, 0);
    }
  }
  if (!ok) {
    if (tid == 0) {
      grace_period();
      if (a.err) atomicExch(a.err, 1);
    }
    return;
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < N / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = (warp + 8 * m) * 16 + g + 8 * (e >> 1), col = j0 + n * 8 + 2 * t4 + (e & 1);
        if (key < dk && col < dv) st[(size_t)col * dk + key] = S[m][n][e];
      }
}

template <typename K>
int dp_raise(K kernel, bool* flags, size_t smem) {
  const int dev = af_current_device();
  if (dev < 0) return -1;
  if (af_first_on_device(flags, dev)) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return af_fail((int)e, "af_delta_prompt: %s", cudaGetErrorString(e));
  }
  return 0;
}

constexpr size_t DP_SMEM = 220 * 1024;      // (dynamic; a block has a few KB of its own besides)

template <int NE>
int dp_launch_chunks(const DeltaPromptArgs& a, int n_chunks, cudaStream_t stream) {
  static bool raised[AF_MAX_DEVICES];
  if (int e = dp_raise(delta_chunk_kernel<NE>, raised, dp_prep_smem(32 * NE))) return e;
  af_launch(delta_chunk_kernel<NE>, dim3(n_chunks, a.H), dim3(256), dp_prep_smem(a.dk), stream, a);
  AF_COUNT_LAUNCH("af_delta_prompt (chunks)");
  return 0;
}

template <int N, int MT>
int dp_launch_walk(const DeltaPromptArgs& a, int n_seqs, cudaStream_t stream) {
  static bool raised[AF_MAX_DEVICES];
  if (int e = dp_raise(delta_walk_kernel<N, MT>, raised, DP_SMEM)) return e;
  const int stages = dp_walk_smem(a.dk, N, 2) <= DP_SMEM ? 2 : 1;
  af_launch(delta_walk_kernel<N, MT>, dim3((a.dv + N - 1) / N, a.H, n_seqs), dim3(256), dp_walk_smem(a.dk, N, stages), stream, a,
            stages);
  AF_CHECK_LAUNCH("af_delta_prompt (walk)");
}

}  // namespace

// Whether af_delta_prompt takes heads of these sizes (whole tiles of 16 keys, up to 256; whole pieces of 16 values).
AF_EXPORT int af_delta_prompt_supported(int dk, int dv) {
  return dk >= 16 && dk <= 256 && dk % 16 == 0 && dv >= 16 && dv % 16 == 0 ? 1 : 0;
}
AF_EXPORT int af_delta_prompt_chunk() { return DP_C; }

// A prefill step's recurrence.  q, k rows of G heads of dk, v rows of H heads of dv (qkv_ts elements between tokens), beta a
// number per token and head, z the decays' logits [tokens][H * dk].  chunk_starts [n_chunks + 1], seq_first_chunk [n_seqs + 1]:
// chunks of up to 32 tokens.  out float [tokens][H * dv]; state float [slots][H][dv][dk] is read and left updated.
// Scratch of af_delta_prompt_scratch(dk, dv, tile, 0 / 1) bytes a chunk and head, 16-byte aligned: blob and u0.  tile: value
// columns of a block of the second kernel (16 or 32).
AF_EXPORT long long af_delta_prompt_scratch(int dk, int dv, int tile, int which) {
  return which == 0 ? (long long)dp_blob(dk).size * 2 : (long long)((dv + tile - 1) / tile) * DP_C * (tile + 4) * 4;
}
AF_EXPORT int af_delta_prompt(float* out, const float* q, const float* k, const float* v, long long qkv_ts, const float* beta,
                              long long beta_ts, const float* z, long long z_ts, const float* dt_bias, const float* rate,
                              float* state, void* blob, float* u0, int tile, const int* chunk_starts,
                              const int* seq_first_chunk, const int* slots, int n_chunks, int n_seqs, int G, int H, int dk,
                              int dv, int* err, cudaStream_t stream) {
  if (n_chunks == 0) return 0;
  AF_REQUIRE(af_delta_prompt_supported(dk, dv), "af_delta_prompt: heads of %d keys and %d values", dk, dv);
  AF_REQUIRE(n_chunks > 0 && n_seqs > 0 && n_seqs < 65536 && G > 0 && H > 0 && H < 65536 && H % G == 0, "af_delta_prompt: bad sizes");
  AF_REQUIRE(qkv_ts % 4 == 0 && z_ts % 4 == 0 &&
                 (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)z | (uintptr_t)dt_bias | (uintptr_t)rate | (uintptr_t)blob |
                   (uintptr_t)u0 | (uintptr_t)out | (uintptr_t)state) & 15) == 0,
             "af_delta_prompt: rows of whole 16-byte pieces");
  AF_REQUIRE(tile == 16 || tile == 32, "af_delta_prompt: tiles of %d value columns", tile);
  DeltaPromptArgs a{q, k, v, beta, z, qkv_ts, beta_ts, z_ts, dt_bias, rate, (__nv_bfloat16*)blob, u0, tile,
                    state, out, chunk_starts, seq_first_chunk, slots, G, H, dk, dv, err};
  int e;
  if (dk <= 32) e = dp_launch_chunks<1>(a, n_chunks, stream);
  else if (dk <= 64) e = dp_launch_chunks<2>(a, n_chunks, stream);
  else if (dk <= 128) e = dp_launch_chunks<4>(a, n_chunks, stream);
  else e = dp_launch_chunks<8>(a, n_chunks, stream);
  if (e) return e;
  if (tile == 16) return dk <= 128 ? dp_launch_walk<16, 1>(a, n_seqs, stream) : dp_launch_walk<16, 2>(a, n_seqs, stream);
  return dk <= 128 ? dp_launch_walk<32, 1>(a, n_seqs, stream) : dp_launch_walk<32, 2>(a, n_seqs, stream);
}
