// Retention: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head with a fixed decay, q and k rotated by their
// positions, each head's output over its root mean square and times a gate.  Two ways:
//
//   a step of single tokens (retention_step): one kernel rotates, updates the state and makes the gated output;
//   a prompt on the tensor cores (retention_prompt): the sequence is cut into chunks,
//     states   B(c) = sum over the chunk's tokens of decay^(last - t) k_t v_t^T, all chunks side by side;
//     carry    S_in(c + 1) = decay^length S_in(c) + B(c), from the cached state and back to it;
//     outputs  o_t = decay^(t + 1) S_in^T q_t + sum over s <= t of the chunk of decay^(t - s) (q_t . k_s) v_s.
//   The state, the scores, their weights and every sum are 32-bit.  The tensor cores' 16-bit operands come in pairs: a
//   32-bit value is hi + lo, both bfloat16, and a product is hi hi + hi lo + lo hi (16 to 17 bits of mantissa; what
//   is dropped is lo lo), so that rotated keys, weighted scores and carried states enter as what they are.
//
// A state of one sequence, run and head is stored [value column][key channel].
#include <cooperative_groups.h>

#include "mma_pairs.cuh"

namespace {

constexpr int RT_TILE = 64;        // tokens of a tile

struct RtArgs {
  const float *q, *k, *v;            // float rows, head h's piece h * dk (h * dv) behind the pointer
  long long q_ts, k_ts, v_ts;
  const float2* table;               // [tokens][n_rot] cosines and sines of the step, or null (n_rot 0)
  int n_rot, adjacent;
  float magnitude;
  const float* powers;               // [heads][chunk + 1]: decay^0 .. decay^chunk
  int chunk;                         // tokens of a chunk (a multiple of RT_TILE)
  float* local;                      // [chunks][heads][dv][dk]: B(c)
  __nv_bfloat16 *k_hi, *k_lo;        // [tokens][heads][dkp]: the rotated keys in two parts
  __nv_bfloat16 *v_hi, *v_lo;        // [tokens][heads][dvp]: the values
  __nv_bfloat16 *s_hi, *s_lo;        // [chunks][heads][dv][dkp]: S_in(c)
  const int* chunk_starts;           // [chunks + 1] first rows
  const int* tiles;                  // [tiles][4]: first row, rows, chunk, the tile's first token in its chunk
  int heads, dk, dv, dkp, dvp;       // dkp, dvp: rounded up to whole groups of 16
  const float* gate;                 // float rows [tokens][heads * dv] (null: plain float outputs)
  long long gate_ts;
  int gate_act;                      // 0: sigmoid, 1: x sigmoid(x)
  float key_scale, eps;
  void* out;                         // [tokens][heads * dv]
  long long out_ts;
  int vec;                           // rows may be read in 16-byte pieces
  int vec2;                          // gates and outputs may be read and written in pairs
};

// Four neighbouring channels c .. c + 3 of a head's query or key row of token t, rotated.
__device__ __forceinline__ void rt_rotated4(const RtArgs& a, const float* row, int t, int c, float* y) {
  const int n = a.n_rot;
  if (a.vec) {
    const float4 x4 = *reinterpret_cast<const float4*>(row + c);
    y[0] = x4.x, y[1] = x4.y, y[2] = x4.z, y[3] = x4.w;
    if (c >= 2 * n) return;                        // (n is a multiple of four here)
    if (a.adjacent) {
      const float4 cs = *reinterpret_cast<const float4*>(a.table + (size_t)t * n + c / 2);
      const float c0 = cs.x * a.magnitude, s0 = cs.y * a.magnitude, c1 = cs.z * a.magnitude, s1 = cs.w * a.magnitude;
      const float u0 = y[0], v0 = y[1], u1 = y[2], v1 = y[3];
      y[0] = u0 * c0 - v0 * s0, y[1] = v0 * c0 + u0 * s0, y[2] = u1 * c1 - v1 * s1, y[3] = v1 * c1 + u1 * s1;
      return;
    }
    const bool second = c >= n;
    const int e = second ? c - n : c;
    const float4 p4 = *reinterpret_cast<const float4*>(row + (second ? e : c + n));
    const float4 ca = *reinterpret_cast<const float4*>(a.table + (size_t)t * n + e);
    const float4 cb = *reinterpret_cast<const float4*>(a.table + (size_t)t * n + e + 2);
    const float pv[4] = {p4.x, p4.y, p4.z, p4.w};
    const float cv[4] = {ca.x, ca.z, cb.x, cb.z}, sv[4] = {ca.y, ca.w, cb.y, cb.w};
    const float m = a.magnitude, sgn = second ? m : -m;
#pragma unroll
    for (int u = 0; u < 4; ++u) y[u] = y[u] * (cv[u] * m) + pv[u] * (sv[u] * sgn);
    return;
  }
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int i = c + u;
    float x = 0.f;
    if (i < a.dk) {
      x = row[i];
      if (i < 2 * n) {
        const int e = a.adjacent ? i >> 1 : (i < n ? i : i - n);
        const bool second = a.adjacent ? (i & 1) : i >= n;
        const int p = a.adjacent ? (i ^ 1) : (second ? i - n : i + n);
        const float2 cs = a.table[(size_t)t * n + e];
        x = x * (cs.x * a.magnitude) + row[p] * (second ? cs.y : -cs.y) * a.magnitude;
      }
    }
    y[u] = x;
  }
}

__device__ __forceinline__ void rt_plain4(const float* row, int c, int size, int vec, float* y) {
  if (vec && c + 3 < size) {
    const float4 x4 = *reinterpret_cast<const float4*>(row + c);
    y[0] = x4.x, y[1] = x4.y, y[2] = x4.z, y[3] = x4.w;
    return;
  }
#pragma unroll
  for (int u = 0; u < 4; ++u) y[u] = c + u < size ? row[c + u] : 0.f;
}

// ---------------------------------------------------------------- single tokens

struct RtStep {
  RtArgs a;                          // q, k, v, rotation, gate, norm, out; a.powers null
  const float* decay;                // [heads]
  float* state;                      // [slots][heads][dv][dk]
  const int *slots, *seq_starts;
  int lanes;                         // P lanes share a value column, R key channels each (P R >= dk, P <= 32)
  int cols;                          // value columns of a block
};

// A cluster of blocks per (head, sequence), each with `cols` value columns of the head: 256 threads, P lanes a
// column.  The state's tile is asked for before the wait for the projection; the head's mean square is joined over the
// cluster through distributed shared memory.
template <int R, typename TO>
__global__ void __launch_bounds__(256)
retention_step_kernel(RtStep p) {
  pdl_launch_dependents();
  namespace cg = cooperative_groups;
  extern __shared__ __align__(16) float o_s[];     // [cols rounded up to 4], then the rotated query and key
  __shared__ float scratch[33];
  __shared__ float part_s;
  RtArgs a = p.a;
  const int P = p.lanes, per = 256 / P, tid = threadIdx.x, part = tid % P, col = tid / P;
  const int h = blockIdx.y, b = blockIdx.z, c0 = part * R;
  const int first = blockIdx.x * p.cols, n_cols = max(0, min(p.cols, a.dv - first));
  const int slot = p.slots[b];
  const int t = p.seq_starts[b];
  TO* dst = reinterpret_cast<TO*>(a.out) + (size_t)t * a.out_ts + (size_t)h * a.dv + first;
  if (slot < 0) {
    pdl_wait();
    for (int i = tid; i < n_cols; i += 256) dst[i] = from_f32<TO>(0.f);
    return;                          // (the whole cluster)
  }
  float* st = p.state + (((size_t)slot * a.heads + h) * a.dv + first) * a.dk + c0;
  float S[R];
  constexpr int RP = R + (R == 4 ? 0 : 4);   // (a lane's run of channels, apart from the next one's in the banks)
  float* q_s = o_s + (p.cols + 3) / 4 * 4;
  float* k_s = q_s + P * RP;
  auto read_state = [&](int j) {
    const float* src = st + (size_t)j * a.dk;
    if (a.vec) {
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < n_cols && c0 + i < a.dk) x = *reinterpret_cast<const float4*>(src + i);
        S[i] = x.x, S[i + 1] = x.y, S[i + 2] = x.z, S[i + 3] = x.w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < R; ++i) S[i] = (j < n_cols && c0 + i < a.dk) ? src[i] : 0.f;
    }
  };
  read_state(col);                   // (what the step before left: it does not wait for the kernel in front)
  const float dec = p.decay[h];
  pdl_wait();
  a.q = pdl_fresh(a.q), a.k = pdl_fresh(a.k), a.v = pdl_fresh(a.v), a.table = pdl_fresh(a.table), a.gate = pdl_fresh(a.gate);
  const float* qr = a.q + (size_t)t * a.q_ts + (size_t)h * a.dk;
  const float* kr = a.k + (size_t)t * a.k_ts + (size_t)h * a.dk;
  for (int i = tid; i < P * R / 2; i += 256) {     // four channels of the query or of the key a thread
    const bool key = i >= P * R / 4;
    const int c = (key ? i - P * R / 4 : i) * 4;
    float y[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < a.dk) rt_rotated4(a, key ? kr : qr, t, c, y);
    *reinterpret_cast<float4*>((key ? k_s : q_s) + (c / R) * RP + c % R) = make_float4(y[0], y[1], y[2], y[3]);
  }
  __syncthreads();
  const float* qv = q_s + part * RP;
  const float* kv = k_s + part * RP;
  const float* vr = a.v + (size_t)t * a.v_ts + (size_t)h * a.dv + first;
  float ss = 0.f;
  for (int j0 = 0; j0 < n_cols; j0 += per) {
    const int j = j0 + col;
    if (j0 > 0) read_state(j);
    const float vj = j < n_cols ? vr[j] : 0.f;
    float o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int i = 0; i < R; i += 4) {
      const float4 kq = *reinterpret_cast<const float4*>(kv + i), qq = *reinterpret_cast<const float4*>(qv + i);
      S[i] = dec * S[i] + kq.x * vj;
      S[i + 1] = dec * S[i + 1] + kq.y * vj;
      S[i + 2] = dec * S[i + 2] + kq.z * vj;
      S[i + 3] = dec * S[i + 3] + kq.w * vj;
      o0 += qq.x * S[i];
      o1 += qq.y * S[i + 1];
      o0 += qq.z * S[i + 2];
      o1 += qq.w * S[i + 3];
    }
    float o = o0 + o1;
    for (int w = 1; w < P; w <<= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
    o *= a.key_scale;
    if (j < n_cols) {
      if (part == 0) o_s[j] = o, ss += o * o;
      float* s_dst = st + (size_t)j * a.dk;
      if (a.vec) {
#pragma unroll
        for (int i = 0; i < R; i += 4)
          if (c0 + i < a.dk) *reinterpret_cast<float4*>(s_dst + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
      } else {
#pragma unroll
        for (int i = 0; i < R; ++i)
          if (c0 + i < a.dk) s_dst[i] = S[i];
      }
    }
  }
  ss = block_sum(ss, scratch);       // (its barriers also publish o_s)
  if (gridDim.x > 1) {
    cg::cluster_group cluster = cg::this_cluster();
    if (tid == 0) part_s = ss;
    cluster.sync();
    float total = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) total += *cluster.map_shared_rank(&part_s, r);
    ss = total;
    cluster.sync();                  // (no block leaves while another still reads its sum)
  }
  const float inv = rsqrtf(ss / (float)a.dv + a.eps);
  const float* gr = a.gate + (size_t)t * a.gate_ts + (size_t)h * a.dv + first;
  for (int i = tid; i < n_cols; i += 256) {
    const float z = gr[i], sg = 1.f / (1.f + expf(-z));
    dst[i] = from_f32<TO>(o_s[i] * inv * (a.gate_act ? z * sg : sg));
  }
}

template <int R, typename TO>
int rt_launch_step(const RtStep& p, int blocks, int heads, int n_seqs, cudaStream_t stream) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(blocks, heads, n_seqs);
  cfg.blockDim = dim3(256);
  cfg.dynamicSmemBytes = ((size_t)(p.cols + 3) / 4 * 4 + (size_t)2 * p.lanes * (R + 4)) * sizeof(float);
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_af_pdl ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = blocks, attr[1].val.clusterDim.y = 1, attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  cudaLaunchKernelEx(&cfg, retention_step_kernel<R, TO>, p);
  AF_CHECK_LAUNCH("af_retention_step");
}

// ---------------------------------------------------------------- a chunk's own state

// Block (chunk, head, value slice x key slice), 256 threads: S[v][c] = sum_t decay^(last - t) v_t[v] k_t[c] for a slice of
// DVT value columns and DKT key channels; 8 warps as 4 (value rows) x 2 (key channels).
template <int DVT, int DKT>
__global__ void __launch_bounds__(256, 2)
retention_states_kernel(RtArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char raw[];
  constexpr int PK = DKT + 8, PV = DVT + 8;
  __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(raw);
  __nv_bfloat16* k_lo = k_hi + RT_TILE * PK;
  __nv_bfloat16* v_hi = k_lo + RT_TILE * PK;
  __nv_bfloat16* v_lo = v_hi + RT_TILE * PV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp >> 1, wn = warp & 1;
  const int ch = blockIdx.x, h = blockIdx.y;
  const int k_slices = (a.dk + DKT - 1) / DKT;
  const int c0 = (blockIdx.z % k_slices) * DKT, j0 = (blockIdx.z / k_slices) * DVT;
  const int first = a.chunk_starts[ch], last = a.chunk_starts[ch + 1];
  const float* pw = a.powers + (size_t)h * (a.chunk + 1);
  constexpr int MT = DVT / 64, NT = DKT / 16;         // m16 tiles and n8 tiles of a warp
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  pdl_wait();
  a.q = pdl_fresh(a.q), a.k = pdl_fresh(a.k), a.v = pdl_fresh(a.v), a.table = pdl_fresh(a.table);
  // (the keys of a slice are kept by the blocks of the first value slice, the values by those of the first key slice)
  const bool keep_k = j0 == 0, keep_v = c0 == 0;
  for (int t0 = first; t0 < last; t0 += RT_TILE) {
    const int rows = min(RT_TILE, last - t0);
    __syncthreads();
    // four groups of four values at a time: their loads are in flight together
    constexpr int KQ = DKT / 4, VQ = DVT / 4;
#pragma unroll 1
    for (int i0 = 0; i0 < RT_TILE * KQ; i0 += 1024) {
      float y[4][4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256 + tid, r = min(i / KQ, rows - 1), c = c0 + (i % KQ) * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) y[u][e] = 0.f;
        if (c < a.dk) rt_rotated4(a, a.k + (size_t)(t0 + r) * a.k_ts + (size_t)h * a.dk, t0 + r, c, y[u]);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256 + tid, r = i / KQ, c = (i % KQ) * 4;
        const bool on = r < rows;
        if (on && keep_k && c0 + c < a.dkp) {
          const size_t dst = ((size_t)(t0 + r) * a.heads + h) * a.dkp + c0 + c;
          mp_put4(a.k_hi + dst, a.k_lo + dst, y[u]);
        }
        const float w = on ? pw[last - 1 - t0 - r] : 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) y[u][e] *= w;
        mp_put4(k_hi + r * PK + c, k_lo + r * PK + c, y[u]);
      }
    }
#pragma unroll 1
    for (int i0 = 0; i0 < RT_TILE * VQ; i0 += 1024) {
      float y[4][4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256 + tid, r = min(i / VQ, rows - 1), c = j0 + (i % VQ) * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) y[u][e] = 0.f;
        if (c < a.dv) rt_plain4(a.v + (size_t)(t0 + r) * a.v_ts + (size_t)h * a.dv, c, a.dv, a.vec, y[u]);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256 + tid, r = i / VQ, c = (i % VQ) * 4;
        if (r < rows) {
          if (keep_v && j0 + c < a.dvp) {
            const size_t dst = ((size_t)(t0 + r) * a.heads + h) * a.dvp + j0 + c;
            mp_put4(a.v_hi + dst, a.v_lo + dst, y[u]);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) y[u][e] = 0.f;
        }
        mp_put4(v_hi + r * PV + c, v_lo + r * PV + c, y[u]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < RT_TILE / 16; ++ks) {
      // A = v^T: rows are value columns, stored as [token][column]: transposed loads
      uint32_t ah[MT][4], al[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int col = (wm * MT + m) * 16 + ((lane >> 3) & 1) * 8;
        const int row = ks * 16 + (lane & 7) + (lane >> 4) * 8;
        mp_ldm4t(ah[m], v_hi + row * PV + col);
        mp_ldm4t(al[m], v_lo + row * PV + col);
      }
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        uint32_t bh[4], bl[4];
        const int col = wn * (DKT / 2) + n2 * 16 + (lane >> 4) * 8;
        const int row = ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
        mp_ldm4t(bh, k_hi + row * PK + col);
        mp_ldm4t(bl, k_lo + row * PK + col);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mp_mma(acc[m][2 * n2], ah[m], bh[0], bh[1]);
          mp_mma(acc[m][2 * n2 + 1], ah[m], bh[2], bh[3]);
          mp_mma(acc[m][2 * n2], ah[m], bl[0], bl[1]);
          mp_mma(acc[m][2 * n2 + 1], ah[m], bl[2], bl[3]);
          mp_mma(acc[m][2 * n2], al[m], bh[0], bh[1]);
          mp_mma(acc[m][2 * n2 + 1], al[m], bh[2], bh[3]);
        }
      }
    }
  }
  float* S = a.local + ((size_t)ch * a.heads + h) * a.dv * a.dk;
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int v = j0 + (wm * MT + m) * 16 + g + 8 * half, c = c0 + wn * (DKT / 2) + n * 8 + 2 * t;
        if (v >= a.dv) continue;
        float* dst = S + (size_t)v * a.dk + c;
        if (a.vec && c + 1 < a.dk) {
          *reinterpret_cast<float2*>(dst) = make_float2(acc[m][n][2 * half], acc[m][n][2 * half + 1]);
        } else {
          if (c < a.dk) dst[0] = acc[m][n][2 * half];
          if (c + 1 < a.dk) dst[1] = acc[m][n][2 * half + 1];
        }
      }
}

// ---------------------------------------------------------------- states from chunk to chunk

// One thread V state elements of a (sequence, head); the loads of four chunks are in flight at a time.  The state that
// enters a chunk goes out in two bfloat16 parts.
template <int V>
__global__ void __launch_bounds__(256)
retention_carry_kernel(RtArgs a, float* __restrict__ state, const int* __restrict__ seq_first_chunk,
                       const int* __restrict__ slots) {
  pdl_launch_dependents();
  const int per_head = a.dv * a.dk;
  const int e = (blockIdx.x * 256 + threadIdx.x) * V, h = blockIdx.y, b = blockIdx.z;
  const int slot = slots[b], ch0 = seq_first_chunk[b], ch1 = seq_first_chunk[b + 1];
  const float* pw = a.powers + (size_t)h * (a.chunk + 1);
  const size_t at16 = (size_t)(e / a.dk) * a.dkp + e % a.dk;
  pdl_wait();
  if (e >= per_head || slot < 0) return;
  float* st = state + ((size_t)slot * a.heads + h) * per_head + e;
  const size_t step = (size_t)a.heads * per_head, step16 = (size_t)a.heads * a.dv * a.dkp;
  const float* p = pdl_fresh(a.local) + (size_t)ch0 * step + (size_t)h * per_head + e;
  size_t o = (size_t)ch0 * step16 + (size_t)h * a.dv * a.dkp + at16;
  float S[V];
  auto get = [](const float* src, float* dst) {
    if constexpr (V == 4) {
      const float4 q = *reinterpret_cast<const float4*>(src);
      dst[0] = q.x, dst[1] = q.y, dst[2] = q.z, dst[3] = q.w;
    } else {
      dst[0] = src[0];
    }
  };
  get(st, S);
  for (int c = ch0; c < ch1; c += 4) {
    float B[4][V];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (c + u < ch1) get(p + (size_t)u * step, B[u]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (c + u >= ch1) continue;
      const float w = pw[a.chunk_starts[c + u + 1] - a.chunk_starts[c + u]];
      if constexpr (V == 4) {
        mp_put4(a.s_hi + o + (size_t)u * step16, a.s_lo + o + (size_t)u * step16, S);
      } else {
        const __nv_bfloat16 hi = __float2bfloat16_rn(S[0]);
        a.s_hi[o + (size_t)u * step16] = hi;
        a.s_lo[o + (size_t)u * step16] = __float2bfloat16_rn(S[0] - __bfloat162float(hi));
      }
#pragma unroll
      for (int i = 0; i < V; ++i) S[i] = fmaf(w, S[i], B[u][i]);
    }
    p += 4 * step;
    o += 4 * step16;
  }
  if constexpr (V == 4) *reinterpret_cast<float4*>(st) = make_float4(S[0], S[1], S[2], S[3]);
  else st[0] = S[0];
}

// ---------------------------------------------------------------- outputs

// Block (tile, head, value slice), eight warps: four groups of 16 tokens by two halves of the slice's value columns (both
// halves work the scores out for themselves).  Keys, values and the entering state come in two parts as the kernels
// in front left them, in whole 16-byte pieces without a register in between; the queries are rotated here.
template <int DVT, typename TO, bool NORM>
__global__ void __launch_bounds__(256, 2)
retention_outputs_kernel(RtArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char raw[];
  const int PQ = a.dkp + 8;
  constexpr int PV = DVT + 8;
  __nv_bfloat16* q_hi = reinterpret_cast<__nv_bfloat16*>(raw);
  __nv_bfloat16* q_lo = q_hi + RT_TILE * PQ;
  __nv_bfloat16* work = q_lo + RT_TILE * PQ;
  __nv_bfloat16 *s_hi = work, *s_lo = work + DVT * PQ;                                  // the entering state, or
  __nv_bfloat16 *k_hi = work, *k_lo = work + RT_TILE * PQ;                              // a tile of keys and
  __nv_bfloat16 *v_hi = work + 2 * RT_TILE * PQ, *v_lo = v_hi + RT_TILE * PV;           // values
  __shared__ float pw[257];                        // decay^0 .. decay^chunk (chunks of up to 256 tokens)
  __shared__ float sq[2][RT_TILE];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int rg = warp & 3, half = warp >> 2;
  const int h = blockIdx.y, j0 = blockIdx.z * DVT;
  const int row0 = a.tiles[4 * blockIdx.x], rows = a.tiles[4 * blockIdx.x + 1], ch = a.tiles[4 * blockIdx.x + 2];
  const int at = a.tiles[4 * blockIdx.x + 3];      // the tile's first token in its chunk
  for (int i = tid; i <= a.chunk; i += 256) pw[i] = a.powers[(size_t)h * (a.chunk + 1) + i];
  pdl_wait();
  a.q = pdl_fresh(a.q), a.table = pdl_fresh(a.table), a.gate = pdl_fresh(a.gate);
  const int pieces = a.dkp / 8, quads = a.dkp / 4;
  {
    const size_t base = ((size_t)ch * a.heads + h) * a.dv;
    for (int i = tid; i < DVT * pieces; i += 256) {
      const int v = i / pieces, c = (i - v * pieces) * 8;
      const bool on = j0 + v < a.dv;
      const size_t src = (base + (on ? j0 + v : 0)) * a.dkp + c;
      mp_cp16(s_hi + v * PQ + c, a.s_hi + src, on);
      mp_cp16(s_lo + v * PQ + c, a.s_lo + src, on);
    }
  }
  for (int i0 = 0; i0 < RT_TILE * quads; i0 += 1024) {      // (RT_TILE * quads is a multiple of 256)
    float y[4][4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = min(i0 + u * 256 + tid, RT_TILE * quads - 1), r = min(i / quads, rows - 1), c = (i % quads) * 4;
#pragma unroll
      for (int e = 0; e < 4; ++e) y[u][e] = 0.f;
      if (c < a.dk) rt_rotated4(a, a.q + (size_t)(row0 + r) * a.q_ts + (size_t)h * a.dk, row0 + r, c, y[u]);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = i0 + u * 256 + tid, r = i / quads, c = (i % quads) * 4;
      if (i < RT_TILE * quads) mp_put4(q_hi + r * PQ + c, q_lo + r * PQ + c, y[u]);
    }
  }
  constexpr int NT = DVT / 16;                     // n8 tiles of a warp
  const int n0 = half * (DVT / 2);
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  mp_cp_commit();
  mp_cp_wait();
  __syncthreads();
  // ---- what the state that enters the chunk gives
  for (int kk = 0; kk < a.dkp; kk += 16) {
    uint32_t ah[4], al[4];
    const int qa = (rg * 16 + (lane & 15)) * PQ + kk + (lane >> 4) * 8;
    mp_ldm4(ah, q_hi + qa);
    mp_ldm4(al, q_lo + qa);
#pragma unroll
    for (int n2 = 0; n2 < NT / 2; ++n2) {
      uint32_t bh[4], bl[4];
      const int sa = (n0 + n2 * 16 + (lane & 7) + (lane >> 4) * 8) * PQ + kk + ((lane >> 3) & 1) * 8;
      mp_ldm4(bh, s_hi + sa);
      mp_ldm4(bl, s_lo + sa);
      mp_mma(o[2 * n2], ah, bh[0], bh[1]);
      mp_mma(o[2 * n2 + 1], ah, bh[2], bh[3]);
      mp_mma(o[2 * n2], ah, bl[0], bl[1]);
      mp_mma(o[2 * n2 + 1], ah, bl[2], bl[3]);
      mp_mma(o[2 * n2], al, bh[0], bh[1]);
      mp_mma(o[2 * n2 + 1], al, bh[2], bh[3]);
    }
  }
  const int lr0 = rg * 16 + g, lr1 = lr0 + 8;      // this lane's rows of the tile
  {
    const float w0 = pw[min(at + lr0 + 1, a.chunk)], w1 = pw[min(at + lr1 + 1, a.chunk)];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] *= w0, o[n][1] *= w0, o[n][2] *= w1, o[n][3] *= w1;
  }
  // ---- what the chunk's own tokens give, tile by tile up to this one
  for (int kt = 0; kt <= at; kt += RT_TILE) {
    const int krow0 = row0 - at + kt;
    const bool own = kt == at;
    const int krows = own ? rows : RT_TILE;
    __syncthreads();                               // (what lay in the work area is done with)
    for (int i = tid; i < RT_TILE * pieces; i += 256) {
      const int r = i / pieces, c = (i - r * pieces) * 8;
      const bool on = r < krows;
      const size_t src = ((size_t)(krow0 + (on ? r : 0)) * a.heads + h) * a.dkp + c;
      mp_cp16(k_hi + r * PQ + c, a.k_hi + src, on);
      mp_cp16(k_lo + r * PQ + c, a.k_lo + src, on);
    }
    for (int i = tid; i < RT_TILE * (DVT / 8); i += 256) {
      const int r = i / (DVT / 8), c = (i - r * (DVT / 8)) * 8;
      const bool on = r < krows && j0 + c < a.dvp;
      const size_t src = ((size_t)(krow0 + (on ? r : 0)) * a.heads + h) * a.dvp + (on ? j0 + c : 0);
      mp_cp16(v_hi + r * PV + c, a.v_hi + src, on);
      mp_cp16(v_lo + r * PV + c, a.v_lo + src, on);
    }
    mp_cp_commit();
    mp_cp_wait();
    __syncthreads();
    const int groups = own ? rg + 1 : RT_TILE / 16;        // groups of 16 keys that this warp's tokens see
    float s[RT_TILE / 8][4];
#pragma unroll
    for (int n = 0; n < RT_TILE / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
    for (int kk = 0; kk < a.dkp; kk += 16) {
      uint32_t ah[4], al[4];
      const int qa = (rg * 16 + (lane & 15)) * PQ + kk + (lane >> 4) * 8;
      mp_ldm4(ah, q_hi + qa);
      mp_ldm4(al, q_lo + qa);
#pragma unroll
      for (int n2 = 0; n2 < RT_TILE / 16; ++n2) {
        if (n2 >= groups) continue;
        uint32_t bh[4], bl[4];
        const int ka = (n2 * 16 + (lane & 7) + (lane >> 4) * 8) * PQ + kk + ((lane >> 3) & 1) * 8;
        mp_ldm4(bh, k_hi + ka);
        mp_ldm4(bl, k_lo + ka);
        mp_mma(s[2 * n2], ah, bh[0], bh[1]);
        mp_mma(s[2 * n2 + 1], ah, bh[2], bh[3]);
        mp_mma(s[2 * n2], ah, bl[0], bl[1]);
        mp_mma(s[2 * n2 + 1], ah, bl[2], bl[3]);
        mp_mma(s[2 * n2], al, bh[0], bh[1]);
        mp_mma(s[2 * n2 + 1], al, bh[2], bh[3]);
      }
    }
    // the weights decay^(t - s); keys behind the token get none
    const int d0 = at + lr0 - kt, d1 = d0 + 8;
#pragma unroll
    for (int n = 0; n < RT_TILE / 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = n * 8 + 2 * t4 + e;
        s[n][e] = d0 >= key ? s[n][e] * pw[d0 - key] : 0.f;
        s[n][2 + e] = d1 >= key ? s[n][2 + e] * pw[d1 - key] : 0.f;
      }
#pragma unroll
    for (int ks = 0; ks < RT_TILE / 16; ++ks) {
      if (ks >= groups) continue;
      uint32_t ph[4], pl[4];
      mp_split2(s[2 * ks][0], s[2 * ks][1], ph[0], pl[0]);
      mp_split2(s[2 * ks][2], s[2 * ks][3], ph[1], pl[1]);
      mp_split2(s[2 * ks + 1][0], s[2 * ks + 1][1], ph[2], pl[2]);
      mp_split2(s[2 * ks + 1][2], s[2 * ks + 1][3], ph[3], pl[3]);
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        uint32_t bh[4], bl[4];
        const int va = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PV + n0 + n2 * 16 + (lane >> 4) * 8;
        mp_ldm4t(bh, v_hi + va);
        mp_ldm4t(bl, v_lo + va);
        mp_mma(o[2 * n2], ph, bh[0], bh[1]);
        mp_mma(o[2 * n2 + 1], ph, bh[2], bh[3]);
        mp_mma(o[2 * n2], ph, bl[0], bl[1]);
        mp_mma(o[2 * n2 + 1], ph, bl[2], bl[3]);
        mp_mma(o[2 * n2], pl, bh[0], bh[1]);
        mp_mma(o[2 * n2 + 1], pl, bh[2], bh[3]);
      }
    }
  }
  // ---- the head's norm and gate (the slice holds the whole head), or the output as it is
  float inv[2] = {a.key_scale, a.key_scale};
  if (NORM) {
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) ss[e >> 1] += (o[n][e] * a.key_scale) * (o[n][e] * a.key_scale);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
      ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
      if (t4 == 0) sq[half][r ? lr1 : lr0] = ss[r];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int lr = r ? lr1 : lr0;
      inv[r] *= rsqrtf((sq[0][lr] + sq[1][lr]) / (float)a.dv + a.eps);
    }
  }
  auto gated = [&](float y, float z) {
    const float sg = 1.f / (1.f + expf(-z));
    return y * (a.gate_act ? z * sg : sg);
  };
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int lr = r ? lr1 : lr0;
    if (lr >= rows) continue;
    const size_t tok = (size_t)(row0 + lr);
    TO* dst = reinterpret_cast<TO*>(a.out) + tok * a.out_ts + (size_t)h * a.dv;
    const float* gr = NORM ? a.gate + tok * a.gate_ts + (size_t)h * a.dv : nullptr;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int c = j0 + n0 + n * 8 + 2 * t4;
      float y0 = o[n][2 * r] * inv[r], y1 = o[n][2 * r + 1] * inv[r];
      if (a.vec2) {                                // (dv is even: a pair lies inside or outside)
        if (c >= a.dv) continue;
        if (NORM) {
          const float2 z = *reinterpret_cast<const float2*>(gr + c);
          y0 = gated(y0, z.x), y1 = gated(y1, z.y);
        }
        if constexpr (sizeof(TO) == 2) *reinterpret_cast<__nv_bfloat162*>(dst + c) = __floats2bfloat162_rn(y0, y1);
        else *reinterpret_cast<float2*>(dst + c) = make_float2(y0, y1);
      } else {
        if (c < a.dv) dst[c] = from_f32<TO>(NORM ? gated(y0, gr[c]) : y0);
        if (c + 1 < a.dv) dst[c + 1] = from_f32<TO>(NORM ? gated(y1, gr[c + 1]) : y1);
      }
    }
  }
}

size_t rt_outputs_smem(int dkp, int dvt) {
  const size_t q = (size_t)2 * RT_TILE * (dkp + 8), kv = (size_t)2 * RT_TILE * (dkp + 8) + (size_t)2 * RT_TILE * (dvt + 8);
  const size_t s = (size_t)2 * dvt * (dkp + 8);
  return (q + (kv > s ? kv : s)) * sizeof(__nv_bfloat16);
}

template <typename K>
int rt_raise(K kernel, bool* flags, size_t smem) {
  const int dev = af_current_device();
  if (dev < 0) return -1;
  if (af_first_on_device(flags, dev)) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return af_fail((int)e, "af_retention_prompt: %s", cudaGetErrorString(e));
  }
  return 0;
}

template <int DVT, int DKT>
int rt_launch_states(const RtArgs& a, int n_chunks, cudaStream_t stream) {
  static bool raised[AF_MAX_DEVICES];
  const size_t smem = (size_t)2 * RT_TILE * (DKT + 8 + DVT + 8) * sizeof(__nv_bfloat16);
  if (int e = rt_raise(retention_states_kernel<DVT, DKT>, raised, smem)) return e;
  const int slices = ((a.dk + DKT - 1) / DKT) * ((a.dv + DVT - 1) / DVT);
  af_launch(retention_states_kernel<DVT, DKT>, dim3(n_chunks, a.heads, slices), dim3(256), smem, stream, a);
  AF_COUNT_LAUNCH("af_retention_prompt (states)");
  return 0;
}

template <int DVT, typename TO, bool NORM>
int rt_launch_outputs(const RtArgs& a, int n_tiles, cudaStream_t stream) {
  static bool raised[AF_MAX_DEVICES];
  if (int e = rt_raise(retention_outputs_kernel<DVT, TO, NORM>, raised, rt_outputs_smem(256, DVT))) return e;
  af_launch(retention_outputs_kernel<DVT, TO, NORM>, dim3(n_tiles, a.heads, (a.dv + DVT - 1) / DVT), dim3(256),
            rt_outputs_smem(a.dkp, DVT), stream, a);
  AF_COUNT_LAUNCH("af_retention_prompt (outputs)");
  return 0;
}

}  // namespace

// 1 when the prompt's kernels take these sizes.
AF_EXPORT int af_retention_prompt_supported(int dk, int dv) { return dk >= 1 && dk <= 256 && dv >= 1 ? 1 : 0; }

// y (bfloat16, contiguous [tokens][heads * dv]) = norm per head (key_scale o) * gate, for dv <= 128; with gate null, out is
// float [tokens][heads * dv] = key_scale o.  Scratch: local float [n_chunks][heads][dv][dk]; with the head sizes rounded
// up to 16, kv16 bfloat16 2 x [n_tokens][heads][dkp] (keys) then 2 x [n_tokens][heads][dvp] (values), s16 2 x
// [n_chunks][heads][dv][dkp] (zeros behind dk on entry).
AF_EXPORT int af_retention_prompt(void* out, const float* q, long long q_ts, const float* k, long long k_ts, const float* v,
                                  long long v_ts, const float* gate, long long gate_ts, int gate_act, const float* table,
                                  int n_rot, int adjacent, float magnitude, const float* powers, int chunk, float* local,
                                  void* kv16, void* s16, float* state, const int* chunk_starts, const int* seq_first_chunk, const int* tiles,
                                  const int* slots, int n_tokens, int n_chunks, int n_seqs, int n_tiles, int heads,
                                  int dk, int dv, float key_scale, float eps, cudaStream_t stream) {
  if (n_tiles == 0) return 0;
  AF_REQUIRE(n_chunks > 0 && n_seqs > 0 && heads > 0 && heads < 65536 && n_seqs < 65536, "af_retention_prompt: bad sizes");
  AF_REQUIRE(af_retention_prompt_supported(dk, dv), "af_retention_prompt: heads of %d keys and %d values", dk, dv);
  AF_REQUIRE(chunk >= RT_TILE && chunk % RT_TILE == 0 && chunk <= 256, "af_retention_prompt: chunks of %d tokens", chunk);
  AF_REQUIRE(n_rot >= 0 && 2 * n_rot <= dk && (n_rot == 0 || table != nullptr), "af_retention_prompt: %d rotated pairs", n_rot);
  AF_REQUIRE(gate == nullptr || dv <= 128, "af_retention_prompt: the norm and gate are made with heads of up to 128 values");
  RtArgs a;
  a.q = q, a.k = k, a.v = v, a.q_ts = q_ts, a.k_ts = k_ts, a.v_ts = v_ts, a.table = (const float2*)table, a.n_rot = n_rot;
  a.adjacent = adjacent, a.magnitude = magnitude, a.powers = powers, a.chunk = chunk, a.local = local;
  a.chunk_starts = chunk_starts, a.tiles = tiles, a.heads = heads, a.dk = dk, a.dv = dv, a.dkp = (dk + 15) / 16 * 16;
  a.gate = gate, a.gate_ts = gate_ts, a.gate_act = gate_act, a.key_scale = key_scale, a.eps = eps, a.out = out;
  a.out_ts = (long long)heads * dv;
  a.dvp = (dv + 15) / 16 * 16;
  const size_t nk = (size_t)n_tokens * heads * a.dkp, nv = (size_t)n_tokens * heads * a.dvp;
  a.k_hi = (__nv_bfloat16*)kv16, a.k_lo = a.k_hi + nk, a.v_hi = a.k_lo + nk, a.v_lo = a.v_hi + nv;
  a.s_hi = (__nv_bfloat16*)s16, a.s_lo = a.s_hi + (size_t)n_chunks * heads * dv * a.dkp;
  AF_REQUIRE((((uintptr_t)kv16 | (uintptr_t)s16) & 15) == 0, "af_retention_prompt: 16-byte aligned scratch");
  a.vec2 = dv % 2 == 0 && (gate_ts & 1) == 0 && (((uintptr_t)gate | (uintptr_t)out) & 7) == 0;
  a.vec = dk % 4 == 0 && dv % 4 == 0 && n_rot % 4 == 0 && ((q_ts | k_ts | v_ts) & 3) == 0 &&
          (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)table | (uintptr_t)local | (uintptr_t)state) & 15) == 0;
  int e = 0;
  if (dv <= 64) e = dk <= 64 ? rt_launch_states<64, 64>(a, n_chunks, stream) : rt_launch_states<64, 128>(a, n_chunks, stream);
  else e = dk <= 64 ? rt_launch_states<128, 64>(a, n_chunks, stream) : rt_launch_states<128, 128>(a, n_chunks, stream);
  if (e) return e;
  const int per_head = dk * dv;
  if (a.vec)
    af_launch(retention_carry_kernel<4>, dim3((per_head / 4 + 255) / 256, heads, n_seqs), dim3(256), 0, stream, a, state,
              seq_first_chunk, slots);
  else
    af_launch(retention_carry_kernel<1>, dim3((per_head + 255) / 256, heads, n_seqs), dim3(256), 0, stream, a, state,
              seq_first_chunk, slots);
  AF_COUNT_LAUNCH("af_retention_prompt (carry)");
  if (gate != nullptr)
    return dv <= 64 ? rt_launch_outputs<64, __nv_bfloat16, true>(a, n_tiles, stream)
                    : rt_launch_outputs<128, __nv_bfloat16, true>(a, n_tiles, stream);
  return dv <= 64 ? rt_launch_outputs<64, float, false>(a, n_tiles, stream)
                  : rt_launch_outputs<128, float, false>(a, n_tiles, stream);
}

// A step in which every sequence brings one token: out (of `out_dtype`, contiguous [tokens][heads * dv]) = norm per head
// (key_scale o) * gate, the states updated.
AF_EXPORT int af_retention_step(void* out, int out_dtype, const float* q, long long q_ts, const float* k, long long k_ts,
                                const float* v, long long v_ts, const float* gate, long long gate_ts, int gate_act,
                                const float* table, int n_rot, int adjacent, float magnitude, const float* decay,
                                float* state, const int* slots, const int* seq_starts, int n_seqs, int heads, int dk, int dv,
                                float key_scale, float eps, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  AF_REQUIRE(n_seqs > 0 && n_seqs < 65536 && heads > 0 && heads < 65536 && dk > 0 && dk <= 1024 && dv > 0,
             "af_retention_step: bad sizes (key size up to 1024)");
  AF_REQUIRE(n_rot >= 0 && 2 * n_rot <= dk && (n_rot == 0 || table != nullptr), "af_retention_step: %d rotated pairs", n_rot);
  AF_REQUIRE(gate != nullptr && decay != nullptr && state != nullptr, "af_retention_step: a gate, decays and states");
  RtStep p;
  RtArgs& a = p.a;
  a = RtArgs{};
  a.q = q, a.k = k, a.v = v, a.q_ts = q_ts, a.k_ts = k_ts, a.v_ts = v_ts, a.table = (const float2*)table, a.n_rot = n_rot;
  a.adjacent = adjacent, a.magnitude = magnitude, a.heads = heads, a.dk = dk, a.dv = dv, a.gate = gate, a.gate_ts = gate_ts;
  a.gate_act = gate_act, a.key_scale = key_scale, a.eps = eps, a.out = out, a.out_ts = (long long)heads * dv;
  a.vec = dk % 4 == 0 && n_rot % 4 == 0 && ((q_ts | k_ts) & 3) == 0 &&
          (((uintptr_t)q | (uintptr_t)k | (uintptr_t)table | (uintptr_t)state) & 15) == 0;
  p.decay = decay, p.state = state, p.slots = slots, p.seq_starts = seq_starts;
  // R key channels a lane, eight lanes a column where that holds the head
  int r = 4, lanes = 1;
  for (;; r *= 2) {
    lanes = 1;
    while (lanes * r < dk && lanes < 32) lanes *= 2;
    if (r == 32 || (lanes * r >= dk && lanes <= 8)) break;
  }
  p.lanes = lanes;
  const int per = 256 / lanes;
  int blocks = (dv + per - 1) / per;
  if (blocks > 8) blocks = 8;
  while (blocks & (blocks - 1)) --blocks;                     // (clusters of 1, 2, 4 or 8 blocks)
  p.cols = (dv + blocks - 1) / blocks;
  AF_REQUIRE(p.cols <= 8192, "af_retention_step: heads of %d values", dv);
#define RT_STEP(R) AF_DISPATCH_DTYPE(out_dtype, TO, return (rt_launch_step<R, TO>(p, blocks, heads, n_seqs, stream)))
  switch (r) {
    case 4: RT_STEP(4); break;
    case 8: RT_STEP(8); break;
    case 16: RT_STEP(16); break;
    default: RT_STEP(32); break;
  }
#undef RT_STEP
  return 0;
}
