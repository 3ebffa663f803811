// A layer whose norm stands behind the residual sum, and what goes with it, all sums in 32 bits:
//
//   layer_norm    y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b, row by row;
//   norm_of_sum   x <- layer_norm(alpha x + gate * (scale_a a + scale_b b)), the terms tensors or split-K partial sums,
//                 gate = sigmoid(z + z_bias) per element or nothing; in the same pass a copy of the new row in the
//                 compute dtype for the sublayer that reads it next, and, for single tokens, that row shifted;
//   add_layer_norm  x <- x + layer_norm(scale_a a + scale_b b) (the norm on the sublayer's output alone): the same
//                 kernels with the stream added behind the norm instead of in front of it;
//   token_shift   h_t = x_t + (x_(t-1) - x_t) mu, the row before a sequence's first row of the step from its state
//                 (zeros before the first token), which keeps the sequence's last row.
#include "common.cuh"

namespace {

// A term of a sum: rows [n_rows, hidden] of the compute dtype, or `parts` of them as floats, `stride` elements apart.
struct LnTerm {
  const void* p;
  int dtype, parts;
  size_t stride;
  float scale;
};

struct LnSumArgs {
  float* x;
  LnTerm a, b;                 // b.p null: one term
  LnTerm z;                    // the gate before its sigmoid (z.p null: no gate)
  const float* z_bias;
  float alpha;
  const float *w, *bias;
  float eps;
  void* y;                     // the new row in the compute dtype, or null
  void* hs;                    // single tokens: the new row shifted, in the compute dtype, or null
  const float* mu;
  float* prev;                 // [slots][hidden]
  const int* slots;            // row -> slot, -1: a padding row (its state is neither read nor written)
  int n_rows, hidden;
};

__device__ __forceinline__ float ln_term1(const LnTerm& t, size_t at) {
  if (t.dtype == AF_BF16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(t.p)[at]) * t.scale;
  const float* p = reinterpret_cast<const float*>(t.p) + at;
  float s = p[0];
  for (int i = 1; i < t.parts; ++i) s += p[(size_t)i * t.stride];
  return s * t.scale;
}

__device__ __forceinline__ void ln_term4(const LnTerm& t, size_t at, float* v) {
  if (t.dtype == AF_BF16) {
    const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(t.p) + at);
    v[0] = __uint_as_float(raw.x << 16) * t.scale;
    v[1] = __uint_as_float(raw.x & 0xffff0000u) * t.scale;
    v[2] = __uint_as_float(raw.y << 16) * t.scale;
    v[3] = __uint_as_float(raw.y & 0xffff0000u) * t.scale;
    return;
  }
  const float* p = reinterpret_cast<const float*>(t.p) + at;
  float4 s = *reinterpret_cast<const float4*>(p);
  for (int i0 = 1; i0 < t.parts; i0 += 4) {                 // (partial sums: four loads in flight, added in order)
    float4 q[4];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      q[u] = i0 + u < t.parts ? *reinterpret_cast<const float4*>(p + (size_t)(i0 + u) * t.stride)
                              : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int u = 0; u < 4; ++u) s.x += q[u].x, s.y += q[u].y, s.z += q[u].z, s.w += q[u].w;
  }
  v[0] = s.x * t.scale, v[1] = s.y * t.scale, v[2] = s.z * t.scale, v[3] = s.w * t.scale;
}

template <typename TY>
__device__ __forceinline__ void ln_store4(TY* dst, const float* v) {
  if constexpr (sizeof(TY) == 2) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(dst) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
    *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
  }
}

__device__ __forceinline__ float ln_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// ---------------------------------------------------------------- the norm alone

template <typename TY>
__global__ void __launch_bounds__(256)
layer_norm_kernel(TY* __restrict__ y, const float* __restrict__ x, const float* __restrict__ w,
                  const float* __restrict__ b, const int* __restrict__ rows, int hidden, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];
  __shared__ float scratch[33];
  const size_t r = blockIdx.x;
  const float* xr = x + (rows != nullptr ? (size_t)rows[r] : r) * hidden;
  float s = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) row[i] = xr[i], s += xr[i];
  const float mean = block_sum(s, scratch) / (float)hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) ss += (row[i] - mean) * (row[i] - mean);
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
  for (int i = threadIdx.x; i < hidden; i += blockDim.x)
    y[r * hidden + i] = from_f32<TY>((row[i] - mean) * inv * w[i] + b[i]);
}

// Rows of whole groups of four: a thread keeps NV groups in registers, the weights are asked for before the wait (they
// are cold in a decode step: the step's other weights have pushed them out of L2).
template <typename TY, int NV>
__global__ void __launch_bounds__(1024)
layer_norm_row_kernel(TY* __restrict__ y, const float* __restrict__ x, const float* __restrict__ w,
                      const float* __restrict__ b, const int* __restrict__ rows, int hidden, float eps) {
  pdl_launch_dependents();
  __shared__ float scratch[33];
  const size_t r = blockIdx.x;
  float4 wv[NV], bv[NV], v[NV];
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
    wv[n] = bv[n] = v[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < hidden) wv[n] = *reinterpret_cast<const float4*>(w + i), bv[n] = *reinterpret_cast<const float4*>(b + i);
  }
  const size_t src = rows != nullptr ? (size_t)rows[r] : r;
  pdl_wait();
  x = pdl_fresh(x);
  float s = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
    if (i < hidden) v[n] = *reinterpret_cast<const float4*>(x + src * hidden + i);
    s += v[n].x + v[n].y + v[n].z + v[n].w;
  }
  const float mean = block_sum(s, scratch) / (float)hidden;
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    v[n].x -= mean, v[n].y -= mean, v[n].z -= mean, v[n].w -= mean;
    if ((threadIdx.x + n * blockDim.x) * 4 < hidden)
      ss += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
    if (i >= hidden) continue;
    const float o[4] = {v[n].x * inv * wv[n].x + bv[n].x, v[n].y * inv * wv[n].y + bv[n].y,
                        v[n].z * inv * wv[n].z + bv[n].z, v[n].w * inv * wv[n].w + bv[n].w};
    ln_store4(y + r * hidden + i, o);
  }
}

// ---------------------------------------------------------------- the norm of the residual sum

// Any row size: the row waits in shared memory between the passes.
// POST: the stream is added to the norm's result, not to its input.
template <typename TY, bool POST>
__global__ void __launch_bounds__(256)
norm_of_sum_kernel(LnSumArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];
  __shared__ float scratch[33];
  const int r = blockIdx.x, hidden = p.hidden;
  const size_t base = (size_t)r * hidden;
  float s = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float v = ln_term1(p.a, base + i);
    if (p.b.p != nullptr) v += ln_term1(p.b, base + i);
    if (p.z.p != nullptr) v *= ln_sigmoid(ln_term1(p.z, base + i) + p.z_bias[i]);
    if (!POST) v = fmaf(p.alpha, p.x[base + i], v);
    row[i] = v;
    s += v;
  }
  const float mean = block_sum(s, scratch) / (float)hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) ss += (row[i] - mean) * (row[i] - mean);
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)hidden + p.eps);
  const int slot = p.hs != nullptr ? p.slots[r] : -1;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float v = (row[i] - mean) * inv * p.w[i] + p.bias[i];
    if (POST) v += p.x[base + i];
    p.x[base + i] = v;
    if (p.y != nullptr) reinterpret_cast<TY*>(p.y)[base + i] = from_f32<TY>(v);
    if (p.hs != nullptr) {
      float before = 0.f;
      if (slot >= 0) before = p.prev[(size_t)slot * hidden + i], p.prev[(size_t)slot * hidden + i] = v;
      reinterpret_cast<TY*>(p.hs)[base + i] = from_f32<TY>(v + (before - v) * p.mu[i]);
    }
  }
}

// Rows of whole groups of four: a thread keeps NV groups in registers and every load of a group is in flight before
// the first sum.  Few rows (a decode step): one group a thread, the weights and the state asked for before the wait for
// the kernel in front; many rows (MANY): two groups a thread, the weights read where they are used (L1 holds them).
template <typename TY, int NV, bool MANY, bool POST>
__global__ void __launch_bounds__(MANY ? 512 : 1024, MANY ? 3 : 1)
norm_of_sum_row_kernel(LnSumArgs p) {
  pdl_launch_dependents();
  __shared__ float scratch[33];
  const int r = blockIdx.x, hidden = p.hidden;
  const size_t base = (size_t)r * hidden;
  float v[NV][4], wv[NV][4], bv[NV][4], zb[NV][4], mu[NV][4], pv[NV][4], xs[POST ? NV : 1][4];
  const int slot = p.hs != nullptr ? p.slots[r] : -1;
  auto get4 = [](const float* src, float* dst) {
    const float4 q = *reinterpret_cast<const float4*>(src);
    dst[0] = q.x, dst[1] = q.y, dst[2] = q.z, dst[3] = q.w;
  };
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
#pragma unroll
    for (int u = 0; u < 4; ++u) v[n][u] = wv[n][u] = bv[n][u] = zb[n][u] = mu[n][u] = pv[n][u] = 0.f;
    if (i >= hidden || MANY) continue;
    get4(p.w + i, wv[n]);
    get4(p.bias + i, bv[n]);
    if (p.z.p != nullptr) get4(p.z_bias + i, zb[n]);
    if (p.hs != nullptr) get4(p.mu + i, mu[n]);
    // (the state is what the step before left: no kernel of this step has touched it)
    if (slot >= 0) get4(p.prev + (size_t)slot * hidden + i, pv[n]);
  }
  pdl_wait();
  p.a.p = pdl_fresh(p.a.p), p.b.p = pdl_fresh(p.b.p), p.z.p = pdl_fresh(p.z.p), p.x = pdl_fresh(p.x);
  float s = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
    if (i >= hidden) continue;
    float xv[4], bt[4] = {0.f, 0.f, 0.f, 0.f}, zt[4];
    get4(p.x + base + i, xv);
    ln_term4(p.a, base + i, v[n]);
    if (p.b.p != nullptr) ln_term4(p.b, base + i, bt);
    if (p.z.p != nullptr) {
      ln_term4(p.z, base + i, zt);
      if (MANY) get4(p.z_bias + i, zb[n]);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      float t = v[n][u] + bt[u];
      if (p.z.p != nullptr) t *= ln_sigmoid(zt[u] + zb[n][u]);
      if (POST) xs[n][u] = xv[u], v[n][u] = t;
      else v[n][u] = fmaf(p.alpha, xv[u], t);
      s += v[n][u];
    }
  }
  const float mean = block_sum(s, scratch) / (float)hidden;
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const bool on = (threadIdx.x + n * blockDim.x) * 4 < hidden;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      v[n][u] -= mean;
      ss += on ? v[n][u] * v[n][u] : 0.f;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)hidden + p.eps);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = (threadIdx.x + n * blockDim.x) * 4;
    if (i >= hidden) continue;
    if (MANY) get4(p.w + i, wv[n]), get4(p.bias + i, bv[n]);
#pragma unroll
    for (int u = 0; u < 4; ++u) v[n][u] = v[n][u] * inv * wv[n][u] + bv[n][u] + (POST ? xs[n][u] : 0.f);
    ln_store4(p.x + base + i, v[n]);
    if (p.y != nullptr) ln_store4(reinterpret_cast<TY*>(p.y) + base + i, v[n]);
    if (p.hs != nullptr) {
      if (MANY) {
        get4(p.mu + i, mu[n]);
        if (slot >= 0) get4(p.prev + (size_t)slot * hidden + i, pv[n]);
      }
      if (slot >= 0) ln_store4(p.prev + (size_t)slot * hidden + i, v[n]);
      float h[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) h[u] = v[n][u] + (pv[n][u] - v[n][u]) * mu[n][u];
      ln_store4(reinterpret_cast<TY*>(p.hs) + base + i, h);
    }
  }
}

// ---------------------------------------------------------------- the shift alone

// One thread a group of V channels of a row.  A sequence's first row of the step takes the row before it from the
// sequence's state and leaves the sequence's last row there (the same thread does both, so nothing is overtaken).
template <typename TY, int V>
__global__ void __launch_bounds__(256)
token_shift_kernel(TY* __restrict__ hs, TY* __restrict__ y, const float* __restrict__ x, const float* __restrict__ mu,
                   float* __restrict__ prev, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                   const int* __restrict__ seq_starts, const int* __restrict__ slots, int hidden) {
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const int seq = seq_of_token[t], slot = slots[seq], first = seq_starts[seq], last = seq_starts[seq + 1] - 1;
  const bool start = positions[t] == 0;
  pdl_wait();
  if (c >= hidden) return;
  x = pdl_fresh(x);
  float v[V], b[V], m[V];
#pragma unroll
  for (int u = 0; u < V; ++u) v[u] = x[(size_t)t * hidden + c + u], m[u] = mu[c + u], b[u] = 0.f;
  if (t != first) {
#pragma unroll
    for (int u = 0; u < V; ++u) b[u] = x[(size_t)(t - 1) * hidden + c + u];
  } else if (slot >= 0) {
    float* st = prev + (size_t)slot * hidden + c;
    const float* end = x + (size_t)last * hidden + c;
#pragma unroll
    for (int u = 0; u < V; ++u) {
      if (!start) b[u] = st[u];
      st[u] = end[u];
    }
  }
  float h[V];
#pragma unroll
  for (int u = 0; u < V; ++u) h[u] = v[u] + (b[u] - v[u]) * m[u];
  const size_t at = (size_t)t * hidden + c;
  if constexpr (V == 4) {
    ln_store4(hs + at, h);
    if (y != nullptr) ln_store4(y + at, v);
  } else {
    hs[at] = from_f32<TY>(h[0]);
    if (y != nullptr) y[at] = from_f32<TY>(v[0]);
  }
}

constexpr int LN_MAX_ROW = 16384;

// Rows that do not fit the default limit of shared memory: raised once a device.
template <typename K>
int ln_raise(K kernel, bool* flags, int hidden) {
  if (hidden * sizeof(float) <= 40 * 1024) return 0;
  const int dev = af_current_device();
  if (dev < 0) return -1;
  if (af_first_on_device(flags, dev)) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LN_MAX_ROW * (int)sizeof(float));
    if (e != cudaSuccess) return af_fail((int)e, "af_layer_norm: %s", cudaGetErrorString(e));
  }
  return 0;
}

template <typename TY>
int ln_launch(void* y, const float* x, const float* w, const float* b, const int* rows, int n_rows, int hidden, float eps,
              cudaStream_t stream) {
  if (hidden % 4 == 0 && hidden <= 8192 && (((uintptr_t)y | (uintptr_t)x | (uintptr_t)w | (uintptr_t)b) & 15) == 0) {
    const int nv = hidden > 4096 ? 2 : 1, threads = ((hidden / 4 + nv - 1) / nv + 31) / 32 * 32;
    if (nv == 2)
      af_launch(layer_norm_row_kernel<TY, 2>, dim3(n_rows), dim3(threads), 0, stream, (TY*)y, x, w, b, rows, hidden, eps);
    else
      af_launch(layer_norm_row_kernel<TY, 1>, dim3(n_rows), dim3(threads), 0, stream, (TY*)y, x, w, b, rows, hidden, eps);
    AF_CHECK_LAUNCH("af_layer_norm");
  }
  static bool raised[AF_MAX_DEVICES];
  if (int e = ln_raise(layer_norm_kernel<TY>, raised, hidden)) return e;
  af_launch(layer_norm_kernel<TY>, dim3(n_rows), dim3(256), (size_t)hidden * sizeof(float), stream, (TY*)y, x, w, b, rows,
            hidden, eps);
  AF_CHECK_LAUNCH("af_layer_norm");
}

template <typename TY, bool POST>
int ln_launch_sum(const LnSumArgs& p, cudaStream_t stream) {
  static bool raised[AF_MAX_DEVICES];
  if (int e = ln_raise(norm_of_sum_kernel<TY, POST>, raised, p.hidden)) return e;
  af_launch(norm_of_sum_kernel<TY, POST>, dim3(p.n_rows), dim3(256), (size_t)p.hidden * sizeof(float), stream, p);
  AF_CHECK_LAUNCH("af_norm_of_sum");
}

int ln_term_check(const LnTerm& t, const char* who, const char* what) {
  AF_REQUIRE(t.p == nullptr || (t.parts >= 1 && (t.dtype == AF_F32 || (t.dtype == AF_BF16 && t.parts == 1))),
             "%s: %s must be floats, or one tensor of bfloat16", who, what);
  return 0;
}

bool ln_term_vec(const LnTerm& t) {
  return t.p == nullptr || (((uintptr_t)t.p & 15) == 0 && t.stride % 4 == 0);
}

}  // namespace

AF_EXPORT int af_layer_norm(void* y, int y_dtype, const float* x, const float* w, const float* b, const int* rows,
                            int n_rows, int hidden, float eps, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  AF_REQUIRE(n_rows > 0 && hidden > 0 && hidden <= LN_MAX_ROW, "af_layer_norm: rows of 1 to %d values", LN_MAX_ROW);
  AF_DISPATCH_DTYPE(y_dtype, TY, return ln_launch<TY>(y, x, w, b, rows, n_rows, hidden, eps, stream));
  return 0;
}

// y_dtype: of y and hs.  The terms' partial sums lie n_rows * hidden elements apart.  `post`: the stream is added
// behind the norm (alpha, the gate and the shift belong to the other form).
AF_EXPORT int af_norm_of_sum(float* x, const void* a, int a_dtype, int a_parts, float scale_a, const void* b, int b_dtype,
                             int b_parts, float scale_b, const void* z, int z_dtype, int z_parts, const float* z_bias,
                             float alpha, const float* w, const float* bias, float eps, void* y, void* hs, int y_dtype,
                             const float* mu, float* prev, const int* slots, int n_rows, int hidden, int post,
                             cudaStream_t stream) {
  if (n_rows == 0) return 0;
  AF_REQUIRE(!post || (z == nullptr && hs == nullptr), "af_norm_of_sum: a norm in front of the sum has no gate and no shift");
  AF_REQUIRE(n_rows > 0 && hidden > 0 && hidden <= LN_MAX_ROW, "af_norm_of_sum: rows of 1 to %d values", LN_MAX_ROW);
  AF_REQUIRE(x != nullptr && a != nullptr && w != nullptr && bias != nullptr && (z == nullptr || z_bias != nullptr),
             "af_norm_of_sum: a stream, a term, the norm's weight and bias, a bias with a gate");
  AF_REQUIRE(hs == nullptr || (mu != nullptr && prev != nullptr && slots != nullptr),
             "af_norm_of_sum: a shifted row needs its factors, the state and the slots");
  const size_t stride = (size_t)n_rows * hidden;
  LnSumArgs p;
  p.x = x;
  p.a = LnTerm{a, a_dtype, a_parts, stride, scale_a};
  p.b = LnTerm{b, b_dtype, b_parts, stride, scale_b};
  p.z = LnTerm{z, z_dtype, z_parts, stride, 1.f};
  p.z_bias = z_bias, p.alpha = alpha, p.w = w, p.bias = bias, p.eps = eps, p.y = y, p.hs = hs, p.mu = mu, p.prev = prev;
  p.slots = slots, p.n_rows = n_rows, p.hidden = hidden;
  if (int e = ln_term_check(p.a, "af_norm_of_sum", "the first term")) return e;
  if (int e = ln_term_check(p.b, "af_norm_of_sum", "the second term")) return e;
  if (int e = ln_term_check(p.z, "af_norm_of_sum", "the gate")) return e;
  const uintptr_t all = (uintptr_t)x | (uintptr_t)w | (uintptr_t)bias | (uintptr_t)z_bias | (uintptr_t)y | (uintptr_t)hs |
                        (uintptr_t)mu | (uintptr_t)prev;
  if (hidden % 4 == 0 && hidden <= 8192 && (all & 15) == 0 && ln_term_vec(p.a) && ln_term_vec(p.b) && ln_term_vec(p.z)) {
    const bool many = n_rows >= 256 && hidden >= 1024 && hidden <= 4096;
    const int nv = many || hidden > 4096 ? 2 : 1;
    const int threads = ((hidden / 4 + nv - 1) / nv + 31) / 32 * 32;
#define LN_LAUNCH(TY, P)                                                                                              \
  do {                                                                                                                \
    if (many) af_launch(norm_of_sum_row_kernel<TY, 2, true, P>, dim3(n_rows), dim3(threads), 0, stream, p);           \
    else if (nv == 2) af_launch(norm_of_sum_row_kernel<TY, 2, false, P>, dim3(n_rows), dim3(threads), 0, stream, p);  \
    else af_launch(norm_of_sum_row_kernel<TY, 1, false, P>, dim3(n_rows), dim3(threads), 0, stream, p);               \
  } while (0)
    if (post) AF_DISPATCH_DTYPE(y_dtype, TY, LN_LAUNCH(TY, true));
    else AF_DISPATCH_DTYPE(y_dtype, TY, LN_LAUNCH(TY, false));
#undef LN_LAUNCH
    AF_CHECK_LAUNCH("af_norm_of_sum");
  }
  if (post) AF_DISPATCH_DTYPE(y_dtype, TY, return (ln_launch_sum<TY, true>(p, stream)));
  AF_DISPATCH_DTYPE(y_dtype, TY, return (ln_launch_sum<TY, false>(p, stream)));
  return 0;
}

AF_EXPORT int af_token_shift(void* hs, void* y, int dtype, const float* x, const float* mu, float* prev,
                             const int* positions, const int* seq_of_token, const int* seq_starts, const int* slots,
                             int n_tokens, int hidden, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  AF_REQUIRE(n_tokens > 0 && hidden > 0, "af_token_shift: bad sizes");
  const bool vec = hidden % 4 == 0 &&
                   (((uintptr_t)hs | (uintptr_t)y | (uintptr_t)x | (uintptr_t)mu | (uintptr_t)prev) & 15) == 0;
  const int groups = vec ? hidden / 4 : hidden;
  const int threads = groups >= 256 ? 256 : ((groups + 31) / 32) * 32;
  const dim3 grid(n_tokens, (groups + threads - 1) / threads);
#define TS_LAUNCH(TY, V)                                                                                            \
  af_launch(token_shift_kernel<TY, V>, grid, dim3(threads), 0, stream, (TY*)hs, (TY*)y, x, mu, prev, positions,     \
            seq_of_token, seq_starts, slots, hidden)
  if (vec) AF_DISPATCH_DTYPE(dtype, TY, TS_LAUNCH(TY, 4));
  else AF_DISPATCH_DTYPE(dtype, TY, TS_LAUNCH(TY, 1));
#undef TS_LAUNCH
  AF_CHECK_LAUNCH("af_token_shift");
}
