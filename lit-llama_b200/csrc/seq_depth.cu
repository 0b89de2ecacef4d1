// Norms with a bias, the residual step of layers that read a learned average over the results of all earlier layers, the
// plain residual step fused with the next norm (or with the operand of a product that replaces the stream), that product
// for a few tokens, and ungated feed-forward activations.  Sums, means and the average are f32; `act_t` is only the storage type of
// sublayer results, weights and the normed output.
#include "seq_common.cuh"

namespace b2l {

constexpr int DEPTH_THREADS = 256;

// mean and 1 / sqrt(variance + eps) (layer norm) or 0 and 1 / sqrt(mean square + eps) (RMS norm) of a row held as
// `n` register values per thread.  Two passes over the registers: the variance is the mean of the squared deviations.
template <int EPT>
__device__ __forceinline__ void row_moments(const float (&v)[EPT], int D, int kind, float eps, float* red, float& mean, float& rinv) {
  mean = 0.f;
  if (kind == B2L_SEQ_NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < EPT; ++e) s += v[e];                       // entries beyond D are 0
    mean = block_sum(s, red) / (float)D;
    __syncthreads();
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = threadIdx.x + e * DEPTH_THREADS;
    const float d = i < D ? v[e] - mean : 0.f;
    ss += d * d;
  }
  ss = block_sum(ss, red);
  rinv = 1.0f / sqrtf(ss / (float)D + eps);
}

template <typename act_t, int EPT>
__global__ void __launch_bounds__(DEPTH_THREADS) seq_norm_kernel(const float* __restrict__ x, const act_t* __restrict__ w,
                                                                 const act_t* __restrict__ b, int kind, float eps,
                                                                 act_t* __restrict__ out, const int* __restrict__ rows, int D) {
  __shared__ float red[32];
  const int r = rows ? rows[blockIdx.x] : blockIdx.x;
  const float* xr = x + (size_t)r * D;
  float v[EPT];
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = threadIdx.x + e * DEPTH_THREADS;
    v[e] = i < D ? xr[i] : 0.f;
  }
  float mean, rinv;
  row_moments<EPT>(v, D, kind, eps, red, mean, rinv);
  act_t* o = out + (size_t)blockIdx.x * D;
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = threadIdx.x + e * DEPTH_THREADS;
    if (i < D) st_act(o, i, (v[e] - mean) * rinv * ld_act(w, i) + (b ? ld_act(b, i) : 0.f));
  }
}

// Rows wider than the register form takes: three passes over global memory.
template <typename act_t>
__global__ void __launch_bounds__(DEPTH_THREADS) seq_norm_wide_kernel(const float* __restrict__ x, const act_t* __restrict__ w,
                                                                      const act_t* __restrict__ b, int kind, float eps,
                                                                      act_t* __restrict__ out, const int* __restrict__ rows, int D) {
  __shared__ float red[32];
  const int r = rows ? rows[blockIdx.x] : blockIdx.x;
  const float* xr = x + (size_t)r * D;
  float mean = 0.f;
  if (kind == B2L_SEQ_NORM_LAYER) {
    float s = 0.f;
    for (int i = threadIdx.x; i < D; i += DEPTH_THREADS) s += xr[i];
    mean = block_sum(s, red) / (float)D;
    __syncthreads();
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < D; i += DEPTH_THREADS) ss += (xr[i] - mean) * (xr[i] - mean);
  ss = block_sum(ss, red);
  const float rinv = 1.0f / sqrtf(ss / (float)D + eps);
  act_t* o = out + (size_t)blockIdx.x * D;
  for (int i = threadIdx.x; i < D; i += DEPTH_THREADS) st_act(o, i, (xr[i] - mean) * rinv * ld_act(w, i) + (b ? ld_act(b, i) : 0.f));
}

// One CTA per token: own result = x_in + y1 + y2 -> hist[n_hist-1]; x_out = sum_j avg[j] hist[j]; h = norm(x_out).
// The row stays in registers from the sum to the normed output; the earlier entries of hist are each read once.
template <typename act_t, int EPT>
__global__ void __launch_bounds__(DEPTH_THREADS) seq_depth_step_kernel(const act_t* __restrict__ y1, const act_t* __restrict__ y2,
                                                                       const float* x_in, float* __restrict__ hist, int n_hist,
                                                                       const float* __restrict__ avg, float* x_out,
                                                                       const act_t* __restrict__ wn, const act_t* __restrict__ bn, int kind,
                                                                       float eps, act_t* __restrict__ h, int T, int D) {
  __shared__ float red[32];
  const size_t row = (size_t)blockIdx.x * D, plane = (size_t)T * D;
  float v[EPT];
  float* own = hist + (size_t)(n_hist - 1) * plane + row;
  if (y1) {
#pragma unroll
    for (int e = 0; e < EPT; ++e) {
      const int i = threadIdx.x + e * DEPTH_THREADS;
      v[e] = 0.f;
      if (i < D) {
        float add = ld_act(y1, row + i);
        if (y2) add += ld_act(y2, row + i);
        v[e] = x_in[row + i] + add;
        own[i] = v[e];
      }
    }
  } else {
#pragma unroll
    for (int e = 0; e < EPT; ++e) {
      const int i = threadIdx.x + e * DEPTH_THREADS;
      v[e] = i < D ? own[i] : 0.f;
    }
  }
  if (avg) {
    const float last = avg[n_hist - 1];
#pragma unroll
    for (int e = 0; e < EPT; ++e) v[e] *= last;
    for (int j = 0; j + 1 < n_hist; ++j) {
      const float a = avg[j];
      const float* hj = hist + (size_t)j * plane + row;
#pragma unroll
      for (int e = 0; e < EPT; ++e) {
        const int i = threadIdx.x + e * DEPTH_THREADS;
        if (i < D) v[e] = fmaf(a, hj[i], v[e]);
      }
    }
  }
  if (x_out) {
#pragma unroll
    for (int e = 0; e < EPT; ++e) {
      const int i = threadIdx.x + e * DEPTH_THREADS;
      if (i < D) x_out[row + i] = v[e];
    }
  }
  if (wn == nullptr) return;
  float mean, rinv;
  row_moments<EPT>(v, D, kind, eps, red, mean, rinv);
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = threadIdx.x + e * DEPTH_THREADS;
    if (i < D) st_act(h, row + i, (v[e] - mean) * rinv * ld_act(wn, i) + (bn ? ld_act(bn, i) : 0.f));
  }
}

// ---- residual step: x_out = x_in + base + vec + (y1 + y2), h = norm(x_out), split = x_out as a pair of act numbers ----
// One CTA per token; a thread holds EPT groups of VEC neighbouring entries in registers from the sum to the normed output.
template <typename act_t, int VEC>
struct RowIO;
template <typename act_t>
struct RowIO<act_t, 1> {
  static __device__ __forceinline__ void ld(const act_t* p, float (&v)[1]) { v[0] = ld_act(p, 0); }
  static __device__ __forceinline__ void st(act_t* p, const float (&v)[1]) { st_act(p, 0, v[0]); }
};
template <>
struct RowIO<float, 4> {
  static __device__ __forceinline__ void ld(const float* p, float (&v)[4]) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
  }
  static __device__ __forceinline__ void st(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <>
struct RowIO<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void ld(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(w.x << 16); v[1] = __uint_as_float(w.x & 0xffff0000u);
    v[2] = __uint_as_float(w.y << 16); v[3] = __uint_as_float(w.y & 0xffff0000u);
  }
  static __device__ __forceinline__ void st(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
};

// The pair (hi, lo) with hi = round(v), lo = round(v - hi): together they carry twice the digits of the storage type.
template <typename act_t, int VEC>
__device__ __forceinline__ void store_split(act_t* hi_p, act_t* lo_p, const float (&v)[VEC]) {
  float hi[VEC], lo[VEC];
#pragma unroll
  for (int u = 0; u < VEC; ++u) {
    act_t tmp[1];
    st_act(tmp, 0, v[u]);
    hi[u] = ld_act(tmp, 0);
    lo[u] = v[u] - hi[u];
  }
  RowIO<act_t, VEC>::st(hi_p, hi);
  RowIO<act_t, VEC>::st(lo_p, lo);
}

template <typename act_t, int VEC, int EPT>
__global__ void __launch_bounds__(DEPTH_THREADS) seq_residual_step_kernel(b2l_seq_residual_args a) {
  __shared__ float red[32];
  const int D = a.D;
  const size_t row = (size_t)blockIdx.x * D;
  const act_t* y1 = (const act_t*)a.y1;
  const act_t* y2 = (const act_t*)a.y2;
  const act_t* vec = (const act_t*)a.vec;
  float v[EPT][VEC];
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = (threadIdx.x + e * DEPTH_THREADS) * VEC;
#pragma unroll
    for (int u = 0; u < VEC; ++u) v[e][u] = 0.f;
    if (i >= D) continue;
    float t[VEC];
    if (y1) {
      RowIO<act_t, VEC>::ld(y1 + row + i, v[e]);
      if (y2) {
        RowIO<act_t, VEC>::ld(y2 + row + i, t);
#pragma unroll
        for (int u = 0; u < VEC; ++u) v[e][u] += t[u];
      }
    }
    if (vec) {
      RowIO<act_t, VEC>::ld(vec + i, t);
#pragma unroll
      for (int u = 0; u < VEC; ++u) v[e][u] += t[u];
    }
    if (a.base) {
      RowIO<float, VEC>::ld(a.base + row + i, t);
#pragma unroll
      for (int u = 0; u < VEC; ++u) v[e][u] += t[u];
    }
    RowIO<float, VEC>::ld(a.x_in + row + i, t);
#pragma unroll
    for (int u = 0; u < VEC; ++u) v[e][u] += t[u];
    if (a.x_out) RowIO<float, VEC>::st(a.x_out + row + i, v[e]);
    if (a.split) store_split<act_t, VEC>((act_t*)a.split + 2 * row + i, (act_t*)a.split + 2 * row + D + i, v[e]);
  }
  if (a.w == nullptr) return;
  float mean = 0.f;
  if (a.norm_kind == B2L_SEQ_NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < EPT; ++e)
#pragma unroll
      for (int u = 0; u < VEC; ++u) s += v[e][u];                    // entries beyond D are 0
    mean = block_sum(s, red) / (float)D;
    __syncthreads();
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    if ((threadIdx.x + e * DEPTH_THREADS) * VEC >= D) continue;
#pragma unroll
    for (int u = 0; u < VEC; ++u) ss += (v[e][u] - mean) * (v[e][u] - mean);
  }
  ss = block_sum(ss, red);
  const float rinv = 1.0f / sqrtf(ss / (float)D + a.eps);
#pragma unroll
  for (int e = 0; e < EPT; ++e) {
    const int i = (threadIdx.x + e * DEPTH_THREADS) * VEC;
    if (i >= D) continue;
    float w[VEC], b[VEC], o[VEC];
    RowIO<act_t, VEC>::ld((const act_t*)a.w + i, w);
#pragma unroll
    for (int u = 0; u < VEC; ++u) b[u] = 0.f;
    if (a.b) RowIO<act_t, VEC>::ld((const act_t*)a.b + i, b);
#pragma unroll
    for (int u = 0; u < VEC; ++u) o[u] = (v[e][u] - mean) * rinv * w[u] + b[u];
    RowIO<act_t, VEC>::st((act_t*)a.h + row + i, o);
  }
}

// Rows wider than the register form takes: the new row is read back from x_out (every thread reads what it wrote).
template <typename act_t>
__global__ void __launch_bounds__(DEPTH_THREADS) seq_residual_step_wide_kernel(b2l_seq_residual_args a) {
  __shared__ float red[32];
  const int D = a.D;
  const size_t row = (size_t)blockIdx.x * D;
  float* xo = a.x_out + row;
  float s = 0.f;
  for (int i = threadIdx.x; i < D; i += DEPTH_THREADS) {
    float v = a.y1 ? ld_act((const act_t*)a.y1, row + i) : 0.f;
    if (a.y2) v += ld_act((const act_t*)a.y2, row + i);
    if (a.vec) v += ld_act((const act_t*)a.vec, i);
    if (a.base) v += a.base[row + i];
    v += a.x_in[row + i];
    xo[i] = v;
    s += v;
    const float one[1] = {v};
    if (a.split) store_split<act_t, 1>((act_t*)a.split + 2 * row + i, (act_t*)a.split + 2 * row + D + i, one);
  }
  if (a.w == nullptr) return;
  float mean = 0.f;
  if (a.norm_kind == B2L_SEQ_NORM_LAYER) {
    mean = block_sum(s, red) / (float)D;
    __syncthreads();
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < D; i += DEPTH_THREADS) ss += (xo[i] - mean) * (xo[i] - mean);
  ss = block_sum(ss, red);
  const float rinv = 1.0f / sqrtf(ss / (float)D + a.eps);
  for (int i = threadIdx.x; i < D; i += DEPTH_THREADS)
    st_act((act_t*)a.h, row + i, (xo[i] - mean) * rinv * ld_act((const act_t*)a.w, i) + (a.b ? ld_act((const act_t*)a.b, i) : 0.f));
}

// A product of an f32 row with a weight matrix for a few tokens, f32 throughout: out[t, i] = W[i, :] . x[t, :] + base[t, i] +
// vec[i].  A warp per output, the row in shared memory.  grid (T, chunks of outputs).
template <typename act_t>
__global__ void __launch_bounds__(256) seq_linear_few_kernel(const act_t* __restrict__ w, const float* __restrict__ x, const float* __restrict__ base,
                                                             const act_t* __restrict__ vec, float* __restrict__ out, int N, int K, int v16) {
  extern __shared__ float few_x[];
  const int t = blockIdx.x, wpc = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < K; i += blockDim.x) few_x[i] = x[(size_t)t * K + i];
  __syncthreads();
  for (int i = blockIdx.y * wpc + warp; i < N; i += gridDim.y * wpc) {
    float v = row_dot(w + (size_t)i * K, few_x, K, lane, v16 != 0);
    if (base) v += base[(size_t)t * N + i];
    if (vec) v += ld_act(vec, i);
    if (lane == 0) out[(size_t)t * N + i] = v;
  }
}

static DynSmemCache g_few_smem[2];

// exp(z) - 1 - z for z <= 0 without the cancellation of the plain form: the series z^2/2 + ... + z^7/5040 near zero (its
// first missing term is below 2^-23 of the sum for |z| < 1/4), exp(z) - 1 - z elsewhere, where the difference is at least
// 0.028 and an absolute error of 1e-7 is at most 4e-6 of it.  No branch: both forms are a handful of operations.
__device__ __forceinline__ float expm1_minus_z(float z) {
  const float series = z * z * fmaf(z, fmaf(z, fmaf(z, fmaf(z, fmaf(z, 1.0f / 5040.0f, 1.0f / 720.0f), 1.0f / 120.0f), 1.0f / 24.0f), 1.0f / 6.0f), 0.5f);
  const float plain = (expf(z) - 1.0f) - z;
  return z > -0.25f ? series : plain;
}

__device__ __forceinline__ float unary_act(float z, int act, float a, float b) {
  switch (act) {
    case B2L_SEQ_ACT_GELU_TANH: return gelu_tanh_f(z);
    case B2L_SEQ_ACT_SILU: return silu_f(z);
    case B2L_SEQ_ACT_SIGMOID: return sigmoid_f(z);
    case B2L_SEQ_ACT_RELU2: { const float r = fmaxf(z, 0.f); return r * r; }
    case B2L_SEQ_ACT_XIELU: return (z > 0.f ? a * z * z : b * expm1_minus_z(fminf(z, 0.f))) + 0.5f * z;
    default: return z;
  }
}

template <typename act_t>
__global__ void seq_unary_act_kernel(const act_t* __restrict__ in, int ldin, act_t* __restrict__ out, int ldout, int F, int act,
                                     const float* __restrict__ coef) {
  const float a = coef ? coef[0] : 0.f, b = coef ? coef[1] : 0.f;
  const act_t* p = in + (size_t)blockIdx.x * ldin;
  act_t* q = out + (size_t)blockIdx.x * ldout;
  for (int j = blockIdx.y * blockDim.x + threadIdx.x; j < F; j += gridDim.y * blockDim.x) st_act(q, j, unary_act(ld_act(p, j), act, a, b));
}

// 16-byte form: eight bf16 or four f32 numbers per load (F and the leading dimensions multiples of that, aligned pointers).
template <typename act_t>
__global__ void seq_unary_act_vec_kernel(const act_t* __restrict__ in, int ldin, act_t* __restrict__ out, int ldout, int F, int act,
                                         const float* __restrict__ coef) {
  constexpr int PER = 16 / sizeof(act_t);
  const float a = coef ? coef[0] : 0.f, b = coef ? coef[1] : 0.f;
  const act_t* p = in + (size_t)blockIdx.x * ldin;
  act_t* q = out + (size_t)blockIdx.x * ldout;
  for (int j = (blockIdx.y * blockDim.x + threadIdx.x) * PER; j < F; j += gridDim.y * blockDim.x * PER) {
    const uint4 u = *reinterpret_cast<const uint4*>(p + j);
    uint4 r;
    if (sizeof(act_t) == 2) {
      const uint32_t uw[4] = {u.x, u.y, u.z, u.w};
      uint32_t rw[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const __nv_bfloat162 t = __floats2bfloat162_rn(unary_act(__uint_as_float(uw[k] << 16), act, a, b),
                                                       unary_act(__uint_as_float(uw[k] & 0xffff0000u), act, a, b));
        rw[k] = *reinterpret_cast<const uint32_t*>(&t);
      }
      r = make_uint4(rw[0], rw[1], rw[2], rw[3]);
    } else {
      r.x = __float_as_uint(unary_act(__uint_as_float(u.x), act, a, b));
      r.y = __float_as_uint(unary_act(__uint_as_float(u.y), act, a, b));
      r.z = __float_as_uint(unary_act(__uint_as_float(u.z), act, a, b));
      r.w = __float_as_uint(unary_act(__uint_as_float(u.w), act, a, b));
    }
    *reinterpret_cast<uint4*>(q + j) = r;
  }
}

}  // namespace b2l

using namespace b2l;

extern "C" int b2l_seq_norm(const float* x, const void* w, const void* b, int kind, float eps, void* out, const int* rows, int n_rows,
                            int D, int act_dtype, b2l_stream_t stream) {
  B2L_CHECK_ARG(x && w && out, "b2l_seq_norm: null pointer");
  B2L_CHECK_ARG(kind == B2L_SEQ_NORM_RMS || kind == B2L_SEQ_NORM_LAYER, "b2l_seq_norm: unknown norm %d", kind);
  B2L_CHECK_ARG(n_rows >= 0 && D > 0, "b2l_seq_norm: bad size");
  if (n_rows == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
#define B2L_NORM_ARGS x, (const act_t*)w, (const act_t*)b, kind, eps, (act_t*)out, rows, D
  B2L_SEQ_DISPATCH(act_dtype, {
    if (D <= 1 * DEPTH_THREADS) seq_norm_kernel<act_t, 1><<<n_rows, DEPTH_THREADS, 0, s>>>(B2L_NORM_ARGS);
    else if (D <= 4 * DEPTH_THREADS) seq_norm_kernel<act_t, 4><<<n_rows, DEPTH_THREADS, 0, s>>>(B2L_NORM_ARGS);
    else if (D <= 8 * DEPTH_THREADS) seq_norm_kernel<act_t, 8><<<n_rows, DEPTH_THREADS, 0, s>>>(B2L_NORM_ARGS);
    else if (D <= 16 * DEPTH_THREADS) seq_norm_kernel<act_t, 16><<<n_rows, DEPTH_THREADS, 0, s>>>(B2L_NORM_ARGS);
    else seq_norm_wide_kernel<act_t><<<n_rows, DEPTH_THREADS, 0, s>>>(B2L_NORM_ARGS);
  });
#undef B2L_NORM_ARGS
  B2L_LAUNCH_CHECK("seq_norm_kernel");
  return 0;
}

extern "C" int b2l_seq_depth_step(const void* y1, const void* y2, const float* x_in, float* hist, int n_hist, const float* avg,
                                  float* x_out, const void* w_next, const void* b_next, int norm_kind, float eps, void* h, int T, int D,
                                  int act_dtype, b2l_stream_t stream) {
  B2L_CHECK_ARG(hist != nullptr && n_hist >= 1, "b2l_seq_depth_step: no history");
  B2L_CHECK_ARG(y1 != nullptr || y2 == nullptr, "b2l_seq_depth_step: a second result without the first");
  B2L_CHECK_ARG(y1 == nullptr || x_in != nullptr, "b2l_seq_depth_step: results without the layer's input");
  B2L_CHECK_ARG((w_next == nullptr) == (h == nullptr) && (w_next != nullptr || b_next == nullptr), "b2l_seq_depth_step: a norm needs its weight and its output");
  B2L_CHECK_ARG(norm_kind == B2L_SEQ_NORM_RMS || norm_kind == B2L_SEQ_NORM_LAYER, "b2l_seq_depth_step: unknown norm %d", norm_kind);
  B2L_CHECK_ARG(T >= 0 && D > 0, "b2l_seq_depth_step: bad size");
  B2L_CHECK_SUPPORTED(D <= 16 * DEPTH_THREADS, "b2l_seq_depth_step: width %d above %d", D, 16 * DEPTH_THREADS);
  if (T == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
#define B2L_DEPTH_ARGS (const act_t*)y1, (const act_t*)y2, x_in, hist, n_hist, avg, x_out, (const act_t*)w_next, (const act_t*)b_next, norm_kind, eps, (act_t*)h, T, D
  B2L_SEQ_DISPATCH(act_dtype, {
    if (D <= 1 * DEPTH_THREADS) seq_depth_step_kernel<act_t, 1><<<T, DEPTH_THREADS, 0, s>>>(B2L_DEPTH_ARGS);
    else if (D <= 4 * DEPTH_THREADS) seq_depth_step_kernel<act_t, 4><<<T, DEPTH_THREADS, 0, s>>>(B2L_DEPTH_ARGS);
    else if (D <= 8 * DEPTH_THREADS) seq_depth_step_kernel<act_t, 8><<<T, DEPTH_THREADS, 0, s>>>(B2L_DEPTH_ARGS);
    else seq_depth_step_kernel<act_t, 16><<<T, DEPTH_THREADS, 0, s>>>(B2L_DEPTH_ARGS);
  });
#undef B2L_DEPTH_ARGS
  B2L_LAUNCH_CHECK("seq_depth_step_kernel");
  return 0;
}

extern "C" int b2l_seq_unary_act(const void* in, int ldin, void* out, int ldout, int T, int F, int act, const float* coef, int act_dtype,
                                 b2l_stream_t stream) {
  B2L_CHECK_ARG(in && out, "b2l_seq_unary_act: null pointer");
  B2L_CHECK_ARG(T >= 0 && F > 0 && ldin >= F && ldout >= F, "b2l_seq_unary_act: bad size");
  B2L_CHECK_ARG(act == B2L_SEQ_ACT_GELU_TANH || act == B2L_SEQ_ACT_SILU || act == B2L_SEQ_ACT_SIGMOID || act == B2L_SEQ_ACT_XIELU ||
                act == B2L_SEQ_ACT_RELU2,
                "b2l_seq_unary_act: unknown activation %d", act);
  B2L_CHECK_ARG(act != B2L_SEQ_ACT_XIELU || coef != nullptr, "b2l_seq_unary_act: xIELU without its two coefficients");
  if (T == 0) return 0;
  B2L_SEQ_DISPATCH(act_dtype, {
    const int per = 16 / (int)sizeof(act_t);
    const bool vec = F % per == 0 && ldin % per == 0 && ldout % per == 0 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0;
    if (vec) {
      dim3 grid((unsigned)T, (unsigned)std::min((F / per + 255) / 256, 64));
      seq_unary_act_vec_kernel<act_t><<<grid, 256, 0, (cudaStream_t)stream>>>((const act_t*)in, ldin, (act_t*)out, ldout, F, act, coef);
    } else {
      dim3 grid((unsigned)T, (unsigned)std::min((F + 255) / 256, 64));
      seq_unary_act_kernel<act_t><<<grid, 256, 0, (cudaStream_t)stream>>>((const act_t*)in, ldin, (act_t*)out, ldout, F, act, coef);
    }
  });
  B2L_LAUNCH_CHECK("seq_unary_act_kernel");
  return 0;
}

extern "C" int b2l_seq_residual_step(const b2l_seq_residual_args* a, b2l_stream_t stream) {
  B2L_CHECK_ARG(a != nullptr && a->x_in != nullptr, "b2l_seq_residual_step: null pointer");
  B2L_CHECK_ARG(a->y1 != nullptr || a->y2 == nullptr, "b2l_seq_residual_step: a second result without the first");
  B2L_CHECK_ARG((a->w == nullptr) == (a->h == nullptr) && (a->w != nullptr || a->b == nullptr), "b2l_seq_residual_step: a norm needs its weight and its output");
  B2L_CHECK_ARG(a->norm_kind == B2L_SEQ_NORM_RMS || a->norm_kind == B2L_SEQ_NORM_LAYER, "b2l_seq_residual_step: unknown norm %d", a->norm_kind);
  B2L_CHECK_ARG(a->T >= 0 && a->D > 0, "b2l_seq_residual_step: bad size");
  if (a->T == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int D = a->D;
  const bool aligned = D % 4 == 0 && ((((uintptr_t)a->y1 | (uintptr_t)a->y2 | (uintptr_t)a->vec | (uintptr_t)a->base | (uintptr_t)a->x_in | (uintptr_t)a->x_out |
                                         (uintptr_t)a->split | (uintptr_t)a->w | (uintptr_t)a->b | (uintptr_t)a->h) & 15) == 0);
#define B2L_RES(VEC, EPT) seq_residual_step_kernel<act_t, VEC, EPT><<<a->T, DEPTH_THREADS, 0, s>>>(*a)
  B2L_SEQ_DISPATCH(a->act_dtype, {
    if (aligned && D > DEPTH_THREADS && D <= 32 * DEPTH_THREADS) {
      if (D <= 4 * DEPTH_THREADS) B2L_RES(4, 1);
      else if (D <= 8 * DEPTH_THREADS) B2L_RES(4, 2);
      else if (D <= 16 * DEPTH_THREADS) B2L_RES(4, 4);
      else B2L_RES(4, 8);
    } else if (D <= DEPTH_THREADS) B2L_RES(1, 1);
    else if (D <= 4 * DEPTH_THREADS) B2L_RES(1, 4);
    else if (D <= 16 * DEPTH_THREADS) B2L_RES(1, 16);
    else {
      B2L_CHECK_SUPPORTED(a->x_out != nullptr, "b2l_seq_residual_step: rows of %d entries need x_out", D);
      seq_residual_step_wide_kernel<act_t><<<a->T, DEPTH_THREADS, 0, s>>>(*a);
    }
  });
#undef B2L_RES
  B2L_LAUNCH_CHECK("seq_residual_step_kernel");
  return 0;
}

extern "C" int b2l_seq_linear_few(const void* w, const float* x, const float* base, const void* vec, float* out, int T, int N, int K, int act_dtype,
                                  b2l_stream_t stream) {
  B2L_CHECK_ARG(w && x && out && x != out, "b2l_seq_linear_few: null pointer, or the output is the input");
  B2L_CHECK_ARG(T >= 0 && N > 0 && K > 0, "b2l_seq_linear_few: bad size");
  const size_t smem = sizeof(float) * (size_t)K;
  B2L_CHECK_SUPPORTED(smem <= 200 * 1024, "b2l_seq_linear_few: rows of %d entries are too long", K);
  if (T == 0) return 0;
  B2L_SEQ_DISPATCH(act_dtype, {
    constexpr int PER = 16 / sizeof(act_t);
    const int rc = ensure_dyn_smem(seq_linear_few_kernel<act_t>, smem, g_few_smem[sizeof(act_t) == 2 ? 0 : 1]);
    if (rc != 0) return rc;
    seq_linear_few_kernel<act_t><<<dim3(T, (N + 7) / 8), 256, smem, (cudaStream_t)stream>>>((const act_t*)w, x, base, (const act_t*)vec, out, N, K,
                                                                                            K % PER == 0 && al16(w));
  });
  B2L_LAUNCH_CHECK("seq_linear_few_kernel");
  return 0;
}
