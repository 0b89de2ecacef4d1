// Matrix memory with exponential gates (mLSTM): per head a matrix S [K x V], a normaliser n [K] and a running maximum m
// of the log gates; S and n are kept divided by exp(m), so every factor below is at most 1.
//   portions: the gate kernel turns the two gate projections into keep = exp(log_f + m' - m), put = exp(log_i - m) and
//     exp(-m) per token (a scan with (max, +) over the portion), the framework's scan kernel runs the recurrence with
//     n as a column of ones beside the value columns, and the read-out kernel divides, normalises, gates and stores;
//   a single token: one launch.  A cluster of CTAs owns a head, each CTA a range of value columns; S streams through the
//     CTA once (read, advanced, read out against q, written), the head's root mean square is summed through distributed
//     shared memory.
// All arithmetic is f32; only the weights, biases and the output have the storage type.
#include "seq_common.cuh"

namespace b2l {

__device__ __forceinline__ float soft_cap_f(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <typename act_t>
__device__ __forceinline__ void log_gates(const b2l_seq_mlstm_args& a, int t, int h, float& li, float& lf) {
  const float* row = a.proj + (size_t)t * a.ld;
  li = soft_cap_f(row[a.i_off + h] + (a.b_i ? ld_act((const act_t*)a.b_i, h) : 0.f), a.gate_cap);
  lf = log_sigmoid_f(soft_cap_f(row[a.f_off + h] + (a.b_f ? ld_act((const act_t*)a.b_f, h) : 0.f), a.gate_cap));
}

// ---- gates of a portion: one CTA per head, tiles of GATE_THREADS * GATE_E tokens.  A run of tokens maps m to
// max(m + add, top); the maps compose associatively: a thread composes its GATE_E tokens, the CTA scans the threads'
// maps, and every thread replays its own tokens from its start.  The first token of a thread takes the m before it as its
// neighbour wrote it, so keep is always the quotient of the two stored maxima whatever their last bits are.
constexpr int GATE_THREADS = 256, GATE_E = 4;

template <typename act_t>
__global__ void __launch_bounds__(GATE_THREADS) seq_mlstm_gates_kernel(b2l_seq_mlstm_args a) {
  __shared__ float w_add[GATE_THREADS / 32], w_top[GATE_THREADS / 32], ends[GATE_THREADS + 1];
  const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* sm = a.state_m + (size_t)a.meta[0] * a.heads + h;
  float carry = *sm;                                   // m before the tile
  for (int t0 = 0; t0 < a.T; t0 += GATE_THREADS * GATE_E) {
    const int mine = t0 + tid * GATE_E, n = max(0, min(GATE_E, a.T - mine));
    float li[GATE_E], lf[GATE_E];
#pragma unroll
    for (int e = 0; e < GATE_E; ++e) {
      li[e] = -INFINITY;                               // beyond the portion: the identity map
      lf[e] = 0.f;
      if (e < n) log_gates<act_t>(a, mine + e, h, li[e], lf[e]);
    }
    float add = 0.f, top = -INFINITY;
#pragma unroll
    for (int e = 0; e < GATE_E; ++e) {
      add += lf[e];
      top = fmaxf(top + lf[e], li[e]);
    }
    float ia = add, it = top;                          // inclusive scan over the warp
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, ia, o), pt = __shfl_up_sync(0xffffffffu, it, o);
      if (lane >= o) {
        it = fmaxf(pt + ia, it);
        ia = pa + ia;
      }
    }
    if (lane == 31) {
      w_add[warp] = ia;
      w_top[warp] = it;
    }
    float xa = __shfl_up_sync(0xffffffffu, ia, 1), xt = __shfl_up_sync(0xffffffffu, it, 1);
    if (lane == 0) {
      xa = 0.f;
      xt = -INFINITY;
    }
    __syncthreads();
    float m = carry;
    for (int w = 0; w < warp; ++w) m = fmaxf(m + w_add[w], w_top[w]);
    m = fmaxf(m + xa, xt);
    float ms[GATE_E];
    {
      float r = m;
#pragma unroll
      for (int e = 0; e < GATE_E; ++e) {
        r = fmaxf(lf[e] + r, li[e]);
        ms[e] = r;
      }
      ends[tid + 1] = r;
      if (tid == 0) ends[0] = carry;
    }
    __syncthreads();
    float prev = ends[tid];
#pragma unroll
    for (int e = 0; e < GATE_E; ++e) {
      if (e < n) {
        const size_t at = (size_t)(mine + e) * a.heads + h;
        a.keep[at] = expf(lf[e] + prev - ms[e]);
        a.put[at] = expf(li[e] - ms[e]);
        a.floor[at] = expf(-ms[e]);
      }
      prev = ms[e];
    }
    carry = ends[GATE_THREADS];
    __syncthreads();                                   // ends, w_add and w_top are reused by the next tile
  }
  if (tid == 0) *sm = carry;
}

// ---- read-out of a portion: one warp per (token, head), the head's values in registers.
constexpr int RO_MAX = 16;             // values per lane: V <= 512 (larger heads re-read)

template <typename act_t>
__global__ void __launch_bounds__(128) seq_mlstm_readout_kernel(b2l_seq_mlstm_args a) {
  const int id = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (id >= a.T * a.heads) return;
  const int t = id / a.heads, h = id - t * a.heads, V = a.V;
  const float* o = a.o + (size_t)t * a.ldr + (size_t)h * V;
  const float* g = a.proj + (size_t)t * a.ld + a.g_off + (size_t)h * V;
  const act_t* w = (const act_t*)a.w_norm + (size_t)h * V;
  act_t* out = (act_t*)a.out + (size_t)t * a.ldo + (size_t)h * V;
  const float inv = 1.f / (fmaxf(fabsf(a.nq[id]), a.floor[id]) + a.den_add);
  float v[RO_MAX], ss = 0.f;
#pragma unroll
  for (int c = 0; c < RO_MAX; ++c) {
    const int i = c * 32 + lane;
    v[c] = i < V ? o[i] * inv : 0.f;
    ss += v[c] * v[c];
  }
  for (int i = RO_MAX * 32 + lane; i < V; i += 32) {
    const float x = o[i] * inv;
    ss += x * x;
  }
  ss = warp_sum(ss);
  const float r = 1.f / sqrtf(ss / (float)V + a.eps);
#pragma unroll
  for (int c = 0; c < RO_MAX; ++c) {
    const int i = c * 32 + lane;
    if (i < V) st_act(out, i, v[c] * r * ld_act(w, i) * sigmoid_f(g[i]));
  }
  for (int i = RO_MAX * 32 + lane; i < V; i += 32) st_act(out, i, o[i] * inv * r * ld_act(w, i) * sigmoid_f(g[i]));
}

// ---- a single token: cluster = one head, CTA rank r = value columns [r * per, (r + 1) * per).
constexpr int STEP_THREADS = 512, STEP_CLUSTER = 8, STEP_U = 4;      // STEP_THREADS: the most a CTA gets

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire;" ::: "memory"); }
__device__ __forceinline__ void store_to_rank(float* local, int rank, float v) {
  unsigned at = (unsigned)__cvta_generic_to_shared(local), remote;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(at), "r"(rank));
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
}

// G lanes share a column of S (4 entries each per round when VEC, else one), 32 / G columns per warp and round.
template <typename act_t, bool VEC>
__global__ void __launch_bounds__(STEP_THREADS) seq_mlstm_step_kernel(b2l_seq_mlstm_args a, int per, int G) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32], part[STEP_CLUSTER];
  const int rank = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, threads = blockDim.x;
  const int K = a.K, V = a.V, Kp = (K + 3) & ~3, slot = a.meta[0];
  float* sq = smem;                                    // [Kp] q times q_mult
  float* sk = sq + Kp;                                 // [Kp] put * k
  float* so = sk + Kp;                                 // [per] read-outs of this CTA's columns
  cluster_arrive();                                    // every CTA of the cluster has started before shared memory is written across
  const float* row = a.proj;
  float li, lf;
  log_gates<act_t>(a, 0, h, li, lf);
  float* pm = a.state_m + (size_t)slot * a.heads + h;
  const float m0 = *pm, m = fmaxf(lf + m0, li), keep = expf(lf + m0 - m), put = expf(li - m);

  float* pn = a.state_n + ((size_t)slot * a.heads + h) * K;
  float nq = 0.f;
  for (int i = tid; i < Kp; i += threads) {
    const float q = i < K ? row[a.q_off + (size_t)h * K + i] * a.q_mult : 0.f;
    const float k = i < K ? put * row[a.k_off + (size_t)h * K + i] : 0.f;
    sq[i] = q;
    sk[i] = k;
    if (i < K) nq = fmaf(fmaf(keep, pn[i], k), q, nq);
  }
  nq = block_sum(nq, red);                             // its barriers also publish sq and sk
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + a.den_add);

  const int c0 = rank * per, nc = max(0, min(per, V - c0));
  float* S = a.state_S + (((size_t)slot * a.heads + h) * V + c0) * K;
  const float* v = row + a.v_off + (size_t)h * V + c0;
  // A lane group owns column cb + sub; STEP_U columns, cpw * warps apart, are in flight at once.
  const int cpw = 32 / G, sub = lane / G, r = lane - sub * G, stride = (threads >> 5) * cpw;
  for (int cb = warp * cpw; cb < nc; cb += stride * STEP_U) {
    float dot[STEP_U], vc[STEP_U];
    float* Sc[STEP_U];
    bool on[STEP_U];
#pragma unroll
    for (int u = 0; u < STEP_U; ++u) {
      const int c = cb + sub + u * stride;
      on[u] = c < nc;
      vc[u] = on[u] ? v[c] : 0.f;
      Sc[u] = S + (size_t)(on[u] ? c : 0) * K;
      dot[u] = 0.f;
    }
    if (VEC) {
      for (int i = r * 4; i < K; i += G * 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(sk + i), q4 = *reinterpret_cast<const float4*>(sq + i);
        float4 s[STEP_U];
#pragma unroll
        for (int u = 0; u < STEP_U; ++u) s[u] = on[u] ? *reinterpret_cast<const float4*>(Sc[u] + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < STEP_U; ++u) {
          s[u].x = fmaf(keep, s[u].x, k4.x * vc[u]); s[u].y = fmaf(keep, s[u].y, k4.y * vc[u]);
          s[u].z = fmaf(keep, s[u].z, k4.z * vc[u]); s[u].w = fmaf(keep, s[u].w, k4.w * vc[u]);
          if (on[u]) *reinterpret_cast<float4*>(Sc[u] + i) = s[u];
          dot[u] = fmaf(s[u].x, q4.x, dot[u]); dot[u] = fmaf(s[u].y, q4.y, dot[u]);
          dot[u] = fmaf(s[u].z, q4.z, dot[u]); dot[u] = fmaf(s[u].w, q4.w, dot[u]);
        }
      }
    } else {
      for (int i = r; i < K; i += G) {
#pragma unroll
        for (int u = 0; u < STEP_U; ++u) {
          if (on[u]) {
            const float s = fmaf(keep, Sc[u][i], sk[i] * vc[u]);
            Sc[u][i] = s;
            dot[u] = fmaf(s, sq[i], dot[u]);
          }
        }
      }
    }
    for (int o = 1; o < G; o <<= 1) {
#pragma unroll
      for (int u = 0; u < STEP_U; ++u) dot[u] += __shfl_xor_sync(0xffffffffu, dot[u], o);
    }
#pragma unroll
    for (int u = 0; u < STEP_U; ++u)
      if (r == 0 && on[u]) so[cb + sub + u * stride] = dot[u] * inv;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < nc; c += threads) ss += so[c] * so[c];
  ss = block_sum(ss, red);
  cluster_wait();
  if (tid < (int)gridDim.x) store_to_rank(part + rank, tid, ss);
  cluster_arrive();
  cluster_wait();                                      // all sums have arrived; m and n have been read by every CTA
  if (rank == 0) {
    for (int i = tid; i < K; i += threads) pn[i] = fmaf(keep, pn[i], sk[i]);
    if (tid == 0) *pm = m;
  }
  ss = 0.f;
  for (int i = 0; i < (int)gridDim.x; ++i) ss += part[i];
  const float rr = 1.f / sqrtf(ss / (float)V + a.eps);
  const float* g = row + a.g_off + (size_t)h * V + c0;
  const act_t* w = (const act_t*)a.w_norm + (size_t)h * V + c0;
  for (int c = tid; c < nc; c += threads) st_act((act_t*)a.out, (size_t)h * V + c0 + c, so[c] * rr * ld_act(w, c) * sigmoid_f(g[c]));
}

static DynSmemCache g_step_smem[4];

template <typename act_t, bool VEC>
static int launch_step(const b2l_seq_mlstm_args* a, int per, int C, int G, int threads, size_t smem, cudaStream_t s, DynSmemCache& cache) {
  int rc = ensure_dyn_smem(seq_mlstm_step_kernel<act_t, VEC>, smem, cache);
  if (rc) return rc;
  LaunchCfg cfg(dim3((unsigned)C, (unsigned)a->heads), dim3((unsigned)threads), smem, s, false, C);
  B2L_CUDA(cudaLaunchKernelEx(&cfg.cfg, seq_mlstm_step_kernel<act_t, VEC>, *a, per, G));
  return 0;
}

static int check_mlstm(const b2l_seq_mlstm_args* a, const char* what) {
  B2L_CHECK_ARG(a != nullptr, "%s: null argument block", what);
  B2L_CHECK_ARG(a->T >= 0 && a->heads > 0 && a->K > 0 && a->V > 0 && a->ld > 0, "%s: bad size", what);
  B2L_CHECK_ARG(a->gate_cap > 0.f && a->den_add >= 0.f, "%s: the gate cap must be positive", what);
  B2L_CHECK_ARG(a->proj && a->meta && a->state_m, "%s: null pointer", what);
  B2L_CHECK_ARG(a->i_off >= 0 && a->i_off + a->heads <= a->ld && a->f_off >= 0 && a->f_off + a->heads <= a->ld, "%s: gate columns outside the projection", what);
  B2L_CHECK_ARG(a->g_off >= 0 && a->g_off + a->heads * a->V <= a->ld, "%s: output gate outside the projection", what);
  return 0;
}

}  // namespace b2l

using namespace b2l;

extern "C" int b2l_seq_mlstm_gates(const b2l_seq_mlstm_args* a, b2l_stream_t stream) {
  int rc = check_mlstm(a, "b2l_seq_mlstm_gates");
  if (rc) return rc;
  B2L_CHECK_ARG(a->keep && a->put && a->floor, "b2l_seq_mlstm_gates: null pointer");
  if (a->T == 0) return 0;
  B2L_SEQ_DISPATCH(a->act_dtype, (seq_mlstm_gates_kernel<act_t><<<a->heads, GATE_THREADS, 0, (cudaStream_t)stream>>>(*a)));
  B2L_LAUNCH_CHECK("seq_mlstm_gates_kernel");
  return 0;
}

extern "C" int b2l_seq_mlstm_readout(const b2l_seq_mlstm_args* a, b2l_stream_t stream) {
  int rc = check_mlstm(a, "b2l_seq_mlstm_readout");
  if (rc) return rc;
  B2L_CHECK_ARG(a->o && a->nq && a->floor && a->w_norm && a->out && a->ldr >= a->heads * a->V && a->ldo >= a->heads * a->V,
                "b2l_seq_mlstm_readout: null pointer or bad size");
  if (a->T == 0) return 0;
  const int ids = a->T * a->heads;
  B2L_SEQ_DISPATCH(a->act_dtype, (seq_mlstm_readout_kernel<act_t><<<(ids + 3) / 4, 128, 0, (cudaStream_t)stream>>>(*a)));
  B2L_LAUNCH_CHECK("seq_mlstm_readout_kernel");
  return 0;
}

extern "C" int b2l_seq_mlstm_step(const b2l_seq_mlstm_args* a, b2l_stream_t stream) {
  int rc = check_mlstm(a, "b2l_seq_mlstm_step");
  if (rc) return rc;
  B2L_CHECK_ARG(a->T == 1, "b2l_seq_mlstm_step: one token, not %d", a->T);
  B2L_CHECK_ARG(a->state_S && a->state_n && a->w_norm && a->out && a->ldo >= a->heads * a->V, "b2l_seq_mlstm_step: null pointer or bad size");
  B2L_CHECK_ARG(a->q_off >= 0 && a->q_off + a->heads * a->K <= a->ld && a->k_off >= 0 && a->k_off + a->heads * a->K <= a->ld && a->v_off >= 0 &&
                a->v_off + a->heads * a->V <= a->ld, "b2l_seq_mlstm_step: q, k or v outside the projection");
  int C = 1;                                           // CTAs of the cluster: at least 16 value columns each
  while (C < STEP_CLUSTER && a->V >= 32 * C) C <<= 1;
  const int per = (a->V + C - 1) / C;
  const bool vec = a->K % 4 == 0 && ((uintptr_t)a->state_S & 15) == 0;
  const int want = vec ? (a->K + 3) / 4 : a->K;
  int G = 1;
  while (G < 32 && G < want) G <<= 1;
  // a warp takes STEP_U rounds of 32 / G columns at once
  const int threads = per * G > 32 * STEP_U * 8 ? STEP_THREADS : STEP_THREADS / 2;
  const size_t smem = sizeof(float) * (2 * (size_t)((a->K + 3) & ~3) + per);
  B2L_CHECK_SUPPORTED(smem <= 200 * 1024, "b2l_seq_mlstm_step: head of %d x %d too large", a->K, a->V);
  cudaStream_t s = (cudaStream_t)stream;
  if (a->act_dtype == B2L_BF16) {
    rc = vec ? launch_step<__nv_bfloat16, true>(a, per, C, G, threads, smem, s, g_step_smem[0]) : launch_step<__nv_bfloat16, false>(a, per, C, G, threads, smem, s, g_step_smem[1]);
  } else if (a->act_dtype == B2L_F32) {
    rc = vec ? launch_step<float, true>(a, per, C, G, threads, smem, s, g_step_smem[2]) : launch_step<float, false>(a, per, C, G, threads, smem, s, g_step_smem[3]);
  } else {
    set_error("b2l_seq_mlstm_step: act_dtype %d unsupported", a->act_dtype);
    return B2L_E_UNSUPPORTED;
  }
  if (rc) return rc;
  B2L_LAUNCH_CHECK("seq_mlstm_step_kernel");
  return 0;
}
