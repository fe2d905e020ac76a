// The gated delta rule with a decay per key channel (sm_100a), float32 and bfloat16 inputs; short convolutions' sums,
// unit norms, step sizes, decays and their logarithms, exponentials, states and all sums of the recurrence are 32-bit.
//
// Per head h (which reads q/k head g = h / (H / G)), with q, k of D and v of V elements, step size b and decays a (D):
//   q, k, v = silu(conv(u)),  conv(u)_t = sum_j w[c, j] u_(t - taps + 1 + j) per channel (u: the projection's columns, zeros
//                             before position 0),  q, k <- x / sqrt(sum(x^2) + unit_eps),  q <- q * q_scale,
//   b = sigmoid(zb),  a = exp(-exp(A_log_h) softplus(za + c)),
//   S <- diag(a) S,   u = b (v - S^T k),   S <- S + k u^T,   o = S^T q,
//   out = o / sqrt(mean(o^2) + eps) * gain * sigmoid(zg)            (mean over the head's V elements, gain [V])
// S [slots, H, D, V] is a sequence's state, moved on; so is the ring of its last `taps` projected rows
// (hist [slots, taps, 2 G D + H V]; the row of position p lies at p mod taps, so that a single token's step may write its own
// row while other blocks still read the rows before it).
//
//   delta_step_kernel     single tokens: ONE kernel, a block a (head, sequence): convolutions, norms, (optionally) the
//                         second halves of the two low-rank projections, decays, the recurrence with S in registers,
//                         output norm and gate.
//   delta_prepare_kernel  otherwise: convolutions, activations and unit norms into q, k, v (32-bit), a warp a (run of
//                         tokens, head); delta_history_kernel then moves the rings on.
//   delta_walk_kernel     short portions: a block a (head, sequence) walks the tokens with S in shared memory.
//   chunks of 32 tokens (long portions): with G_t the running sums of log a inside a chunk,
//     u_t = b_t (v_t - S_0^T (e^(G_t) k_t) - sum_(s<t) (k_t . e^(G_t - G_s) k_s) u_s)
//   is one triangular system per chunk whose right side is linear in the state S_0 at the chunk's begin:
//     delta_intra_kernel  a block a (chunk, head): the system's matrix, its solution X for the right side b e^G k and Y for
//                         b v (so u = Y - X S_0), the weights P_ts = q_t . e^(G_t - G_s) k_s (s <= t), e^(G_t) q_t,
//                         e^(G_end - G_t) k_t and e^(G_end).  No exponent is ever positive: pairs of tokens within 16 take
//                         e^(G_t - G_s) itself, pairs across take it in two factors around the border between them.
//     delta_scan_kernel   a block a (slice of V, head, sequence) walks the chunks: u = Y - X S (left in Y's place), the state
//                         at the chunk's begin (left for the next kernel), S <- diag(e^(G_end)) S + (e^(G_end - G) k)^T u.
//     delta_out_kernel    a block a (chunk, head): o = (e^G q) S_begin + P u, output norm, gain, gate.
#include "common.cuh"

#define DL_THREADS 256
#define DL_C 32                     // tokens a chunk
#define DL_LD (DL_C + 4)

__device__ __forceinline__ float dl_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float dl_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float dl_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float dl_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
#define DL_LOG2E 1.4426950408889634f
// A decay below 2^-40 empties its channel as far as 32-bit sums can tell (1e-12 of the state stays).  In the chunks the
// logarithms are cut off there, and they are summed from the begin of each half of a chunk: a difference of two running
// sums, of which decays between two tokens are made, then keeps its last bits whatever strong decays came before.
#define DL_LOG_MIN -40.f
__device__ __forceinline__ void dl_cp16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dl_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void dl_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

struct DlArgs {
  const void* proj; int row, col, b_col;     // q, k, v columns from col on (2 G D + H V of them), step sizes' from b_col on
  const float* taps_w; int taps;             // [2 G D + H V, taps]
  float* hist;                               // [slots, taps, 2 G D + H V]
  const float* z; int z_ld;                  // pre-activations: decays in columns h D + d, output gates in H D + h V + c
  const float* a_log;                        // [H]
  const float* dt_bias;                      // [H D]
  const float* gain;                         // [V]
  float q_scale, unit_eps, eps;
  float* S;                                  // [slots, H, D, V]
  void* out;                                 // [T, H V]
  const int* positions; const int* seq_of_token; const int* cu_seqlens; const int* seq_past; const int* seq_lens;
  const int* seq_slots;
  int H, G, D, V;
};

// ---------------------------------------------------------------------------------------------------------------
// convolution, activation, unit norm.  Units of a token: G query heads, G key heads (D channels each), H value heads (V).
// ---------------------------------------------------------------------------------------------------------------
struct DlPrep { float* q; float* k; float* v; };          // [T, G D], [T, G D], [T, H V]

__device__ __forceinline__ void dl_unit(const DlArgs& a, int unit, int& c0, int& n, int& kind) {
  if (unit < a.G) { c0 = unit * a.D; n = a.D; kind = 0; }
  else if (unit < 2 * a.G) { c0 = unit * a.D; n = a.D; kind = 1; }
  else { c0 = 2 * a.G * a.D + (unit - 2 * a.G) * a.V; n = a.V; kind = 2; }
}
__device__ __forceinline__ float* dl_prep_dst(const DlArgs& a, const DlPrep& w, int t, int unit, int kind) {
  const size_t gd = (size_t)a.G * a.D;
  if (kind == 0) return w.q + (size_t)t * gd + (size_t)unit * a.D;
  if (kind == 1) return w.k + (size_t)t * gd + (size_t)(unit - a.G) * a.D;
  return w.v + (size_t)t * a.H * a.V + (size_t)(unit - 2 * a.G) * a.V;
}

// any sizes: a warp a (token, unit)
template <typename T>
__global__ void __launch_bounds__(DL_THREADS) delta_prepare_kernel(DlArgs a, DlPrep w, int n_tokens) {
  pdl_wait();
  pdl_trigger();
  const int units = 2 * a.G + a.H, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (DL_THREADS / 32) + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * units) return;
  const int t = (int)(item / units), unit = (int)(item % units);
  int c0, n, kind;
  dl_unit(a, unit, c0, n, kind);
  const int s = a.seq_of_token[t], pos = a.positions[t], past = a.seq_past[s], C = 2 * a.G * a.D + a.H * a.V;
  const T* proj = (const T*)a.proj;
  const float* hs = a.hist + (size_t)a.seq_slots[s] * a.taps * C;
  float* dst = dl_prep_dst(a, w, t, unit, kind);
  float ss = 0.f;
  for (int i = lane; i < n; i += 32) {
    const int c = c0 + i;
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
      const int p = pos - a.taps + 1 + j;
      if (p < 0) continue;
      const float u = p >= past ? to_f32(proj[(size_t)(t - (pos - p)) * a.row + a.col + c]) : hs[(size_t)(p % a.taps) * C + c];
      acc = fmaf(a.taps_w[(size_t)c * a.taps + j], u, acc);
    }
    const float y = dl_silu(acc);
    dst[i] = y;
    ss += y * y;
  }
  if (kind == 2) return;
  const float f = rsqrtf(warp_sum(ss) + a.unit_eps) * (kind == 0 ? a.q_scale : 1.f);
  for (int i = lane; i < n; i += 32) dst[i] *= f;            // a lane reads what it wrote itself
}

// N = 32 * CPL channels a unit, TAPS known: a warp a (run of DL_RUN tokens, unit), a lane CPL neighbouring channels, the
// rows before a token kept in registers
#define DL_RUN 8
template <int CPL> __device__ __forceinline__ void dl_ld_f32(const float* p, float (&v)[CPL]) {
  if (CPL % 4 == 0) {
#pragma unroll
    for (int i = 0; i < CPL / 4; ++i) {
      const float4 f = reinterpret_cast<const float4*>(p)[i];
      v[4 * i] = f.x; v[(4 * i + 1) % CPL] = f.y; v[(4 * i + 2) % CPL] = f.z; v[(4 * i + 3) % CPL] = f.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < CPL; ++i) v[i] = p[i];
  }
}
template <typename T, int CPL> struct DlLd;
template <int CPL> struct DlLd<float, CPL> {
  static __device__ __forceinline__ void go(const float* p, float (&v)[CPL]) { dl_ld_f32<CPL>(p, v); }
};
template <int CPL> struct DlLd<bf16, CPL> {
  static __device__ __forceinline__ void go(const bf16* p, float (&v)[CPL]) {
    if (CPL == 4) {
      const uint2 u = *reinterpret_cast<const uint2*>(p);
      const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&u.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
      v[0] = __low2float(lo); v[1 % CPL] = __high2float(lo); v[2 % CPL] = __low2float(hi); v[3 % CPL] = __high2float(hi);
    } else {
#pragma unroll
      for (int i = 0; i < CPL; ++i) v[i] = __bfloat162float(p[i]);
    }
  }
};

// the activation where the result is rounded to 16 bits' worth anyway (bfloat16 projections), and the precise one
template <typename T> __device__ __forceinline__ float dl_silu_of(float z);
template <> __device__ __forceinline__ float dl_silu_of<float>(float z) { return dl_silu(z); }
template <> __device__ __forceinline__ float dl_silu_of<bf16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }

template <typename T, int CPL, int TAPS>
__device__ __forceinline__ void dl_prepare_run(const DlArgs& a, const DlPrep& w, int t0, int t1, int unit, int c0, int kind, int lane) {
  const int C = 2 * a.G * a.D + a.H * a.V, c = c0 + lane * CPL;
  const T* src = (const T*)a.proj + a.col + c;
  float wt[CPL][TAPS], win[TAPS][CPL];            // win[j]: the row that tap j reads
  float raw[DL_RUN][CPL];                         // the run's rows, all asked for at once
#pragma unroll
  for (int r = 0; r < DL_RUN; ++r) DlLd<T, CPL>::go(src + (size_t)min(t0 + r, t1 - 1) * a.row, raw[r]);
  const int s = a.seq_of_token[t0], pos = a.positions[t0], past = a.seq_past[s];
  const float* hs = a.hist + (size_t)a.seq_slots[s] * TAPS * C + c;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int p = pos - TAPS + 1 + j;             // goes to place j + 1: the shift below brings it to place j
    if (p < 0) {
#pragma unroll
      for (int i = 0; i < CPL; ++i) win[j + 1][i] = 0.f;
    } else if (p >= past) {
      DlLd<T, CPL>::go(src + (size_t)(t0 - (pos - p)) * a.row, win[j + 1]);
    } else {
      dl_ld_f32<CPL>(hs + (size_t)(p % TAPS) * C, win[j + 1]);
    }
  }
#pragma unroll
  for (int i = 0; i < CPL; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[i][j] = a.taps_w[(size_t)(c + i) * TAPS + j];
  float* dst = dl_prep_dst(a, w, t0, unit, kind) + lane * CPL;
  const size_t ld = kind == 2 ? (size_t)a.H * a.V : (size_t)a.G * a.D;
#pragma unroll
  for (int r = 0; r < DL_RUN; ++r) {
    if (t0 + r >= t1) break;
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int i = 0; i < CPL; ++i) win[j][i] = win[j + 1][i];
#pragma unroll
    for (int i = 0; i < CPL; ++i) win[TAPS - 1][i] = raw[r][i];
    float y[CPL], ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[i][j], win[j][i], acc);
      y[i] = dl_silu_of<T>(acc);
      ss += y[i] * y[i];
    }
    if (kind != 2) {
      const float f = rsqrtf(warp_sum(ss) + a.unit_eps) * (kind == 0 ? a.q_scale : 1.f);
#pragma unroll
      for (int i = 0; i < CPL; ++i) y[i] *= f;
    }
    if (CPL % 4 == 0) {
#pragma unroll
      for (int i = 0; i < CPL / 4; ++i)
        reinterpret_cast<float4*>(dst)[i] = make_float4(y[4 * i], y[(4 * i + 1) % CPL], y[(4 * i + 2) % CPL], y[(4 * i + 3) % CPL]);
    } else {
#pragma unroll
      for (int i = 0; i < CPL; ++i) dst[i] = y[i];
    }
    dst += ld;
  }
}

// WIDE: some heads have 256 channels
template <typename T, int TAPS, bool WIDE>
__global__ void __launch_bounds__(DL_THREADS) delta_prepare_run_kernel(DlArgs a, DlPrep w, int n_tokens) {
  pdl_wait();
  pdl_trigger();
  const int unit = blockIdx.y * (DL_THREADS / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= 2 * a.G + a.H) return;
  const int begin = blockIdx.x * DL_RUN, end = min(n_tokens, begin + DL_RUN);
  int c0, n, kind;
  dl_unit(a, unit, c0, n, kind);
  // a run that lies in one sequence goes through whole, others in stretches of a sequence each
  for (int t0 = begin; t0 < end;) {
    const int t1 = min(end, a.cu_seqlens[a.seq_of_token[t0] + 1]);
    switch (n) {
      case 32: dl_prepare_run<T, 1, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
      case 64: dl_prepare_run<T, 2, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
      case 128: dl_prepare_run<T, 4, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
      default: if (WIDE) dl_prepare_run<T, 8, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
    }
    t0 = t1;
  }
}

// the rings after the portion: a thread a channel of a sequence
template <typename T>
__global__ void __launch_bounds__(256) delta_history_kernel(DlArgs a) {
  pdl_wait();
  pdl_trigger();
  const int C = 2 * a.G * a.D + a.H * a.V, s = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C) return;
  const int past = a.seq_past[s], len = a.seq_lens[s], t0 = a.cu_seqlens[s];
  float* hs = a.hist + (size_t)a.seq_slots[s] * a.taps * C + c;
  const T* proj = (const T*)a.proj + a.col + c;
  for (int p = max(past, len - a.taps); p < len; ++p) hs[(size_t)(p % a.taps) * C] = to_f32(proj[(size_t)(t0 + p - past) * a.row]);
}

// ---------------------------------------------------------------------------------------------------------------
// token by token: a block a (head, sequence).  One pass over S a token: the write of the token before is applied on the
// way (S <- a (S + k_prev u_prev^T)), and o = S'^T q + (k . q) u needs no second pass.
// ---------------------------------------------------------------------------------------------------------------
template <typename TP, typename TO>
__global__ void __launch_bounds__(DL_THREADS) delta_walk_kernel(DlArgs a, DlPrep w, int in_place) {
  extern __shared__ float sm[];
  const int D = a.D, V = a.V, H = a.H;
  constexpr int NW = DL_THREADS / 32;
  float* S = sm;
  float* q = in_place ? sm : S + D * V;
  float* k = q + D;
  float* g = k + D;
  float* kp = g + D;                 // the token before: its key
  float* up = kp + D;                // its update u
  float* pr = up + V;                // NW * V: partial S'^T k
  float* pp = pr + NW * V;           // NW * V: partial S'^T q
  __shared__ float red[33];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = h / (H / a.G);
  const int t0 = a.cu_seqlens[s], t1 = a.cu_seqlens[s + 1];
  float* Sg = a.S + ((size_t)a.seq_slots[s] * H + h) * D * V;
  if (in_place) S = Sg;
  else
    for (int i = tid; i < D * V; i += DL_THREADS) S[i] = Sg[i];
  for (int i = tid; i < D; i += DL_THREADS) kp[i] = 0.f;
  for (int i = tid; i < V; i += DL_THREADS) up[i] = 0.f;
  const float ea = expf(a.a_log[h]);
  __syncthreads();
  for (int t = t0; t < t1; ++t) {
    float kq = 0.f;
    for (int i = tid; i < D; i += DL_THREADS) {
      const float qi = w.q[(size_t)t * a.G * D + gq * D + i], ki = w.k[(size_t)t * a.G * D + gq * D + i];
      q[i] = qi; k[i] = ki;
      kq = fmaf(qi, ki, kq);
      g[i] = expf(-ea * dl_softplus(a.z[(size_t)t * a.z_ld + h * D + i] + a.dt_bias[h * D + i]));
    }
    const float beta = dl_sigmoid(to_f32(((const TP*)a.proj)[(size_t)t * a.row + a.b_col + h]));
    kq = block_sum(kq, red);                       // also orders q, k, g before the reads below
    for (int c0 = 0; c0 < V; c0 += 32) {
      const int c = c0 + lane;
      if (c < V) {
        const float uc = up[c];
        float r = 0.f, p = 0.f;
        for (int d = warp; d < D; d += NW) {
          const float x = g[d] * fmaf(kp[d], uc, S[d * V + c]);
          S[d * V + c] = x;
          r = fmaf(x, k[d], r);
          p = fmaf(x, q[d], p);
        }
        pr[warp * V + c] = r;
        pp[warp * V + c] = p;
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < V; c += DL_THREADS) {
      float r = 0.f, p = 0.f;
#pragma unroll
      for (int x = 0; x < NW; ++x) { r += pr[x * V + c]; p += pp[x * V + c]; }
      const float u = beta * (w.v[(size_t)t * H * V + h * V + c] - r);
      up[c] = u;
      const float o = fmaf(kq, u, p);
      pp[c] = o;                                   // this thread's column of the first partial row: read by nobody else
      ss += o * o;
    }
    for (int i = tid; i < D; i += DL_THREADS) kp[i] = k[i];
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)V + a.eps);
    for (int c = tid; c < V; c += DL_THREADS)
      ((TO*)a.out)[(size_t)t * H * V + h * V + c] =
          from_f32<TO>(pp[c] * inv * a.gain[c] * dl_sigmoid(a.z[(size_t)t * a.z_ld + H * D + h * V + c]));
    __syncthreads();
  }
  for (int i = tid; i < D * V; i += DL_THREADS) Sg[i] = fmaf(kp[i / V], up[i % V], S[i]);
}

static size_t dl_walk_smem(int D, int V, bool in_place) {
  return (size_t)((in_place ? 0 : D * V) + 4 * D + V + 2 * (DL_THREADS / 32) * V) * sizeof(float);
}

// ---------------------------------------------------------------------------------------------------------------
// single tokens: everything behind the stacked projection in one kernel.  V a power of two from 4 to 256: the row of S is
// V / 4 float4, a thread owns one of them in rows r0, r0 + RP, ... (RP = 1024 / V rows a pass, NI passes).
// low rank: the second halves of the two low-rank projections run here: wz [H D + H V, ra + rg] (row h D + d: a2 in the
// first ra columns; row H D + h V + c: g2 in the last rg), their inputs in the projection's columns lr_col .. + ra + rg.
// staged: this head's rows of it come to shared memory (rows of max(ra, rg) padded to whole 16-byte pieces) ahead of the wait.
// What no kernel of this layer's chain has written (the state, the ring's earlier rows, constants) is asked for ahead of
// the wait for the kernel before; the state and the ring were written a step (many launches) ago.
// ---------------------------------------------------------------------------------------------------------------
struct DlLowRank { const void* wz; int ra, rg, lr_col, staged; };

template <typename TW> __host__ __device__ __forceinline__ int dl_lr_ld(int ra, int rg) {
  const int m = ra > rg ? ra : rg, q = 16 / (int)sizeof(TW);
  return (m + q - 1) / q * q;
}

// rows dot x: 8 lanes a row, 16-byte loads where the row's start and length allow
template <typename TW>
__device__ __forceinline__ float dl_row_dot(const TW* wr, const float* x, int n, int sub, bool vec) {
  float acc = 0.f;
  constexpr int VE = 16 / sizeof(TW);
  if (vec) {
#pragma unroll 2
    for (int e = sub * VE; e < n; e += 8 * VE) {
      if (sizeof(TW) == 2) {
        const uint4 u = *reinterpret_cast<const uint4*>(wr + e);
        const __nv_bfloat162* hp = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(hp[i]);
          acc = fmaf(f.x, x[e + 2 * i], acc);
          acc = fmaf(f.y, x[e + 2 * i + 1], acc);
        }
      } else {
        const float4 f = *reinterpret_cast<const float4*>(wr + e);
        acc = fmaf(f.x, x[e], fmaf(f.y, x[e + 1], fmaf(f.z, x[e + 2], fmaf(f.w, x[e + 3], acc))));
      }
    }
  } else {
    for (int e = sub; e < n; e += 8) acc = fmaf(to_f32(wr[e]), x[e], acc);
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  return acc;
}

#define DL_STEP_CH 4                 // convolved channels a thread: 2 D + V <= 1024

template <typename TP, typename TO, int NI>
__global__ void __launch_bounds__(DL_THREADS, NI <= 16 ? 2 : 1) delta_step_kernel(DlArgs a, DlLowRank lr) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.D, V = a.V, H = a.H, G = a.G;
  float* q = sm;                     // D
  float* k = q + D;                  // D
  float* g = k + D;                  // D: decays
  float* v = g + D;                  // V
  float* og = v + V;                 // V: output gates (after the sigmoid)
  float* xs = og + V;                // ra + rg
  float* pr = sm + ((3 * D + 2 * V + lr.ra + lr.rg + 3) & ~3);       // 1024: RP rows of V partial sums
  float* pp = pr + 1024;             // 1024
  float* us = pp + 1024;             // V: updates
  TO* wsm = (TO*)(us + V);           // (D + V) rows, if staged
  __shared__ float red[33];
  __shared__ float sc[3];
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int V4 = V >> 2, RP = 1024 / V, c4 = (tid % V4) * 4, r0 = tid / V4;
  const int slot = a.seq_slots[s];
  float* Sg = a.S + ((size_t)slot * H + h) * D * V + c4;
  float4 S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = r0 + i * RP;
    S[i] = d < D ? *reinterpret_cast<const float4*>(Sg + (size_t)d * V) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const TO* wz = (const TO*)lr.wz;
  constexpr int VE = 16 / sizeof(TO);
  const int ld = lr.ra + lr.rg, wld = dl_lr_ld<TO>(lr.ra, lr.rg);
  if (lr.staged) {
    const int pa = lr.ra / VE, pg = lr.rg / VE;
    const int sub = lane & 15;                       // half a warp a row
#pragma unroll 4
    for (int r = warp * 2 + (lane >> 4); r < D + V; r += DL_THREADS / 16) {
      const bool dec = r < D;
      const TO* wr = dec ? wz + (size_t)(h * D + r) * ld : wz + (size_t)(H * D + h * V + (r - D)) * ld + lr.ra;
      for (int e = sub; e < (dec ? pa : pg); e += 16) dl_cp16((float*)(wsm + r * wld + e * VE), (const float*)(wr + e * VE));
    }
  }
  dl_commit();
  const int rep = H / G, gq = h / rep, t = s, pos = a.positions[t], taps = a.taps;
  const int C = 2 * G * D + H * V, GD = G * D;
  float* hs = a.hist + (size_t)slot * taps * C;
  // the rows before this one: the loads of up to four of them all on their way before any is used
  float past[DL_STEP_CH], w_now[DL_STEP_CH], hr[DL_STEP_CH][4], hw[DL_STEP_CH][4];
  int ring[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int p = pos - 1 - j;                       // j + 1 rows back, tap taps - 2 - j
    ring[j] = (j < taps - 1 && p >= 0) ? p % taps : -1;
  }
#pragma unroll
  for (int x = 0; x < DL_STEP_CH; ++x) {
    const int i = tid + x * DL_THREADS;
    w_now[x] = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) hr[x][j] = hw[x][j] = 0.f;
    if (i < 2 * D + V) {
      const int c = i < D ? gq * D + i : (i < 2 * D ? GD + gq * D + (i - D) : 2 * GD + h * V + (i - 2 * D));
      const float* wt = a.taps_w + (size_t)c * taps;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (ring[j] >= 0) { hr[x][j] = hs[(size_t)ring[j] * C + c]; hw[x][j] = wt[taps - 2 - j]; }
      w_now[x] = wt[taps - 1];
    }
  }
#pragma unroll
  for (int x = 0; x < DL_STEP_CH; ++x) {
    const int i = tid + x * DL_THREADS;
    past[x] = 0.f;
    if (taps > 5 && i < 2 * D + V) {                 // more rows than that: the older ones one after the other
      const int c = i < D ? gq * D + i : (i < 2 * D ? GD + gq * D + (i - D) : 2 * GD + h * V + (i - 2 * D));
      for (int j = 0; j < taps - 5; ++j) {
        const int p = pos - taps + 1 + j;
        if (p >= 0) past[x] = fmaf(a.taps_w[(size_t)c * taps + j], hs[(size_t)(p % taps) * C + c], past[x]);
      }
    }
#pragma unroll
    for (int j = 3; j >= 0; --j) past[x] = fmaf(hw[x][j], hr[x][j], past[x]);
  }
  pdl_wait();
  pdl_trigger();
  const TP* pj = (const TP*)a.proj + (size_t)t * a.row;
#pragma unroll
  for (int x = 0; x < DL_STEP_CH; ++x) {
    const int i = tid + x * DL_THREADS;
    if (i < 2 * D + V) {
      const bool is_v = i >= 2 * D;
      const int c = i < D ? gq * D + i : (is_v ? 2 * GD + h * V + (i - 2 * D) : GD + gq * D + (i - D));
      const float now = to_f32(pj[a.col + c]);
      if (is_v || h % rep == 0) hs[(size_t)(pos % taps) * C + c] = now;      // the ring's free row
      const float y = dl_silu(fmaf(w_now[x], now, past[x]));
      if (i < D) q[i] = y; else if (is_v) v[i - 2 * D] = y; else k[i - D] = y;
    }
  }
  if (lr.wz)
    for (int i = tid; i < ld; i += DL_THREADS) xs[i] = to_f32(pj[lr.lr_col + i]);
  const float beta = dl_sigmoid(to_f32(pj[a.b_col + h]));
  const float ea = expf(a.a_log[h]);
  dl_wait<0>();
  __syncthreads();
  if (warp == 0) {
    float sq = 0.f, sk = 0.f, kq = 0.f;
    for (int i = lane; i < D; i += 32) { sq = fmaf(q[i], q[i], sq); sk = fmaf(k[i], k[i], sk); kq = fmaf(q[i], k[i], kq); }
    sq = warp_sum(sq); sk = warp_sum(sk); kq = warp_sum(kq);
    const float fq = rsqrtf(sq + a.unit_eps) * a.q_scale, fk = rsqrtf(sk + a.unit_eps);
    if (lane == 0) { sc[0] = fq; sc[1] = fk; sc[2] = kq * fq * fk; }
  }
  if (lr.wz) {
    const int grp = tid >> 3, sub = tid & 7;
    const bool va = lr.ra % VE == 0 && lr.rg % VE == 0;
#pragma unroll 2
    for (int r = grp; r < D + V; r += DL_THREADS / 8) {           // D + V is a multiple of the warps' 4 rows (checked by the host)
      const bool dec = r < D;
      const TO* wr = lr.staged ? wsm + r * wld : (dec ? wz + (size_t)(h * D + r) * ld : wz + (size_t)(H * D + h * V + (r - D)) * ld + lr.ra);
      const float zz = dl_row_dot<TO>(wr, dec ? xs : xs + lr.ra, dec ? lr.ra : lr.rg, sub, va);
      if (sub == 0) {
        if (dec) g[r] = expf(-ea * dl_softplus(zz + a.dt_bias[h * D + r]));
        else og[r - D] = dl_sigmoid(zz);
      }
    }
  } else {
    for (int i = tid; i < D; i += DL_THREADS) g[i] = expf(-ea * dl_softplus(a.z[(size_t)t * a.z_ld + h * D + i] + a.dt_bias[h * D + i]));
    for (int i = tid; i < V; i += DL_THREADS) og[i] = dl_sigmoid(a.z[(size_t)t * a.z_ld + H * D + h * V + i]);
  }
  __syncthreads();
  float4 r = make_float4(0.f, 0.f, 0.f, 0.f), p = r;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = r0 + i * RP;
    if (d < D) {
      const float gd = g[d], kd = k[d], qd = q[d];
      S[i].x *= gd; S[i].y *= gd; S[i].z *= gd; S[i].w *= gd;
      r.x = fmaf(S[i].x, kd, r.x); r.y = fmaf(S[i].y, kd, r.y); r.z = fmaf(S[i].z, kd, r.z); r.w = fmaf(S[i].w, kd, r.w);
      p.x = fmaf(S[i].x, qd, p.x); p.y = fmaf(S[i].y, qd, p.y); p.z = fmaf(S[i].z, qd, p.z); p.w = fmaf(S[i].w, qd, p.w);
    }
  }
  *reinterpret_cast<float4*>(pr + r0 * V + c4) = r;
  *reinterpret_cast<float4*>(pp + r0 * V + c4) = p;
  __syncthreads();
  const float fq = sc[0], fk = sc[1], kq = sc[2];
  float o = 0.f;
  if (tid < V) {
    float rr = 0.f, po = 0.f;
    for (int x = 0; x < RP; ++x) { rr += pr[x * V + tid]; po += pp[x * V + tid]; }
    const float u = beta * (v[tid] - rr * fk);
    us[tid] = u;
    o = fmaf(kq, u, po * fq);
  }
  const float ss = block_sum(o * o, red);            // also orders us before the reads below
  if (tid < V)
    ((TO*)a.out)[(size_t)t * H * V + h * V + tid] = from_f32<TO>(o * rsqrtf(ss / (float)V + a.eps) * a.gain[tid] * og[tid]);
  const float4 u4 = *reinterpret_cast<const float4*>(us + c4);
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = r0 + i * RP;
    if (d < D) {
      const float kd = k[d] * fk;
      *reinterpret_cast<float4*>(Sg + (size_t)d * V) = make_float4(fmaf(kd, u4.x, S[i].x), fmaf(kd, u4.y, S[i].y), fmaf(kd, u4.z, S[i].z), fmaf(kd, u4.w, S[i].w));
    }
  }
}

static bool dl_step_fits(int D, int V, int ra, int rg) {
  if (V < 4 || V > 256 || (V & (V - 1)) || D <= 0 || (D + V) % 4) return false;
  const int NI = (D * V + 1023) / 1024;
  return NI <= 32 && 2 * D + V <= DL_STEP_CH * DL_THREADS && (size_t)(3 * D + 3 * V + ra + rg + 4 + 2048) * sizeof(float) <= 48 * 1024;
}
extern "C" int sx_delta_step_fits(int D, int V, int ra, int rg) { return dl_step_fits(D, V, ra, rg) ? 1 : 0; }

// ---------------------------------------------------------------------------------------------------------------
// chunks, numbered through the step: chunk p of sequence s is number cu_seqlens[s] / 32 + s + p, so that sequences of
// unequal lengths need no more than (tokens / 32 + sequences) of them.  Scratch per (chunk, head): x, qg, kd [32, D] each, y [32, V], p [32, 32], ge [D], sb [D, V] (the state
// at the chunk's begin).
// ---------------------------------------------------------------------------------------------------------------
struct DlChunks { float* x; float* qg; float* kd; float* y; float* p; float* ge; float* sb; int P; };

template <typename TP>
__global__ void __launch_bounds__(DL_THREADS, 3) delta_intra_kernel(DlArgs a, DlPrep w, DlChunks ch) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.D, V = a.V, H = a.H, DS = D + 4, G = a.G;
  float* ks = sm;                        // 32 * DS
  float* qs = ks + DL_C * DS;            // 32 * DS
  float* Gs = qs + DL_C * DS;            // 32 * DS: running sums of the decays' logarithms, base 2, from token 0 and from token 16 on
  float* As = Gs + DL_C * DS;            // 32 * DL_LD
  float* bs = As + DL_C * DL_LD;         // 32
  pdl_wait();
  pdl_trigger();
  const int p = blockIdx.x, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x, gq = h / (H / G);
  const int t0 = a.cu_seqlens[s] + p * DL_C, len = a.cu_seqlens[s + 1] - t0;
  if (len <= 0) return;
  const int L = min(DL_C, len);
  const size_t ci = (size_t)(a.cu_seqlens[s] / DL_C + s + p) * H + h;
  const int D4 = D >> 2;
  for (int i = tid; i < DL_C * D4; i += DL_THREADS) {
    const int t = i / D4, d = (i - t * D4) * 4;
    if (t < L) {
      const size_t at = (size_t)(t0 + t) * G * D + gq * D + d;
      dl_cp16(ks + t * DS + d, w.k + at);
      dl_cp16(qs + t * DS + d, w.q + at);
    } else {
      *reinterpret_cast<float4*>(ks + t * DS + d) = make_float4(0.f, 0.f, 0.f, 0.f);
      *reinterpret_cast<float4*>(qs + t * DS + d) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  dl_commit();
  if (tid < DL_C) bs[tid] = tid < L ? dl_sigmoid(to_f32(((const TP*)a.proj)[(size_t)(t0 + tid) * a.row + a.b_col + h])) : 0.f;
  for (int i = tid; i < DL_C * DL_LD; i += DL_THREADS) As[i] = 0.f;
  // the right sides of the value columns come early too: their loads run beside the others
  float rhs[DL_C];
  if (tid >= D && tid < D + V) {
    const float* vp = w.v + (size_t)t0 * H * V + h * V + (tid - D);
#pragma unroll
    for (int t = 0; t < DL_C; ++t) {
      rhs[t] = *vp;                                  // rows behind the chunk's end: its last row again, times 0 below
      if (t + 1 < L) vp += (size_t)H * V;
    }
  }
  {   // running sums: a thread a channel and half of the chunk (D <= 128) or a channel
    const int parts = D <= DL_THREADS / 2 ? 2 : 1, part = parts == 2 && tid >= DL_THREADS / 2 ? 1 : 0, d = tid - part * (DL_THREADS / 2);
    if (d < D) {
      const float ea = -expf(a.a_log[h]) * DL_LOG2E, c = a.dt_bias[h * D + d];
      for (int half = part; half < (parts == 2 ? part + 1 : 2); ++half) {
        const float* z = a.z + (size_t)(t0 + half * 16) * a.z_ld + h * D + d;
        const int n = L - half * 16;                 // rows of this half
        float zz[16], acc = 0.f;
#pragma unroll
        for (int t = 0; t < 16; ++t) zz[t] = t < n ? z[(size_t)t * a.z_ld] : 0.f;
#pragma unroll
        for (int t = 0; t < 16; ++t) {
          if (t < n) acc += fmaxf(ea * dl_softplus(zz[t] + c), DL_LOG_MIN);
          Gs[(half * 16 + t) * DS + d] = acc;
        }
      }
    }
    dl_wait<0>();
  }
  __syncthreads();
  // pairs within 16 tokens: thread (i, j): j < i the first half's pair (i, j), j > i the second half's (16 + j, 16 + i)
  const int i16 = tid >> 4, j16 = tid & 15;
  float* Pg = ch.p + ci * DL_C * DL_C;
  if (i16 != j16) {
    const int t = j16 < i16 ? i16 : 16 + j16, u = j16 < i16 ? j16 : 16 + i16;
    const float *kt = ks + t * DS, *qt = qs + t * DS, *ku = ks + u * DS, *gt = Gs + t * DS, *gu = Gs + u * DS;
    float sa = 0.f, sp = 0.f;
    for (int d = 0; d < D; d += 4) {
      const float4 x = *reinterpret_cast<const float4*>(gt + d), y = *reinterpret_cast<const float4*>(gu + d);
      const float4 b = *reinterpret_cast<const float4*>(ku + d), c = *reinterpret_cast<const float4*>(kt + d);
      const float4 e = *reinterpret_cast<const float4*>(qt + d);
      const float b0 = b.x * dl_exp2(x.x - y.x), b1 = b.y * dl_exp2(x.y - y.y), b2 = b.z * dl_exp2(x.z - y.z), b3 = b.w * dl_exp2(x.w - y.w);
      sa = fmaf(c.x, b0, fmaf(c.y, b1, fmaf(c.z, b2, fmaf(c.w, b3, sa))));
      sp = fmaf(e.x, b0, fmaf(e.y, b1, fmaf(e.z, b2, fmaf(e.w, b3, sp))));
    }
    As[t * DL_LD + u] = bs[t] * sa;
    Pg[t * DL_C + u] = sp;
    Pg[u * DL_C + t] = 0.f;
  } else {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = half * 16 + i16;
      const float *kt = ks + t * DS, *qt = qs + t * DS;
      float sp = 0.f;
      for (int d = 0; d < D; d += 4) {
        const float4 c = *reinterpret_cast<const float4*>(kt + d), e = *reinterpret_cast<const float4*>(qt + d);
        sp = fmaf(e.x, c.x, fmaf(e.y, c.y, fmaf(e.z, c.z, fmaf(e.w, c.w, sp))));
      }
      Pg[t * DL_C + t] = sp;
    }
  }
  __syncthreads();
  // a thread a channel: what the scan reads, the right side b e^G k in registers, then k and q around the border (token 15)
  float* X = ch.x + ci * DL_C * D;
  if (tid < D) {
    float* Q = ch.qg + ci * DL_C * D + tid;
    float* K = ch.kd + ci * DL_C * D + tid;
    float *gp = Gs + tid, *kp = ks + tid, *qp = qs + tid;      // walked row by row: 32 addresses held at once would spill
    const float gm = Gs[15 * DS + tid], gl = Gs[(DL_C - 1) * DS + tid];        // the two halves' whole sums
    ch.ge[ci * D + tid] = dl_exp2(gm + gl);
#pragma unroll
    for (int t = 0; t < DL_C; ++t) {
      asm volatile("" ::: "memory");
      const float gt = *gp, kt = *kp, qt = *qp;
      const float e = dl_exp2(t < 16 ? gt : gm + gt);
      rhs[t] = bs[t] * e * kt;
      *Q = e * qt;
      *K = dl_exp2(t < 16 ? (gm - gt) + gl : gl - gt) * kt;
      const float f = dl_exp2(t < 16 ? gm - gt : gt);
      *kp = f * kt;
      *qp = f * qt;
      Q += D; K += D; gp += DS; kp += DS; qp += DS;
    }
  } else if (tid < D + V) {
#pragma unroll
    for (int t = 0; t < DL_C; ++t) rhs[t] *= bs[t];          // 0 behind the chunk's end
  }
  __syncthreads();
  {   // pairs across the border: row 16 + i, column j
    const float *kt = ks + (16 + i16) * DS, *qt = qs + (16 + i16) * DS, *ku = ks + j16 * DS;
    float sa = 0.f, sp = 0.f;
    for (int d = 0; d < D; d += 4) {
      const float4 b = *reinterpret_cast<const float4*>(ku + d), c = *reinterpret_cast<const float4*>(kt + d);
      const float4 e = *reinterpret_cast<const float4*>(qt + d);
      sa = fmaf(c.x, b.x, fmaf(c.y, b.y, fmaf(c.z, b.z, fmaf(c.w, b.w, sa))));
      sp = fmaf(e.x, b.x, fmaf(e.y, b.y, fmaf(e.z, b.z, fmaf(e.w, b.w, sp))));
    }
    As[(16 + i16) * DL_LD + j16] = bs[16 + i16] * sa;
    Pg[(16 + i16) * DL_C + j16] = sp;
    Pg[j16 * DL_C + 16 + i16] = 0.f;
  }
  __syncthreads();
  // forward substitution, a thread a column
  float* Y = ch.y + ci * DL_C * V;
  for (int col = tid; col < D + V; col += DL_THREADS) {
    if (col != tid) {                    // columns beyond the first round: value columns
      const float* vp = w.v + (size_t)t0 * H * V + h * V + (col - D);
#pragma unroll
      for (int t = 0; t < DL_C; ++t) {
        rhs[t] = t < L ? bs[t] * *vp : 0.f;
        if (t + 1 < L) vp += (size_t)H * V;
      }
    }
#pragma unroll
    for (int t = 1; t < DL_C; ++t) {
      asm volatile("" ::: "memory");       // a row's loads stay in their row: hoisted all together they spill
      float acc = rhs[t];
#pragma unroll
      for (int u = 0; u < t; u += 4) {
        const float4 m = *reinterpret_cast<const float4*>(As + t * DL_LD + u);       // zero from column t on
        acc = fmaf(-m.x, rhs[u], acc);
        if (u + 1 < t) acc = fmaf(-m.y, rhs[u + 1], acc);
        if (u + 2 < t) acc = fmaf(-m.z, rhs[u + 2], acc);
        if (u + 3 < t) acc = fmaf(-m.w, rhs[u + 3], acc);
      }
      rhs[t] = acc;
    }
    float* dst = col < D ? X + col : Y + (col - D);
    const int ld = col < D ? D : V;
#pragma unroll
    for (int t = 0; t < DL_C; ++t) {
      asm volatile("" ::: "memory");
      *dst = rhs[t];
      dst += ld;
    }
  }
}

static size_t dl_intra_smem(int D) { return (size_t)(3 * DL_C * (D + 4) + DL_C * DL_LD + DL_C) * sizeof(float); }


// VS: columns of the state a block owns (8, 16 or 32); ND: tiles of the state a thread owns (D <= 128 ND).
#define DL_SCAN_THREADS 256
template <int VS, int ND>
__global__ void __launch_bounds__(DL_SCAN_THREADS) delta_scan_kernel(DlArgs a, DlChunks ch) {
  extern __shared__ __align__(16) float sm[];
  constexpr int SS = VS + 4;
  constexpr int CG = VS / 4;                       // groups of four columns in the product with S
  constexpr int KSPLIT = DL_SCAN_THREADS / (8 * CG);   // 16, 8 or 4: parts of D in that product
  constexpr int CP = VS / 8;                       // columns a thread of u and of the state's tiles
  const int D = a.D, V = a.V, H = a.H, DS = D + 4;
  float* xs = sm;                                  // 2 * 32 * DS: X, two chunks
  float* kd = xs + 2 * DL_C * DS;                  // 2 * 32 * DS: e^(G_end - G) k
  float* S = kd + 2 * DL_C * DS;                   // D * SS
  float* U = S + D * SS;                           // 32 * SS
  float* part = U + DL_C * SS;                     // KSPLIT * 32 * SS
  pdl_wait();
  pdl_trigger();
  const int v0 = blockIdx.x * VS, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int tok0 = a.cu_seqlens[s], n = a.cu_seqlens[s + 1] - tok0, np = (n + DL_C - 1) / DL_C;
  if (np <= 0) return;
  float* Sg = a.S + ((size_t)a.seq_slots[s] * H + h) * D * V;
  const int D4 = D >> 2;
  const size_t c0 = (size_t)(tok0 / DL_C + s) * H + h;      // the first chunk; the next lies H further
  // pointers that walk from chunk to chunk
  const float *xg = ch.x + c0 * DL_C * D + (tid >> 5) * D + (tid & 31) * 4, *kg_ = ch.kd + c0 * DL_C * D + (tid >> 5) * D + (tid & 31) * 4;
  const size_t step_x = (size_t)H * DL_C * D;
  const int soff = (tid >> 5) * DS + (tid & 31) * 4;
  auto load = [&](int p) {                         // called for 0, 1, 2, ... in order
    float *xd = xs + (p & 1) * DL_C * DS + soff, *kk = kd + (p & 1) * DL_C * DS + soff;
    for (int d = (tid & 31) * 4, o = 0; d < D; d += 128, o += 128)
#pragma unroll
      for (int t = 0; t < DL_C; t += DL_SCAN_THREADS / 32) {
        dl_cp16(xd + t * DS + o, xg + t * D + o);
        dl_cp16(kk + t * DS + o, kg_ + t * D + o);
      }
    xg += step_x;
    kg_ += step_x;
  };
  // this thread's place in u (row ur, CP columns from uc on) and in the state (rows 4 sd .., the same columns)
  const int ur = tid >> 3, uc = (tid & 7) * CP, sd = tid >> 3;
  float st[ND][4][CP], y[CP], ge[ND][4];
  float* yg = ch.y + c0 * DL_C * V + (size_t)ur * V + v0 + uc;         // this chunk's right side (and then its u)
  const float* gg = ch.ge + c0 * D;
  float* sb = ch.sb + c0 * D * V + (size_t)sd * 4 * V + v0 + uc;
  const size_t step_y = (size_t)H * DL_C * V, step_s = (size_t)H * D * V;
  auto load_small = [&](const float* yg, const float* gg) {            // u's right side and the chunk's whole decay, to registers
#pragma unroll
    for (int j = 0; j < CP; ++j) y[j] = v0 + uc + j < V ? yg[j] : 0.f;
#pragma unroll
    for (int b = 0; b < ND; ++b) {
      const int d = (sd + 32 * b) * 4;
      if (d < D) {
        const float4 f = *reinterpret_cast<const float4*>(gg + d);
        ge[b][0] = f.x; ge[b][1] = f.y; ge[b][2] = f.z; ge[b][3] = f.w;
      }
    }
  };
  load(0);
  dl_commit();
  load_small(yg, gg);
#pragma unroll
  for (int b = 0; b < ND; ++b)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = (sd + 32 * b) * 4 + i;
#pragma unroll
      for (int j = 0; j < CP; ++j) st[b][i][j] = d < D && v0 + uc + j < V ? Sg[(size_t)d * V + v0 + uc + j] : 0.f;
    }
  const int kg = tid / (8 * CG), rem = tid - kg * 8 * CG, rg = rem / CG, cg = rem - rg * CG;
  const int dper = (D4 + KSPLIT - 1) / KSPLIT * 4, da = kg * dper, db = min(D, da + dper);
  for (int p = 0; p < np; ++p) {
    // the state at the chunk's begin: to shared memory for the product, to memory for the output kernel
#pragma unroll
    for (int b = 0; b < ND; ++b)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = (sd + 32 * b) * 4 + i;
        if (d < D) {
#pragma unroll
          for (int j = 0; j < CP; ++j) S[d * SS + uc + j] = st[b][i][j];
          float* sr = sb + (b * 128 + i) * V;
          if ((V & 3) == 0 && v0 + uc + CP <= V) {
            if (CP == 4) *reinterpret_cast<float4*>(sr) = make_float4(st[b][i][0], st[b][i][1 % CP], st[b][i][2 % CP], st[b][i][3 % CP]);
            else if (CP == 2) *reinterpret_cast<float2*>(sr) = make_float2(st[b][i][0], st[b][i][1 % CP]);
            else *sr = st[b][i][0];
          } else {
#pragma unroll
            for (int j = 0; j < CP; ++j)
              if (v0 + uc + j < V) sr[j] = st[b][i][j];
          }
        }
      }
    dl_wait<0>();
    __syncthreads();                               // X, k of this chunk and S are in place; the other buffers are read out
    if (p + 1 < np) load(p + 1);
    dl_commit();
    const float *xd = xs + (p & 1) * DL_C * DS, *kk = kd + (p & 1) * DL_C * DS;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 2
    for (int d = da; d < db; d += 4) {             // rows rg, rg + 8, rg + 16, rg + 24
      float4 b[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) b[x] = *reinterpret_cast<const float4*>(S + (d + x) * SS + cg * 4);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 m = *reinterpret_cast<const float4*>(xd + (rg + 8 * i) * DS + d);
        acc[i][0] = fmaf(m.x, b[0].x, fmaf(m.y, b[1].x, fmaf(m.z, b[2].x, fmaf(m.w, b[3].x, acc[i][0]))));
        acc[i][1] = fmaf(m.x, b[0].y, fmaf(m.y, b[1].y, fmaf(m.z, b[2].y, fmaf(m.w, b[3].y, acc[i][1]))));
        acc[i][2] = fmaf(m.x, b[0].z, fmaf(m.y, b[1].z, fmaf(m.z, b[2].z, fmaf(m.w, b[3].z, acc[i][2]))));
        acc[i][3] = fmaf(m.x, b[0].w, fmaf(m.y, b[1].w, fmaf(m.z, b[2].w, fmaf(m.w, b[3].w, acc[i][3]))));
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      *reinterpret_cast<float4*>(part + (kg * DL_C + rg + 8 * i) * SS + cg * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    __syncthreads();
    {   // u = Y - X S, left in Y's place for the output kernel
      float u[CP];
#pragma unroll
      for (int j = 0; j < CP; ++j) u[j] = y[j];
#pragma unroll
      for (int x = 0; x < KSPLIT; ++x)
#pragma unroll
        for (int j = 0; j < CP; ++j) u[j] -= part[(x * DL_C + ur) * SS + uc + j];
#pragma unroll
      for (int j = 0; j < CP; ++j) {
        U[ur * SS + uc + j] = u[j];
        if (v0 + uc + j < V) yg[j] = u[j];
      }
    }
#pragma unroll
    for (int b = 0; b < ND; ++b)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < CP; ++j) st[b][i][j] *= ge[b][i];
    yg += step_y;
    gg += (size_t)H * D;
    sb += step_s;
    if (p + 1 < np) load_small(yg, gg);
    __syncthreads();
#pragma unroll
    for (int b = 0; b < ND; ++b) {
      const int d = (sd + 32 * b) * 4;
      if (d < D) {
#pragma unroll 8
        for (int t = 0; t < DL_C; ++t) {
          const float4 f = *reinterpret_cast<const float4*>(kk + t * DS + d);
          float u[CP];
#pragma unroll
          for (int j = 0; j < CP; ++j) u[j] = U[t * SS + uc + j];
#pragma unroll
          for (int j = 0; j < CP; ++j) {
            st[b][0][j] = fmaf(f.x, u[j], st[b][0][j]);
            st[b][1][j] = fmaf(f.y, u[j], st[b][1][j]);
            st[b][2][j] = fmaf(f.z, u[j], st[b][2][j]);
            st[b][3][j] = fmaf(f.w, u[j], st[b][3][j]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int b = 0; b < ND; ++b)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = (sd + 32 * b) * 4 + i;
#pragma unroll
      for (int j = 0; j < CP; ++j)
        if (d < D && v0 + uc + j < V) Sg[(size_t)d * V + v0 + uc + j] = st[b][i][j];
    }
}

static size_t dl_scan_smem(int D, int VS) {
  const int SS = VS + 4, ksplit = DL_SCAN_THREADS / (2 * VS);
  return (size_t)(4 * DL_C * (D + 4) + D * SS + DL_C * SS + ksplit * DL_C * SS) * sizeof(float);
}

// a block a (chunk, head): o = [e^G q | P] [S_begin; u], then the output norm, gain and gate.  A warp owns four rows of all
// columns (NT tiles of 128), so the norm is a warp's business; both factors lie in shared memory whole, in two portions
// that arrive one after the other.
template <typename TO, int NT>
__global__ void __launch_bounds__(DL_THREADS, 2) delta_out_kernel(DlArgs a, DlChunks ch) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.D, V = a.V, H = a.H, DS = D + DL_C + 4, BS = ((V + 3) & ~3) + 4;
  float* A = sm;                                   // 32 * DS: e^G q, then P
  float* B = A + DL_C * DS;                        // (D + 32) * BS: S_begin, then u
  pdl_wait();
  pdl_trigger();
  const int p = blockIdx.x, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int t0 = a.cu_seqlens[s] + p * DL_C, len = a.cu_seqlens[s + 1] - t0;
  if (len <= 0) return;
  const int L = min(DL_C, len);
  const size_t ci = (size_t)(a.cu_seqlens[s] / DL_C + s + p) * H + h;
  const float *qg = ch.qg + ci * DL_C * D, *pg = ch.p + ci * DL_C * DL_C, *sb = ch.sb + ci * D * V, *ug = ch.y + ci * DL_C * V;
  const int warp = tid >> 5, lane = tid & 31;
  auto load_rows = [&](float* dst, const float* src, int rows) {        // rows of V columns
    if ((V & 3) == 0) {
      for (int c = lane * 4; c < V; c += 128)
        for (int r = warp; r < rows; r += DL_THREADS / 32) dl_cp16(dst + r * BS + c, src + (size_t)r * V + c);
    } else {
      for (int c = lane; c < V; c += 32)
        for (int r = warp; r < rows; r += DL_THREADS / 32) dst[r * BS + c] = src[(size_t)r * V + c];
    }
  };
  const int half = D / 2 & ~3;
  for (int d = lane * 4; d < D; d += 128)
    for (int t = warp; t < DL_C; t += DL_THREADS / 32) dl_cp16(A + t * DS + d, qg + t * D + d);
  load_rows(B, sb, half);
  dl_commit();
  dl_cp16(A + (tid >> 3) * DS + D + (tid & 7) * 4, pg + tid * 4);
  load_rows(B + half * BS, sb + (size_t)half * V, D - half);
  load_rows(B + D * BS, ug, DL_C);
  dl_commit();
  float acc[NT][4][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[n][i][j] = 0.f;
  auto product = [&](int k0, int k1) {
#pragma unroll 4
    for (int k = k0; k < k1; k += 4) {
      float4 m[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) m[i] = *reinterpret_cast<const float4*>(A + (warp * 4 + i) * DS + k);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int c = n * 128 + lane * 4;
        if (c < V) {
          float4 x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = *reinterpret_cast<const float4*>(B + (k + e) * BS + c);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            acc[n][i][0] = fmaf(m[i].x, x[0].x, fmaf(m[i].y, x[1].x, fmaf(m[i].z, x[2].x, fmaf(m[i].w, x[3].x, acc[n][i][0]))));
            acc[n][i][1] = fmaf(m[i].x, x[0].y, fmaf(m[i].y, x[1].y, fmaf(m[i].z, x[2].y, fmaf(m[i].w, x[3].y, acc[n][i][1]))));
            acc[n][i][2] = fmaf(m[i].x, x[0].z, fmaf(m[i].y, x[1].z, fmaf(m[i].z, x[2].z, fmaf(m[i].w, x[3].z, acc[n][i][2]))));
            acc[n][i][3] = fmaf(m[i].x, x[0].w, fmaf(m[i].y, x[1].w, fmaf(m[i].z, x[2].w, fmaf(m[i].w, x[3].w, acc[n][i][3]))));
          }
        }
      }
    }
  };
  dl_wait<1>();
  __syncthreads();
  product(0, half);
  dl_wait<0>();
  __syncthreads();
  float z[NT][4][4];                               // the gates' pre-activations: on their way during the second product
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = n * 128 + lane * 4, r = min(warp * 4 + i, L - 1);
      const float* zr = a.z + (size_t)(t0 + r) * a.z_ld + H * D + h * V + c;
#pragma unroll
      for (int j = 0; j < 4; ++j) z[n][i][j] = c + j < V ? zr[j] : 0.f;
    }
  product(half, D + DL_C);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = warp * 4 + i;
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n * 128 + lane * 4 + j < V) ss += acc[n][i][j] * acc[n][i][j];
    const float inv = rsqrtf(warp_sum(ss) / (float)V + a.eps);
    if (r < L) {
      TO* out = (TO*)a.out + (size_t)(t0 + r) * H * V + h * V;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int c = n * 128 + lane * 4 + j;
          if (c < V) out[c] = from_f32<TO>(acc[n][i][j] * inv * a.gain[c] * dl_sigmoid(z[n][i][j]));
        }
    }
  }
}

static size_t dl_out_smem(int D, int V) { return (size_t)(DL_C * (D + DL_C + 4) + (D + DL_C) * (((V + 3) & ~3) + 4)) * sizeof(float); }

extern "C" int sx_delta_chunk_tokens() { return DL_C; }
extern "C" int sx_delta_chunks_fit(int D, int V) {
  return (D % 4 == 0 && D <= DL_THREADS && V <= 256 && dl_intra_smem(D) <= 220 * 1024 && dl_scan_smem(D, 32) <= 220 * 1024 &&
          dl_scan_smem(D, 16) <= 220 * 1024 && dl_scan_smem(D, 8) <= 220 * 1024 && dl_out_smem(D, V) <= 220 * 1024) ? 1 : 0;
}

// ---------------------------------------------------------------------------------------------------------------
static DlArgs dl_args(const void* proj, int row, int col, int b_col, const float* taps_w, int taps, float* hist, const float* z,
                      int z_ld, const float* a_log, const float* dt_bias, const float* gain, float q_scale, float unit_eps,
                      float eps, float* S, void* out, const int* positions, const int* seq_of_token, const int* cu_seqlens,
                      const int* seq_past, const int* seq_lens, const int* seq_slots, int H, int G, int D, int V) {
  DlArgs a = {proj, row, col, b_col, taps_w, taps, hist, z, z_ld, a_log, dt_bias, gain, q_scale, unit_eps, eps, S, out,
              positions, seq_of_token, cu_seqlens, seq_past, seq_lens, seq_slots, H, G, D, V};
  return a;
}

#define DL_FORMALS                                                                                                           \
  const void *proj, int row, int col, int b_col, const float *taps_w, int taps, float *hist, const float *z, int z_ld,        \
      const float *a_log, const float *dt_bias, const float *gain, float q_scale, float unit_eps, float eps, float *S,        \
      void *out, const int *positions, const int *seq_of_token, const int *cu_seqlens, const int *seq_past,                   \
      const int *seq_lens, const int *seq_slots, int n_tokens, int n_seqs, int H, int G, int D, int V, int proj_dt, int out_dt
#define DL_ACTUALS                                                                                                           \
  proj, row, col, b_col, taps_w, taps, hist, z, z_ld, a_log, dt_bias, gain, q_scale, unit_eps, eps, S, out, positions,        \
      seq_of_token, cu_seqlens, seq_past, seq_lens, seq_slots, H, G, D, V

static int dl_check(int n_seqs, int H, int G, int D, int V, int taps) {
  return (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || taps <= 0 || H > 65535 || n_seqs > 65535) ? SX_ERR_SIZE : 0;
}

template <typename TP, typename TO>
static int dl_step_launch(const DlArgs& a, DlLowRank lr, int n_seqs, cudaStream_t stream) {
  size_t smem = (size_t)(((3 * a.D + 2 * a.V + lr.ra + lr.rg + 3) & ~3) + 2048 + a.V) * sizeof(float);
  constexpr int VE = 16 / sizeof(TO);
  if (lr.wz && lr.ra % VE == 0 && lr.rg % VE == 0) {
    const size_t w = (size_t)(a.D + a.V) * dl_lr_ld<TO>(lr.ra, lr.rg) * sizeof(TO);
    if (smem + w <= 100 * 1024) { lr.staged = 1; smem += w; }
  }
  const int NI = (a.D * a.V + 1023) / 1024;
  const dim3 grid(a.H, n_seqs), block(DL_THREADS);
#define DL_STEP(N)                                                                                                              \
  do {                                                                                                                          \
    if (smem > 48 * 1024) cudaFuncSetAttribute(delta_step_kernel<TP, TO, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    return sx_launch(delta_step_kernel<TP, TO, N>, grid, block, smem, stream, a, lr);                                           \
  } while (0)
  if (NI <= 2) DL_STEP(2);
  if (NI <= 4) DL_STEP(4);
  if (NI <= 8) DL_STEP(8);
  if (NI <= 16) DL_STEP(16);
  DL_STEP(32);
#undef DL_STEP
}

// single tokens, a sequence each (n_seqs of them); wz null: z holds the pre-activations
extern "C" int sx_delta_step(DL_FORMALS, const void* wz, int ra, int rg, int lr_col, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (n_tokens != n_seqs || dl_check(n_seqs, H, G, D, V, taps) || !dl_step_fits(D, V, wz ? ra : 0, wz ? rg : 0)) return SX_ERR_SIZE;
  if (wz == nullptr && z == nullptr) return SX_ERR_SIZE;
  if ((uintptr_t)S % 16 || (uintptr_t)wz % 16) return SX_ERR_ALIGN;
  const DlArgs a = dl_args(DL_ACTUALS);
  const DlLowRank lr = {wz, wz ? ra : 0, wz ? rg : 0, lr_col, 0};
  if (proj_dt == SX_F32 && out_dt == SX_F32) return dl_step_launch<float, float>(a, lr, n_seqs, stream);
  if (proj_dt == SX_F32 && out_dt == SX_BF16) return dl_step_launch<float, bf16>(a, lr, n_seqs, stream);
  if (proj_dt == SX_BF16 && out_dt == SX_BF16) return dl_step_launch<bf16, bf16>(a, lr, n_seqs, stream);
  return SX_ERR_DTYPE;
}

template <typename TP>
static int dl_prepare_launch(const DlArgs& a, const DlPrep& w, int n_tokens, int n_seqs, cudaStream_t stream) {
  const int units = 2 * a.G + a.H, C = 2 * a.G * a.D + a.H * a.V;
  auto lane_vec = [](int n) { return n == 32 || n == 64 || n == 128 || n == 256; };
  const bool aligned = a.row % 4 == 0 && a.col % 4 == 0 && (uintptr_t)a.proj % 16 == 0 && (uintptr_t)a.hist % 16 == 0;
  int rc;
  if (lane_vec(a.D) && lane_vec(a.V) && aligned && a.taps >= 2 && a.taps <= 4) {
    const dim3 grid((n_tokens + DL_RUN - 1) / DL_RUN, (units + DL_THREADS / 32 - 1) / (DL_THREADS / 32));
    const bool wide = a.D == 256 || a.V == 256;
#define DL_RUN_GO(N)                                                                                                     \
  rc = wide ? sx_launch(delta_prepare_run_kernel<TP, N, true>, grid, dim3(DL_THREADS), 0, stream, a, w, n_tokens)        \
            : sx_launch(delta_prepare_run_kernel<TP, N, false>, grid, dim3(DL_THREADS), 0, stream, a, w, n_tokens)
    if (a.taps == 2) DL_RUN_GO(2);
    else if (a.taps == 3) DL_RUN_GO(3);
    else DL_RUN_GO(4);
#undef DL_RUN_GO
  } else {
    const long long items = (long long)n_tokens * units;
    rc = sx_launch(delta_prepare_kernel<TP>, dim3((unsigned)((items + DL_THREADS / 32 - 1) / (DL_THREADS / 32))), dim3(DL_THREADS), 0, stream, a, w, n_tokens);
  }
  if (rc) return rc;
  return sx_launch(delta_history_kernel<TP>, dim3((C + 255) / 256, n_seqs), dim3(256), 0, stream, a);
}

// convolutions, activations, unit norms into q, k [T, G D], v [T, H V] (float32); the rings are moved on
extern "C" int sx_delta_prepare(DL_FORMALS, float* q, float* k, float* v, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (dl_check(n_seqs, H, G, D, V, taps)) return SX_ERR_SIZE;
  const DlArgs a = dl_args(DL_ACTUALS);
  const DlPrep w = {q, k, v};
  (void)out_dt;
  if (proj_dt == SX_F32) return dl_prepare_launch<float>(a, w, n_tokens, n_seqs, stream);
  if (proj_dt == SX_BF16) return dl_prepare_launch<bf16>(a, w, n_tokens, n_seqs, stream);
  return SX_ERR_DTYPE;
}

template <typename TP, typename TO>
static int dl_walk_launch(const DlArgs& a, const DlPrep& w, int n_seqs, cudaStream_t stream) {
  const int in_place = dl_walk_smem(a.D, a.V, false) > 200 * 1024 ? 1 : 0;
  const size_t smem = dl_walk_smem(a.D, a.V, in_place != 0);
  if (smem > 200 * 1024) return SX_ERR_SIZE;
  if (smem > 48 * 1024) cudaFuncSetAttribute(delta_walk_kernel<TP, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return sx_launch(delta_walk_kernel<TP, TO>, dim3(a.H, n_seqs), dim3(DL_THREADS), smem, stream, a, w, in_place);
}

extern "C" int sx_delta_walk(DL_FORMALS, float* q, float* k, float* v, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (dl_check(n_seqs, H, G, D, V, taps)) return SX_ERR_SIZE;
  const DlArgs a = dl_args(DL_ACTUALS);
  const DlPrep w = {q, k, v};
  if (proj_dt == SX_F32 && out_dt == SX_F32) return dl_walk_launch<float, float>(a, w, n_seqs, stream);
  if (proj_dt == SX_F32 && out_dt == SX_BF16) return dl_walk_launch<float, bf16>(a, w, n_seqs, stream);
  if (proj_dt == SX_BF16 && out_dt == SX_BF16) return dl_walk_launch<bf16, bf16>(a, w, n_seqs, stream);
  return SX_ERR_DTYPE;
}

template <typename TP, typename TO>
static int dl_chunks_launch(const DlArgs& a, const DlPrep& w, const DlChunks& ch, int n_seqs, int slice, cudaStream_t stream) {
  const size_t si = dl_intra_smem(a.D);
  if (si > 48 * 1024) cudaFuncSetAttribute(delta_intra_kernel<TP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)si);
  int rc = sx_launch(delta_intra_kernel<TP>, dim3(ch.P, a.H, n_seqs), dim3(DL_THREADS), si, stream, a, w, ch);
  if (rc) return rc;
  const size_t ss = dl_scan_smem(a.D, slice);
  const dim3 grid((a.V + slice - 1) / slice, a.H, n_seqs);
#define DL_SCAN(VS, ND)                                                                                                       \
  do {                                                                                                                        \
    if (ss > 48 * 1024) cudaFuncSetAttribute(delta_scan_kernel<VS, ND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ss); \
    rc = sx_launch(delta_scan_kernel<VS, ND>, grid, dim3(DL_SCAN_THREADS), ss, stream, a, ch);                                      \
  } while (0)
  if (slice == 32) { if (a.D <= 128) DL_SCAN(32, 1); else DL_SCAN(32, 2); }
  else if (slice == 16) { if (a.D <= 128) DL_SCAN(16, 1); else DL_SCAN(16, 2); }
  else { if (a.D <= 128) DL_SCAN(8, 1); else DL_SCAN(8, 2); }
#undef DL_SCAN
  if (rc) return rc;
  const size_t so = dl_out_smem(a.D, a.V);
  if (a.V <= 128) {
    if (so > 48 * 1024) cudaFuncSetAttribute(delta_out_kernel<TO, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);
    return sx_launch(delta_out_kernel<TO, 1>, dim3(ch.P, a.H, n_seqs), dim3(DL_THREADS), so, stream, a, ch);
  }
  if (so > 48 * 1024) cudaFuncSetAttribute(delta_out_kernel<TO, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);
  return sx_launch(delta_out_kernel<TO, 2>, dim3(ch.P, a.H, n_seqs), dim3(DL_THREADS), so, stream, a, ch);
}

// chunks of DL_C tokens (the caller has asked sx_delta_chunks_fit); slice: columns of the state a block of the scan owns
extern "C" int sx_delta_chunks(DL_FORMALS, float* q, float* k, float* v, float* x, float* qg, float* kd, float* y, float* p,
                               float* ge, float* sb, int chunks, int slice, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (dl_check(n_seqs, H, G, D, V, taps) || !sx_delta_chunks_fit(D, V) || (slice != 8 && slice != 16 && slice != 32) || chunks <= 0) return SX_ERR_SIZE;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)x | (uintptr_t)qg | (uintptr_t)kd | (uintptr_t)y | (uintptr_t)p | (uintptr_t)ge | (uintptr_t)sb) % 16)
    return SX_ERR_ALIGN;
  const DlArgs a = dl_args(DL_ACTUALS);
  const DlPrep w = {q, k, v};
  const DlChunks ch = {x, qg, kd, y, p, ge, sb, chunks};
  if (proj_dt == SX_F32 && out_dt == SX_F32) return dl_chunks_launch<float, float>(a, w, ch, n_seqs, slice, stream);
  if (proj_dt == SX_F32 && out_dt == SX_BF16) return dl_chunks_launch<float, bf16>(a, w, ch, n_seqs, slice, stream);
  if (proj_dt == SX_BF16 && out_dt == SX_BF16) return dl_chunks_launch<bf16, bf16>(a, w, ch, n_seqs, slice, stream);
  return SX_ERR_DTYPE;
}
