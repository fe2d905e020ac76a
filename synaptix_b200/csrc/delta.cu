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
//     delta_scan_kernel   a block a (slice of V, head, sequence) walks the chunks: u = Y - X S, o = (e^G q) S + P u,
//                         S <- diag(e^(G_end)) S + (e^(G_end - G) k)^T u.
//     delta_finish_kernel a warp a (token, head): output norm, gain, gate.
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

template <typename T, int CPL, int TAPS>
__device__ __forceinline__ void dl_prepare_run(const DlArgs& a, const DlPrep& w, int t0, int t1, int unit, int c0, int kind, int lane) {
  const int C = 2 * a.G * a.D + a.H * a.V, c = c0 + lane * CPL;
  const T* src = (const T*)a.proj + a.col + c;
  float wt[CPL][TAPS], win[TAPS][CPL];            // win[j]: the row that tap j reads
#pragma unroll
  for (int i = 0; i < CPL; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[i][j] = a.taps_w[(size_t)(c + i) * TAPS + j];
  int seq = -1, pos = 0;
  for (int t = t0; t < t1; ++t) {
    const int s = a.seq_of_token[t];
    if (s != seq) {                               // the run's first token, or another sequence's: fetch the rows before it
      seq = s;
      pos = a.positions[t];
      const int past = a.seq_past[s];
      const float* hs = a.hist + (size_t)a.seq_slots[s] * TAPS * C + c;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int p = pos - TAPS + 1 + j;         // goes to place j + 1: the shift below brings it to place j
        if (p < 0) {
#pragma unroll
          for (int i = 0; i < CPL; ++i) win[j + 1][i] = 0.f;
        } else if (p >= past) {
          DlLd<T, CPL>::go(src + (size_t)(t - (pos - p)) * a.row, win[j + 1]);
        } else {
          dl_ld_f32<CPL>(hs + (size_t)(p % TAPS) * C, win[j + 1]);
        }
      }
    } else {
      ++pos;
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int i = 0; i < CPL; ++i) win[j][i] = win[j + 1][i];
    DlLd<T, CPL>::go(src + (size_t)t * a.row, win[TAPS - 1]);
    float y[CPL], ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[i][j], win[j][i], acc);
      y[i] = dl_silu(acc);
      ss += y[i] * y[i];
    }
    if (kind != 2) {
      const float f = rsqrtf(warp_sum(ss) + a.unit_eps) * (kind == 0 ? a.q_scale : 1.f);
#pragma unroll
      for (int i = 0; i < CPL; ++i) y[i] *= f;
    }
    float* dst = dl_prep_dst(a, w, t, unit, kind) + lane * CPL;
    if (CPL % 4 == 0) {
#pragma unroll
      for (int i = 0; i < CPL / 4; ++i)
        reinterpret_cast<float4*>(dst)[i] = make_float4(y[4 * i], y[(4 * i + 1) % CPL], y[(4 * i + 2) % CPL], y[(4 * i + 3) % CPL]);
    } else {
#pragma unroll
      for (int i = 0; i < CPL; ++i) dst[i] = y[i];
    }
  }
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(DL_THREADS) delta_prepare_run_kernel(DlArgs a, DlPrep w, int n_tokens) {
  pdl_wait();
  pdl_trigger();
  const int unit = blockIdx.y * (DL_THREADS / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= 2 * a.G + a.H) return;
  const int t0 = blockIdx.x * DL_RUN, t1 = min(n_tokens, t0 + DL_RUN);
  int c0, n, kind;
  dl_unit(a, unit, c0, n, kind);
  switch (n) {
    case 32: dl_prepare_run<T, 1, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
    case 64: dl_prepare_run<T, 2, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
    case 128: dl_prepare_run<T, 4, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;
    default: dl_prepare_run<T, 8, TAPS>(a, w, t0, t1, unit, c0, kind, lane); break;      // 256
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
// ---------------------------------------------------------------------------------------------------------------
struct DlLowRank { const void* wz; int ra, rg, lr_col; };

// rows dot x: 8 lanes a row, 16-byte loads where the row's start and length allow
template <typename TW>
__device__ __forceinline__ float dl_row_dot(const TW* wr, const float* x, int n, int sub, bool vec) {
  float acc = 0.f;
  constexpr int VE = 16 / sizeof(TW);
  if (vec) {
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

template <typename TP, typename TO, int NI>
__global__ void __launch_bounds__(DL_THREADS) delta_step_kernel(DlArgs a, DlLowRank lr) {
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
  __shared__ float red[33];
  __shared__ float sc[3];
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int V4 = V >> 2, RP = 1024 / V, c4 = (tid % V4) * 4, r0 = tid / V4;
  const int slot = a.seq_slots[s];
  float* Sg = a.S + ((size_t)slot * H + h) * D * V + c4;
  float4 S[NI];
  // the state was written by a kernel of an earlier step (several launches back): asked for before the wait
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = r0 + i * RP;
    S[i] = d < D ? *reinterpret_cast<const float4*>(Sg + (size_t)d * V) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  pdl_trigger();
  const int rep = H / G, gq = h / rep, t = s, pos = a.positions[t], taps = a.taps;
  const int C = 2 * G * D + H * V, GD = G * D;
  const TP* pj = (const TP*)a.proj + (size_t)t * a.row;
  float* hs = a.hist + (size_t)slot * taps * C;
  for (int i = tid; i < 2 * D + V; i += DL_THREADS) {
    const bool is_v = i >= 2 * D;
    const int c = i < D ? gq * D + i : (is_v ? 2 * GD + h * V + (i - 2 * D) : GD + gq * D + (i - D));
    const float* wt = a.taps_w + (size_t)c * taps;
    const float now = to_f32(pj[a.col + c]);
    float acc = 0.f;
    for (int j = 0; j < taps - 1; ++j) {
      const int p = pos - taps + 1 + j;
      if (p >= 0) acc = fmaf(wt[j], hs[(size_t)(p % taps) * C + c], acc);
    }
    acc = fmaf(wt[taps - 1], now, acc);
    if (is_v || h % rep == 0) hs[(size_t)(pos % taps) * C + c] = now;        // the ring's free row
    const float y = dl_silu(acc);
    if (i < D) q[i] = y; else if (is_v) v[i - 2 * D] = y; else k[i - D] = y;
  }
  if (lr.wz)
    for (int i = tid; i < lr.ra + lr.rg; i += DL_THREADS) xs[i] = to_f32(pj[lr.lr_col + i]);
  __syncthreads();
  if (warp == 0) {
    float sq = 0.f, sk = 0.f, kq = 0.f;
    for (int i = lane; i < D; i += 32) { sq = fmaf(q[i], q[i], sq); sk = fmaf(k[i], k[i], sk); kq = fmaf(q[i], k[i], kq); }
    sq = warp_sum(sq); sk = warp_sum(sk); kq = warp_sum(kq);
    const float fq = rsqrtf(sq + a.unit_eps) * a.q_scale, fk = rsqrtf(sk + a.unit_eps);
    if (lane == 0) { sc[0] = fq; sc[1] = fk; sc[2] = kq * fq * fk; }
  }
  const float ea = expf(a.a_log[h]);
  if (lr.wz) {
    const TO* wz = (const TO*)lr.wz;
    const int ld = lr.ra + lr.rg, grp = tid >> 3, sub = tid & 7;
    constexpr int VE = 16 / sizeof(TO);
    const bool va = lr.ra % VE == 0 && lr.rg % VE == 0;
    for (int r = grp; r < D + V; r += DL_THREADS / 8) {           // D + V is a multiple of the warps' 4 rows (checked by the host)
      const bool dec = r < D;
      const TO* wr = dec ? wz + (size_t)(h * D + r) * ld : wz + (size_t)(H * D + h * V + (r - D)) * ld + lr.ra;
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
  const float beta = dl_sigmoid(to_f32(pj[a.b_col + h]));
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
  return NI <= 32 && (size_t)(3 * D + 3 * V + ra + rg + 4 + 2048) * sizeof(float) <= 48 * 1024;
}
extern "C" int sx_delta_step_fits(int D, int V, int ra, int rg) { return dl_step_fits(D, V, ra, rg) ? 1 : 0; }

// ---------------------------------------------------------------------------------------------------------------
// chunks.  Scratch per (sequence, chunk, head): x, qg, kd [32, D] each, y [32, V], p [32, 32], ge [D].
// ---------------------------------------------------------------------------------------------------------------
struct DlChunks { float* x; float* qg; float* kd; float* y; float* p; float* ge; float* o; int P; };     // o [T, H V]

template <typename TP>
__global__ void __launch_bounds__(DL_THREADS, 2) delta_intra_kernel(DlArgs a, DlPrep w, DlChunks ch) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.D, V = a.V, H = a.H, DS = D + 4, G = a.G;
  float* ks = sm;                        // 32 * DS
  float* qs = ks + DL_C * DS;            // 32 * DS
  float* Gs = qs + DL_C * DS;            // 32 * DS: running sums of the decays' logarithms, base 2
  float* As = Gs + DL_C * DS;            // 32 * DL_LD
  float* bs = As + DL_C * DL_LD;         // 32
  pdl_wait();
  pdl_trigger();
  const int p = blockIdx.x, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x, gq = h / (H / G);
  const int t0 = a.cu_seqlens[s] + p * DL_C, len = a.cu_seqlens[s + 1] - t0;
  if (len <= 0) return;
  const int L = min(DL_C, len);
  const size_t ci = ((size_t)s * ch.P + p) * H + h;
  const int D4 = D >> 2;
  for (int i = tid; i < DL_C * D4; i += DL_THREADS) {
    const int t = i / D4, d = (i - t * D4) * 4;
    float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv;
    if (t < L) {
      const size_t at = (size_t)(t0 + t) * G * D + gq * D + d;
      kv = *reinterpret_cast<const float4*>(w.k + at);
      qv = *reinterpret_cast<const float4*>(w.q + at);
    }
    *reinterpret_cast<float4*>(ks + t * DS + d) = kv;
    *reinterpret_cast<float4*>(qs + t * DS + d) = qv;
  }
  if (tid < DL_C) bs[tid] = tid < L ? dl_sigmoid(to_f32(((const TP*)a.proj)[(size_t)(t0 + tid) * a.row + a.b_col + h])) : 0.f;
  for (int i = tid; i < DL_C * DL_LD; i += DL_THREADS) As[i] = 0.f;
  if (tid < D) {
    const float ea = -expf(a.a_log[h]) * DL_LOG2E, c = a.dt_bias[h * D + tid];
    const float* z = a.z + (size_t)t0 * a.z_ld + h * D + tid;
    float acc = 0.f;
#pragma unroll 8
    for (int t = 0; t < DL_C; ++t) {
      if (t < L) acc = fmaf(ea, dl_softplus(z[(size_t)t * a.z_ld] + c), acc);
      Gs[t * DS + tid] = acc;
    }
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
  float rhs[DL_C];
  float* X = ch.x + ci * DL_C * D;
  if (tid < D) {
    float* Q = ch.qg + ci * DL_C * D + tid;
    float* K = ch.kd + ci * DL_C * D + tid;
    float *gp = Gs + tid, *kp = ks + tid, *qp = qs + tid;      // walked row by row: 32 addresses held at once would spill
    const float gm = Gs[15 * DS + tid], ge = Gs[(DL_C - 1) * DS + tid];
    ch.ge[ci * D + tid] = dl_exp2(ge);
#pragma unroll
    for (int t = 0; t < DL_C; ++t) {
      asm volatile("" ::: "memory");
      const float gt = *gp, kt = *kp, qt = *qp;
      const float e = dl_exp2(gt);
      rhs[t] = bs[t] * e * kt;
      *Q = e * qt;
      *K = dl_exp2(ge - gt) * kt;
      const float f = dl_exp2(t < 16 ? gm - gt : gt - gm);
      *kp = f * kt;
      *qp = f * qt;
      Q += D; K += D; gp += DS; kp += DS; qp += DS;
    }
  } else if (tid < D + V) {
    const float* vp = w.v + (size_t)t0 * H * V + h * V + (tid - D);
#pragma unroll
    for (int t = 0; t < DL_C; ++t) {
      rhs[t] = t < L ? bs[t] * *vp : 0.f;
      if (t + 1 < L) vp += (size_t)H * V;
    }
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

__device__ __forceinline__ void dl_cp16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dl_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void dl_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// VS: columns of the state a block owns (32 or 16)
template <int VS>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(DlArgs a, DlChunks ch) {
  extern __shared__ __align__(16) float sm[];
  constexpr int SS = VS + 4;
  constexpr int CG = VS / 4;                       // groups of four columns
  constexpr int KSPLIT = DL_THREADS / (16 * CG);   // 2 or 4: parts of D in the products with S
  const int D = a.D, V = a.V, H = a.H, DS = D + 4;
  float* xq = sm;                                  // 64 * DS: X above e^G q
  float* kd = xq + 2 * DL_C * DS;                  // 32 * DS
  float* S = kd + DL_C * DS;                       // D * SS
  float* P = S + D * SS;                           // 32 * DL_LD
  float* U = P + DL_C * DL_LD;                     // 32 * SS: u of the chunk
  float* O = U + DL_C * SS;                        // 32 * SS: (e^G q) S
  float* part = O + DL_C * SS;                     // (KSPLIT - 1) * 64 * SS
  float* ge = part + (KSPLIT - 1) * 64 * SS;       // D
  pdl_wait();
  pdl_trigger();
  const int v0 = blockIdx.x * VS, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
  const int tok0 = a.cu_seqlens[s], n = a.cu_seqlens[s + 1] - tok0, np = (n + DL_C - 1) / DL_C;
  float* Sg = a.S + ((size_t)a.seq_slots[s] * H + h) * D * V;
  const int D4 = D >> 2;
  auto load_xq = [&](int p) {
    const size_t ci = ((size_t)s * ch.P + p) * H + h;
    const float *x = ch.x + ci * DL_C * D, *q = ch.qg + ci * DL_C * D;
    for (int i = tid; i < DL_C * D4; i += DL_THREADS) {
      const int t = i / D4, d = (i - t * D4) * 4;
      dl_cp16(xq + t * DS + d, x + (size_t)t * D + d);
      dl_cp16(xq + (DL_C + t) * DS + d, q + (size_t)t * D + d);
    }
    dl_commit();
  };
  auto load_kp = [&](int p) {
    const size_t ci = ((size_t)s * ch.P + p) * H + h;
    const float *k = ch.kd + ci * DL_C * D, *pg = ch.p + ci * DL_C * DL_C, *g = ch.ge + ci * D;
    for (int i = tid; i < DL_C * D4; i += DL_THREADS) {
      const int t = i / D4, d = (i - t * D4) * 4;
      dl_cp16(kd + t * DS + d, k + (size_t)t * D + d);
    }
    for (int i = tid; i < DL_C * DL_C / 4; i += DL_THREADS) dl_cp16(P + (i >> 3) * DL_LD + (i & 7) * 4, pg + i * 4);
    for (int i = tid; i < D4; i += DL_THREADS) dl_cp16(ge + i * 4, g + i * 4);
    dl_commit();
  };
  if (np > 0) { load_xq(0); load_kp(0); }
  for (int i = tid; i < D * VS; i += DL_THREADS) {
    const int d = i / VS, c = i - d * VS;
    S[d * SS + c] = v0 + c < V ? Sg[(size_t)d * V + v0 + c] : 0.f;
  }
  const int kg = tid / (16 * CG), rem = tid - kg * 16 * CG, rg = rem / CG, cg = rem - rg * CG;
  const int dper = (D4 + KSPLIT - 1) / KSPLIT * 4, da = kg * dper, db = min(D, da + dper);
  for (int p = 0; p < np; ++p) {
    const size_t ci = ((size_t)s * ch.P + p) * H + h;
    const int L = min(DL_C, n - p * DL_C);
    dl_wait<1>();
    __syncthreads();                               // X, q of this chunk and S of the last are in place
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int d = da; d < db; d += 4) {             // rows rg, rg + 16, rg + 32, rg + 48
      float4 b[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) b[x] = *reinterpret_cast<const float4*>(S + (d + x) * SS + cg * 4);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 m = *reinterpret_cast<const float4*>(xq + (rg + 16 * i) * DS + d);
        acc[i][0] = fmaf(m.x, b[0].x, fmaf(m.y, b[1].x, fmaf(m.z, b[2].x, fmaf(m.w, b[3].x, acc[i][0]))));
        acc[i][1] = fmaf(m.x, b[0].y, fmaf(m.y, b[1].y, fmaf(m.z, b[2].y, fmaf(m.w, b[3].y, acc[i][1]))));
        acc[i][2] = fmaf(m.x, b[0].z, fmaf(m.y, b[1].z, fmaf(m.z, b[2].z, fmaf(m.w, b[3].z, acc[i][2]))));
        acc[i][3] = fmaf(m.x, b[0].w, fmaf(m.y, b[1].w, fmaf(m.z, b[2].w, fmaf(m.w, b[3].w, acc[i][3]))));
      }
    }
    if (kg > 0) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float4*>(part + ((kg - 1) * 64 + rg + 16 * i) * SS + cg * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    }
    __syncthreads();                               // X and q are read out
    if (p + 1 < np) load_xq(p + 1); else dl_commit();
    if (kg == 0) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = rg + 16 * i;
        float4 v = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
#pragma unroll
        for (int x = 0; x < KSPLIT - 1; ++x) {
          const float4 o = *reinterpret_cast<const float4*>(part + (x * 64 + r) * SS + cg * 4);
          v.x += o.x; v.y += o.y; v.z += o.z; v.w += o.w;
        }
        if (i < 2) {                               // u = Y - X S
          const float* Y = ch.y + ci * DL_C * V + (size_t)r * V + v0 + cg * 4;
          const int left = V - (v0 + cg * 4);
          float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
          if (left >= 4 && (V & 3) == 0) y = *reinterpret_cast<const float4*>(Y);
          else {
            if (left > 0) y.x = Y[0];
            if (left > 1) y.y = Y[1];
            if (left > 2) y.z = Y[2];
            if (left > 3) y.w = Y[3];
          }
          *reinterpret_cast<float4*>(U + r * SS + cg * 4) = make_float4(y.x - v.x, y.y - v.y, y.z - v.z, y.w - v.w);
        } else {
          *reinterpret_cast<float4*>(O + (r - DL_C) * SS + cg * 4) = v;
        }
      }
    }
    dl_wait<1>();
    __syncthreads();                               // u, the first half of o, and this chunk's k, P, e^(G_end)
    {   // o: a thread two rows and VS / 16 columns
      constexpr int OC = VS / 16;
      const int r = (tid >> 4) * 2, c = (tid & 15) * OC;
      float o[2][OC];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < OC; ++j) o[i][j] = O[(r + i) * SS + c + j];
      for (int u = 0; u <= r + 1; u += 4) {        // P is zero above its diagonal
        const float4 p0 = *reinterpret_cast<const float4*>(P + r * DL_LD + u), p1 = *reinterpret_cast<const float4*>(P + (r + 1) * DL_LD + u);
#pragma unroll
        for (int j = 0; j < OC; ++j) {
          const float u0 = U[u * SS + c + j], u1 = U[(u + 1) * SS + c + j], u2 = U[(u + 2) * SS + c + j], u3 = U[(u + 3) * SS + c + j];
          o[0][j] = fmaf(p0.x, u0, fmaf(p0.y, u1, fmaf(p0.z, u2, fmaf(p0.w, u3, o[0][j]))));
          o[1][j] = fmaf(p1.x, u0, fmaf(p1.y, u1, fmaf(p1.z, u2, fmaf(p1.w, u3, o[1][j]))));
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (r + i < L) {
          float* og = ch.o + (size_t)(tok0 + p * DL_C + r + i) * H * V + h * V;
#pragma unroll
          for (int j = 0; j < OC; ++j)
            if (v0 + c + j < V) og[v0 + c + j] = o[i][j];
        }
    }
    {   // S: tiles of RT rows x 4 columns
      constexpr int RT = VS == 32 ? 4 : 2;
      const int tiles = (D / RT) * CG;
      for (int tile = tid; tile < tiles; tile += DL_THREADS) {
        const int d = (tile / CG) * RT, c = (tile % CG) * 4;
        float4 x[RT];
#pragma unroll
        for (int i = 0; i < RT; ++i) {
          const float e = ge[d + i];
          x[i] = *reinterpret_cast<const float4*>(S + (d + i) * SS + c);
          x[i].x *= e; x[i].y *= e; x[i].z *= e; x[i].w *= e;
        }
#pragma unroll 8
        for (int t = 0; t < DL_C; ++t) {
          const float4 u = *reinterpret_cast<const float4*>(U + t * SS + c);
          float kk[4];
          if (RT == 4) {
            const float4 f = *reinterpret_cast<const float4*>(kd + t * DS + d);
            kk[0] = f.x; kk[1] = f.y; kk[2] = f.z; kk[3] = f.w;
          } else {
            const float2 f = *reinterpret_cast<const float2*>(kd + t * DS + d);
            kk[0] = f.x; kk[1] = f.y;
          }
#pragma unroll
          for (int i = 0; i < RT; ++i) {
            x[i].x = fmaf(kk[i], u.x, x[i].x); x[i].y = fmaf(kk[i], u.y, x[i].y);
            x[i].z = fmaf(kk[i], u.z, x[i].z); x[i].w = fmaf(kk[i], u.w, x[i].w);
          }
        }
#pragma unroll
        for (int i = 0; i < RT; ++i) *reinterpret_cast<float4*>(S + (d + i) * SS + c) = x[i];
      }
    }
    __syncthreads();                               // k, P and u are read out
    if (p + 1 < np) load_kp(p + 1); else dl_commit();
  }
  dl_wait<0>();
  __syncthreads();
  for (int i = tid; i < D * VS; i += DL_THREADS) {
    const int d = i / VS, c = i - d * VS;
    if (v0 + c < V) Sg[(size_t)d * V + v0 + c] = S[d * SS + c];
  }
}

static size_t dl_scan_smem(int D, int VS) {
  const int SS = VS + 4, ksplit = DL_THREADS / (16 * (VS / 4));
  return (size_t)(3 * DL_C * (D + 4) + D * SS + DL_C * DL_LD + 2 * DL_C * SS + (ksplit - 1) * 64 * SS + D) * sizeof(float);
}

// a warp a (token, head): o / rms(o) * gain * sigmoid(gate)
template <typename TO>
__global__ void __launch_bounds__(DL_THREADS) delta_finish_kernel(DlArgs a, const float* __restrict__ o, int n_tokens) {
  pdl_wait();
  pdl_trigger();
  const int V = a.V, H = a.H, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (DL_THREADS / 32) + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * H) return;
  const int t = (int)(item / H), h = (int)(item % H);
  const float* x = o + (size_t)item * V;
  const float* z = a.z + (size_t)t * a.z_ld + H * a.D + h * V;
  TO* out = (TO*)a.out + (size_t)item * V;
  if (V == 128) {
    const float4 f = reinterpret_cast<const float4*>(x)[lane];
    const float4 gt = make_float4(z[lane * 4], z[lane * 4 + 1], z[lane * 4 + 2], z[lane * 4 + 3]);
    const float inv = rsqrtf(warp_sum(f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w) / 128.f + a.eps);
    const float* gn = a.gain + lane * 4;
    out[lane * 4] = from_f32<TO>(f.x * inv * gn[0] * dl_sigmoid(gt.x));
    out[lane * 4 + 1] = from_f32<TO>(f.y * inv * gn[1] * dl_sigmoid(gt.y));
    out[lane * 4 + 2] = from_f32<TO>(f.z * inv * gn[2] * dl_sigmoid(gt.z));
    out[lane * 4 + 3] = from_f32<TO>(f.w * inv * gn[3] * dl_sigmoid(gt.w));
    return;
  }
  float ss = 0.f;
  for (int c = lane; c < V; c += 32) ss += x[c] * x[c];
  const float inv = rsqrtf(warp_sum(ss) / (float)V + a.eps);
  for (int c = lane; c < V; c += 32) out[c] = from_f32<TO>(x[c] * inv * a.gain[c] * dl_sigmoid(z[c]));
}

extern "C" int sx_delta_chunk_tokens() { return DL_C; }
extern "C" int sx_delta_chunks_fit(int D, int V) {
  return (D % 4 == 0 && D <= DL_THREADS && dl_intra_smem(D) <= 220 * 1024 && dl_scan_smem(D, 32) <= 220 * 1024 &&
          dl_scan_smem(D, 16) <= 220 * 1024 && V > 0) ? 1 : 0;
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
static int dl_step_launch(const DlArgs& a, const DlLowRank& lr, int n_seqs, cudaStream_t stream) {
  const size_t smem = (size_t)(3 * a.D + 3 * a.V + lr.ra + lr.rg + 4 + 2048) * sizeof(float);
  const int NI = (a.D * a.V + 1023) / 1024;
  const dim3 grid(a.H, n_seqs), block(DL_THREADS);
#define DL_STEP(N) return sx_launch(delta_step_kernel<TP, TO, N>, grid, block, smem, stream, a, lr)
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
  const DlLowRank lr = {wz, wz ? ra : 0, wz ? rg : 0, lr_col};
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
    if (a.taps == 2) rc = sx_launch(delta_prepare_run_kernel<TP, 2>, grid, dim3(DL_THREADS), 0, stream, a, w, n_tokens);
    else if (a.taps == 3) rc = sx_launch(delta_prepare_run_kernel<TP, 3>, grid, dim3(DL_THREADS), 0, stream, a, w, n_tokens);
    else rc = sx_launch(delta_prepare_run_kernel<TP, 4>, grid, dim3(DL_THREADS), 0, stream, a, w, n_tokens);
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
static int dl_chunks_launch(const DlArgs& a, const DlPrep& w, const DlChunks& ch, int n_tokens, int n_seqs, int slice, cudaStream_t stream) {
  const size_t si = dl_intra_smem(a.D);
  if (si > 48 * 1024) cudaFuncSetAttribute(delta_intra_kernel<TP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)si);
  int rc = sx_launch(delta_intra_kernel<TP>, dim3(ch.P, a.H, n_seqs), dim3(DL_THREADS), si, stream, a, w, ch);
  if (rc) return rc;
  const size_t ss = dl_scan_smem(a.D, slice);
  const dim3 grid((a.V + slice - 1) / slice, a.H, n_seqs);
  if (slice == 32) {
    if (ss > 48 * 1024) cudaFuncSetAttribute(delta_scan_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ss);
    rc = sx_launch(delta_scan_kernel<32>, grid, dim3(DL_THREADS), ss, stream, a, ch);
  } else {
    if (ss > 48 * 1024) cudaFuncSetAttribute(delta_scan_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ss);
    rc = sx_launch(delta_scan_kernel<16>, grid, dim3(DL_THREADS), ss, stream, a, ch);
  }
  if (rc) return rc;
  const long long items = (long long)n_tokens * a.H;
  return sx_launch(delta_finish_kernel<TO>, dim3((unsigned)((items + DL_THREADS / 32 - 1) / (DL_THREADS / 32))), dim3(DL_THREADS), 0, stream, a,
                   (const float*)ch.o, n_tokens);
}

// chunks of DL_C tokens (the caller has asked sx_delta_chunks_fit); slice: columns of the state a block of the scan owns
extern "C" int sx_delta_chunks(DL_FORMALS, float* q, float* k, float* v, float* x, float* qg, float* kd, float* y, float* p,
                               float* ge, float* o, int chunks, int slice, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (dl_check(n_seqs, H, G, D, V, taps) || !sx_delta_chunks_fit(D, V) || (slice != 16 && slice != 32) || chunks <= 0) return SX_ERR_SIZE;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)x | (uintptr_t)qg | (uintptr_t)kd | (uintptr_t)y | (uintptr_t)p | (uintptr_t)ge | (uintptr_t)o) % 16)
    return SX_ERR_ALIGN;
  const DlArgs a = dl_args(DL_ACTUALS);
  const DlPrep w = {q, k, v};
  const DlChunks ch = {x, qg, kd, y, p, ge, o, chunks};
  if (proj_dt == SX_F32 && out_dt == SX_F32) return dl_chunks_launch<float, float>(a, w, ch, n_tokens, n_seqs, slice, stream);
  if (proj_dt == SX_F32 && out_dt == SX_BF16) return dl_chunks_launch<float, bf16>(a, w, ch, n_tokens, n_seqs, slice, stream);
  if (proj_dt == SX_BF16 && out_dt == SX_BF16) return dl_chunks_launch<bf16, bf16>(a, w, ch, n_tokens, n_seqs, slice, stream);
  return SX_ERR_DTYPE;
}
