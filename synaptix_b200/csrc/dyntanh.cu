// The norm without statistics behind the sum into the residual stream, in 32-bit:
//
//   v = h[t] (+ delta[t] + dbias);  if write_h: h[t] = v;  y[r] = tanh(alpha v) * w + b
//
// Rows: r = 0..R-1, t = rows ? rows[r] : r.  Every element stands on its own (no mean, no variance), so the work is split
// over elements and not over rows.  It is the form for where no product ends in the stream (a sequence's first norm, rows
// picked out for the output head, 32-bit); elsewhere the products finish this norm in their epilogues (dyn_tanh).
// delta may be float32 or bfloat16 whatever y is.
#include "common.cuh"

#define DT_THREADS 256

// V elements a thread (4 where the width is a multiple of 4 and all arrays are 16-byte aligned)
template <typename TO, typename TD, int V>
__global__ void __launch_bounds__(DT_THREADS) add_dyn_tanh_kernel(float* __restrict__ h, const TD* __restrict__ delta,
                                                                  const float* __restrict__ dbias, float alpha,
                                                                  const float* __restrict__ w, const float* __restrict__ b,
                                                                  TO* __restrict__ y, const int* __restrict__ rows, int W,
                                                                  int write_h, size_t total) {
  const size_t idx = (size_t)blockIdx.x * DT_THREADS + threadIdx.x;
  const int per = W / V;
  const size_t r = idx / per;
  const int c = (int)(idx - r * per) * V;
  float g[V], s[V], e[V];
#pragma unroll
  for (int i = 0; i < V; ++i) e[i] = 0.f;
  if (idx < total) {                       // weights: asked for ahead of the wait
#pragma unroll
    for (int i = 0; i < V; ++i) { g[i] = __ldg(w + c + i); s[i] = __ldg(b + c + i); }
    if (dbias)
#pragma unroll
      for (int i = 0; i < V; ++i) e[i] = __ldg(dbias + c + i);
  }
  pdl_wait();
  pdl_trigger();
  if (idx >= total) return;
  const size_t t = rows ? (size_t)rows[r] : r;
  float* hp = h + t * W + c;
  float v[V];
  if (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(hp);
    v[0] = f.x; v[V > 1 ? 1 : 0] = f.y; v[V > 2 ? 2 : 0] = f.z; v[V > 3 ? 3 : 0] = f.w;
  } else {
    v[0] = *hp;
  }
  if (delta) {
    const TD* d = delta + t * W + c;
    float f[V];
    if (V == 4 && sizeof(TD) == 2) {
      const uint2 u = *reinterpret_cast<const uint2*>(d);
      const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
      const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
      f[0] = lo.x; f[V > 1 ? 1 : 0] = lo.y; f[V > 2 ? 2 : 0] = hi.x; f[V > 3 ? 3 : 0] = hi.y;
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = to_f32(d[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] += f[i] + e[i];
    if (write_h) {
      if (V == 4) *reinterpret_cast<float4*>(hp) = make_float4(v[0], v[V > 1 ? 1 : 0], v[V > 2 ? 2 : 0], v[V > 3 ? 3 : 0]);
      else *hp = v[0];
    }
  }
  __align__(16) TO o[V];
#pragma unroll
  for (int i = 0; i < V; ++i) o[i] = from_f32<TO>(dyn_tanh(v[i], alpha, g[i], s[i]));
  TO* yp = y + r * W + c;
  if (V == 4 && sizeof(TO) == 2) *reinterpret_cast<uint2*>(yp) = *reinterpret_cast<const uint2*>(o);
  else if (V == 4) *reinterpret_cast<uint4*>(yp) = *reinterpret_cast<const uint4*>(o);
  else *yp = o[0];
}

template <typename TO, typename TD>
static int dyn_tanh_launch(float* h, const void* delta, const float* dbias, float alpha, const float* w, const float* b, void* y,
                           const int* rows, int R, int W, int write_h, bool vec, cudaStream_t stream) {
  const size_t total = (size_t)R * (vec ? W / 4 : W);
  const size_t blocks = (total + DT_THREADS - 1) / DT_THREADS;
  if (blocks > 0x7fffffffULL) return SX_ERR_SIZE;
  if (vec)
    return sx_launch(add_dyn_tanh_kernel<TO, TD, 4>, dim3((unsigned)blocks), dim3(DT_THREADS), 0, stream, h, (const TD*)delta, dbias,
                     alpha, w, b, (TO*)y, rows, W, write_h, total);
  return sx_launch(add_dyn_tanh_kernel<TO, TD, 1>, dim3((unsigned)blocks), dim3(DT_THREADS), 0, stream, h, (const TD*)delta, dbias,
                   alpha, w, b, (TO*)y, rows, W, write_h, total);
}

extern "C" int sx_add_dyn_tanh(float* h, const void* delta, int delta_dt, const float* dbias, float alpha, const float* w,
                               const float* b, void* y, int out_dt, const int* rows, int R, int W, int write_h,
                               cudaStream_t stream) {
  if (R <= 0) return 0;
  if (W <= 0 || (rows && write_h)) return SX_ERR_SIZE;
  const bool vec = W % 4 == 0 && (((uintptr_t)h | (uintptr_t)delta | (uintptr_t)y) & 15) == 0;
  if (delta && delta_dt != SX_F32 && delta_dt != SX_BF16) return SX_ERR_DTYPE;
  const bool d16 = delta && delta_dt == SX_BF16;
  if (out_dt == SX_F32)
    return d16 ? dyn_tanh_launch<float, bf16>(h, delta, dbias, alpha, w, b, y, rows, R, W, write_h, vec, stream)
               : dyn_tanh_launch<float, float>(h, delta, dbias, alpha, w, b, y, rows, R, W, write_h, vec, stream);
  if (out_dt == SX_BF16)
    return d16 ? dyn_tanh_launch<bf16, bf16>(h, delta, dbias, alpha, w, b, y, rows, R, W, write_h, vec, stream)
               : dyn_tanh_launch<bf16, float>(h, delta, dbias, alpha, w, b, y, rows, R, W, write_h, vec, stream);
  return SX_ERR_DTYPE;
}
