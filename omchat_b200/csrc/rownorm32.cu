// Row kernels of decoders whose residual stream is fp32: scaled embedding gather, RMS norm of fp32 rows, and the
// output-side norm + residual add (x <- x + y / rms(y) * (1 + g)) that also emits the rounded copy the next sublayer reads.
// One CTA per row; the row is read once into registers / shared memory, the statistics are fp32. HBM-bound row work.
#include "seq_common.cuh"

namespace omc {

template <typename TT, typename TB>
__global__ void __launch_bounds__(256) embed_scale_kernel(const int32_t* __restrict__ ids, const TT* __restrict__ table, int C,
                                                          int vocab, float scale, float* __restrict__ h32, long long ldh,
                                                          TB* __restrict__ xb, long long ldxb) {
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float v = ok ? ldf(table + (long long)id * C + c) * scale : 0.f;
    h32[(long long)t * ldh + c] = v;
    if (xb != nullptr) stf(xb + (long long)t * ldxb + c, v);
  }
}

// Embedding row plus a row chosen by the hashed pair (previous token, token) of the same sequence: row (prev mul_prev + cur mul_cur) mod
// buckets of the second table, for a sequence's first token its row number `buckets` (the last one). The previous token is the row
// before when that belongs to the same request, else the slot's state prev[slot]. The row goes to the fp32 stream, and its RMS
// norm with weight nw, rounded, to xb (what the first sublayer reads). save_here: every row of the step is a request of its own, so
// the slot's state is updated from here; else last_token_save_kernel does that behind this launch.
template <typename TT, typename TB>
__global__ void __launch_bounds__(256) embed_bigram_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ pos,
                                                           const int32_t* __restrict__ slot, const TT* __restrict__ table, int C, int vocab,
                                                           const TT* __restrict__ bigram, int buckets, int mul_prev, int mul_cur,
                                                           int32_t* __restrict__ prev, const TT* __restrict__ nw, float eps,
                                                           float* __restrict__ h32, long long ldh, TB* __restrict__ xb, long long ldxb, int save_here, int vec) {
  extern __shared__ __align__(16) float erow[];  // [C]
  float* row = erow;
  __shared__ float red[33];
  __shared__ int s_row;
  const int t = blockIdx.x, id = ids[t];
  if (threadIdx.x == 0) {
    const int s = slot[t];
    long long b = buckets;
    if (pos[t] > 0) {
      const long long before = (t > 0 && slot[t - 1] == s) ? ids[t - 1] : prev[s];
      b = (before * mul_prev + (long long)id * mul_cur) % buckets;
      if (b < 0) b += buckets;
    }
    s_row = (int)b;
    if (save_here) prev[s] = id;   // read above by this thread, and by no other
  }
  __syncthreads();
  const bool ok = id >= 0 && id < vocab;
  const TT* br = bigram + (long long)s_row * C;
  float ss = 0.f;
  if (vec) {   // four neighbouring columns at a time
    for (int c = threadIdx.x * 4; c < C; c += blockDim.x * 4) {
      float v[4] = {0.f, 0.f, 0.f, 0.f}, b[4];
      if (ok) ld4(table + (long long)id * C + c, v);
      ld4(br + c, b);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] += b[e], ss = fmaf(v[e], v[e], ss);
      st4(h32 + (long long)t * ldh + c, v);
      st4(row + c, v);
    }
    if (xb == nullptr) return;
    ss = block_sum(ss, red);
    const float rstd = 1.f / sqrtf(ss / (float)C + eps);
    for (int c = threadIdx.x * 4; c < C; c += blockDim.x * 4) {
      float v[4], w[4];
      ld4(row + c, v);
      ld4(nw + c, w);
      const float o[4] = {v[0] * rstd * w[0], v[1] * rstd * w[1], v[2] * rstd * w[2], v[3] * rstd * w[3]};
      st4(xb + (long long)t * ldxb + c, o);
    }
    return;
  }
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float v = (ok ? ldf(table + (long long)id * C + c) : 0.f) + ldf(br + c);
    h32[(long long)t * ldh + c] = v;
    row[c] = v;
    ss = fmaf(v, v, ss);
  }
  if (xb == nullptr) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)C + eps);
  for (int c = threadIdx.x; c < C; c += blockDim.x) stf(xb + (long long)t * ldxb + c, row[c] * rstd * ldf(nw + c));   // every thread rereads only what it wrote
}

__global__ void __launch_bounds__(256) last_token_save_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ slot, int T,
                                                              int32_t* __restrict__ prev) {
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t < T && (t + 1 == T || slot[t + 1] != slot[t])) prev[slot[t]] = ids[t];
}

// Embedding row plus the sinusoidal position vector: entry 2i is sin(p * f_i), entry 2i + 1 is cos(p * f_i). The angle is formed
// and reduced in double precision (f_i arrives as a double table), so it is exact to fp32 at any position.
template <typename TT>
__global__ void __launch_bounds__(256) embed_sinusoid_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ pos,
                                                             const TT* __restrict__ table, int C, int vocab, float scale,
                                                             const double* __restrict__ freq, float* __restrict__ h32, long long ldh) {
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  const double p = (double)pos[t];
  for (int i = threadIdx.x; 2 * i < C; i += blockDim.x) {
    double sn, cs;
    sincos(p * freq[i], &sn, &cs);
    const int c = 2 * i;
    h32[(long long)t * ldh + c] = (ok ? ldf(table + (long long)id * C + c) * scale : 0.f) + (float)sn;
    if (c + 1 < C) h32[(long long)t * ldh + c + 1] = (ok ? ldf(table + (long long)id * C + c + 1) * scale : 0.f) + (float)cs;
  }
}

template <typename TW, typename TY>
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* __restrict__ x, long long ldx, const TW* __restrict__ w,
                                                       int one_plus, float eps, TY* __restrict__ y, long long ldy, int n) {
  __shared__ float red[33];
  const float* xr = x + (long long)blockIdx.x * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float v = xr[c];
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)n + eps);
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    float g = 1.f;
    if (w != nullptr) g = one_plus ? 1.f + ldf(w + c) : ldf(w + c);
    stf(y + (long long)blockIdx.x * ldy + c, xr[c] * rstd * g);
  }
}

template <typename TW, typename TB>
__global__ void __launch_bounds__(256) norm_residual_kernel(const float* __restrict__ y, long long ldy, const TW* __restrict__ w,
                                                            float eps, float* __restrict__ h32, long long ldh,
                                                            TB* __restrict__ xb, long long ldxb, int C) {
  __shared__ float red[33];
  const float* yr = y + (long long)blockIdx.x * ldy;
  float ss = 0.f;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float v = yr[c];
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)C + eps);
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float v = h32[(long long)blockIdx.x * ldh + c] + yr[c] * rstd * (1.f + ldf(w + c));
    h32[(long long)blockIdx.x * ldh + c] = v;
    if (xb != nullptr) stf(xb + (long long)blockIdx.x * ldxb + c, v);
  }
}


// Sublayer output -> residual stream -> next sublayer's input, one CTA per row, the row staged in shared memory:
//   y = y1                                               (y2 == NULL)
//   y = (y1 / rms(y1) * wa + y2 / rms(y2) * wb) / 2      (two mixers side by side, each normed with a plain weight first)
//   h32 += mult * y / rms(y) * (1 + w_post)
//   xb = h32 / rms(h32) * (1 + w_next)   (w_next == NULL: xb = round(h32); xb == NULL: nothing)
template <typename TW, typename TB>
__global__ void __launch_bounds__(256) post_norm_residual_kernel(const float* __restrict__ y1, long long ld1, const TW* __restrict__ wa,
                                                                 const float* __restrict__ y2, long long ld2, const TW* __restrict__ wb,
                                                                 const TW* __restrict__ w_post, float eps, float mult,
                                                                 float* __restrict__ h32, long long ldh, const TW* __restrict__ w_next,
                                                                 TB* __restrict__ xb, long long ldxb, int C) {
  extern __shared__ float row[];  // [C]
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float s1 = 0.f, s2 = 0.f;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    const float a = y1[t * ld1 + c];
    s1 = fmaf(a, a, s1);
    if (y2 != nullptr) {
      const float b = y2[t * ld2 + c];
      s2 = fmaf(b, b, s2);
    }
  }
  s1 = block_sum(s1, red);
  float ss = 0.f;
  if (y2 != nullptr) {
    s2 = block_sum(s2, red);
    const float r1 = 1.f / sqrtf(s1 / (float)C + eps), r2 = 1.f / sqrtf(s2 / (float)C + eps);
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
      const float v = 0.5f * (y1[t * ld1 + c] * r1 * ldf(wa + c) + y2[t * ld2 + c] * r2 * ldf(wb + c));
      row[c] = v;
      ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
  } else {
    for (int c = threadIdx.x; c < C; c += blockDim.x) row[c] = y1[t * ld1 + c];
    ss = s1;
  }
  const float rstd = 1.f / sqrtf(ss / (float)C + eps);
  float sh = 0.f;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {   // every thread rereads only what it wrote
    const float v = h32[t * ldh + c] + mult * (row[c] * rstd * (1.f + ldf(w_post + c)));
    h32[t * ldh + c] = v;
    row[c] = v;
    sh = fmaf(v, v, sh);
  }
  if (xb == nullptr) return;
  if (w_next == nullptr) {
    for (int c = threadIdx.x; c < C; c += blockDim.x) stf(xb + t * ldxb + c, row[c]);
    return;
  }
  sh = block_sum(sh, red);
  const float rn = 1.f / sqrtf(sh / (float)C + eps);
  for (int c = threadIdx.x; c < C; c += blockDim.x) stf(xb + t * ldxb + c, row[c] * rn * (1.f + ldf(w_next + c)));
}

// out = act(gate) * up over the two halves of a stacked projection: z [rows, 2 * n] -> out [rows, n]; the arithmetic is fp32.
// Four neighbouring columns per thread (8- or 16-byte accesses) when the rows are laid out for it, else one.
struct GluParams {
  int act;
  float limit, slope, shift;   // OMC_ACT_CLAMP_SWISH only
};
__device__ __forceinline__ float glu_pair(float g, float u, const GluParams& p) {
  if (p.act == OMC_ACT_CLAMP_SWISH) {
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    return g / (1.f + expf(-p.slope * g)) * (u + p.shift);
  }
  if (p.act == OMC_ACT_GELU_TANH) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  if (p.act == OMC_ACT_GELU_ERF) return 0.5f * g * (1.f + erff(g * 0.70710678118654752f)) * u;
  if (p.act == OMC_ACT_RELU2) return fmaxf(g, 0.f) * fmaxf(g, 0.f) * u;
  if (p.act == OMC_ACT_SILU) return g / (1.f + expf(-g)) * u;
  return g * u;
}

template <typename TZ, typename TY, int VEC>
__global__ void __launch_bounds__(256) glu_mul_kernel(const TZ* __restrict__ z, long long ldz, int n, GluParams gp, TY* __restrict__ y,
                                                      long long ldy, long long total, const int32_t* __restrict__ tile_group, int tile) {
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;   // one thread per VEC columns
  if (e >= total) return;
  const int per_row = n / VEC;
  const long long t = e / per_row;
  const int c = (int)(e - t * per_row) * VEC;
  if (tile_group != nullptr && tile_group[t / tile] < 0) return;   // a tile of the expert-sorted layout that no expert uses
  if (VEC == 4) {
    float g[4], u[4];
    ld4(z + t * ldz + c, g);
    ld4(z + t * ldz + n + c, u);
#pragma unroll
    for (int i = 0; i < 4; ++i) g[i] = glu_pair(g[i], u[i], gp);
    st4(y + t * ldy + c, g);
  } else {
    stf(y + t * ldy + c, glu_pair(ldf(z + t * ldz + c), ldf(z + t * ldz + n + c), gp));
  }
}


// y[t, c] = tanh(alpha * x[t, c]) * w[c] + b[c]: a norm without statistics (alpha one scalar in device memory).
template <typename TW, typename TY>
__global__ void __launch_bounds__(256) dyt_rows_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ alpha_p,
                                                       const TW* __restrict__ w, const TW* __restrict__ b, TY* __restrict__ y, long long ldy,
                                                       int C, long long total) {
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= total) return;
  const long long t = e / C;
  const int c = (int)(e - t * C);
  stf(y + t * ldy + c, fmaf(tanhf(*alpha_p * x[t * ldx + c]), ldf(w + c), ldf(b + c)));
}

// x[t, c] <- cap * tanh(x[t, c] / cap), in place.
__global__ void __launch_bounds__(256) tanh_cap_rows_kernel(float* __restrict__ x, long long ldx, int cols, long long total, float cap) {
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= total) return;
  const long long t = e / cols;
  float* p = x + t * ldx + (e - t * cols);
  *p = cap * tanhf(*p / cap);
}

// ---- layer norm after the residual sum --------------------------------------------------------------------------------------
//   v = alpha * x[t] + y[t] + sum_j w[t, j] * ys[slot_of[t, j]]        (y, ys: absent terms are zero)
//   o = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * nw + nb    -> x_out[t] (fp32 stream), xb[t] (rounded: the next input)
// RMS: the norm stands before the sublayer instead. The sum v itself is the stream (x_out[t] = v), and what the next sublayer reads is
// xb[t] = v / sqrt(mean(v^2) + eps) * nw.
// One CTA per row; a thread keeps its NV float4 pieces of the row in registers (the variance is taken about the mean, two block
// reductions with one barrier each). Rows that are not laid out for float4 or too wide go through shared memory instead (VEC false).
struct LnResArgs {
  const float* x;
  long long ldx;
  float alpha;
  const float* y;
  long long ldy;
  const float* ys;
  long long ldys;
  const int32_t* slot_of;
  const float* w;
  int top;
  const void* nw;
  const void* nb;
  float eps;
  float* x_out;
  long long ldxo;
  void* xb;
  long long ldxb;
  int C;
};

template <int NT>
__device__ __forceinline__ float row_sum(float v, float* red) {  // red: a [NT / 32] piece of shared memory no other reduction uses
  v = seq_warp_sum(v);
  if (NT == 32) return v;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) s += red[i];
  return s;
}

template <typename TW, typename TB, int NT, int NV, bool RMS>
__global__ void __launch_bounds__(NT) ln_residual_kernel(LnResArgs a) {
  __shared__ float red[2][NT / 32];
  const long long t = blockIdx.x;
  float4 v[NV];
  const float* xr = a.x + t * a.ldx;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * NT + threadIdx.x) * 4;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < a.C) {
      const float4 q = *reinterpret_cast<const float4*>(xr + c);
      v[i] = make_float4(a.alpha * q.x, a.alpha * q.y, a.alpha * q.z, a.alpha * q.w);
      if (a.y != nullptr) {
        const float4 u = *reinterpret_cast<const float4*>(a.y + t * a.ldy + c);
        v[i].x += u.x, v[i].y += u.y, v[i].z += u.z, v[i].w += u.w;
      }
    }
  }
  if (a.ys != nullptr) {
#pragma unroll 4
    for (int k = 0; k < a.top; ++k) {
      const int sl = a.slot_of[t * a.top + k];
      if (sl < 0) continue;
      const float wk = a.w[t * a.top + k];
      const float* yr = a.ys + (long long)sl * a.ldys;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * NT + threadIdx.x) * 4;
        if (c < a.C) {
          const float4 u = *reinterpret_cast<const float4*>(yr + c);
          v[i].x = fmaf(wk, u.x, v[i].x), v[i].y = fmaf(wk, u.y, v[i].y), v[i].z = fmaf(wk, u.z, v[i].z), v[i].w = fmaf(wk, u.w, v[i].w);
        }
      }
    }
  }
  float s = 0.f;
  if (RMS) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + threadIdx.x) * 4;
      if (a.x_out != nullptr && c < a.C) *reinterpret_cast<float4*>(a.x_out + t * a.ldxo + c) = v[i];
      s = fmaf(v[i].x, v[i].x, s), s = fmaf(v[i].y, v[i].y, s), s = fmaf(v[i].z, v[i].z, s), s = fmaf(v[i].w, v[i].w, s);
    }
    if (a.xb == nullptr) return;
    const float rstd = 1.f / sqrtf(row_sum<NT>(s, red[0]) / (float)a.C + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * NT + threadIdx.x) * 4;
      if (c < a.C) {
        float w4[4];
        ld4(static_cast<const TW*>(a.nw) + c, w4);
        const float o[4] = {v[i].x * rstd * w4[0], v[i].y * rstd * w4[1], v[i].z * rstd * w4[2], v[i].w * rstd * w4[3]};
        st4(static_cast<TB*>(a.xb) + t * a.ldxb + c, o);
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  const float mean = row_sum<NT>(s, red[0]) / (float)a.C;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if ((i * NT + (int)threadIdx.x) * 4 < a.C) {
      v[i].x -= mean, v[i].y -= mean, v[i].z -= mean, v[i].w -= mean;
      s = fmaf(v[i].x, v[i].x, s), s = fmaf(v[i].y, v[i].y, s), s = fmaf(v[i].z, v[i].z, s), s = fmaf(v[i].w, v[i].w, s);
    }
  }
  const float rstd = 1.f / sqrtf(row_sum<NT>(s, red[1]) / (float)a.C + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * NT + threadIdx.x) * 4;
    if (c < a.C) {
      float w4[4], b4[4];
      ld4(static_cast<const TW*>(a.nw) + c, w4);
      ld4(static_cast<const TW*>(a.nb) + c, b4);
      const float o[4] = {fmaf(v[i].x * rstd, w4[0], b4[0]), fmaf(v[i].y * rstd, w4[1], b4[1]), fmaf(v[i].z * rstd, w4[2], b4[2]),
                          fmaf(v[i].w * rstd, w4[3], b4[3])};
      if (a.x_out != nullptr) st4(a.x_out + t * a.ldxo + c, o);
      if (a.xb != nullptr) st4(static_cast<TB*>(a.xb) + t * a.ldxb + c, o);
    }
  }
}

template <typename TW, typename TB, bool RMS>
__global__ void __launch_bounds__(256) ln_residual_any_kernel(LnResArgs a) {
  extern __shared__ float row[];  // [C]
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float s = 0.f;
  for (int c = threadIdx.x; c < a.C; c += blockDim.x) {
    float v = a.alpha * a.x[t * a.ldx + c];
    if (a.y != nullptr) v += a.y[t * a.ldy + c];
    if (a.ys != nullptr)
      for (int k = 0; k < a.top; ++k) {
        const int sl = a.slot_of[t * a.top + k];
        if (sl >= 0) v = fmaf(a.w[t * a.top + k], a.ys[(long long)sl * a.ldys + c], v);
      }
    row[c] = v;
    s += RMS ? v * v : v;
    if (RMS && a.x_out != nullptr) a.x_out[t * a.ldxo + c] = v;
  }
  if (RMS) {
    if (a.xb == nullptr) return;
    const float rstd = 1.f / sqrtf(block_sum(s, red) / (float)a.C + a.eps);
    for (int c = threadIdx.x; c < a.C; c += blockDim.x) stf(static_cast<TB*>(a.xb) + t * a.ldxb + c, row[c] * rstd * ldf(static_cast<const TW*>(a.nw) + c));
    return;
  }
  const float mean = block_sum(s, red) / (float)a.C;
  s = 0.f;
  for (int c = threadIdx.x; c < a.C; c += blockDim.x) {   // every thread rereads only what it wrote
    const float d = row[c] - mean;
    s = fmaf(d, d, s);
  }
  const float rstd = 1.f / sqrtf(block_sum(s, red) / (float)a.C + a.eps);
  for (int c = threadIdx.x; c < a.C; c += blockDim.x) {
    const float o = fmaf((row[c] - mean) * rstd, ldf(static_cast<const TW*>(a.nw) + c), ldf(static_cast<const TW*>(a.nb) + c));
    if (a.x_out != nullptr) a.x_out[t * a.ldxo + c] = o;
    if (a.xb != nullptr) stf(static_cast<TB*>(a.xb) + t * a.ldxb + c, o);
  }
}

template <typename TW, typename TB, bool RMS>
static int launch_ln_residual(const LnResArgs& a, int rows, cudaStream_t st) {
  auto al = [](const void* p, size_t n) { return p == nullptr || reinterpret_cast<uintptr_t>(p) % n == 0; };
  const bool vec = a.C % 4 == 0 && a.C <= 8192 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.ldys % 4 == 0 && a.ldxo % 4 == 0 && a.ldxb % 4 == 0 &&
                   al(a.x, 16) && al(a.y, 16) && al(a.ys, 16) && al(a.x_out, 16) && al(a.nw, 4 * sizeof(TW)) && al(a.nb, 4 * sizeof(TW)) &&
                   al(a.xb, 4 * sizeof(TB));
  if (vec) {
    if (a.C <= 256) ln_residual_kernel<TW, TB, 64, 1, RMS><<<rows, 64, 0, st>>>(a);
    else if (a.C <= 512) ln_residual_kernel<TW, TB, 128, 1, RMS><<<rows, 128, 0, st>>>(a);
    else if (a.C <= 1024) ln_residual_kernel<TW, TB, 256, 1, RMS><<<rows, 256, 0, st>>>(a);
    else if (a.C <= 2048) ln_residual_kernel<TW, TB, 256, 2, RMS><<<rows, 256, 0, st>>>(a);
    else if (a.C <= 4096) ln_residual_kernel<TW, TB, 256, 4, RMS><<<rows, 256, 0, st>>>(a);
    else ln_residual_kernel<TW, TB, 256, 8, RMS><<<rows, 256, 0, st>>>(a);
  } else {
    const size_t smem = (size_t)a.C * sizeof(float);
    if (smem > 200 * 1024) return set_error(OMC_ERR_SHAPE, "omc_ln_residual: row too wide for shared memory");
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(ln_residual_any_kernel<TW, TB, RMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return set_error(OMC_ERR_CUDA, cudaGetErrorString(e));
    }
    ln_residual_any_kernel<TW, TB, RMS><<<rows, 256, smem, st>>>(a);
  }
  return check_launch("omc_ln_residual");
}

}  // namespace omc

using namespace omc;

extern "C" int omc_embed_scale(const int32_t* ids, int T, const void* table, int t_dt, int C, int vocab, float scale, float* h32,
                               long long ldh, void* xb, int xb_dt, long long ldxb, void* stream) {
  if (ids == nullptr || table == nullptr || h32 == nullptr || T < 0 || C <= 0) return set_error(OMC_ERR_ARG, "omc_embed_scale: bad argument");
  if (T == 0) return OMC_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(t_dt, TT, OMC_DT_SWITCH(xb_dt, TB, {
    embed_scale_kernel<TT, TB><<<T, 256, 0, st>>>(ids, static_cast<const TT*>(table), C, vocab, scale, h32, ldh,
                                                   static_cast<TB*>(xb), ldxb);
  }))
  return check_launch("omc_embed_scale");
}

extern "C" int omc_rms_rows(const float* x, long long ldx, const void* w, int w_dt, int one_plus, float eps, void* y, int y_dt,
                            long long ldy, int rows, int n, void* stream) {
  if (x == nullptr || y == nullptr || rows < 0 || n <= 0) return set_error(OMC_ERR_ARG, "omc_rms_rows: bad argument");
  if (rows == 0) return OMC_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(y_dt, TY, {
    rms_rows_kernel<TW, TY><<<rows, 256, 0, st>>>(x, ldx, static_cast<const TW*>(w), one_plus, eps, static_cast<TY*>(y), ldy, n);
  }))
  return check_launch("omc_rms_rows");
}

extern "C" int omc_norm_residual(const float* y, long long ldy, const void* w, int w_dt, float eps, float* h32, long long ldh,
                                 void* xb, int xb_dt, long long ldxb, int rows, int C, void* stream) {
  if (y == nullptr || w == nullptr || h32 == nullptr || rows < 0 || C <= 0) return set_error(OMC_ERR_ARG, "omc_norm_residual: bad argument");
  if (rows == 0) return OMC_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(xb_dt, TB, {
    norm_residual_kernel<TW, TB><<<rows, 256, 0, st>>>(y, ldy, static_cast<const TW*>(w), eps, h32, ldh, static_cast<TB*>(xb), ldxb, C);
  }))
  return check_launch("omc_norm_residual");
}

extern "C" int omc_post_norm_residual(const float* y1, long long ld1, const void* wa, const float* y2, long long ld2, const void* wb,
                                      const void* w_post, int w_dt, float eps, float mult, float* h32, long long ldh,
                                      const void* w_next, void* xb, int xb_dt, long long ldxb, int rows, int C, void* stream) {
  if (y1 == nullptr || w_post == nullptr || h32 == nullptr || rows < 0 || C <= 0 || (y2 != nullptr && (wa == nullptr || wb == nullptr)))
    return set_error(OMC_ERR_ARG, "omc_post_norm_residual: bad argument");
  if (rows == 0) return OMC_OK;
  const size_t smem = (size_t)C * sizeof(float);
  if (smem > 200 * 1024) return set_error(OMC_ERR_SHAPE, "omc_post_norm_residual: row too wide for shared memory");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(xb_dt, TB, {
    if (smem > 48 * 1024) cudaFuncSetAttribute(post_norm_residual_kernel<TW, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    post_norm_residual_kernel<TW, TB><<<rows, 256, smem, st>>>(y1, ld1, static_cast<const TW*>(wa), y2, ld2, static_cast<const TW*>(wb),
                                                               static_cast<const TW*>(w_post), eps, mult, h32, ldh,
                                                               static_cast<const TW*>(w_next), static_cast<TB*>(xb), ldxb, C);
  }))
  return check_launch("omc_post_norm_residual");
}

extern "C" int omc_glu_mul(const void* z, int z_dt, long long ldz, int rows, int n, int act, float limit, float slope, float shift,
                           void* y, int y_dt, long long ldy, const int32_t* tile_group, int tile, void* stream) {
  if (z == nullptr || y == nullptr || rows < 0 || n <= 0 || (tile_group != nullptr && tile <= 0)) return set_error(OMC_ERR_ARG, "omc_glu_mul: bad argument");
  if (rows == 0) return OMC_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long total = (long long)rows * n;
  const bool vec = n % 4 == 0 && ldz % 4 == 0 && ldy % 4 == 0 && reinterpret_cast<uintptr_t>(z) % 16 == 0 && reinterpret_cast<uintptr_t>(y) % 16 == 0;
  const GluParams gp{act, limit, slope, shift};
  OMC_DT_SWITCH(z_dt, TZ, OMC_DT_SWITCH(y_dt, TY, {
    if (vec) glu_mul_kernel<TZ, TY, 4><<<(unsigned)((total / 4 + 255) / 256), 256, 0, st>>>(static_cast<const TZ*>(z), ldz, n, gp, static_cast<TY*>(y), ldy, total / 4, tile_group, tile);
    else glu_mul_kernel<TZ, TY, 1><<<(unsigned)((total + 255) / 256), 256, 0, st>>>(static_cast<const TZ*>(z), ldz, n, gp, static_cast<TY*>(y), ldy, total, tile_group, tile);
  }))
  return check_launch("omc_glu_mul");
}

extern "C" int omc_embed_sinusoid(const int32_t* ids, const int32_t* pos, int T, const void* table, int t_dt, int C, int vocab, float scale,
                                  const double* freq, float* h32, long long ldh, void* stream) {
  if (ids == nullptr || pos == nullptr || table == nullptr || freq == nullptr || h32 == nullptr || T < 0 || C <= 0)
    return set_error(OMC_ERR_ARG, "omc_embed_sinusoid: bad argument");
  if (T == 0) return OMC_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(t_dt, TT, {
    embed_sinusoid_kernel<TT><<<T, 256, 0, st>>>(ids, pos, static_cast<const TT*>(table), C, vocab, scale, freq, h32, ldh);
  })
  return check_launch("omc_embed_sinusoid");
}

extern "C" int omc_dyt_rows(const float* x, long long ldx, const float* alpha, const void* w, const void* b, int w_dt, void* y, int y_dt,
                            long long ldy, int rows, int C, void* stream) {
  if (x == nullptr || alpha == nullptr || w == nullptr || b == nullptr || y == nullptr || rows < 0 || C <= 0)
    return set_error(OMC_ERR_ARG, "omc_dyt_rows: bad argument");
  if (rows == 0) return OMC_OK;
  const long long total = (long long)rows * C;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(y_dt, TY, {
    dyt_rows_kernel<TW, TY><<<(unsigned)((total + 255) / 256), 256, 0, st>>>(x, ldx, alpha, static_cast<const TW*>(w), static_cast<const TW*>(b),
                                                                            static_cast<TY*>(y), ldy, C, total);
  }))
  return check_launch("omc_dyt_rows");
}

extern "C" int omc_tanh_cap_rows(float* x, long long ldx, int rows, int cols, float cap, void* stream) {
  if (x == nullptr || rows < 0 || cols <= 0 || !(cap > 0.f)) return set_error(OMC_ERR_ARG, "omc_tanh_cap_rows: bad argument");
  if (rows == 0) return OMC_OK;
  const long long total = (long long)rows * cols;
  tanh_cap_rows_kernel<<<(unsigned)((total + 255) / 256), 256, 0, static_cast<cudaStream_t>(stream)>>>(x, ldx, cols, total, cap);
  return check_launch("omc_tanh_cap_rows");
}

extern "C" int omc_ln_residual(const float* x, long long ldx, float alpha, const float* y, long long ldy, const float* ys, long long ldys,
                               const int32_t* slot_of, const float* w, int top, const void* nw, const void* nb, int w_dt, float eps,
                               float* x_out, long long ldxo, void* xb, int xb_dt, long long ldxb, int rows, int C, void* stream) {
  if (x == nullptr || nw == nullptr || nb == nullptr || (x_out == nullptr && xb == nullptr) || rows < 0 || C <= 0 ||
      (ys != nullptr && (slot_of == nullptr || w == nullptr || top <= 0)))
    return set_error(OMC_ERR_ARG, "omc_ln_residual: bad argument");
  if (rows == 0) return OMC_OK;
  const LnResArgs a{x, ldx, alpha, y, y != nullptr ? ldy : 0, ys, ys != nullptr ? ldys : 0, slot_of, w, top, nw, nb, eps, x_out,
                    x_out != nullptr ? ldxo : 0, xb, xb != nullptr ? ldxb : 0, C};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(xb_dt, TB, { return (launch_ln_residual<TW, TB, false>(a, rows, st)); }))
}

extern "C" int omc_rms_residual(const float* x, long long ldx, const float* y, long long ldy, const float* ys, long long ldys, const int32_t* slot_of,
                                const float* w, int top, const void* nw, int w_dt, float eps, float* x_out, long long ldxo, void* xb, int xb_dt,
                                long long ldxb, int rows, int C, void* stream) {
  if (x == nullptr || (xb != nullptr && nw == nullptr) || (x_out == nullptr && xb == nullptr) || rows < 0 || C <= 0 ||
      (ys != nullptr && (slot_of == nullptr || w == nullptr || top <= 0)))
    return set_error(OMC_ERR_ARG, "omc_rms_residual: bad argument");
  if (rows == 0) return OMC_OK;
  const LnResArgs a{x, ldx, 1.f, y, y != nullptr ? ldy : 0, ys, ys != nullptr ? ldys : 0, slot_of, w, top, nw, nullptr, eps, x_out,
                    x_out != nullptr ? ldxo : 0, xb, xb != nullptr ? ldxb : 0, C};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(w_dt, TW, OMC_DT_SWITCH(xb_dt, TB, { return (launch_ln_residual<TW, TB, true>(a, rows, st)); }))
}

extern "C" int omc_embed_bigram(const int32_t* ids, const int32_t* pos, const int32_t* slot, int T, const void* table, int t_dt, int C, int vocab,
                                const void* bigram, int buckets, int mul_prev, int mul_cur, int32_t* prev, const void* nw, float eps, float* h32,
                                long long ldh, void* xb, int xb_dt, long long ldxb, int single_rows, void* stream) {
  if (ids == nullptr || pos == nullptr || slot == nullptr || table == nullptr || bigram == nullptr || prev == nullptr || h32 == nullptr || T < 0 || C <= 0 ||
      buckets <= 0 || mul_prev < 0 || mul_cur < 0 || (xb != nullptr && nw == nullptr))
    return set_error(OMC_ERR_ARG, "omc_embed_bigram: bad argument");
  if (T == 0) return OMC_OK;
  const size_t smem = (size_t)C * sizeof(float);
  if (smem > 200 * 1024) return set_error(OMC_ERR_SHAPE, "omc_embed_bigram: row too wide for shared memory");
  auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int vec = C % 4 == 0 && ldh % 4 == 0 && ldxb % 4 == 0 && al16(table) && al16(bigram) && al16(nw) && al16(h32) && al16(xb) ? 1 : 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  OMC_DT_SWITCH(t_dt, TT, OMC_DT_SWITCH(xb_dt, TB, {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(embed_bigram_kernel<TT, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return set_error(OMC_ERR_CUDA, cudaGetErrorString(e));
    }
    embed_bigram_kernel<TT, TB><<<T, 256, smem, st>>>(ids, pos, slot, static_cast<const TT*>(table), C, vocab, static_cast<const TT*>(bigram), buckets,
                                                      mul_prev, mul_cur, prev, static_cast<const TT*>(nw), eps, h32, ldh, static_cast<TB*>(xb), ldxb,
                                                      single_rows, vec);
  }))
  if (!single_rows) last_token_save_kernel<<<(T + 255) / 256, 256, 0, st>>>(ids, slot, T, prev);
  return check_launch("omc_embed_bigram");
}
