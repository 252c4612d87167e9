// parallel_mixers.cu — ragged-batch kernels for layers that add a mixer and a feed-forward of the SAME fp32 stream, and for
// mixers that run side by side: softmax attention with rotated keys and the delta rule with separate removal and decay
// vectors.
//
// Conventions as in seq_mixers.cu: `tok_seq[t]` / `tok_pos[t]` give each batch row's sequence in the batch and position,
// `seq_info[s] = {first row, rows, tokens already seen, state slot}`, `T` is the activation type (bf16 or float); the
// stream, norms, filters, angles, gates and the recurrence are fp32 in both.
//
//   resid_sum_step       stream += y + mult (a / rms(a) wa + b / rms(b) wb);  1 / rms of the new row, or its norm, or -- for
//                        batches of one row per sequence -- both norms of the next layer and its input filter
//   norm_filter_rows     rows of several tokens: mixer input h + filter(h) with h = norm1(x), feed-forward input norm2(x)
//   rope_append          whole-row RMS norm and rotation of q and k, q times a number per head -> fp32, k / v -> paged cache
//   removal_prepare      decay, unit key, removal rate and scaled value of the delta rule from its projections
//   removal_recurrence / removal_step   S <- diag(w) S - (a u) (u^T S) + k v^T,  o = S^T r;  state per slot
#include <algorithm>
#include <initializer_list>
#include "seq_common.cuh"
#include <cuda_pipeline.h>

namespace sxb {
namespace seqmix {

// ------------------------------------------------------------------------------------------------ stream + norms
// One CTA per row.  x = resid + y + mult * (a / rms(a) * wa + b / rms(b) * wb); without wa: + a as it is; any of y, a, b may
// be absent.  The new row goes back to resid (unless `rows` selects rows: then row rows[i] is only read).
//   rstd:  1 / rms of the new row
//   out:   x / rms * w1
//   FILTER (one batch row per sequence): out = h + sum_j filt[j] h[taps-1-j tokens back], h = x / rms * w1, earlier h from the
//   sequence's slot (state fp32 [slots, taps-1, width], last row = most recent), which moves on by one; out2 = x / rms * w2.
// filt is stored [taps, width], its last row multiplies the current token.
struct ResidSum {
  float* resid;
  const void *y, *a, *wa, *b, *wb;
  float mult, eps;
  float* rstd;
  const int* rows;
  const void* w1;
  void* out;
  const void* w2;
  void* out2;
  const void* filt;
  float* state;
  const int *seq_info, *tok_seq;
  int taps, width;
};

template <typename T, bool FILTER>
__global__ void __launch_bounds__(1024)
resid_sum_vec_kernel(const ResidSum p) {        // eight consecutive channels per thread, blockDim.x * 8 >= width
  __shared__ float2 red2[32];
  __shared__ float red[32];
  const long long t = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  const int c0 = threadIdx.x * 8;
  const bool live = c0 < p.width;
  const long long base = t * p.width + c0, ob = (long long)blockIdx.x * p.width + c0;
  const float wn = (float)p.width;
  float x[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) x[e] = 0.f;
  if (live) load8_f32<float>(p.resid + base, x);
  if (p.y != nullptr && live) {
    float v[8];
    load8_f32<T>((const T*)p.y + base, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] += v[e];
  }
  if (p.a != nullptr) {
    float av[8], bv[8], wv[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) av[e] = bv[e] = wv[e] = 0.f;
    if (live) load8_f32<T>((const T*)p.a + base, av);
    if (p.b != nullptr && live) load8_f32<T>((const T*)p.b + base, bv);
    if (p.wa != nullptr) {
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) sa += av[e] * av[e], sb += bv[e] * bv[e];
      const float2 s = block_sum2(sa, sb, red2);
      const float ia = p.mult / sqrtf(s.x / wn + p.eps), ib = p.mult / sqrtf(s.y / wn + p.eps);
      if (live) {
        load8_f32<T>((const T*)p.wa + c0, wv);
#pragma unroll
        for (int e = 0; e < 8; ++e) av[e] *= ia * wv[e];
        if (p.b != nullptr) {
          load8_f32<T>((const T*)p.wb + c0, wv);
#pragma unroll
          for (int e = 0; e < 8; ++e) av[e] += bv[e] * ib * wv[e];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] += av[e];
  }
  if (p.rows == nullptr && live && (p.y != nullptr || p.a != nullptr)) store8_f32<float>(p.resid + base, x);
  if (p.rstd == nullptr && p.out == nullptr) return;
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / wn + p.eps);
  if (p.rstd != nullptr && threadIdx.x == 0) p.rstd[blockIdx.x] = inv;
  if (p.out == nullptr || !live) return;
  float w[8], h[8];
  load8_f32<T>((const T*)p.w1 + c0, w);
#pragma unroll
  for (int e = 0; e < 8; ++e) h[e] = x[e] * inv * w[e];
  if (FILTER) {
    const int* si = p.seq_info + 4 * p.tok_seq[t];
    const int seen = si[2], keep = p.taps - 1;
    float* st = p.state + (long long)si[3] * keep * p.width + c0;
    float acc[8], f[8];
    load8_f32<T>((const T*)p.filt + (long long)keep * p.width + c0, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = h[e] + f[e] * h[e];
    for (int j = 0; j < keep; ++j) {          // carried row j lies keep - j tokens back
      float s[8];
      load8_f32<float>(st + (long long)j * p.width, s);
      if (seen >= keep - j) {
        load8_f32<T>((const T*)p.filt + (long long)j * p.width + c0, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] += f[e] * s[e];
      }
      if (j > 0) store8_f32<float>(st + (long long)(j - 1) * p.width, s);
    }
    if (keep > 0) store8_f32<float>(st + (long long)(keep - 1) * p.width, h);
    if (p.out2 != nullptr) {
      load8_f32<T>((const T*)p.w2 + c0, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] *= x[e] * inv;
      store8_f32<T>((T*)p.out2 + ob, w);
    }
    store8_f32<T>((T*)p.out + ob, acc);
  } else {
    store8_f32<T>((T*)p.out + ob, h);
  }
}

template <typename T, bool FILTER>
__global__ void __launch_bounds__(256)
resid_sum_kernel(const ResidSum p) {            // any width
  __shared__ float2 red2[32];
  __shared__ float red[32];
  const long long t = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  const long long base = t * p.width, ob = (long long)blockIdx.x * p.width;
  const float wn = (float)p.width;
  const T *y = (const T*)p.y, *a = (const T*)p.a, *b = (const T*)p.b, *wa = (const T*)p.wa, *wb = (const T*)p.wb;
  float ia = 1.f, ib = 0.f;
  if (a != nullptr && wa != nullptr) {
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      const float u = to_f32<T>(a[base + c]), v = b ? to_f32<T>(b[base + c]) : 0.f;
      sa += u * u, sb += v * v;
    }
    const float2 s = block_sum2(sa, sb, red2);
    ia = p.mult / sqrtf(s.x / wn + p.eps), ib = p.mult / sqrtf(s.y / wn + p.eps);
  }
  auto value = [&](int c) {
    float x = p.resid[base + c];
    if (y != nullptr) x += to_f32<T>(y[base + c]);
    if (a != nullptr) {
      float v = to_f32<T>(a[base + c]) * ia * (wa ? to_f32<T>(wa[c]) : 1.f);
      if (b != nullptr) v += to_f32<T>(b[base + c]) * ib * to_f32<T>(wb[c]);
      x += v;
    }
    return x;
  };
  const bool write = p.rows == nullptr && (y != nullptr || a != nullptr);
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const float x = value(c);
    if (write) p.resid[base + c] = x;
    ss += x * x;
  }
  if (p.rstd == nullptr && p.out == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / wn + p.eps);
  if (p.rstd != nullptr && threadIdx.x == 0) p.rstd[blockIdx.x] = inv;
  if (p.out == nullptr) return;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const float x = write ? p.resid[base + c] : value(c);
    const float h = x * inv * to_f32<T>(((const T*)p.w1)[c]);
    float acc = h;
    if (FILTER) {
      const int* si = p.seq_info + 4 * p.tok_seq[t];
      const int seen = si[2], keep = p.taps - 1;
      float* st = p.state + (long long)si[3] * keep * p.width + c;
      const T* f = (const T*)p.filt + c;
      acc += to_f32<T>(f[(long long)keep * p.width]) * h;
      for (int j = 0; j < keep; ++j) {
        const float s = st[(long long)j * p.width];
        if (seen >= keep - j) acc += to_f32<T>(f[(long long)j * p.width]) * s;
        if (j > 0) st[(long long)(j - 1) * p.width] = s;
      }
      if (keep > 0) st[(long long)(keep - 1) * p.width] = h;
      if (p.out2 != nullptr) ((T*)p.out2)[ob + c] = from_f32<T>(x * inv * to_f32<T>(((const T*)p.w2)[c]));
    }
    ((T*)p.out)[ob + c] = from_f32<T>(acc);
  }
}

// ------------------------------------------------------------------------------------------------ norm + input filter
// h[t] = x[t] * rstd[t] * w1;  out[t] = h[t] + sum_j filt[taps-1-j] h[t-j];  out2[t] = x[t] * rstd[t] * w2 (optional).  Rows of a
// sequence before this batch come from its slot, rows before its start are zero; the slot then holds the last taps-1 h.
// A thread takes 8 channels and walks kNfRows batch rows with the last taps-1 h in registers.  A sequence's first taps-1 rows
// all belong to the thread of its first row: that thread alone reads the slot, before it writes the slot's new contents.
constexpr int kNfRows = 8;

template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
norm_filter_vec_kernel(const float* __restrict__ x, const float* __restrict__ rstd, const T* __restrict__ w1,
                       const T* __restrict__ filt, float* __restrict__ state, const int* __restrict__ seq_info,
                       const int* __restrict__ tok_seq, T* __restrict__ out, const T* __restrict__ w2,
                       T* __restrict__ out2, int C, int n_tokens) {
  constexpr int KEEP = TAPS - 1;
  const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (c0 >= C) return;
  const int t0 = blockIdx.x * kNfRows, t1 = min(t0 + kNfRows, n_tokens);
  float w1v[8], w2v[8], wt[TAPS][8], hist[TAPS][8];      // hist[j]: h of j rows back
  load8_f32<T>(w1 + c0, w1v);
#pragma unroll
  for (int e = 0; e < 8; ++e) w2v[e] = 0.f;
  if (w2 != nullptr) load8_f32<T>(w2 + c0, w2v);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    load8_f32<T>(filt + (long long)j * C + c0, wt[j]);
#pragma unroll
    for (int e = 0; e < 8; ++e) hist[j][e] = 0.f;
  }
  auto h_row = [&](int t, float* h) {
    load8_f32<float>(x + (long long)t * C + c0, h);
    const float r = rstd[t];
#pragma unroll
    for (int e = 0; e < 8; ++e) h[e] *= r * w1v[e];
  };
  bool need = true;
  int first = 0, end = 0;                                // the current sequence's rows in the batch
  const int* si = seq_info;
  float nx[8], nr = rstd[t0];                            // the next row, fetched one row ahead
  load8_f32<float>(x + (long long)t0 * C + c0, nx);
  for (int t = t0; t < n_tokens; ++t) {
    if (t >= end) {
      si = seq_info + 4 * tok_seq[t];
      first = si[0], end = first + si[1];
    }
    const int local = t - first;
    const bool head = local > 0 && local < KEEP;         // belongs to the thread of the sequence's first row
    if (t >= t1 && !(head && first >= t0)) break;
    float xv[8], o[8];
    const float r = nr;
#pragma unroll
    for (int e = 0; e < 8; ++e) xv[e] = nx[e];
    if (t + 1 < n_tokens) {
      load8_f32<float>(x + (long long)(t + 1) * C + c0, nx);
      nr = rstd[t + 1];
    }
    if (head && first < t0) continue;
    if (local == 0) {
      const int n = si[1], seen = si[2];
      float* st = state + (long long)si[3] * KEEP * C + c0;
#pragma unroll
      for (int j = 1; j < TAPS; ++j) {
        if (seen >= j) {
          load8_f32<float>(st + (long long)(KEEP - j) * C, hist[j]);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) hist[j][e] = 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < KEEP; ++j) {                   // new carried row j: row n + j of (carried rows ++ this batch's)
        float v[8];
        const int i = n + j;
        if (i >= KEEP) {
          h_row(first + i - KEEP, v);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) v[e] = 0.f;
#pragma unroll
          for (int m = 1; m < TAPS; ++m)
            if (KEEP - i == m) {
#pragma unroll
              for (int e = 0; e < 8; ++e) v[e] = hist[m][e];
            }
        }
        store8_f32<float>(st + (long long)j * C, v);
      }
    } else if (need) {
#pragma unroll
      for (int j = 1; j < TAPS; ++j) h_row(t - j, hist[j]);
    } else {
#pragma unroll
      for (int j = TAPS - 1; j >= 1; --j)
#pragma unroll
        for (int e = 0; e < 8; ++e) hist[j][e] = hist[j - 1][e];
    }
    need = false;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      xv[e] *= r;
      hist[0][e] = xv[e] * w1v[e];
      o[e] = hist[0][e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) o[e] += wt[TAPS - 1 - j][e] * hist[j][e];
    }
    store8_f32<T>(out + (long long)t * C + c0, o);
    if (out2 != nullptr) {
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[e] *= w2v[e];
      store8_f32<T>(out2 + (long long)t * C + c0, xv);
    }
  }
}

// Any width and any number of taps: one thread per element, the slots moved on by a second kernel.
template <typename T>
__global__ void __launch_bounds__(256)
norm_filter_kernel(const float* __restrict__ x, const float* __restrict__ rstd, const T* __restrict__ w1,
                   const T* __restrict__ filt, const float* __restrict__ state, const int* __restrict__ seq_info,
                   const int* __restrict__ tok_seq, T* __restrict__ out, const T* __restrict__ w2,
                   T* __restrict__ out2, int C, int taps) {
  const int t = blockIdx.x, keep = taps - 1;
  const int* si = seq_info + 4 * tok_seq[t];
  const int local = t - si[0], seen = si[2];
  const float* st = state + (long long)si[3] * keep * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    const float w = to_f32<T>(w1[c]), xr = x[(long long)t * C + c] * rstd[t];
    float o = xr * w;
    for (int j = 0; j < taps; ++j) {
      const int src = local - j;
      float h = 0.f;
      if (src >= 0) h = x[(long long)(t - j) * C + c] * rstd[t - j] * w;
      else if (seen + src >= 0) h = st[(long long)(keep + src) * C + c];
      o += to_f32<T>(filt[(long long)(keep - j) * C + c]) * h;
    }
    out[(long long)t * C + c] = from_f32<T>(o);
    if (out2 != nullptr) out2[(long long)t * C + c] = from_f32<T>(xr * to_f32<T>(w2[c]));
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
norm_filter_state_kernel(const float* __restrict__ x, const float* __restrict__ rstd, const T* __restrict__ w1,
                         float* __restrict__ state, const int* __restrict__ seq_info, int C, int taps) {
  const int* si = seq_info + 4 * blockIdx.x;
  const int first = si[0], n = si[1], keep = taps - 1;
  float* st = state + (long long)si[3] * keep * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
    for (int j = 0; j < keep; ++j) {           // row n + j of (carried ++ new); n >= 1, so ascending order never overwrites a source
      const int i = n + j;
      float v;
      if (i >= keep) v = x[(long long)(first + i - keep) * C + c] * rstd[first + i - keep] * to_f32<T>(w1[c]);
      else v = st[(long long)i * C + c];
      st[(long long)j * C + c] = v;
    }
}

// ------------------------------------------------------------------------------------------------ rotated attention rows
// One CTA per token.  q (Hq d channels at column q0), k (G d at k0) and v (G dv at v0; v0 may be k0: the values are then the
// projected keys as they are) of a fused projection row.  q_w / k_w (Hq d / G d entries): the WHOLE row of q / of k is divided by
// its root mean square and multiplied by the weight.  The first n_rot channels of every head turn by pos * inv_freq[i] in
// pairs (2i, 2i+1) (interleaved) or (i, i + n_rot/2), cos and sin times amp.  q -> fp32 [tokens, Hq, d], times q_scale[h]; k, v -> paged caches.
// VEC 4: all columns, sizes and the rotated part's pieces are multiples of 4 channels.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
rope_append_kernel(const T* __restrict__ proj, long long ld, int q0, int k0, int v0, const T* __restrict__ q_w,
                   const T* __restrict__ k_w, const float* __restrict__ inv_freq, const float* __restrict__ q_scale,
                   float* __restrict__ q_out, T* __restrict__ kcache, T* __restrict__ vcache,
                   const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, const int* __restrict__ tables,
                   int max_blocks, int block_size, int Hq, int G, int d, int dv, int n_rot, int interleaved, float eps,
                   float amp) {
  extern __shared__ __align__(16) float cs[];   // cos [n_rot / 2] | sin [n_rot / 2]
  __shared__ float2 red[32];
  const int t = blockIdx.x, half = n_rot >> 1;
  const T* row = proj + (long long)t * ld;
  const int pos = tok_pos[t];
  const long long slot = (long long)tables[(long long)tok_seq[t] * max_blocks + pos / block_size] * block_size + pos % block_size;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, co;
    sincosf((float)pos * inv_freq[i], &sn, &co);
    cs[i] = co * amp, cs[half + i] = sn * amp;
  }
  float iq = 1.f, ik = 1.f;
  if (q_w != nullptr || k_w != nullptr) {
    float sq = 0.f, sk = 0.f;
    if (q_w != nullptr)
      for (int c = threadIdx.x * VEC; c < Hq * d; c += blockDim.x * VEC) {
        if (VEC == 4) {
          const float4 v = load4_f32<T>(row + q0 + c);
          sq += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        } else {
          const float v = to_f32<T>(row[q0 + c]);
          sq += v * v;
        }
      }
    if (k_w != nullptr)
      for (int c = threadIdx.x * VEC; c < G * d; c += blockDim.x * VEC) {
        if (VEC == 4) {
          const float4 v = load4_f32<T>(row + k0 + c);
          sk += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        } else {
          const float v = to_f32<T>(row[k0 + c]);
          sk += v * v;
        }
      }
    const float2 s = block_sum2(sq, sk, red);
    if (q_w != nullptr) iq = 1.f / sqrtf(s.x / (float)(Hq * d) + eps);
    if (k_w != nullptr) ik = 1.f / sqrtf(s.y / (float)(G * d) + eps);
  }
  __syncthreads();
  // items of a head: rotated ones (a pair, or VEC / 2 or VEC pairs), then VEC passing channels each
  const int n_turn = VEC == 4 ? (interleaved ? n_rot >> 2 : half >> 2) : half;
  const int per = n_turn + (d - n_rot) / VEC;
  for (int idx = threadIdx.x; idx < (Hq + G) * per; idx += blockDim.x) {
    const int s = idx / per, i = idx % per;
    const bool is_q = s < Hq;
    const int hc = (is_q ? s : s - Hq) * d;              // the head's first column in q or k
    const T* src = row + (is_q ? q0 : k0) + hc;
    const T* wrow = is_q ? q_w : k_w;
    const T* w = wrow ? wrow + hc : nullptr;
    const float m = is_q ? iq : ik, qs = (is_q && q_scale) ? q_scale[s] : 1.f;
    float* qd = is_q ? q_out + ((long long)t * Hq + s) * d : nullptr;
    T* kd = is_q ? nullptr : kcache + (slot * G + (s - Hq)) * d;
    if (VEC == 4) {
      auto get = [&](int c) {
        float4 v = load4_f32<T>(src + c);
        if (w != nullptr) {
          const float4 g = load4_f32<T>(w + c);
          v.x *= m * g.x, v.y *= m * g.y, v.z *= m * g.z, v.w *= m * g.w;
        }
        return v;
      };
      auto put = [&](int c, float4 v) {
        if (is_q) store4_f32<float>(qd + c, make_float4(v.x * qs, v.y * qs, v.z * qs, v.w * qs));
        else store4_f32<T>(kd + c, v);
      };
      if (i >= n_turn) {
        const int c = n_rot + (i - n_turn) * 4;
        put(c, get(c));
      } else if (interleaved) {
        const int c = i * 4;
        const float4 v = get(c);
        const float c0 = cs[2 * i], c1 = cs[2 * i + 1], s0 = cs[half + 2 * i], s1 = cs[half + 2 * i + 1];
        put(c, make_float4(v.x * c0 - v.y * s0, v.y * c0 + v.x * s0, v.z * c1 - v.w * s1, v.w * c1 + v.z * s1));
      } else {
        const int c = i * 4;
        const float4 u = get(c), v = get(c + half);
        const float4 co = *reinterpret_cast<const float4*>(cs + c), si = *reinterpret_cast<const float4*>(cs + half + c);
        put(c, make_float4(u.x * co.x - v.x * si.x, u.y * co.y - v.y * si.y, u.z * co.z - v.z * si.z, u.w * co.w - v.w * si.w));
        put(c + half, make_float4(v.x * co.x + u.x * si.x, v.y * co.y + u.y * si.y, v.z * co.z + u.z * si.z,
                                  v.w * co.w + u.w * si.w));
      }
    } else {
      auto get = [&](int c) { return to_f32<T>(src[c]) * (w != nullptr ? m * to_f32<T>(w[c]) : 1.f); };
      auto put = [&](int c, float v) {
        if (is_q) qd[c] = v * qs;
        else kd[c] = from_f32<T>(v);
      };
      if (i >= n_turn) {
        const int c = n_rot + (i - n_turn);
        put(c, get(c));
      } else {
        const int ca = interleaved ? 2 * i : i, cb = interleaved ? 2 * i + 1 : i + half;
        const float u = get(ca), v = get(cb);
        put(ca, u * cs[i] - v * cs[half + i]);
        put(cb, v * cs[i] + u * cs[half + i]);
      }
    }
  }
  for (int c = threadIdx.x * VEC; c < G * dv; c += blockDim.x * VEC) {
    if (VEC == 4) store4_f32<T>(vcache + slot * G * dv + c, load4_f32<T>(row + v0 + c));
    else vcache[slot * G * dv + c] = row[v0 + c];
  }
}

// ------------------------------------------------------------------------------------------------ delta rule with removal
// From the projection rows (columns r0, k0, v0, a0: H n channels each; w0c: `rank` channels), per token, head and channel:
//   w = exp(-rate * sigmoid(w2^T tanh(low) + w0)),  u = k / sqrt(sum k^2 + eps),  a = sigmoid(a_raw + a_bias),  r,
//   v' = v * sqrt(sum k^2 + eps)      (so k v^T = u v'^T)
// buf fp32 [tokens, H, 5, n] = w | u | a | r | v'.  One CTA per (TT tokens, head); a thread takes CPT channels of the head and
// reads its entries of w2 ([rank, H n]) once for all TT tokens.
template <typename T, int TT, int CPT>
__global__ void __launch_bounds__(256)
removal_prepare_kernel(const T* __restrict__ proj, long long ld, int r0, int k0, int v0, int a0, int low0,
                       const T* __restrict__ w2, const float* __restrict__ w0, const float* __restrict__ a_bias,
                       float* __restrict__ buf, int n_tokens, int H, int n, int rank, float rate, float eps) {
  extern __shared__ __align__(16) float low[];             // tanh of the inner projection, [rank][TT]
  __shared__ float part[8][TT];
  const int t0 = blockIdx.x * TT, nt = min(TT, n_tokens - t0), h = blockIdx.y;
  for (int i = threadIdx.x; i < rank * TT; i += blockDim.x) {
    const int j = i % rank, tt = i / rank;
    low[j * TT + tt] = tt < nt ? tanhf(to_f32<T>(proj[(long long)(t0 + tt) * ld + low0 + j])) : 0.f;
  }
  const int c = threadIdx.x * CPT, hc = h * n + c;
  const bool live = c < n;
  struct alignas(sizeof(T) * CPT) Vt { T v[CPT]; };
  struct alignas(4 * CPT) Vf { float v[CPT]; };
  auto load = [&](const T* p) { return *reinterpret_cast<const Vt*>(p); };
  float kk[TT][CPT], acc[TT][CPT], ss[TT];
#pragma unroll
  for (int tt = 0; tt < TT; ++tt) {
    ss[tt] = 0.f;
    Vt kv;
    if (live && tt < nt) kv = load(proj + (long long)(t0 + tt) * ld + k0 + hc);
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
      kk[tt][e] = (live && tt < nt) ? to_f32<T>(kv.v[e]) : 0.f;
      acc[tt][e] = live ? w0[hc + e] : 0.f;
      ss[tt] += kk[tt][e] * kk[tt][e];
    }
  }
#pragma unroll
  for (int tt = 0; tt < TT; ++tt) ss[tt] = warp_sum(ss[tt]);
  if ((threadIdx.x & 31) == 0) {
#pragma unroll
    for (int tt = 0; tt < TT; ++tt) part[threadIdx.x >> 5][tt] = ss[tt];
  }
  __syncthreads();
  if (!live) return;
  const int Hn = H * n;
#pragma unroll 4
  for (int j = 0; j < rank; ++j) {
    const Vt wv = load(w2 + (long long)j * Hn + hc);
    float th[TT];
    if (TT % 4 == 0) {
#pragma unroll
      for (int q = 0; q < TT / 4; ++q) {
        const float4 f = *reinterpret_cast<const float4*>(low + j * TT + 4 * q);
        th[4 * q] = f.x, th[4 * q + 1] = f.y, th[4 * q + 2] = f.z, th[4 * q + 3] = f.w;
      }
    } else {
#pragma unroll
      for (int tt = 0; tt < TT; ++tt) th[tt] = low[j * TT + tt];
    }
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
      const float w = to_f32<T>(wv.v[e]);
#pragma unroll
      for (int tt = 0; tt < TT; ++tt) acc[tt][e] += w * th[tt];
    }
  }
  const int nw = blockDim.x >> 5;
#pragma unroll
  for (int tt = 0; tt < TT; ++tt) {
    if (tt >= nt) break;
    float s = 0.f;
    for (int w = 0; w < nw; ++w) s += part[w][tt];
    const float len = sqrtf(s + eps);
    const T* row = proj + (long long)(t0 + tt) * ld + hc;
    const Vt rv = load(row + r0), vv = load(row + v0), av = load(row + a0);
    Vf ow, ou, oa, orr, ov;
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
      ow.v[e] = expf(-rate * sigmoid_f(acc[tt][e]));
      ou.v[e] = kk[tt][e] / len;
      oa.v[e] = sigmoid_f(to_f32<T>(av.v[e]) + a_bias[hc + e]);
      orr.v[e] = to_f32<T>(rv.v[e]);
      ov.v[e] = to_f32<T>(vv.v[e]) * len;
    }
    float* o = buf + ((long long)(t0 + tt) * H + h) * 5 * n + c;
    *reinterpret_cast<Vf*>(o) = ow;
    *reinterpret_cast<Vf*>(o + n) = ou;
    *reinterpret_cast<Vf*>(o + 2 * n) = oa;
    *reinterpret_cast<Vf*>(o + 3 * n) = orr;
    *reinterpret_cast<Vf*>(o + 4 * n) = ov;
  }
}

// State per (slot, head): n value columns of n key channels each, stored [value][key].  Column v evolves on its own:
//   z = u . s;   s <- w s + u (v' - a z);   o = s . r        (all products per key channel, z from the old s)
// A column is held by LPC lanes (the n-vector as 16-byte chunks, chunk i on lane i mod LPC), 128 / LPC columns per CTA; the
// CTA walks its sequence's rows in order, staging w | u | a | r of TB tokens at a time in shared memory (two buffers, cp.async).
constexpr int kRmThreads = 128, kRmTB = 8;

template <int R, int LPC>
__global__ void __launch_bounds__(kRmThreads)
removal_recurrence_kernel(const float* __restrict__ buf, float* __restrict__ state, float* __restrict__ out,
                          const int* __restrict__ seq_info, int H, int n) {
  constexpr int NP = R * LPC, R4 = R / 4, COLS = kRmThreads / LPC;
  constexpr int stage = 4 * kRmTB * NP + kRmTB * COLS;
  static_assert(LPC >= kRmTB, "lane t of a column writes token t of the group");
  extern __shared__ __align__(16) float sm[];
  const int* si = seq_info + 4 * blockIdx.z;
  const int first = si[0], rows = si[1], seen = si[2], slot = si[3];
  const int h = blockIdx.y, lc = threadIdx.x / LPC, l = threadIdx.x % LPC;
  const int col = blockIdx.x * COLS + lc;
  const bool live = col < n, n4 = (n & 3) == 0;
  if (NP != n) {
    for (int i = threadIdx.x; i < 2 * stage; i += blockDim.x) sm[i] = 0.f;      // the padding stays zero
  }
  float* sp = state + (((long long)slot * H + h) * n + (live ? col : 0)) * n;
  float2 S[R / 2];
#pragma unroll
  for (int r4 = 0; r4 < R4; ++r4) {
    const int i = (r4 * LPC + l) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && seen > 0) {
      if (n4 && i < n) {
        v = *reinterpret_cast<const float4*>(sp + i);
      } else {
        if (i < n) v.x = sp[i];
        if (i + 1 < n) v.y = sp[i + 1];
        if (i + 2 < n) v.z = sp[i + 2];
        if (i + 3 < n) v.w = sp[i + 3];
      }
    }
    S[2 * r4] = make_float2(v.x, v.y), S[2 * r4 + 1] = make_float2(v.z, v.w);
  }
  __syncthreads();
  auto stage_in = [&](int b, int t0) {
    float* sv = sm + b * stage;                 // [TB][4][NP] then values [TB][COLS]
    float* sx = sv + 4 * kRmTB * NP;
    const int nt = min(kRmTB, rows - t0);
    if (n4) {
      const int n4c = n >> 2;
      for (int i = threadIdx.x; i < nt * 4 * n4c; i += blockDim.x) {
        const int tv = i / n4c, c = (i % n4c) * 4, tt = tv >> 2, vec = tv & 3;
        const float* src = buf + (((long long)(first + t0 + tt) * H + h) * 5 + vec) * n + c;
        __pipeline_memcpy_async(sv + tv * NP + c, src, 16);
      }
    } else {
      for (int i = threadIdx.x; i < nt * 4 * n; i += blockDim.x) {
        const int tv = i / n, c = i % n, tt = tv >> 2, vec = tv & 3;
        const float* src = buf + (((long long)(first + t0 + tt) * H + h) * 5 + vec) * n + c;
        __pipeline_memcpy_async(sv + tv * NP + c, src, 4);
      }
    }
    for (int i = threadIdx.x; i < nt * COLS; i += blockDim.x) {
      const int c = min((int)blockIdx.x * COLS + i % COLS, n - 1);
      __pipeline_memcpy_async(sx + i, buf + (((long long)(first + t0 + i / COLS) * H + h) * 5 + 4) * n + c, 4);
    }
    __pipeline_commit();
  };
  struct Tok {                                  // one token's operands, loaded one token ahead of their use
    float v;
    float4 w[R4], u[R4], a[R4], r[R4];
  };
  stage_in(0, 0);
  int b = 0;
  for (int t0 = 0; t0 < rows; t0 += kRmTB, b ^= 1) {
    const int nt = min(kRmTB, rows - t0);
    const bool more = t0 + kRmTB < rows;
    if (more) stage_in(b ^ 1, t0 + kRmTB);
    if (more) __pipeline_wait_prior(1);
    else __pipeline_wait_prior(0);
    __syncthreads();
    const float* sv = sm + b * stage;
    const float* sx = sv + 4 * kRmTB * NP;
    auto fetch = [&](int tt) {
      Tok t;
      t.v = sx[tt * COLS + lc];
      const float4* p = reinterpret_cast<const float4*>(sv + tt * 4 * NP) + l;
#pragma unroll
      for (int r4 = 0; r4 < R4; ++r4) {
        t.w[r4] = p[r4 * LPC], t.u[r4] = p[NP / 4 + r4 * LPC];
        t.a[r4] = p[2 * (NP / 4) + r4 * LPC], t.r[r4] = p[3 * (NP / 4) + r4 * LPC];
      }
      return t;
    };
    auto step = [&](const Tok& t, float& o_lane) {
      float2 z01 = make_float2(0.f, 0.f), z23 = make_float2(0.f, 0.f);
#pragma unroll
      for (int r4 = 0; r4 < R4; ++r4) {
        z01 = __ffma2_rn(S[2 * r4], make_float2(t.u[r4].x, t.u[r4].y), z01);
        z23 = __ffma2_rn(S[2 * r4 + 1], make_float2(t.u[r4].z, t.u[r4].w), z23);
      }
      float z = (z01.x + z01.y) + (z23.x + z23.y);
#pragma unroll
      for (int r4 = 0; r4 < R4; ++r4) {          // the decayed state does not wait for z
        S[2 * r4] = __fmul2_rn(S[2 * r4], make_float2(t.w[r4].x, t.w[r4].y));
        S[2 * r4 + 1] = __fmul2_rn(S[2 * r4 + 1], make_float2(t.w[r4].z, t.w[r4].w));
      }
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
      const float2 nz = make_float2(-z, -z), v2 = make_float2(t.v, t.v);
      float2 o01 = make_float2(0.f, 0.f), o23 = make_float2(0.f, 0.f);
#pragma unroll
      for (int r4 = 0; r4 < R4; ++r4) {
        const float2 c01 = __ffma2_rn(make_float2(t.a[r4].x, t.a[r4].y), nz, v2);
        const float2 c23 = __ffma2_rn(make_float2(t.a[r4].z, t.a[r4].w), nz, v2);
        S[2 * r4] = __ffma2_rn(make_float2(t.u[r4].x, t.u[r4].y), c01, S[2 * r4]);
        S[2 * r4 + 1] = __ffma2_rn(make_float2(t.u[r4].z, t.u[r4].w), c23, S[2 * r4 + 1]);
        o01 = __ffma2_rn(S[2 * r4], make_float2(t.r[r4].x, t.r[r4].y), o01);
        o23 = __ffma2_rn(S[2 * r4 + 1], make_float2(t.r[r4].z, t.r[r4].w), o23);
      }
      o_lane = (o01.x + o01.y) + (o23.x + o23.y);
    };
    float op[kRmTB];
    if (nt == kRmTB) {
      Tok cur = fetch(0);
#pragma unroll
      for (int tt = 0; tt < kRmTB; ++tt) {
        const Tok nxt = fetch(tt + 1 < kRmTB ? tt + 1 : tt);
        step(cur, op[tt]);
        cur = nxt;
      }
    } else {
#pragma unroll
      for (int tt = 0; tt < kRmTB; ++tt) {
        op[tt] = 0.f;
        if (tt < nt) step(fetch(tt), op[tt]);
      }
    }
#pragma unroll
    for (int x = 1; x < LPC; x <<= 1)
#pragma unroll
      for (int tt = 0; tt < kRmTB; ++tt) op[tt] += __shfl_xor_sync(0xffffffffu, op[tt], x);
    float mine = op[0];
#pragma unroll
    for (int tt = 1; tt < kRmTB; ++tt) mine = (l == tt) ? op[tt] : mine;
    if (live && l < nt) out[((long long)(first + t0 + l) * H + h) * n + col] = mine;
    __syncthreads();            // the buffer just walked is the target of the next iteration's copies
  }
  if (live) {
#pragma unroll
    for (int r4 = 0; r4 < R4; ++r4) {
      const int i = (r4 * LPC + l) * 4;
      if (n4 && i < n) {
        *reinterpret_cast<float4*>(sp + i) = make_float4(S[2 * r4].x, S[2 * r4].y, S[2 * r4 + 1].x, S[2 * r4 + 1].y);
      } else {
        if (i < n) sp[i] = S[2 * r4].x;
        if (i + 1 < n) sp[i + 1] = S[2 * r4].y;
        if (i + 2 < n) sp[i + 2] = S[2 * r4 + 1].x;
        if (i + 3 < n) sp[i + 3] = S[2 * r4 + 1].y;
      }
    }
  }
}

// The same for batches of one row per sequence: a warp takes kStepCols columns, lane l the channels 4 l .. 4 l + 3 (+ 128 for
// NV = 2) of each; the token's vectors sit in registers, every column is read and written once.
constexpr int kStepCols = 8, kStepWarps = 4;

template <int NV>
__global__ void __launch_bounds__(32 * kStepWarps)
removal_step_kernel(const float* __restrict__ buf, float* __restrict__ state, float* __restrict__ out,
                    const int* __restrict__ seq_info, int H, int n) {
  const int* si = seq_info + 4 * blockIdx.z;
  const int row = si[0], seen = si[2], slot = si[3];
  const int h = blockIdx.y, lane = threadIdx.x & 31;
  const int col0 = (blockIdx.x * kStepWarps + (threadIdx.x >> 5)) * kStepCols;
  if (col0 >= n) return;
  const float* tok = buf + ((long long)row * H + h) * 5 * n;
  float* sp = state + (((long long)slot * H + h) * n + col0) * n;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 S[kStepCols][NV], w[NV], u[NV], a[NV], r[NV];
#pragma unroll
  for (int j = 0; j < kStepCols; ++j)
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = 128 * v + 4 * lane;
      S[j][v] = (seen > 0 && c < n && col0 + j < n) ? *reinterpret_cast<const float4*>(sp + (long long)j * n + c) : zero;
    }
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int c = 128 * v + 4 * lane;
    w[v] = c < n ? *reinterpret_cast<const float4*>(tok + c) : zero;
    u[v] = c < n ? *reinterpret_cast<const float4*>(tok + n + c) : zero;
    a[v] = c < n ? *reinterpret_cast<const float4*>(tok + 2 * n + c) : zero;
    r[v] = c < n ? *reinterpret_cast<const float4*>(tok + 3 * n + c) : zero;
  }
  const float vall = (lane < kStepCols && col0 + lane < n) ? tok[4 * n + col0 + lane] : 0.f;
  float z[kStepCols], o[kStepCols];
#pragma unroll
  for (int j = 0; j < kStepCols; ++j) {
    z[j] = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
      z[j] += (S[j][v].x * u[v].x + S[j][v].y * u[v].y) + (S[j][v].z * u[v].z + S[j][v].w * u[v].w);
  }
#pragma unroll
  for (int x = 16; x > 0; x >>= 1)
#pragma unroll
    for (int j = 0; j < kStepCols; ++j) z[j] += __shfl_xor_sync(0xffffffffu, z[j], x);
#pragma unroll
  for (int j = 0; j < kStepCols; ++j) {
    const float vj = __shfl_sync(0xffffffffu, vall, j);
    o[j] = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      float4& s = S[j][v];
      s.x = w[v].x * s.x + u[v].x * (vj - a[v].x * z[j]);
      s.y = w[v].y * s.y + u[v].y * (vj - a[v].y * z[j]);
      s.z = w[v].z * s.z + u[v].z * (vj - a[v].z * z[j]);
      s.w = w[v].w * s.w + u[v].w * (vj - a[v].w * z[j]);
      o[j] += (s.x * r[v].x + s.y * r[v].y) + (s.z * r[v].z + s.w * r[v].w);
      const int c = 128 * v + 4 * lane;
      if (c < n && col0 + j < n) *reinterpret_cast<float4*>(sp + (long long)j * n + c) = s;
    }
  }
#pragma unroll
  for (int x = 16; x > 0; x >>= 1)
#pragma unroll
    for (int j = 0; j < kStepCols; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], x);
  float mine = o[0];
#pragma unroll
  for (int j = 1; j < kStepCols; ++j) mine = lane == j ? o[j] : mine;
  if (lane < kStepCols && col0 + lane < n) out[((long long)row * H + h) * n + col0 + lane] = mine;
}

static bool aligned16(std::initializer_list<const void*> ps) {
  uintptr_t x = 0;
  for (const void* p : ps) x |= reinterpret_cast<uintptr_t>(p);
  return (x & 15) == 0;
}

}  // namespace seqmix
}  // namespace sxb

using namespace sxb;
using namespace sxb::seqmix;

/* Row i of the fp32 stream resid [n, width] (row rows[i] when rows, int32, is given; such rows are read, not written):
 * x = resid + y + mult (a / rms(a) wa + b / rms(b) wb), y / a / b / wa / wb `dtype` or null (wa null: + a as it is, no b), written
 * back.  rstd (fp32 [n_rows] or null): 1 / rms of the new row.  out (`dtype` [n_rows, width] or null): x / rms * w1.  With filt
 * (`dtype` [taps, width], last row = current token; every sequence has exactly one batch row): out = h + filter(h), h = x /
 * rms * w1, earlier h from state fp32 [slots, taps-1, width], which moves on; out2 (or null) = x / rms * w2. */
SXB_API int sxb_resid_sum_step(void* resid, const void* y, const void* a, const void* wa, const void* b, const void* wb,
                               float mult, float eps, void* rstd, const void* rows, const void* w1, void* out,
                               const void* w2, void* out2, const void* filt, void* state, const void* seq_info,
                               const void* tok_seq, int taps, int n_rows, int width, int dtype, void* stream) {
  if (n_rows <= 0) return SXB_OK;
  if ((out != nullptr) != (w1 != nullptr) || (b != nullptr && (a == nullptr || wa == nullptr || wb == nullptr)))
    return SXB_ERR_BAD_ARG;
  if (filt != nullptr && (out == nullptr || taps < 1 || rows != nullptr || (taps > 1 && state == nullptr) ||
                          seq_info == nullptr || tok_seq == nullptr))
    return SXB_ERR_BAD_ARG;
  const ResidSum p{(float*)resid, y, a, wa, b, wb, mult, eps, (float*)rstd, (const int*)rows, w1, out, w2, out2, filt,
                   (float*)state, (const int*)seq_info, (const int*)tok_seq, taps, width};
  cudaStream_t s = (cudaStream_t)stream;
  if (width % 8 == 0 && width <= 8192 && aligned16({resid, y, a, wa, b, wb, w1, out, w2, out2, filt, state})) {
    const int nt = (width / 8 + 31) / 32 * 32;
    if (filt != nullptr) SEQMIX_DISPATCH(dtype, (resid_sum_vec_kernel<T, true><<<n_rows, nt, 0, s>>>(p)));
    else SEQMIX_DISPATCH(dtype, (resid_sum_vec_kernel<T, false><<<n_rows, nt, 0, s>>>(p)));
  } else {
    if (filt != nullptr) SEQMIX_DISPATCH(dtype, (resid_sum_kernel<T, true><<<n_rows, 256, 0, s>>>(p)));
    else SEQMIX_DISPATCH(dtype, (resid_sum_kernel<T, false><<<n_rows, 256, 0, s>>>(p)));
  }
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Batch rows of any number per sequence: out `dtype` [n_tokens, width] = h + filter(h) with h = x * rstd * w1 (x fp32, rstd fp32
 * [n_tokens]), filt `dtype` [taps, width] (last row = current token), earlier h from state fp32 [slots, taps-1, width], which is
 * left holding every sequence's last taps-1 rows of h; out2 (or null) = x * rstd * w2. */
SXB_API int sxb_norm_filter_rows(const void* x, const void* rstd, const void* w1, const void* filt, void* state,
                                 const void* seq_info, const void* tok_seq, void* out, const void* w2, void* out2,
                                 int n_tokens, int n_seqs, int width, int taps, int dtype, void* stream) {
  if (n_tokens <= 0) return SXB_OK;
  if (taps < 1 || (taps > 1 && state == nullptr) || (out2 != nullptr && w2 == nullptr)) return SXB_ERR_BAD_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  if (taps <= 4 && width % 8 == 0 && aligned16({x, w1, filt, state, out, w2, out2})) {
    const dim3 grid((n_tokens + kNfRows - 1) / kNfRows, (width / 8 + 127) / 128);
    const int nt = std::min(128, (width / 8 + 31) / 32 * 32);
#define NORM_FILTER(TAPS)                                                                                             \
  SEQMIX_DISPATCH(dtype, (norm_filter_vec_kernel<T, TAPS><<<grid, nt, 0, s>>>(                                        \
                             (const float*)x, (const float*)rstd, (const T*)w1, (const T*)filt, (float*)state,        \
                             (const int*)seq_info, (const int*)tok_seq, (T*)out, (const T*)w2, (T*)out2, width, n_tokens)))
    if (taps == 1) NORM_FILTER(1);
    else if (taps == 2) NORM_FILTER(2);
    else if (taps == 3) NORM_FILTER(3);
    else NORM_FILTER(4);
#undef NORM_FILTER
    SXB_CHECK_LAUNCH();
    return SXB_OK;
  }
  const int gy = (width + 1023) / 1024;
  SEQMIX_DISPATCH(dtype, (norm_filter_kernel<T><<<dim3(n_tokens, gy), 256, 0, s>>>(
                             (const float*)x, (const float*)rstd, (const T*)w1, (const T*)filt, (const float*)state,
                             (const int*)seq_info, (const int*)tok_seq, (T*)out, (const T*)w2, (T*)out2, width, taps)));
  SXB_CHECK_LAUNCH();
  if (taps > 1) {
    SEQMIX_DISPATCH(dtype, (norm_filter_state_kernel<T><<<dim3(n_seqs, gy), 256, 0, s>>>(
                               (const float*)x, (const float*)rstd, (const T*)w1, (float*)state, (const int*)seq_info, width,
                               taps)));
    SXB_CHECK_LAUNCH();
  }
  return SXB_OK;
}

/* Rows of a fused projection (`dtype`, pitch ld): q (Hq d channels at column q0), k (G d at k0), v (G dv at v0, which may be k0).
 * q_w / k_w (`dtype` [Hq d] / [G d] or null): RMS norm over the whole row of q / k with that weight.  The first n_rot channels of
 * every q and k head turn by pos * inv_freq[i] (fp32 [n_rot / 2]) in pairs (2i, 2i+1) (interleaved != 0) or (i, i + n_rot/2), cos
 * and sin multiplied by amp.
 * q -> q_out fp32 [n_tokens, Hq, d] times q_scale[h] (fp32 or null), k -> kcache [pages, block_size, G, d], v -> vcache
 * [pages, block_size, G, dv] at each token's (page, offset). */
SXB_API int sxb_rope_append(const void* proj, long long ld, int q0, int k0, int v0, const void* q_w, const void* k_w,
                            const void* inv_freq, const void* q_scale, void* q_out, void* kcache, void* vcache,
                            const void* tok_seq, const void* tok_pos, const void* tables, int n_tokens, int max_blocks,
                            int block_size, int Hq, int G, int d, int dv, int n_rot, int interleaved, float eps, float amp,
                            int dtype, void* stream) {
  if (n_tokens <= 0) return SXB_OK;
  if (n_rot < 0 || n_rot > d || (n_rot & 1) || (n_rot > 0 && inv_freq == nullptr) || Hq % G) return SXB_ERR_BAD_ARG;
  const int turn = interleaved ? n_rot : n_rot / 2;
  const bool vec = d % 4 == 0 && dv % 4 == 0 && turn % 4 == 0 && ld % 4 == 0 && q0 % 4 == 0 && k0 % 4 == 0 && v0 % 4 == 0 &&
                   aligned16({proj, q_w, k_w, q_out, kcache, vcache});
  const size_t smem = (size_t)n_rot * sizeof(float);
  cudaStream_t s = (cudaStream_t)stream;
#define ROPE_APPEND(VEC)                                                                                               \
  SEQMIX_DISPATCH(dtype, (rope_append_kernel<T, VEC><<<n_tokens, 256, smem, s>>>(                                      \
                             (const T*)proj, ld, q0, k0, v0, (const T*)q_w, (const T*)k_w, (const float*)inv_freq,     \
                             (const float*)q_scale, (float*)q_out, (T*)kcache, (T*)vcache, (const int*)tok_seq,        \
                             (const int*)tok_pos, (const int*)tables, max_blocks, block_size, Hq, G, d, dv, n_rot,     \
                             interleaved, eps, amp)))
  if (vec) ROPE_APPEND(4);
  else ROPE_APPEND(1);
#undef ROPE_APPEND
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Operands of the delta rule with removal from projection rows (`dtype`, pitch ld; r, k, v, a: H n channels at columns r0, k0, v0,
 * a0; the decay's inner projection: rank channels at low0): buf fp32 [n_tokens, H, 5, n] = w | u | a | r | v' with w = exp(-rate
 * sigmoid(w2^T tanh(low) + w0)) (w2 `dtype` [rank, H n], w0 fp32 [H n]), u = k / sqrt(sum k^2 + eps) per head, a = sigmoid(a +
 * a_bias) (fp32 [H n]), v' = v sqrt(sum k^2 + eps). */
SXB_API int sxb_removal_prepare(const void* proj, long long ld, int r0, int k0, int v0, int a0, int low0, const void* w2,
                                const void* w0, const void* a_bias, void* buf, int n_tokens, int H, int n, int rank,
                                float rate, float eps, int dtype, void* stream) {
  if (n_tokens <= 0) return SXB_OK;
  if (n > 256 || n < 1 || rank < 1 || rank > 1024) return SXB_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  const bool pair = n % 2 == 0 && ld % 2 == 0 && r0 % 2 == 0 && k0 % 2 == 0 && v0 % 2 == 0 && a0 % 2 == 0 &&
                    aligned16({proj, w2, buf});
  const int tt = n_tokens >= 512 ? 8 : 1, cpt = pair ? 2 : 1;
  const int threads = ((n + cpt - 1) / cpt + 31) / 32 * 32;
  const dim3 grid((n_tokens + tt - 1) / tt, H);
  const size_t smem = (size_t)rank * tt * sizeof(float);
#define REMOVAL_PREP(TT, CPT)                                                                                           \
  SEQMIX_DISPATCH(dtype, (removal_prepare_kernel<T, TT, CPT><<<grid, threads, smem, s>>>(                               \
                             (const T*)proj, ld, r0, k0, v0, a0, low0, (const T*)w2, (const float*)w0,                  \
                             (const float*)a_bias, (float*)buf, n_tokens, H, n, rank, rate, eps)))
  if (tt == 8) {
    if (pair) REMOVAL_PREP(8, 2);
    else REMOVAL_PREP(8, 1);
  } else {
    if (pair) REMOVAL_PREP(1, 2);
    else REMOVAL_PREP(1, 1);
  }
#undef REMOVAL_PREP
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Per sequence and head, rows in order: S <- diag(w) S - (a u) (u^T S) + u v'^T (both terms read the old S), o = S^T r, with buf from
 * sxb_removal_prepare; state fp32 [slots, H, n (value), n (key)] is taken as zero when the sequence has seen no token and
 * written back; out fp32 [n_tokens, H n].  single_rows != 0: every sequence has exactly one batch row. */
SXB_API int sxb_removal_recurrence(const void* buf, void* state, void* out, const void* seq_info, int n_seqs, int H, int n,
                                   int single_rows, void* stream) {
  if (n_seqs <= 0) return SXB_OK;
  if (n > 256 || n < 1) return SXB_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  if (single_rows && n % 4 == 0 && aligned16({buf, state})) {
    const int per = kStepCols * kStepWarps;
    const dim3 grid((n + per - 1) / per, H, n_seqs);
    if (n <= 128)
      removal_step_kernel<1><<<grid, 32 * kStepWarps, 0, s>>>((const float*)buf, (float*)state, (float*)out,
                                                              (const int*)seq_info, H, n);
    else
      removal_step_kernel<2><<<grid, 32 * kStepWarps, 0, s>>>((const float*)buf, (float*)state, (float*)out,
                                                              (const int*)seq_info, H, n);
    SXB_CHECK_LAUNCH();
    return SXB_OK;
  }
#define REMOVAL_REC(R, LPC)                                                                                            \
  do {                                                                                                                 \
    constexpr int cols = kRmThreads / LPC;                                                                             \
    const size_t smem = (size_t)2 * (4 * kRmTB * (R * LPC) + kRmTB * cols) * sizeof(float);                            \
    if (smem > 48 * 1024) {                                                                                            \
      cudaError_t e = cudaFuncSetAttribute(removal_recurrence_kernel<R, LPC>,                                          \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                    \
      if (e != cudaSuccess) return (int)e;                                                                             \
    }                                                                                                                  \
    removal_recurrence_kernel<R, LPC><<<dim3((n + cols - 1) / cols, H, n_seqs), kRmThreads, smem, s>>>(                \
        (const float*)buf, (float*)state, (float*)out, (const int*)seq_info, H, n);                                    \
  } while (0)
  if (n <= 32) REMOVAL_REC(4, 8);
  else if (n <= 64) REMOVAL_REC(8, 8);
  else if (n <= 128) REMOVAL_REC(16, 8);
  else REMOVAL_REC(32, 8);
#undef REMOVAL_REC
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}
