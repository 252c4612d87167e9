// gated_mixers.cu — ragged-batch kernels for mixers with elementwise-gated recurrences: operands of decayed sums of outer
// products (lightning attention, gated linear attention) for linear_recurrence, and the gated linear recurrent unit.
//
// Conventions as in seq_mixers.cu: `seq_info[s] = {first row, rows, tokens already seen, state slot}`, `T` is the activation type
// (bf16 or float); gates, decays and recurrences are fp32 in both.
//
//   silu_columns         fp32 copy of projection columns behind a SiLU
//   decay_prepare        fp32 q (scaled), k, v and the decay per (head, key channel) from a two-step projection
//   lru_gates            a = exp(rate r), sqrt(1 - a^2) i u with r, i = sigmoid of block-diagonal products of the filtered input u
//   lru_scan / lru_step  s <- a s + g per channel, output s * gelu(y + bias); the unit's carried filter inputs move on
#include <algorithm>
#include <initializer_list>
#include "seq_common.cuh"

namespace sxb {
namespace seqmix {

__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// ------------------------------------------------------------------------------------------------ operand rows
// out[t, c] = silu(x[t, c]), VEC consecutive channels per thread.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
silu_columns_kernel(const T* __restrict__ x, long long ld, float* __restrict__ out, long long total, int C) {
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= total) return;
  const long long t = i / C;
  const int c = (int)(i % C);
  if (VEC == 8) {
    float v[8];
    load8_f32<T>(x + t * ld + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = silu_f(v[e]);
    store8_f32<float>(out + i, v);
  } else {
    out[i] = silu_f(to_f32<T>(x[t * ld + c]));
  }
}

// Per token: q * qscale | k | v as fp32 (buf rows of 2 Hn + Hv), and decay[c] = sigmoid(z)^inv_tau with z = w2^T low + bias over the
// Hn key channels (low: `rank` projection columns, w2 [rank, Hn]).  A CTA takes TT tokens and blockDim.x * CPT columns; a thread
// reads its entries of w2 once for all TT tokens.
template <typename T, int TT, int CPT>
__global__ void __launch_bounds__(128)
decay_prepare_kernel(const T* __restrict__ proj, long long ld, int q0, int k0, int v0, int low0,
                     const T* __restrict__ w2, const float* __restrict__ bias, float* __restrict__ buf,
                     float* __restrict__ decay, int n_tokens, int Hn, int Hv, int rank, float qscale, float inv_tau) {
  extern __shared__ __align__(16) float low[];             // [rank][TT]
  const int t0 = blockIdx.x * TT, nt = min(TT, n_tokens - t0);
  for (int i = threadIdx.x; i < rank * TT; i += blockDim.x) {
    const int j = i % rank, tt = i / rank;
    low[j * TT + tt] = tt < nt ? to_f32<T>(proj[(long long)(t0 + tt) * ld + low0 + j]) : 0.f;
  }
  __syncthreads();
  struct alignas(sizeof(T) * CPT) Vt { T v[CPT]; };
  struct alignas(4 * CPT) Vf { float v[CPT]; };
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * CPT;
  const long long bw = 2LL * Hn + Hv;
  auto copy = [&](int src, int dst, float f) {
    Vt in[TT];
#pragma unroll
    for (int tt = 0; tt < TT; ++tt)
      if (tt < nt) in[tt] = *reinterpret_cast<const Vt*>(proj + (long long)(t0 + tt) * ld + src + c);
#pragma unroll
    for (int tt = 0; tt < TT; ++tt)
      if (tt < nt) {
        Vf o;
#pragma unroll
        for (int e = 0; e < CPT; ++e) o.v[e] = to_f32<T>(in[tt].v[e]) * f;
        *reinterpret_cast<Vf*>(buf + (t0 + tt) * bw + dst + c) = o;
      }
  };
  if (c < Hv) copy(v0, 2 * Hn, 1.f);
  if (c >= Hn) return;
  copy(q0, 0, qscale);
  copy(k0, Hn, 1.f);
  float acc[TT][CPT];
#pragma unroll
  for (int tt = 0; tt < TT; ++tt)
#pragma unroll
    for (int e = 0; e < CPT; ++e) acc[tt][e] = bias[c + e];
#pragma unroll 4
  for (int j = 0; j < rank; ++j) {
    const Vt wv = *reinterpret_cast<const Vt*>(w2 + (long long)j * Hn + c);
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
      const float w = to_f32<T>(wv.v[e]);
#pragma unroll
      for (int tt = 0; tt < TT; ++tt) acc[tt][e] += w * low[j * TT + tt];
    }
  }
#pragma unroll
  for (int tt = 0; tt < TT; ++tt)
    if (tt < nt) {
      Vf o;
#pragma unroll
      for (int e = 0; e < CPT; ++e) {
        const float z = acc[tt][e];
        o.v[e] = expf(inv_tau * (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))));      // log sigmoid(z), no overflow on either side
      }
      *reinterpret_cast<Vf*>(decay + (long long)(t0 + tt) * Hn + c) = o;
    }
}

// ------------------------------------------------------------------------------------------------ gated linear recurrent unit
// u fp32 [tokens, N] in `blocks` parts of S channels.  For output channel c of part b: r = sigmoid(u_b . w[0][b][:, c] + bias[0]),
// i = sigmoid(u_b . w[1][b][:, c] + bias[1]);  a = exp(rate[c] r),  g = sqrt(1 - a^2) i u[c].  w: [2][blocks][S in][S out].
// A CTA holds a tile of 64 tokens x BN channels of one part for BOTH gates: 256 threads, each 4 tokens x BN/16 channels x 2 gates,
// packed pairs (fma.f32x2).  The tiles of u and w for the next KT input channels are fetched into registers while the current
// ones are multiplied.
constexpr int kLruBM = 64, kLruKT = 16;

template <typename T, int BN>
__global__ void __launch_bounds__(256)
lru_gates_kernel(const float* __restrict__ u, const T* __restrict__ w, const float* __restrict__ bias,
                 const float* __restrict__ rate, float* __restrict__ a_out, float* __restrict__ g_out, int n_tokens, int N,
                 int S, int vec) {
  constexpr int BM = kLruBM, KT = kLruKT, CN = BN / 16, NB = 2 * KT * BN / 256;      // NB: weight elements a thread fetches
  static_assert(NB >= 2 && NB % 2 == 0 && (CN == 1 || CN % 2 == 0), "tile shape");
  __shared__ __align__(16) float As[2][KT][BM + 4];
  __shared__ __align__(16) float Bs[2][2][KT][BN];
  const int tiles = (S + BN - 1) / BN, b = blockIdx.y / tiles, n0 = (blockIdx.y % tiles) * BN;
  const int t0 = blockIdx.x * BM, c0 = b * S, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const long long gate_stride = (long long)N * S;
  float ar[4];
  float br[NB];
  const int arow = tid >> 2, ak = (tid & 3) * 4;                      // a thread fetches 4 input channels of one token
  auto fetch = [&](int k0) {
    const int t = t0 + arow, k = k0 + ak;
    const float* p = u + (long long)t * N + c0 + k;
    if (vec && t < n_tokens && k + 3 < S) {
      const float4 v = *reinterpret_cast<const float4*>(p);
      ar[0] = v.x, ar[1] = v.y, ar[2] = v.z, ar[3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) ar[e] = (t < n_tokens && k + e < S) ? p[e] : 0.f;
    }
#pragma unroll
    for (int x = 0; x < NB / 2; ++x)
#pragma unroll
      for (int gate = 0; gate < 2; ++gate) {
        const int i = tid + 256 * x, kk = i / BN, n = i % BN;
        br[2 * x + gate] = (k0 + kk < S && n0 + n < S)
                               ? to_f32<T>(w[gate * gate_stride + ((long long)b * S + k0 + kk) * S + n0 + n])
                               : 0.f;
      }
  };
  auto stash = [&](int buf) {
#pragma unroll
    for (int e = 0; e < 4; ++e) As[buf][ak + e][arow] = ar[e];
#pragma unroll
    for (int x = 0; x < NB / 2; ++x)
#pragma unroll
      for (int gate = 0; gate < 2; ++gate) {
        const int i = tid + 256 * x;
        Bs[buf][gate][i / BN][i % BN] = br[2 * x + gate];
      }
  };
  float2 acc[2][4][(CN + 1) / 2];
#pragma unroll
  for (int gate = 0; gate < 2; ++gate)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < (CN + 1) / 2; ++j) acc[gate][i][j] = make_float2(0.f, 0.f);
  fetch(0);
  stash(0);
  __syncthreads();
  int buf = 0;
  for (int k0 = 0; k0 < S; k0 += KT, buf ^= 1) {
    const bool more = k0 + KT < S;
    if (more) fetch(k0 + KT);
#pragma unroll
    for (int k = 0; k < KT; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&As[buf][k][ty * 4]);
      const float a4[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
      for (int gate = 0; gate < 2; ++gate) {
        float2 bv[(CN + 1) / 2];
        if (CN == 4) {
          const float4 v = *reinterpret_cast<const float4*>(&Bs[buf][gate][k][tx * CN]);
          bv[0] = make_float2(v.x, v.y), bv[(CN + 1) / 2 - 1] = make_float2(v.z, v.w);
        } else {
#pragma unroll
          for (int j = 0; j < (CN + 1) / 2; ++j)
            bv[j] = make_float2(Bs[buf][gate][k][tx * CN + 2 * j], CN == 1 ? 0.f : Bs[buf][gate][k][tx * CN + 2 * j + (CN > 1)]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < (CN + 1) / 2; ++j) acc[gate][i][j] = __ffma2_rn(make_float2(a4[i], a4[i]), bv[j], acc[gate][i][j]);
      }
    }
    if (more) stash(buf ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= n_tokens) continue;
#pragma unroll
    for (int j = 0; j < CN; ++j) {
      const int n = n0 + tx * CN + j;
      if (n >= S) continue;
      const int c = c0 + n;
      const float zr = (j & 1) ? acc[0][i][j / 2].y : acc[0][i][j / 2].x, zi = (j & 1) ? acc[1][i][j / 2].y : acc[1][i][j / 2].x;
      const float la = rate[c] * sigmoid_f(zr + bias[c]);
      const long long o = (long long)t * N + c;
      a_out[o] = expf(la);
      g_out[o] = sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi + bias[N + c]) * u[o];
    }
  }
}

// After the last use of a sequence's carried filter inputs in a batch: row j of the slot becomes row rows + j of (carried ++ new).
template <typename T>
__device__ __forceinline__ void move_inputs(const T* x, long long ld, T* st, int first, int n, int seen, int keep, int C, int c) {
  for (int j = 0; j < keep; ++j) {          // n >= 1, so ascending order never overwrites a source
    const int i = n + j;
    T v = from_f32<T>(0.f);
    if (i >= keep) v = x[(long long)(first + i - keep) * ld + c];
    else if (seen + i - keep >= 0) v = st[(long long)i * C + c];
    st[(long long)j * C + c] = v;
  }
}

// s <- a s + g per channel over the rows of each sequence, s from the slot (zero at its start); out = s * gelu(y + ybias) * scale.
// A CTA takes 32 channels of one sequence (a lane each) and cuts its rows into one segment per warp: every warp multiplies out
// its segment (product of a, result from zero), takes the state in front of it from the segments before, and walks it again.
constexpr int kLruWarps = 32;

template <typename T>
__global__ void __launch_bounds__(32 * kLruWarps)
lru_scan_kernel(const float* __restrict__ a, const float* __restrict__ g, const T* __restrict__ y, long long ldy,
                const T* __restrict__ ybias, const T* __restrict__ x, long long ldx, float* __restrict__ state,
                T* __restrict__ conv_state, const int* __restrict__ seq_info, T* __restrict__ out, long long out_ld, int N,
                int keep, float scale) {
  __shared__ float sa[kLruWarps][32], sg[kLruWarps][32];
  const int* si = seq_info + 4 * blockIdx.y;
  const int first = si[0], rows = si[1], seen = si[2];
  const long long slot = si[3];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane, cc = min(c, N - 1);
  const int seg = (rows + kLruWarps - 1) / kLruWarps;
  const int r0 = min(warp * seg, rows), r1 = min(r0 + seg, rows);
  constexpr int U = 8;                                      // rows in flight
  const float* ap = a + (long long)first * N + cc;
  const float* gp = g + (long long)first * N + cc;
  float pa = 1.f, pg = 0.f;
  for (int r = r0; r < r1; r += U) {
    float av[U], gv[U];
#pragma unroll
    for (int q = 0; q < U; ++q) {
      const bool in = r + q < r1;
      av[q] = in ? ap[(long long)(r + q) * N] : 1.f;
      gv[q] = in ? gp[(long long)(r + q) * N] : 0.f;
    }
#pragma unroll
    for (int q = 0; q < U; ++q) pg = av[q] * pg + gv[q], pa *= av[q];
  }
  sa[warp][lane] = pa, sg[warp][lane] = pg;
  float s = (seen > 0) ? state[slot * N + cc] : 0.f;        // read before the barrier: the last warp writes the new one behind it
  __syncthreads();
  for (int w = 0; w < warp; ++w) s = sa[w][lane] * s + sg[w][lane];
  const float yb = to_f32<T>(ybias[cc]);
  for (int r = r0; r < r1; r += U) {
    float av[U], gv[U], yv[U];
#pragma unroll
    for (int q = 0; q < U; ++q) {
      const bool in = r + q < r1;
      av[q] = in ? ap[(long long)(r + q) * N] : 1.f;
      gv[q] = in ? gp[(long long)(r + q) * N] : 0.f;
      yv[q] = in ? to_f32<T>(y[(long long)(first + r + q) * ldy + cc]) : 0.f;
    }
#pragma unroll
    for (int q = 0; q < U; ++q) {
      s = av[q] * s + gv[q];
      if (r + q < r1 && c < N) out[(long long)(first + r + q) * out_ld + c] = from_f32<T>(s * gelu_tanh_f(yv[q] + yb) * scale);
    }
  }
  if (c >= N) return;
  if (warp == kLruWarps - 1) state[slot * N + c] = s;        // trailing warps without rows carry the final state through
  if (warp == 0 && keep > 0) move_inputs<T>(x, ldx, conv_state + slot * keep * N, first, rows, seen, keep, N, c);
}

// The same for batches of one row per sequence: one thread per (sequence, channel).
template <typename T>
__global__ void __launch_bounds__(256)
lru_step_kernel(const float* __restrict__ a, const float* __restrict__ g, const T* __restrict__ y, long long ldy,
                const T* __restrict__ ybias, const T* __restrict__ x, long long ldx, float* __restrict__ state,
                T* __restrict__ conv_state, const int* __restrict__ seq_info, T* __restrict__ out, long long out_ld, int N,
                int keep, float scale) {
  const int* si = seq_info + 4 * blockIdx.y;
  const int row = si[0], seen = si[2];
  const long long slot = si[3];
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= N) return;
  const long long o = (long long)row * N + c;
  const float s = a[o] * (seen > 0 ? state[slot * N + c] : 0.f) + g[o];
  state[slot * N + c] = s;
  out[(long long)row * out_ld + c] =
      from_f32<T>(s * gelu_tanh_f(to_f32<T>(y[(long long)row * ldy + c]) + to_f32<T>(ybias[c])) * scale);
  if (keep > 0) move_inputs<T>(x, ldx, conv_state + slot * keep * N, row, 1, seen, keep, N, c);
}

static bool words16(std::initializer_list<const void*> ps) {
  uintptr_t x = 0;
  for (const void* p : ps) x |= reinterpret_cast<uintptr_t>(p);
  return (x & 15) == 0;
}

}  // namespace seqmix
}  // namespace sxb

using namespace sxb;
using namespace sxb::seqmix;

/* out fp32 [n_tokens, C] = silu(x) of C columns of `dtype` rows with pitch ld. */
SXB_API int sxb_silu_columns(const void* x, long long ld, void* out, int n_tokens, int C, int dtype, void* stream) {
  const long long total = (long long)n_tokens * C;
  if (total <= 0) return SXB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  if (C % 8 == 0 && ld % 8 == 0 && words16({x, out})) {
    SEQMIX_DISPATCH(dtype, (silu_columns_kernel<T, 8><<<(unsigned)((total / 8 + 255) / 256), 256, 0, s>>>(
                               (const T*)x, ld, (float*)out, total, C)));
  } else {
    SEQMIX_DISPATCH(dtype, (silu_columns_kernel<T, 1><<<(unsigned)((total + 255) / 256), 256, 0, s>>>(
                               (const T*)x, ld, (float*)out, total, C)));
  }
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Projection rows (`dtype`, pitch ld; q and k: Hn channels at columns q0 and k0, v: Hv at v0, low: rank at low0) -> buf fp32
 * [n_tokens, 2 Hn + Hv] = q * qscale | k | v and decay fp32 [n_tokens, Hn] = sigmoid(low w2 + bias)^(1 / tau) with w2 `dtype`
 * [rank, Hn], bias fp32 [Hn], inv_tau = 1 / tau; the inner product is 32-bit. */
SXB_API int sxb_decay_prepare(const void* proj, long long ld, int q0, int k0, int v0, int low0, const void* w2,
                              const void* bias, void* buf, void* decay, int n_tokens, int Hn, int Hv, int rank, float qscale,
                              float inv_tau, int dtype, void* stream) {
  if (n_tokens <= 0) return SXB_OK;
  if (Hn < 1 || Hv < 1 || rank < 1 || rank > 1024) return SXB_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  const bool pair = Hn % 2 == 0 && Hv % 2 == 0 && ld % 2 == 0 && q0 % 2 == 0 && k0 % 2 == 0 && v0 % 2 == 0 &&
                    words16({proj, w2, buf, decay});
  const int tt = n_tokens >= 512 ? 8 : 1, cols = 128 * (pair ? 2 : 1);
  const dim3 grid((n_tokens + tt - 1) / tt, (std::max(Hn, Hv) + cols - 1) / cols);
  const size_t smem = (size_t)rank * tt * sizeof(float);
#define DECAY_PREP(TT, CPT)                                                                                              \
  SEQMIX_DISPATCH(dtype, (decay_prepare_kernel<T, TT, CPT><<<grid, 128, smem, s>>>(                                      \
                             (const T*)proj, ld, q0, k0, v0, low0, (const T*)w2, (const float*)bias, (float*)buf,        \
                             (float*)decay, n_tokens, Hn, Hv, rank, qscale, inv_tau)))
  if (tt == 8) {
    if (pair) DECAY_PREP(8, 2);
    else DECAY_PREP(8, 1);
  } else {
    if (pair) DECAY_PREP(1, 2);
    else DECAY_PREP(1, 1);
  }
#undef DECAY_PREP
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Gates of the linear recurrent unit from its filtered input u fp32 [n_tokens, N] (`blocks` parts of S = N / blocks channels):
 * r, i = sigmoid(u_b w[gate][b] + bias[gate]) (w `dtype` [2, blocks, S in, S out], bias fp32 [2, N]); a_out = exp(rate r)
 * (rate fp32 [N], not positive), g_out = sqrt(1 - a^2) i u; fp32 [n_tokens, N] each, products and sums 32-bit. */
SXB_API int sxb_lru_gates(const void* u, const void* w, const void* bias, const void* rate, void* a_out, void* g_out,
                          int n_tokens, int N, int blocks, int dtype, void* stream) {
  if (n_tokens <= 0) return SXB_OK;
  if (N < 1 || blocks < 1 || N % blocks) return SXB_ERR_BAD_ARG;
  const int S = N / blocks, vec = S % 4 == 0 && words16({u});
  cudaStream_t s = (cudaStream_t)stream;
  // few rows or narrow parts: narrow tiles, so that every SM has one
  const bool wide = n_tokens > 256 && S > 32;
  const int bn = wide ? 64 : 16;
  const dim3 grid((n_tokens + kLruBM - 1) / kLruBM, blocks * ((S + bn - 1) / bn));
#define LRU_GATES(BN)                                                                                          \
  SEQMIX_DISPATCH(dtype, (lru_gates_kernel<T, BN><<<grid, 256, 0, s>>>(                                        \
                             (const float*)u, (const T*)w, (const float*)bias, (const float*)rate, (float*)a_out, \
                             (float*)g_out, n_tokens, N, S, vec)))
  if (wide) LRU_GATES(64);
  else LRU_GATES(16);
#undef LRU_GATES
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}

/* Per sequence and channel, rows in order: s <- a s + g (a, g fp32 [n_tokens, N]); out `dtype` (pitch out_ld) = s * gelu_tanh(y +
 * ybias) * scale with y `dtype` rows of pitch ldy and ybias `dtype` [N].  state fp32 [slots, N] is taken as zero when the sequence
 * has seen no token and written back.  conv_state `dtype` [slots, keep, N] (keep 0: none) moves on: it is left holding the last
 * keep rows of (carried rows ++ this batch's rows of x, `dtype`, pitch ldx).  single_rows != 0: one batch row per sequence. */
SXB_API int sxb_lru_scan(const void* a, const void* g, const void* y, long long ldy, const void* ybias, const void* x,
                         long long ldx, void* state, void* conv_state, const void* seq_info, void* out, long long out_ld,
                         int n_seqs, int N, int keep, float scale, int single_rows, int dtype, void* stream) {
  if (n_seqs <= 0) return SXB_OK;
  if (N < 1 || keep < 0 || (keep > 0 && conv_state == nullptr)) return SXB_ERR_BAD_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  if (single_rows) {
    SEQMIX_DISPATCH(dtype, (lru_step_kernel<T><<<dim3((N + 255) / 256, n_seqs), 256, 0, s>>>(
                               (const float*)a, (const float*)g, (const T*)y, ldy, (const T*)ybias, (const T*)x, ldx,
                               (float*)state, (T*)conv_state, (const int*)seq_info, (T*)out, out_ld, N, keep, scale)));
  } else {
    SEQMIX_DISPATCH(dtype, (lru_scan_kernel<T><<<dim3((N + 31) / 32, n_seqs), 32 * kLruWarps, 0, s>>>(
                               (const float*)a, (const float*)g, (const T*)y, ldy, (const T*)ybias, (const T*)x, ldx,
                               (float*)state, (T*)conv_state, (const int*)seq_info, (T*)out, out_ld, N, keep, scale)));
  }
  SXB_CHECK_LAUNCH();
  return SXB_OK;
}
