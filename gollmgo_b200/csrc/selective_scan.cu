// A selective scan (a state-space layer of the Mamba-1 kind).  I channels evolve alone, each with a state of N
// values in float32, carried in the request's state slot [I, N]:
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
// with A = -exp(A_log) (one value per channel and state, so there is no form in chunks of matrix products), B and C
// the same for all channels, dt = softplus(v + bias) per channel; the result is multiplied by silu(z).
//
//   scan_conv   x = silu(short causal convolution per channel + bias) from the projection's rows and the window of
//               the last taps - 1 inputs carried in the state slot
//   (two products make B, C and v from x)
//   scan_run    the recurrence over every sequence's tokens of the step, from the products' rows to the gated rows;
//               moves the convolution's window on
//   scan_step   the same for steps of single tokens
// A channel's N states lie in L neighbouring lanes, K each.  The exponentials bound the long form: N a token and
// channel at 16 a clock and multiprocessor; the chain from token to token is one multiply-add, so blocks of channels
// walk the whole sequence and nothing is cut along time.  A2 = A log2(e), so that exp is exp2 of one product.
#include "common.cuh"

#define SC_THREADS 128
#define SC_TT 32                    // tokens staged at a time
#define SC_RUN 8                    // tokens a thread of the convolution takes in long steps

__device__ __forceinline__ float sc_silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }
// silu: of bfloat16 rows with the fast exponential and division, of float32 rows exact to rounding
template <typename TA> __device__ __forceinline__ float sc_gate(float z) {
  if constexpr (sizeof(TA) == 4) return z / (1.f + expf(-z));
  return sc_silu(z);
}
// softplus(x) = max(x, 0) + log(1 + e), e = exp(-|x|), with log(1 + e) = 2 atanh(e / (2 + e)) by its power series: the
// argument is at most 1/3, so the terms up to the 17th power leave less than a unit of float32 rounding.
__device__ __forceinline__ float sc_softplus(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = 2.f / 17.f;
  p = fmaf(p, q, 2.f / 15.f); p = fmaf(p, q, 2.f / 13.f); p = fmaf(p, q, 2.f / 11.f); p = fmaf(p, q, 2.f / 9.f);
  p = fmaf(p, q, 2.f / 7.f); p = fmaf(p, q, 2.f / 5.f); p = fmaf(p, q, 2.f / 3.f); p = fmaf(p, q, 2.f);
  return fmaf(s, p, fmaxf(x, 0.f));
}
// two float32 operations in one instruction, each half rounded as the scalar one
__device__ __forceinline__ float2 sc_fma2(float2 a, float2 b, float2 c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(*reinterpret_cast<unsigned long long*>(&a)),
      "l"(*reinterpret_cast<unsigned long long*>(&b)), "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&d);
}
__device__ __forceinline__ float2 sc_mul2(float2 a, float2 b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(*reinterpret_cast<unsigned long long*>(&a)),
      "l"(*reinterpret_cast<unsigned long long*>(&b)));
  return *reinterpret_cast<float2*>(&d);
}

__device__ __forceinline__ int sc_seq_of_token(const int* __restrict__ cu, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

template <int V, typename T> __device__ __forceinline__ void sc_load(float (&o)[V], const T* p) {
  if constexpr (V == 1) o[0] = to_f32(*p);
  else if constexpr (sizeof(T) == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    o[0] = q.x; o[1] = q.y; o[2] = q.z; o[3] = q.w;
  } else {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
    o[0] = lo.x; o[1] = lo.y; o[2] = hi.x; o[3] = hi.y;
  }
}
template <int V> __device__ __forceinline__ void sc_store(float* p, const float (&v)[V]) {
  if constexpr (V == 1) *p = v[0];
  else *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <int V> __device__ __forceinline__ void sc_store(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 1) *p = from_f32<__nv_bfloat16>(v[0]);
  else {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  }
}

// ---------------------------------------------------------------- the convolution
// grid (ceil(T / tt), ceil(C / (128 V))): a thread takes V channels of tt tokens in a row; with TAPS > 0 it keeps the
// last inputs in registers, else every tap is read.
template <typename TA, int TAPS, int V>
__global__ void __launch_bounds__(SC_THREADS)
scan_conv_kernel(const TA* __restrict__ x, long long stride, const float* __restrict__ w, const float* __restrict__ bias,
                 const float* __restrict__ conv_state, const int* __restrict__ cu, const int* __restrict__ context_lens,
                 const int* __restrict__ state_slots, int T, int B, int C, int taps_rt, int tt, TA* __restrict__ out) {
  pdl_trigger();
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  const int c = (blockIdx.y * SC_THREADS + threadIdx.x) * V;
  if (c >= C) return;
  constexpr int WT = TAPS > 0 ? TAPS : 1;
  float wt[WT][V], b[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    b[v] = bias ? bias[c + v] : 0.f;
    if constexpr (TAPS == 4) {                   // (rows of four floats)
      const float4 q = *reinterpret_cast<const float4*>(w + (size_t)(c + v) * 4);
      wt[0][v] = q.x; wt[1][v] = q.y; wt[2][v] = q.z; wt[3][v] = q.w;
    } else if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < WT; ++j) wt[j][v] = w[(size_t)(c + v) * taps + j];
    }
  }
  const int ta = blockIdx.x * tt, tb = min(T, ta + tt);
  int s = sc_seq_of_token(cu, B, ta);
  pdl_wait();
  int s0 = 0, s1 = 0;
  const float* st = nullptr;
  float win[WT][V];
  auto at = [&](int i, float (&o)[V]) {          // the input i tokens into this step's portion (i < 0: carried or before the start)
    if (i >= 0) sc_load<V>(o, x + (size_t)(s0 + i) * stride + c);
    else if (st) sc_load<V>(o, st + (size_t)(taps - 1 + i) * C + c);
    else {
#pragma unroll
      for (int v = 0; v < V; ++v) o[v] = 0.f;
    }
  };
  if constexpr (TAPS > 0) {
    s1 = s < B - 1 ? cu[s + 1] : T;
    if (tt == SC_RUN && tb - ta == SC_RUN && s1 >= tb) {
      // a whole run inside one sequence: every input asked for at once
      s0 = cu[s];
      const int slot = state_slots[s], start = context_lens[s] - (cu[s + 1] - s0);
      st = (slot >= 0 && start > 0 && taps > 1) ? conv_state + (size_t)slot * (taps - 1) * C : nullptr;
      float in[SC_RUN + WT - 1][V];
      if (ta - s0 >= WT - 1) {
        const TA* r = x + (size_t)(ta - (WT - 1)) * stride + c;
#pragma unroll
        for (int i = 0; i < SC_RUN + WT - 1; ++i) sc_load<V>(in[i], r + i * stride);
      } else {
#pragma unroll
        for (int i = 0; i < SC_RUN + WT - 1; ++i) at(ta - s0 - (WT - 1) + i, in[i]);
      }
#pragma unroll
      for (int i = 0; i < SC_RUN; ++i) {
        float acc[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
          acc[v] = b[v];
#pragma unroll
          for (int j = 0; j < WT; ++j) acc[v] = fmaf(wt[j][v], in[i + j][v], acc[v]);
          acc[v] = sc_gate<TA>(acc[v]);
        }
        sc_store<V>(out + (size_t)(ta + i) * C + c, acc);
      }
      return;
    }
    s1 = 0;
  }
  for (int t = ta; t < tb; ++t) {
    if (t >= s1) {                                // the first token here, or of the next sequence
      while (s < B - 1 && cu[s + 1] <= t) ++s;
      s0 = cu[s]; s1 = s < B - 1 ? cu[s + 1] : T;
      const int slot = state_slots[s], start = context_lens[s] - (cu[s + 1] - s0);
      st = (slot >= 0 && start > 0 && taps > 1) ? conv_state + (size_t)slot * (taps - 1) * C : nullptr;
      if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < WT - 1; ++j) at(t - s0 - (WT - 1) + j, win[j]);
      }
    }
    float acc[V];
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = b[v];
    if (TAPS > 0) {
      at(t - s0, win[WT - 1]);
#pragma unroll
      for (int j = 0; j < WT; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = fmaf(wt[j][v], win[j][v], acc[v]);
#pragma unroll
      for (int j = 0; j + 1 < WT; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) win[j][v] = win[j + 1][v];
    } else {
      for (int j = 0; j < taps; ++j) {
        float xv[V];
        at(t - s0 - (taps - 1) + j, xv);
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = fmaf(w[(size_t)(c + v) * taps + j], xv[v], acc[v]);
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = sc_gate<TA>(acc[v]);
    sc_store<V>(out + (size_t)t * C + c, acc);
  }
}

// ---------------------------------------------------------------- the recurrence
struct ScanArgs {
  const void* x;                                   // [T, I] after the convolution
  const void* proj; long long pstride;             // rows [x before it | z]
  const void* low; long long lstride; int bcol;    // rows [.. | B | C], B from column bcol
  const void* v; long long vstride;                // [T, I]: the step sizes before bias and softplus
  const void* w_dt; int rank;                      // scan_step: v is made here, row c of w_dt [I, rank] by low's first columns
  const float *dt_bias, *A2, *D;
  float *state, *conv_state; int taps;
  const int *cu, *context_lens, *state_slots;
  int I, N;
  void* out;                                       // [T, I]
};

// The window of the convolution moved on by qlen tokens, one channel a thread.
template <typename TA>
__device__ __forceinline__ void sc_move_window(const ScanArgs& a, int c, int slot, int t0, int qlen, int start) {
  const int keep = a.taps - 1;
  float* st = a.conv_state + (size_t)slot * keep * a.I + c;
  for (int j = 0; j < keep; ++j) {
    const int i = qlen - keep + j;
    float v = 0.f;
    if (i >= 0) v = to_f32(((const TA*)a.proj)[(size_t)(t0 + i) * a.pstride + c]);
    else if (start > 0) v = st[(size_t)(j + qlen) * a.I];          // j + qlen < keep: not yet overwritten
    st[(size_t)j * a.I] = v;
  }
}

template <typename TA> __device__ __forceinline__ float sc_exp2(float x) {
  if constexpr (sizeof(TA) == 4) return exp2f(x);
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void sc_unpack8(float (&o)[8], const uint4& q) {
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(p[i]); o[2 * i] = f.x; o[2 * i + 1] = f.y; }
}

// grid (B, ceil(I / CH)), CH = 128 / L channels a block, two kinds of warps: four walk the recurrence over tile i (32
// tokens), four others make tile i + 1 ready in shared memory (softplus, B and C in float32) and finish tile i - 1 (D, the
// gate, the store); one barrier a tile.  A walking warp is alone on its scheduler where channels are few, so whatever it
// need not do itself is taken from it.  FAST: bfloat16, N = L K, rows on 16-byte borders and whole blocks of channels: a
// staging thread keeps eight channels of one token in registers, asked for two tiles ahead.
template <typename TA, int L, int K, bool FAST>
__global__ void __launch_bounds__(2 * SC_THREADS) scan_run_kernel(ScanArgs a) {
  constexpr int CH = SC_THREADS / L, NP = L * K, TT = SC_TT, YLD = CH + 4, KP = (K + 1) / 2;
  constexpr int STAGE = 2 * TT * CH + 2 * TT * NP;         // floats of (dt, dt x), B and C of a tile
  extern __shared__ __align__(16) float sc_sm[];
  float* ysum = sc_sm + 2 * STAGE;                         // [2][TT][YLD]
  const int b = blockIdx.x, c0 = blockIdx.y * CH, I = a.I, N = a.N;
  const int t0 = a.cu[b], qlen = a.cu[b + 1] - t0, slot = a.state_slots[b], start = a.context_lens[b] - qlen;
  if (qlen <= 0) { pdl_trigger(); return; }
  const int tiles = (qlen + TT - 1) / TT;
  const TA *x = (const TA*)a.x, *proj = (const TA*)a.proj, *low = (const TA*)a.low, *vv = (const TA*)a.v;
  TA* out = (TA*)a.out;

  if (threadIdx.x >= SC_THREADS) {
    // ------------------------------------------------ staging warps
    const int tid = threadIdx.x - SC_THREADS;
    if constexpr (FAST) {
      constexpr int G8 = CH / 8 > 0 ? CH / 8 : 1, BCN = NP >= 16 ? NP / 16 : 1;
      const int ft = tid / G8, fc = (tid % G8) * 8;
      const bool fon = tid < TT * G8;
      const uint4 zero = make_uint4(0, 0, 0, 0);
      uint4 x0 = zero, z0 = zero, x1 = zero, z1 = zero, x2 = zero, z2 = zero, v2 = zero, bc2[BCN];       // tiles i - 1, i, i + 1
      float bias8[8], d8[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) { bias8[i] = fon ? a.dt_bias[c0 + fc + i] : 0.f; d8[i] = fon ? a.D[c0 + fc + i] : 0.f; }
      auto fetch = [&](int at) {
        const bool on = fon && at + ft < qlen;
        const size_t t = t0 + at + ft;
        x2 = on ? *reinterpret_cast<const uint4*>(x + t * I + c0 + fc) : zero;
        v2 = on ? *reinterpret_cast<const uint4*>(vv + t * a.vstride + c0 + fc) : zero;
        z2 = on ? *reinterpret_cast<const uint4*>(proj + t * a.pstride + I + c0 + fc) : zero;
#pragma unroll
        for (int u = 0; u < BCN; ++u) {
          const int e = tid + u * SC_THREADS, tok = e / (NP / 4), g = (e % (NP / 4)) * 8;      // g < NP: B, else C
          bc2[u] = tok < TT && at + tok < qlen ? *reinterpret_cast<const uint4*>(low + (size_t)(t0 + at + tok) * a.lstride + a.bcol + g) : zero;
        }
      };
      auto stage = [&](int at, float* buf) {
        float2* dtx = reinterpret_cast<float2*>(buf);
        float x8[8], v8[8];
        sc_unpack8(x8, x2); sc_unpack8(v8, v2);
        if (fon) {
          const bool real = at + ft < qlen;        // places past the end: dt = 0 leaves the state as it is
#pragma unroll
          for (int i = 0; i < 8; i += 2) {
            const float d0 = real ? sc_softplus(v8[i] + bias8[i]) : 0.f, d1 = real ? sc_softplus(v8[i + 1] + bias8[i + 1]) : 0.f;
            *reinterpret_cast<float4*>(dtx + ft * CH + fc + i) = make_float4(d0, d0 * x8[i], d1, d1 * x8[i + 1]);
          }
        }
#pragma unroll
        for (int u = 0; u < BCN; ++u) {
          const int e = tid + u * SC_THREADS, tok = e / (NP / 4), g = (e % (NP / 4)) * 8;
          float q[8];
          sc_unpack8(q, bc2[u]);
          float* dst = buf + 2 * TT * CH + (g < NP ? tok * NP + g : (TT + tok) * NP + g - NP);
          if (tok < TT) {
            *reinterpret_cast<float4*>(dst) = make_float4(q[0], q[1], q[2], q[3]);
            *reinterpret_cast<float4*>(dst + 4) = make_float4(q[4], q[5], q[6], q[7]);
          }
        }
      };
      auto finish = [&](int at, const float* ys) {
        if (fon && at + ft < qlen) {
          float x8[8], z8[8];
          sc_unpack8(x8, x0); sc_unpack8(z8, z0);
          const float4 y0 = *reinterpret_cast<const float4*>(ys + ft * YLD + fc), y1 = *reinterpret_cast<const float4*>(ys + ft * YLD + fc + 4);
          const float y8[8] = {y0.x, y0.y, y0.z, y0.w, y1.x, y1.y, y1.z, y1.w};
          uint4 o;
          __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
          for (int i = 0; i < 4; ++i)
            o2[i] = __floats2bfloat162_rn(fmaf(d8[2 * i], x8[2 * i], y8[2 * i]) * sc_silu(z8[2 * i]),
                                          fmaf(d8[2 * i + 1], x8[2 * i + 1], y8[2 * i + 1]) * sc_silu(z8[2 * i + 1]));
          *reinterpret_cast<uint4*>(out + (size_t)(t0 + at + ft) * I + c0 + fc) = o;
        }
      };
      pdl_wait();
      fetch(0);
      stage(0, sc_sm);
      x1 = x2; z1 = z2;
      fetch(TT);
      __syncthreads();
      for (int i = 0; i < tiles; ++i) {
        if (i + 1 < tiles) stage((i + 1) * TT, sc_sm + ((i + 1) & 1) * STAGE);
        if (i > 0) finish((i - 1) * TT, ysum + ((i - 1) & 1) * TT * YLD);
        x0 = x1; z0 = z1; x1 = x2; z1 = z2;
        if (i + 2 < tiles) fetch((i + 2) * TT);
        __syncthreads();
      }
      finish((tiles - 1) * TT, ysum + ((tiles - 1) & 1) * TT * YLD);
    } else {
      auto stage = [&](int at, float* buf) {
        const int n = min(TT, qlen - at);
        float2* dtx = reinterpret_cast<float2*>(buf);
        float *Bs = buf + 2 * TT * CH, *Cs = Bs + TT * NP;
        for (int e = tid; e < TT * CH; e += SC_THREADS) {
          const int tok = e / CH, cc = c0 + e % CH;
          float2 d = make_float2(0.f, 0.f);
          if (tok < n && cc < I) {
            const size_t t = t0 + at + tok;
            d.x = sc_softplus(to_f32(vv[t * a.vstride + cc]) + a.dt_bias[cc]);
            d.y = d.x * to_f32(x[t * I + cc]);
          }
          dtx[e] = d;
        }
        for (int e = tid; e < TT * NP; e += SC_THREADS) {
          const int tok = e / NP, i = e % NP;
          const TA* r = low + (size_t)(t0 + at + tok) * a.lstride + a.bcol + i;
          const bool in = tok < n && i < N;
          Bs[e] = in ? to_f32(r[0]) : 0.f;
          Cs[e] = in ? to_f32(r[N]) : 0.f;
        }
      };
      auto finish = [&](int at, const float* ys) {
        const int n = min(TT, qlen - at);
        for (int e = tid; e < n * CH; e += SC_THREADS) {
          const int tok = e / CH, cc = c0 + e % CH;
          if (cc < I) {
            const size_t t = t0 + at + tok;
            const float y = fmaf(a.D[cc], to_f32(x[t * I + cc]), ys[tok * YLD + e % CH]);
            out[t * I + cc] = from_f32<TA>(y * sc_gate<TA>(to_f32(proj[t * a.pstride + I + cc])));
          }
        }
      };
      pdl_wait();
      stage(0, sc_sm);
      __syncthreads();
      for (int i = 0; i < tiles; ++i) {
        if (i + 1 < tiles) stage((i + 1) * TT, sc_sm + ((i + 1) & 1) * STAGE);
        if (i > 0) finish((i - 1) * TT, ysum + ((i - 1) & 1) * TT * YLD);
        __syncthreads();
      }
      finish((tiles - 1) * TT, ysum + ((tiles - 1) & 1) * TT * YLD);
    }
    pdl_trigger();
    if (slot >= 0 && a.taps > 1 && tid < CH && c0 + tid < I) sc_move_window<TA>(a, c0 + tid, slot, t0, qlen, start);
    return;
  }

  // -------------------------------------------------- walking warps
  const int l = threadIdx.x % L, ch = threadIdx.x / L, c = c0 + ch;
  float2 A[KP], S[KP];
  float* srow = a.state + ((size_t)(slot >= 0 ? slot : 0) * I + (c < I ? c : 0)) * N + l * K;
#pragma unroll
  for (int k = 0; k < 2 * KP; ++k) {
    const bool in = k < K && c < I && l * K + k < N;
    const float av = in ? a.A2[(size_t)c * N + l * K + k] : 0.f;
    const float sv = in && slot >= 0 && start > 0 ? srow[k] : 0.f;
    if (k & 1) { A[k >> 1].y = av; S[k >> 1].y = sv; } else { A[k >> 1].x = av; S[k >> 1].x = sv; }
  }
  pdl_wait();
  __syncthreads();
  for (int i = 0; i < tiles; ++i) {
    const int n = min(TT, qlen - i * TT);
    const float* buf = sc_sm + (i & 1) * STAGE;
    const float2* dtx = reinterpret_cast<const float2*>(buf) + ch;
    const float *Bs = buf + 2 * TT * CH + l * K, *Cs = Bs + TT * NP;
    float* ys = ysum + (i & 1) * TT * YLD + ch;
    // Groups of four tokens.  A group's values are read from shared memory while the group before is worked on, and
    // its sums cross the lanes while the group behind it is: with a warp or two on a scheduler nothing else hides them.
    float2 dn[4];
    float bn[4][2 * KP], cn[4][2 * KP];
    auto grab = [&](int tt) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        dn[j] = dtx[(tt + j) * CH];
        const float *bp = Bs + (tt + j) * NP, *cp = Cs + (tt + j) * NP;
        if constexpr (K % 4 == 0) {
#pragma unroll
          for (int k = 0; k < K; k += 4) {
            const float4 q = *reinterpret_cast<const float4*>(bp + k), r = *reinterpret_cast<const float4*>(cp + k);
            bn[j][k] = q.x; bn[j][k + 1] = q.y; bn[j][k + 2] = q.z; bn[j][k + 3] = q.w;
            cn[j][k] = r.x; cn[j][k + 1] = r.y; cn[j][k + 2] = r.z; cn[j][k + 3] = r.w;
          }
        } else if constexpr (K == 2) {
          const float2 q = *reinterpret_cast<const float2*>(bp), r = *reinterpret_cast<const float2*>(cp);
          bn[j][0] = q.x; bn[j][1] = q.y; cn[j][0] = r.x; cn[j][1] = r.y;
        } else {
          bn[j][0] = *bp; bn[j][1] = 0.f; cn[j][0] = *cp; cn[j][1] = 0.f;
        }
      }
    };
    // the four tokens' sums over the lanes of a channel at once: each exchange halves what a lane still holds, and lane
    // l of four ends with token l
    auto flush = [&](const float (&p)[4], int tt) {
      const bool b0 = l & 1, b1 = l & 2;
      const float q0 = (b0 ? p[1] : p[0]) + __shfl_xor_sync(0xffffffffu, b0 ? p[0] : p[1], 1);
      const float q1 = (b0 ? p[3] : p[2]) + __shfl_xor_sync(0xffffffffu, b0 ? p[2] : p[3], 1);
      float r = (b1 ? q1 : q0) + __shfl_xor_sync(0xffffffffu, b1 ? q0 : q1, 2);
#pragma unroll
      for (int o = 4; o < L; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
      if (l < 4) ys[(tt + l) * YLD] = r;
    };
    grab(0);
    float p[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 2
    for (int tt = 0; tt < n; tt += 4) {
      float2 d[4];
      float bv[4][2 * KP], cv[4][2 * KP], pp[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        d[j] = dn[j]; pp[j] = p[j];
#pragma unroll
        for (int k = 0; k < 2 * KP; ++k) { bv[j][k] = bn[j][k]; cv[j][k] = cn[j][k]; }
      }
      grab(min(tt + 4, TT - 4));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 acc = make_float2(0.f, 0.f);
        const float2 dt2 = make_float2(d[j].x, d[j].x), dx2 = make_float2(d[j].y, d[j].y);
#pragma unroll
        for (int k = 0; k < KP; ++k) {
          const float2 g = sc_mul2(A[k], dt2);
          const float2 e = make_float2(sc_exp2<TA>(g.x), K == 1 ? 0.f : sc_exp2<TA>(g.y));
          S[k] = sc_fma2(e, S[k], sc_mul2(dx2, make_float2(bv[j][2 * k], bv[j][2 * k + 1])));
          acc = sc_fma2(S[k], make_float2(cv[j][2 * k], cv[j][2 * k + 1]), acc);
        }
        p[j] = acc.x + acc.y;
      }
      if (tt > 0) flush(pp, tt - 4);
    }
    flush(p, (n + 3) / 4 * 4 - 4);
    __syncthreads();
  }
  pdl_trigger();                                   // only now: a long kernel of few blocks keeps the machine to itself
  if (slot < 0) return;
#pragma unroll
  for (int k = 0; k < K; ++k)
    if (c < I && l * K + k < N) srow[k] = (k & 1) ? S[k >> 1].y : S[k >> 1].x;
}

// The same window moved on by one token: what is read is read before it is overwritten, four places at a time.
template <typename TA>
__device__ __forceinline__ void sc_push_window(const ScanArgs& a, int c, int slot, int t, bool old) {
  const int keep = a.taps - 1;
  float* st = a.conv_state + (size_t)slot * keep * a.I + c;
  const float x = to_f32(((const TA*)a.proj)[(size_t)t * a.pstride + c]);
  for (int j0 = 0; j0 < keep; j0 += 4) {
    float m[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) m[j] = j0 + j == keep - 1 ? x : (old && j0 + j < keep - 1 ? st[(size_t)(j0 + j + 1) * a.I] : 0.f);
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (j0 + j < keep) st[(size_t)(j0 + j) * a.I] = m[j];
  }
}

// Steps of single tokens.  grid (ceil(B / SEQ), ceil(I / CH)): a block keeps its channels' A and takes SEQ sequences, whose
// states are asked for together; the state is read and written once.  Step size, gate and window of a (sequence, channel)
// are one thread's work.  With w_dt (one sequence a block) the step size's product is made here too: row c of w_dt times
// the first `rank` columns of low, the lanes of a channel taking turns.
template <typename TA, int L, int K, int SEQ>
__global__ void __launch_bounds__(SC_THREADS, (K <= 4 ? 7 : 4)) scan_step_kernel(ScanArgs a, int B) {
  constexpr int CH = SC_THREADS / L, NP = L * K;
  constexpr bool V4 = K % 4 == 0;
  __shared__ float4 prm[SEQ][CH];                  // dt, dt x, D x, silu(z)
  __shared__ __align__(16) float bcs[SEQ][2 * NP]; // B, then C
  const int b0 = blockIdx.x * SEQ, tid = threadIdx.x, l = tid % L, ch = tid / L, c0 = blockIdx.y * CH, c = c0 + ch;
  const int I = a.I, N = a.N;
  pdl_trigger();
  const bool live = c < I;
  const int cc = live ? c : I - 1;
  const bool v4 = V4 && N % 4 == 0;                // whole groups of four states, on 16-byte borders
  auto load = [&](float (&o)[K], const float* p, bool on) {
#pragma unroll
    for (int k = 0; k < K; k += V4 ? 4 : 1) {
      if constexpr (V4) {
        if (v4) {
          const float4 q = on && l * K + k < N ? *reinterpret_cast<const float4*>(p + k) : make_float4(0.f, 0.f, 0.f, 0.f);
          o[k] = q.x; o[k + 1] = q.y; o[k + 2] = q.z; o[k + 3] = q.w;
          continue;
        }
      }
#pragma unroll
      for (int i = k; i < k + (V4 ? 4 : 1); ++i) o[i] = on && l * K + i < N ? p[i] : 0.f;
    }
  };
  float A[K], S[SEQ][K];
  load(A, a.A2 + (size_t)cc * N + l * K, true);
#pragma unroll
  for (int q = 0; q < SEQ; ++q) {
    const int b = min(b0 + q, B - 1), slot = b0 + q < B ? a.state_slots[b] : -1;
    load(S[q], a.state + ((size_t)(slot >= 0 ? slot : 0) * I + cc) * N + l * K, slot >= 0 && a.context_lens[b] > 1);
  }
  pdl_wait();
  const TA* low = (const TA*)a.low;
  for (int e = tid; e < SEQ * 2 * NP; e += SC_THREADS) {
    const int q = e / (2 * NP), i = e % (2 * NP), n = i < NP ? i : i - NP;
    const int t = a.cu[min(b0 + q, B - 1)];
    bcs[q][i] = n < N ? to_f32(low[(size_t)t * a.lstride + a.bcol + (i < NP ? n : N + n)]) : 0.f;
  }
  float v1 = 0.f;
  if (SEQ == 1 && a.w_dt) {
    const TA *w = (const TA*)a.w_dt + (size_t)cc * a.rank, *row = low + (size_t)a.cu[b0] * a.lstride;
    constexpr int VP = 16 / (int)sizeof(TA);
    if (a.rank % VP == 0 && ((size_t)a.low | (size_t)(a.lstride * sizeof(TA)) | (size_t)a.w_dt) % 16 == 0) {
      for (int r = l * VP; r < a.rank; r += L * VP) {
        const uint4 p = *reinterpret_cast<const uint4*>(w + r), m = *reinterpret_cast<const uint4*>(row + r);
        const TA *pw = reinterpret_cast<const TA*>(&p), *pm = reinterpret_cast<const TA*>(&m);
#pragma unroll
        for (int i = 0; i < VP; ++i) v1 = fmaf(to_f32(pw[i]), to_f32(pm[i]), v1);
      }
    } else {
      for (int r = l; r < a.rank; r += L) v1 = fmaf(to_f32(w[r]), to_f32(row[r]), v1);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) v1 += __shfl_xor_sync(0xffffffffu, v1, o);
    if (l == 0) prm[0][ch].x = v1;
    __syncthreads();
  }
  for (int e = tid; e < SEQ * CH; e += SC_THREADS) {
    const int q = e / CH, h = e % CH, cq = c0 + h, b = b0 + q;
    if (b < B && cq < I) {
      const int t = a.cu[b], slot = a.state_slots[b];
      const float x = to_f32(((const TA*)a.x)[(size_t)t * I + cq]), z = to_f32(((const TA*)a.proj)[(size_t)t * a.pstride + I + cq]);
      const float v = SEQ == 1 && a.w_dt ? prm[q][h].x : to_f32(((const TA*)a.v)[(size_t)t * a.vstride + cq]);
      const float dt = sc_softplus(v + a.dt_bias[cq]);
      prm[q][h] = make_float4(dt, dt * x, a.D[cq] * x, sc_gate<TA>(z));
      if (a.taps > 1 && slot >= 0) sc_push_window<TA>(a, cq, slot, t, a.context_lens[b] > 1);
    } else {
      prm[q][h] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  __syncthreads();
#pragma unroll
  for (int q = 0; q < SEQ; ++q) {
    const float4 p = prm[q][ch];
    const float *bq = &bcs[q][l * K], *cq = bq + NP;
    float y = 0.f;
#pragma unroll
    for (int k = 0; k < K; ++k) {
      S[q][k] = fmaf(sc_exp2<TA>(p.x * A[k]), S[q][k], p.y * bq[k]);
      y = fmaf(S[q][k], cq[k], y);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!live || b0 + q >= B) continue;
    if (l == 0) ((TA*)a.out)[(size_t)a.cu[b0 + q] * I + c] = from_f32<TA>((y + p.z) * p.w);
    const int slot = a.state_slots[b0 + q];
    if (slot < 0) continue;
    float* srow = a.state + ((size_t)slot * I + c) * N + l * K;
#pragma unroll
    for (int k = 0; k < K; k += V4 ? 4 : 1) {
      if constexpr (V4) {
        if (v4) {
          if (l * K + k < N) *reinterpret_cast<float4*>(srow + k) = make_float4(S[q][k], S[q][k + 1], S[q][k + 2], S[q][k + 3]);
          continue;
        }
      }
#pragma unroll
      for (int i = k; i < k + (V4 ? 4 : 1); ++i)
        if (l * K + i < N) srow[i] = S[q][i];
    }
  }
}

// ---------------------------------------------------------------- launchers
extern "C" int gg_scan_conv(const void* x, long long stride, int dtype, const float* w, const float* bias, const float* conv_state,
                            const int* cu, const int* context_lens, const int* state_slots, int T, int B, int C, int taps,
                            void* out, cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && B > 0 && C > 0 && taps >= 1 && taps <= 64, "scan_conv: bad sizes T=%d B=%d C=%d taps=%d", T, B, C, taps);
  GG_REQUIRE(x && w && out && (taps == 1 || conv_state) && stride >= C, "scan_conv: a pointer is null or the rows are too short");
  if (T == 0) return GG_OK;
  const bool vec = C % 4 == 0 && stride % 4 == 0 && ((size_t)x | (size_t)out | (size_t)conv_state) % 16 == 0;
  const int per = SC_THREADS * (vec ? 4 : 1), cols = (C + per - 1) / per;
  GG_REQUIRE(cols <= 65535, "scan_conv: too many channels");
  // few tokens: a token a block; more: runs of tokens, whose inputs a thread then reads once
  const int tt = T > 512 ? SC_RUN : (T > 4 * B ? 4 : 1);
  const dim3 grid((T + tt - 1) / tt, cols);
#define SC_CONV(TA, TAPS)                                                                                                 \
  do {                                                                                                                    \
    if (vec) gg_launch(scan_conv_kernel<TA, TAPS, 4>, grid, dim3(SC_THREADS), 0, stream, (const TA*)x, stride, w, bias, conv_state, cu, context_lens, state_slots, T, B, C, taps, tt, (TA*)out); \
    else gg_launch(scan_conv_kernel<TA, TAPS, 1>, grid, dim3(SC_THREADS), 0, stream, (const TA*)x, stride, w, bias, conv_state, cu, context_lens, state_slots, T, B, C, taps, tt, (TA*)out); \
  } while (0)
#define SC_CONV_T(TA) do { if (taps == 4 && (size_t)w % 16 == 0) SC_CONV(TA, 4); else if (taps == 3) SC_CONV(TA, 3); else SC_CONV(TA, 0); } while (0)
  if (dtype == GG_F32) SC_CONV_T(float);
  else if (dtype == GG_BF16) SC_CONV_T(__nv_bfloat16);
  else return gg_fail(GG_ERR_INVALID, "scan_conv: unknown dtype %d", dtype);
#undef SC_CONV
#undef SC_CONV_T
  return gg_check_launch("scan_conv");
}

template <typename TA, int L, int K>
static int scan_go(const ScanArgs& a, int B, bool single, bool long_rows, cudaStream_t stream) {
  constexpr int CH = SC_THREADS / L, NP = L * K;
  const dim3 grid(B, (a.I + CH - 1) / CH);
  GG_REQUIRE(grid.y <= 65535, "scan: too many channels");
  if (single) {
    // several sequences a block where there are blocks enough for the machine anyway
    if (!a.w_dt && (long long)B * grid.y >= 2048) gg_launch(scan_step_kernel<TA, L, K, 4>, dim3((B + 3) / 4, grid.y), dim3(SC_THREADS), 0, stream, a, B);
    else gg_launch(scan_step_kernel<TA, L, K, 1>, grid, dim3(SC_THREADS), 0, stream, a, B);
    return gg_check_launch("scan_step");
  }
  const size_t smem = sizeof(float) * 2 * (2 * SC_TT * CH + 2 * SC_TT * NP + SC_TT * (CH + 4));
  bool fast = false;
  if constexpr (sizeof(TA) == 2 && CH % 8 == 0 && NP <= 64)
    fast = a.N == NP && NP % 8 == 0 && a.I % CH == 0 && a.pstride % 8 == 0 && a.lstride % 8 == 0 && a.vstride % 8 == 0 && a.bcol % 8 == 0 &&
           ((size_t)a.x | (size_t)a.proj | (size_t)a.low | (size_t)a.v | (size_t)a.out) % 16 == 0;
  auto go = [&](void (*kernel)(ScanArgs)) {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "scan_run: %s", cudaGetErrorString(e));
    }
    // blocks that run for as long as their sequence is wait for an empty machine (common.cuh)
    if (long_rows) gg_launch_after(kernel, grid, dim3(2 * SC_THREADS), smem, stream, a);
    else gg_launch(kernel, grid, dim3(2 * SC_THREADS), smem, stream, a);
    return gg_check_launch("scan_run");
  };
  if constexpr (sizeof(TA) == 2 && CH % 8 == 0 && NP <= 64) {
    if (fast) return go(scan_run_kernel<TA, L, K, true>);
  }
  return go(scan_run_kernel<TA, L, K, false>);
}

template <typename TA>
static int scan_sizes(const ScanArgs& a, int B, bool single, bool long_rows, cudaStream_t stream) {
  if (a.N <= 4) return scan_go<TA, 4, 1>(a, B, single, long_rows, stream);
  if (a.N <= 8) return scan_go<TA, 4, 2>(a, B, single, long_rows, stream);
  if (a.N <= 16) return scan_go<TA, 4, 4>(a, B, single, long_rows, stream);
  if (a.N <= 32) return scan_go<TA, 8, 4>(a, B, single, long_rows, stream);
  if (a.N <= 64) return scan_go<TA, 16, 4>(a, B, single, long_rows, stream);
  if (a.N <= 128) return scan_go<TA, 32, 4>(a, B, single, long_rows, stream);
  return scan_go<TA, 32, 8>(a, B, single, long_rows, stream);
}

// single: every sequence of the step has one token; w_dt (or null) is taken only then, else v.
extern "C" int gg_selective_scan(const void* x, const void* proj, long long pstride, const void* low, long long lstride, int bcol,
                                 const void* v, long long vstride, const void* w_dt, int rank, const float* dt_bias, const float* A2,
                                 const float* D, float* state, float* conv_state, int taps, const int* cu, const int* context_lens,
                                 const int* state_slots, int T, int B, int I, int N, int single, void* out, int dtype,
                                 cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && B > 0 && I > 0 && N > 0 && taps >= 1, "selective_scan: bad sizes T=%d B=%d I=%d N=%d taps=%d", T, B, I, N, taps);
  GG_REQUIRE(N <= 256, "selective_scan: %d states a channel are beyond 256", N);
  GG_REQUIRE(x && proj && low && dt_bias && A2 && D && state && out && (taps == 1 || conv_state), "selective_scan: a pointer is null");
  GG_REQUIRE((single && w_dt) ? rank > 0 : v != nullptr, "selective_scan: no step sizes");
  GG_REQUIRE(pstride >= 2ll * I && lstride >= (long long)bcol + 2 * N && (!v || vstride >= I), "selective_scan: the rows are too short");
  GG_REQUIRE(!single || T == B, "selective_scan: %d tokens of %d sequences are not one each", T, B);
  if (T == 0) return GG_OK;
  ScanArgs a = {x, proj, pstride, low, lstride, bcol, v, vstride, single ? w_dt : nullptr, rank, dt_bias, A2, D, state, conv_state,
                taps, cu, context_lens, state_slots, I, N, out};
  const bool long_rows = T > 4 * B;
  if (dtype == GG_F32) return scan_sizes<float>(a, B, single != 0, long_rows, stream);
  if (dtype == GG_BF16) return scan_sizes<__nv_bfloat16>(a, B, single != 0, long_rows, stream);
  return gg_fail(GG_ERR_INVALID, "selective_scan: unknown dtype %d", dtype);
}
