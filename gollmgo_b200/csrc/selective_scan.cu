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

__device__ __forceinline__ float sc_silu(float x) { return x / (1.f + __expf(-x)); }
__device__ __forceinline__ float sc_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
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
    if (TAPS > 0) {
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
    for (int v = 0; v < V; ++v) acc[v] = acc[v] / (1.f + expf(-acc[v]));
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
template <typename TA> __device__ __forceinline__ float sc_gate(float z) {
  if constexpr (sizeof(TA) == 4) return z / (1.f + expf(-z));
  return sc_silu(z);
}
__device__ __forceinline__ void sc_unpack8(float (&o)[8], const uint4& q) {
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(p[i]); o[2 * i] = f.x; o[2 * i + 1] = f.y; }
}

// grid (B, ceil(I / CH)), CH = 128 / L channels a block.  FAST: bfloat16, N = L K, every row on 16-byte borders and
// whole blocks of channels: the next tile's rows are fetched into registers while this one is worked on.
template <typename TA, int L, int K, bool FAST>
__global__ void __launch_bounds__(SC_THREADS) scan_run_kernel(ScanArgs a) {
  constexpr int CH = SC_THREADS / L, NP = L * K, TT = SC_TT, YLD = CH + 8;
  constexpr int KP = (K + 1) / 2;
  extern __shared__ __align__(16) float sc_sm[];
  float2* dtx = reinterpret_cast<float2*>(sc_sm);          // [TT][CH]: (dt, dt x)
  float* Bs = sc_sm + 2 * TT * CH;                         // [TT][NP]
  float* Cs = Bs + TT * NP;
  float* ys = Cs + TT * NP;                                // [TT][YLD]
  const int b = blockIdx.x, tid = threadIdx.x, l = tid % L, ch = tid / L, c0 = blockIdx.y * CH, c = c0 + ch;
  const int I = a.I, N = a.N;
  const int t0 = a.cu[b], qlen = a.cu[b + 1] - t0, slot = a.state_slots[b], start = a.context_lens[b] - qlen;
  if (qlen <= 0) { pdl_trigger(); return; }
  float2 A[KP], S[KP];
  float* srow = a.state + ((size_t)(slot >= 0 ? slot : 0) * I + (c < I ? c : 0)) * N + l * K;
#pragma unroll
  for (int k = 0; k < 2 * KP; ++k) {
    const bool in = k < K && c < I && l * K + k < N;
    const float av = in ? a.A2[(size_t)c * N + l * K + k] : 0.f;
    const float sv = in && slot >= 0 && start > 0 ? srow[k] : 0.f;
    if (k & 1) { A[k >> 1].y = av; S[k >> 1].y = sv; } else { A[k >> 1].x = av; S[k >> 1].x = sv; }
  }
  const TA *x = (const TA*)a.x, *proj = (const TA*)a.proj, *low = (const TA*)a.low, *vv = (const TA*)a.v;
  // FAST: which eight channels of which token this thread stages, and which eight values of B and C
  constexpr int G8 = CH / 8 > 0 ? CH / 8 : 1, BCN = NP >= 16 ? NP / 16 : 1;
  const int ft = tid / G8, fc = (tid % G8) * 8;
  const bool fon = tid < TT * G8;
  uint4 rx, rz, rv, rbc[BCN];
  float bias8[8], d8[8];
  if constexpr (FAST) {
#pragma unroll
    for (int i = 0; i < 8; ++i) { bias8[i] = a.dt_bias[c0 + fc + i]; d8[i] = a.D[c0 + fc + i]; }
  }
  auto fetch = [&](int at) {
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const bool on = fon && at + ft < qlen;
    const size_t t = t0 + at + ft;
    rx = on ? *reinterpret_cast<const uint4*>(x + t * I + c0 + fc) : zero;
    rv = on ? *reinterpret_cast<const uint4*>(vv + t * a.vstride + c0 + fc) : zero;
    rz = on ? *reinterpret_cast<const uint4*>(proj + t * a.pstride + I + c0 + fc) : zero;
#pragma unroll
    for (int u = 0; u < BCN; ++u) {
      const int e = tid + u * SC_THREADS, tok = e / (NP / 4), g = (e % (NP / 4)) * 8;      // g < NP: B, else C
      rbc[u] = tok < TT && at + tok < qlen ? *reinterpret_cast<const uint4*>(low + (size_t)(t0 + at + tok) * a.lstride + a.bcol + g) : zero;
    }
  };
  pdl_wait();
  if constexpr (FAST) fetch(0);
  for (int at = 0; at < qlen; at += TT) {
    const int n = min(TT, qlen - at);
    float x8[8], z8[8];
    if constexpr (FAST) {
      float v8[8];
      sc_unpack8(x8, rx); sc_unpack8(z8, rz); sc_unpack8(v8, rv);
      if (fon) {
        const bool real = ft < n;                  // places past the end: dt = 0 leaves the state as it is
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
        sc_unpack8(q, rbc[u]);
        float* dst = g < NP ? Bs + tok * NP + g : Cs + tok * NP + g - NP;
        if (tok < TT) {
          *reinterpret_cast<float4*>(dst) = make_float4(q[0], q[1], q[2], q[3]);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(q[4], q[5], q[6], q[7]);
        }
      }
      if (at + TT < qlen) fetch(at + TT);
    } else {
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
    }
    __syncthreads();
    for (int tt = 0; tt < n; tt += 4) {
      float p[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 d = dtx[(tt + j) * CH + ch];
        float bv[2 * KP], cv[2 * KP];
        if constexpr (K % 4 == 0) {
#pragma unroll
          for (int k = 0; k < K; k += 4) {
            const float4 q = *reinterpret_cast<const float4*>(Bs + (tt + j) * NP + l * K + k), r = *reinterpret_cast<const float4*>(Cs + (tt + j) * NP + l * K + k);
            bv[k] = q.x; bv[k + 1] = q.y; bv[k + 2] = q.z; bv[k + 3] = q.w;
            cv[k] = r.x; cv[k + 1] = r.y; cv[k + 2] = r.z; cv[k + 3] = r.w;
          }
        } else {
#pragma unroll
          for (int k = 0; k < 2 * KP; ++k) {
            bv[k] = k < K ? Bs[(tt + j) * NP + l * K + k] : 0.f;
            cv[k] = k < K ? Cs[(tt + j) * NP + l * K + k] : 0.f;
          }
        }
        float2 acc = make_float2(0.f, 0.f);
        const float2 dt2 = make_float2(d.x, d.x), dx2 = make_float2(d.y, d.y);
#pragma unroll
        for (int k = 0; k < KP; ++k) {
          const float2 g = sc_mul2(A[k], dt2);
          const float2 e = make_float2(sc_exp2<TA>(g.x), K == 1 ? 0.f : sc_exp2<TA>(g.y));
          S[k] = sc_fma2(e, S[k], sc_mul2(dx2, make_float2(bv[2 * k], bv[2 * k + 1])));
          acc = sc_fma2(S[k], make_float2(cv[2 * k], cv[2 * k + 1]), acc);
        }
        p[j] = acc.x + acc.y;
      }
      // the four tokens' sums over the lanes of a channel at once: each exchange halves what a lane still holds, and
      // lane l of four ends with token l
      const bool b0 = l & 1, b1 = l & 2;
      const float q0 = (b0 ? p[1] : p[0]) + __shfl_xor_sync(0xffffffffu, b0 ? p[0] : p[1], 1);
      const float q1 = (b0 ? p[3] : p[2]) + __shfl_xor_sync(0xffffffffu, b0 ? p[2] : p[3], 1);
      float r = (b1 ? q1 : q0) + __shfl_xor_sync(0xffffffffu, b1 ? q0 : q1, 2);
#pragma unroll
      for (int o = 4; o < L; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
      if (l < 4) ys[(tt + l) * YLD + ch] = r;
    }
    __syncthreads();
    TA* out = (TA*)a.out;
    if constexpr (FAST) {
      if (ft < n && fon) {
        const float4 y0 = *reinterpret_cast<const float4*>(ys + ft * YLD + fc), y1 = *reinterpret_cast<const float4*>(ys + ft * YLD + fc + 4);
        const float y8[8] = {y0.x, y0.y, y0.z, y0.w, y1.x, y1.y, y1.z, y1.w};
        __nv_bfloat162 o[4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
          o[i] = __floats2bfloat162_rn(fmaf(d8[2 * i], x8[2 * i], y8[2 * i]) * sc_silu(z8[2 * i]),
                                       fmaf(d8[2 * i + 1], x8[2 * i + 1], y8[2 * i + 1]) * sc_silu(z8[2 * i + 1]));
        *reinterpret_cast<uint4*>(out + (size_t)(t0 + at + ft) * I + c0 + fc) = *reinterpret_cast<const uint4*>(o);
      }
    } else {
      for (int e = tid; e < n * CH; e += SC_THREADS) {
        const int tok = e / CH, cc = c0 + e % CH;
        if (cc < I) {
          const size_t t = t0 + at + tok;
          const float y = fmaf(a.D[cc], to_f32(x[t * I + cc]), ys[tok * YLD + e % CH]);
          out[t * I + cc] = from_f32<TA>(y * sc_gate<TA>(to_f32(proj[t * a.pstride + I + cc])));
        }
      }
      __syncthreads();
    }
  }
  pdl_trigger();                                   // only now: a long kernel of few blocks keeps the machine to itself
  if (slot < 0) return;
#pragma unroll
  for (int k = 0; k < K; ++k)
    if (c < I && l * K + k < N) srow[k] = (k & 1) ? S[k >> 1].y : S[k >> 1].x;
  if (a.taps > 1 && tid < CH && c0 + tid < I) sc_move_window<TA>(a, c0 + tid, slot, t0, qlen, start);
}

// Steps of single tokens.  grid (B, ceil(I / CH)): the state is read and written once.  With w_dt the step size's
// product is made here too (its row times the first `rank` columns of low, the lanes of a channel taking turns).
template <typename TA, int L, int K>
__global__ void __launch_bounds__(SC_THREADS) scan_step_kernel(ScanArgs a) {
  constexpr int CH = SC_THREADS / L;
  constexpr bool V4 = K % 4 == 0;
  const int b = blockIdx.x, tid = threadIdx.x, l = tid % L, ch = tid / L, c0 = blockIdx.y * CH, c = c0 + ch;
  const int I = a.I, N = a.N;
  pdl_trigger();
  const int t = a.cu[b], slot = a.state_slots[b], start = a.context_lens[b] - 1;
  if (a.cu[b + 1] <= t) return;
  const bool live = c < I;
  const int cc = live ? c : I - 1;
  float* srow = a.state + ((size_t)(slot >= 0 ? slot : 0) * I + cc) * N + l * K;
  const bool v4 = V4 && N % 4 == 0;                // whole groups of four states, on 16-byte borders
  float A[K], S[K];
  const bool old = slot >= 0 && start > 0;
  const float* arow = a.A2 + (size_t)cc * N + l * K;
#pragma unroll
  for (int k = 0; k < K; k += V4 ? 4 : 1) {
    if constexpr (V4) {
      if (v4) {
        const bool in = l * K + k < N;
        const float4 q = in ? *reinterpret_cast<const float4*>(arow + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 s = in && old ? *reinterpret_cast<const float4*>(srow + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        A[k] = q.x; A[k + 1] = q.y; A[k + 2] = q.z; A[k + 3] = q.w;
        S[k] = s.x; S[k + 1] = s.y; S[k + 2] = s.z; S[k + 3] = s.w;
        continue;
      }
    }
#pragma unroll
    for (int i = k; i < k + (V4 ? 4 : 1); ++i) {
      const bool in = l * K + i < N;
      A[i] = in ? arow[i] : 0.f;
      S[i] = in && old ? srow[i] : 0.f;
    }
  }
  pdl_wait();
  const TA* low = (const TA*)a.low + (size_t)t * a.lstride;
  float v = 0.f;
  if (a.w_dt) {
    const TA* w = (const TA*)a.w_dt + (size_t)cc * a.rank;
    constexpr int VP = 16 / (int)sizeof(TA);
    if (a.rank % VP == 0 && ((size_t)a.low | (size_t)(a.lstride * sizeof(TA)) | (size_t)a.w_dt) % 16 == 0) {
      for (int r = l * VP; r < a.rank; r += L * VP) {
        const uint4 p = *reinterpret_cast<const uint4*>(w + r), q = *reinterpret_cast<const uint4*>(low + r);
        const TA *pw = reinterpret_cast<const TA*>(&p), *pq = reinterpret_cast<const TA*>(&q);
#pragma unroll
        for (int i = 0; i < VP; ++i) v = fmaf(to_f32(pw[i]), to_f32(pq[i]), v);
      }
    } else {
      for (int r = l; r < a.rank; r += L) v = fmaf(to_f32(w[r]), to_f32(low[r]), v);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  } else {
    v = to_f32(((const TA*)a.v)[(size_t)t * a.vstride + cc]);
  }
  const float xc = to_f32(((const TA*)a.x)[(size_t)t * I + cc]);
  const float z = to_f32(((const TA*)a.proj)[(size_t)t * a.pstride + I + cc]);
  const float dt = sc_softplus(v + a.dt_bias[cc]), dx = dt * xc;
  float y = 0.f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const bool in = l * K + k < N;
    const float bv = in ? to_f32(low[a.bcol + l * K + k]) : 0.f, cv = in ? to_f32(low[a.bcol + N + l * K + k]) : 0.f;
    S[k] = fmaf(sc_exp2<TA>(dt * A[k]), S[k], dx * bv);
    y = fmaf(S[k], cv, y);
  }
#pragma unroll
  for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (live && l == 0) ((TA*)a.out)[(size_t)t * I + c] = from_f32<TA>(fmaf(a.D[c], xc, y) * sc_gate<TA>(z));
  if (slot < 0) return;
  if (live) {
#pragma unroll
    for (int k = 0; k < K; k += V4 ? 4 : 1) {
      if constexpr (V4) {
        if (v4) {
          if (l * K + k < N) *reinterpret_cast<float4*>(srow + k) = make_float4(S[k], S[k + 1], S[k + 2], S[k + 3]);
          continue;
        }
      }
#pragma unroll
      for (int i = k; i < k + (V4 ? 4 : 1); ++i)
        if (l * K + i < N) srow[i] = S[i];
    }
  }
  if (a.taps > 1 && tid < CH && c0 + tid < I) sc_move_window<TA>(a, c0 + tid, slot, t, 1, start);
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
  const int tt = T > 512 ? 8 : (T > 4 * B ? 4 : 1);
  const dim3 grid((T + tt - 1) / tt, cols);
#define SC_CONV(TA, TAPS)                                                                                                 \
  do {                                                                                                                    \
    if (vec) gg_launch(scan_conv_kernel<TA, TAPS, 4>, grid, dim3(SC_THREADS), 0, stream, (const TA*)x, stride, w, bias, conv_state, cu, context_lens, state_slots, T, B, C, taps, tt, (TA*)out); \
    else gg_launch(scan_conv_kernel<TA, TAPS, 1>, grid, dim3(SC_THREADS), 0, stream, (const TA*)x, stride, w, bias, conv_state, cu, context_lens, state_slots, T, B, C, taps, tt, (TA*)out); \
  } while (0)
#define SC_CONV_T(TA) do { if (taps == 4) SC_CONV(TA, 4); else if (taps == 3) SC_CONV(TA, 3); else SC_CONV(TA, 0); } while (0)
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
    gg_launch(scan_step_kernel<TA, L, K>, grid, dim3(SC_THREADS), 0, stream, a);
    return gg_check_launch("scan_step");
  }
  const size_t smem = sizeof(float) * (2 * SC_TT * CH + 2 * SC_TT * NP + SC_TT * (CH + 8));
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
    if (long_rows) gg_launch_after(kernel, grid, dim3(SC_THREADS), smem, stream, a);
    else gg_launch(kernel, grid, dim3(SC_THREADS), smem, stream, a);
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
