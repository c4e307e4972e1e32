// A residual of several parallel streams x_1 .. x_S per token (float32, [T, S, D]), read through a learned
// contraction and written through a learned mixing:
//     u = sum_s in[s] x_s;  h = u / sqrt(mean(u^2) + eps) * w;  y = sublayer(h);
//     x_t <- sum_s mix[s, t] x_s + out[t] y          (all streams at once from the old ones)
//
// gg_streams_join, one CTA a token, is everything between two sublayers: it adds what the sublayer before
// left (its rows, or a mixture of experts' rows that are not summed yet) with that sublayer's mix and out,
// writes the new streams, contracts them with the next sublayer's in and makes its norm, so that the streams
// are read and written once per sublayer.  Variants by null pointers:
//   x1 given                the streams before the first sublayer: S copies of one row
//   out null                nothing is owed: the streams stay as they are
//   in null                 u is the plain sum of the streams; norm_w null: u itself goes to `u` (float32), and
//                           the streams are not written back (the end of the stretch with several streams)
#include "common.cuh"

#define ST_MAX 16

struct StreamsArgs {
  float* x; const float* x1;
  const void *dense, *y, *same; const int* place; const float* wgt; int top;
  const float *mix, *out, *in, *norm_w; float eps;
  void* h; float* u;
  int S, D, write;
};

template <int V> struct StVec { float v[V]; };
template <int V> __device__ __forceinline__ StVec<V> st_load(const float* p) {
  StVec<V> r;
  if constexpr (V == 4) { const float4 q = *reinterpret_cast<const float4*>(p); r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w; }
  else r.v[0] = *p;
  return r;
}
template <int V> __device__ __forceinline__ StVec<V> st_load(const __nv_bfloat16* p) {
  StVec<V> r;
  if constexpr (V == 4) {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
    r.v[0] = lo.x; r.v[1] = lo.y; r.v[2] = hi.x; r.v[3] = hi.y;
  } else r.v[0] = to_f32(*p);
  return r;
}
template <int V> __device__ __forceinline__ void st_store(float* p, const StVec<V>& a) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
  else *p = a.v[0];
}
template <int V> __device__ __forceinline__ void st_store(__nv_bfloat16* p, const StVec<V>& a) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else *p = from_f32<__nv_bfloat16>(a.v[0]);
}
template <int V> __device__ __forceinline__ void st_axpy(StVec<V>& s, float w, const StVec<V>& a) {
#pragma unroll
  for (int i = 0; i < V; ++i) s.v[i] = fmaf(w, a.v[i], s.v[i]);
}

// SM: the number of streams rounded up to a power of two (the rest are skipped).
template <typename TA, int SM, int V>
__global__ void streams_join_kernel(StreamsArgs a) {
  extern __shared__ __align__(16) float row[];             // [D]
  __shared__ float red[33];
  __shared__ float mix_s[SM * SM], in_s[SM], out_s[SM];
  pdl_trigger();
  const int S = a.S, D = a.D;
  const size_t t = blockIdx.x;
  const bool owed = a.out != nullptr;
  // weights are written by no kernel
  if (owed)
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix_s[(i / S) * SM + i % S] = a.mix[i];
  if (threadIdx.x < S) {
    in_s[threadIdx.x] = a.in ? a.in[threadIdx.x] : 1.f;
    out_s[threadIdx.x] = owed ? a.out[threadIdx.x] : 0.f;
  }
  __syncthreads();
  pdl_wait();
  const TA *dense = (const TA*)a.dense, *y = (const TA*)a.y, *same = (const TA*)a.same;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V) {
    StVec<V> x[SM];
    if (a.x1) {
      const StVec<V> e = st_load<V>(a.x1 + t * D + c);
#pragma unroll
      for (int s = 0; s < SM; ++s) x[s] = e;
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) x[s] = st_load<V>(a.x + (t * S + s) * D + c);
    }
    if (owed) {
      StVec<V> v;
      if (dense) v = st_load<V>(dense + t * D + c);
      else {
#pragma unroll
        for (int i = 0; i < V; ++i) v.v[i] = 0.f;
      }
      for (int j = 0; j < a.top; ++j) {
        const int p = a.place[t * a.top + j];
        st_axpy<V>(v, a.wgt ? a.wgt[t * a.top + j] : 1.f, st_load<V>(p >= 0 ? y + (size_t)p * D + c : same + t * D + c));
      }
      StVec<V> n[SM];
#pragma unroll
      for (int r = 0; r < SM; ++r) {
        if (r < S) {
#pragma unroll
          for (int i = 0; i < V; ++i) n[r].v[i] = out_s[r] * v.v[i];
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (s < S) st_axpy<V>(n[r], mix_s[s * SM + r], x[s]);
        }
      }
#pragma unroll
      for (int r = 0; r < SM; ++r) x[r] = n[r];
    }
    StVec<V> u;
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = 0.f;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S) {
        st_axpy<V>(u, in_s[s], x[s]);
        if (a.write) st_store<V>(a.x + (t * S + s) * D + c, x[s]);
      }
    if (a.norm_w) {
      st_store<V>(row + c, u);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(u.v[i], u.v[i], ss);
    } else st_store<V>(a.u + t * D + c, u);
  }
  if (!a.norm_w) return;
  const float f = rsqrtf(block_sum(ss, red) / (float)D + a.eps);
  TA* h = (TA*)a.h + t * D;
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V) {
    const StVec<V> r = st_load<V>(row + c), w = st_load<V>(a.norm_w + c);
    StVec<V> o;
#pragma unroll
    for (int i = 0; i < V; ++i) o.v[i] = r.v[i] * f * w.v[i];
    st_store<V>(h + c, o);
  }
}

// `same`: the rows that choices with place < 0 (experts that hand on their input) add.  h may be `same`.
extern "C" int gg_streams_join(float* x, const float* x1, const void* dense, const void* y, const int* place, const float* wgt,
                               int top, const void* same, const float* mix, const float* out, const float* in,
                               const float* norm_w, float eps, void* h, float* u, int T, int S, int D, int act_dtype,
                               cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && D > 0 && S >= 1 && S <= ST_MAX && top >= 0, "streams_join: bad sizes T=%d S=%d (at most %d) D=%d top=%d", T, S, ST_MAX, D, top);
  GG_REQUIRE(x && (!out || (mix && (dense || top > 0))) && (top == 0 || (y && place && same)), "streams_join: a pointer is null");
  GG_REQUIRE(norm_w ? h != nullptr : u != nullptr, "streams_join: nowhere to leave the contraction");
  const size_t smem = norm_w ? (size_t)D * sizeof(float) : 0;
  GG_REQUIRE(smem <= 200 * 1024, "streams_join: rows of %d values do not fit in shared memory", D);
  if (T == 0) return GG_OK;
  const size_t at = (size_t)x | (size_t)x1 | (size_t)dense | (size_t)y | (size_t)same | (size_t)norm_w | (size_t)h | (size_t)u;
  const bool vec = D % 4 == 0 && at % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((D + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  StreamsArgs a = {x, x1, dense, y, same, place, wgt, top, mix, out, in, norm_w, eps, h, u, S, D,
                   norm_w != nullptr && out != nullptr};
#define ST_GO(TA, SM, V)                                                                                                   \
  do {                                                                                                                     \
    if (smem > 40 * 1024) cudaFuncSetAttribute(streams_join_kernel<TA, SM, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    gg_launch(streams_join_kernel<TA, SM, V>, dim3(T), dim3(threads), smem, stream, a);                                    \
  } while (0)
#define ST_V(TA, SM) do { if (vec) ST_GO(TA, SM, 4); else ST_GO(TA, SM, 1); } while (0)
#define ST_S(TA)                                                                                         \
  do { if (S <= 2) ST_V(TA, 2); else if (S <= 4) ST_V(TA, 4); else if (S <= 8) ST_V(TA, 8); else ST_V(TA, 16); } while (0)
  if (act_dtype == GG_F32) ST_S(float);
  else if (act_dtype == GG_BF16) ST_S(__nv_bfloat16);
  else return gg_fail(GG_ERR_INVALID, "streams_join: unknown dtype %d", act_dtype);
#undef ST_GO
#undef ST_V
#undef ST_S
  return gg_check_launch("streams_join");
}
