// Retention: linear attention with one fixed decay g per head and no softmax.  Per head a matrix state
// S [d, dv] in float32, carried from token to token in the request's state slot:
//     S <- g S + k v^T;    o = S^T q
// q and k are rotated by their token's position, k is scaled (d^-1/2), and each head's o is then divided
// by its root mean square and multiplied by silu(gate) (csrc/delta_rule.cu: gg_delta_out).
//
// gg_retention_rows: the projection's rows [q: H*d | k: H*d | v: H*dv] (activation type) to float32 rows of
//   the same layout, q and k rotated, k scaled.  Angles are formed and reduced in float64, sines, cosines
//   and the rotation are float32 (as rope_cache.cu), and nothing is rounded to 16 bits afterwards.
#include "common.cuh"

__device__ __forceinline__ void rotation_of(double pos, double inv_freq, float* c, float* s) {
  const double two_pi = 6.283185307179586476925286766559;
  const double ang = pos * inv_freq;
  const float r = (float)(ang - two_pi * rint(ang * (1.0 / two_pi)));
  sincosf(r, s, c);
}

#define RET_HEADS 8          // heads (of q, k or v) a block of the rows kernel takes

// grid (T, ceil(3H / 8)), 256 threads.  vec: four neighbouring values a thread (d, dv and the row stride multiples
// of 4, rot a multiple of 8, half-split pairs, aligned rows)
template <typename TA>
__global__ void __launch_bounds__(256)
retention_rows_kernel(const TA* __restrict__ x, long long x_stride, const int* __restrict__ positions,
                      const double* __restrict__ inv_freq, int H, int d, int dv, int rot, int interleaved, float kscale,
                      int vec, float* __restrict__ out) {
  extern __shared__ float cs[];                    // cos [rot/2], sin [rot/2]
  pdl_trigger();
  const size_t t = blockIdx.x;
  const int half = rot >> 1, h0 = blockIdx.y * RET_HEADS, h1 = min(h0 + RET_HEADS, 3 * H);
  if (h0 < 2 * H)
    for (int p = threadIdx.x; p < half; p += blockDim.x) rotation_of((double)positions[t], inv_freq[p], &cs[p], &cs[half + p]);
  __syncthreads();
  pdl_wait();
  const int C = H * (2 * d + dv);
  const TA* xr = x + t * x_stride;
  float* o = out + t * C;
  const int wmax = max(d, dv);
  if (vec) {
    const int per = wmax >> 2;                     // groups of four values of a head (those past its size do nothing)
    for (int e = threadIdx.x; e < (h1 - h0) * per; e += blockDim.x) {
      const int h = h0 + e / per, c = (e % per) << 2;
      const bool is_v = h >= 2 * H;
      if (c >= (is_v ? dv : d)) continue;
      const size_t base = is_v ? (size_t)2 * H * d + (size_t)(h - 2 * H) * dv : (size_t)h * d;
      const float sc = h >= H && !is_v ? kscale : 1.f;
      if (!is_v && c >= half && c < rot) continue; // the second half of the rotated pairs goes with the first
      float a[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] = to_f32(xr[base + c + j]);
      if (!is_v && c < half) {
        float b[4], ra[4], rb[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          b[j] = to_f32(xr[base + half + c + j]);
          const float co = cs[c + j], si = cs[half + c + j];
          ra[j] = (a[j] * co - b[j] * si) * sc;
          rb[j] = (b[j] * co + a[j] * si) * sc;
        }
        *reinterpret_cast<float4*>(o + base + c) = make_float4(ra[0], ra[1], ra[2], ra[3]);
        *reinterpret_cast<float4*>(o + base + half + c) = make_float4(rb[0], rb[1], rb[2], rb[3]);
      } else {
        *reinterpret_cast<float4*>(o + base + c) = make_float4(a[0] * sc, a[1] * sc, a[2] * sc, a[3] * sc);
      }
    }
    return;
  }
  for (int e = threadIdx.x; e < (h1 - h0) * wmax; e += blockDim.x) {
    const int h = h0 + e / wmax, c = e % wmax;
    const bool is_v = h >= 2 * H;
    if (c >= (is_v ? dv : d)) continue;
    const size_t base = is_v ? (size_t)2 * H * d + (size_t)(h - 2 * H) * dv : (size_t)h * d;
    float y = to_f32(xr[base + c]);
    if (!is_v && c < rot) {
      const int p = interleaved ? c >> 1 : (c < half ? c : c - half);
      const bool second = interleaved ? (c & 1) : c >= half;
      const int mate = interleaved ? (c ^ 1) : (second ? c - half : c + half);
      const float z = to_f32(xr[base + mate]);
      y = second ? y * cs[p] + z * cs[half + p] : y * cs[p] - z * cs[half + p];
    }
    if (h >= H && !is_v) y *= kscale;
    o[base + c] = y;
  }
}

extern "C" int gg_retention_rows(const void* x, long long x_stride, int dtype, const int* positions, const double* inv_freq,
                                 int T, int H, int d, int dv, int rot, int interleaved, float kscale, float* out,
                                 cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && H > 0 && d > 0 && dv > 0, "retention_rows: bad sizes T=%d H=%d d=%d dv=%d", T, H, d, dv);
  GG_REQUIRE(x && out && positions && x_stride >= (long long)H * (2 * d + dv), "retention_rows: rows of %lld values are too short", x_stride);
  GG_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || inv_freq), "retention_rows: %d rotated values of %d", rot, d);
  GG_REQUIRE((3 * H + RET_HEADS - 1) / RET_HEADS <= 65535 && rot <= 8192, "retention_rows: too many heads or rotated values");
  if (T == 0) return GG_OK;
  const int vec = !interleaved && d % 4 == 0 && dv % 4 == 0 && rot % 8 == 0 && ((size_t)out % 16) == 0;
  const dim3 grid(T, (3 * H + RET_HEADS - 1) / RET_HEADS);
  const size_t smem = (size_t)rot * sizeof(float);
  if (dtype == GG_F32)
    gg_launch(retention_rows_kernel<float>, grid, dim3(256), smem, stream, (const float*)x, x_stride, positions, inv_freq, H, d, dv, rot, interleaved, kscale, vec, out);
  else if (dtype == GG_BF16)
    gg_launch(retention_rows_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, (const __nv_bfloat16*)x, x_stride, positions, inv_freq, H, d, dv, rot, interleaved, kscale, vec, out);
  else
    return gg_fail(GG_ERR_INVALID, "retention_rows: unknown dtype %d", dtype);
  return gg_check_launch("retention_rows");
}
