// Retention: linear attention with one fixed decay g per head and no softmax.  Per head a matrix state
// S [d, dv] in float32, carried from token to token in the request's state slot:
//     S <- g S + k v^T;    o = S^T q;    y = o / sqrt(mean(o^2) + eps) * silu(gate)
// q and k are rotated by their token's position and k is scaled (d^-1/2) after that.
//
// Single decoded tokens: gg_retention_decode, one kernel from the projection's row to y: rotation, the state's
//   step, the read-out, the unit norm and the gate.  The columns of a head's state are spread over the CTAs of a
//   cluster, which exchange their sums of squares through distributed shared memory.
// Prompt portions, in chunks of 64 tokens counted from the portion's start (a fixed decay makes a chunk a product):
//   gg_retention_rows    q and k rotated, k scaled, in float32 rows [q | k | v]
//   gg_retention_states  S before every chunk: S' = g^n S + sum_j g^(n-1-j) k_j v_j^T over the n tokens of a chunk;
//                        tiles of the state in parallel, a sequence's chunks one after the other
//   gg_retention_chunks  per chunk and head, all chunks at once: row i = g^(i+1) q_i S + sum_(j<=i) g^(i-j) (q_i . k_j) v_j,
//                        then the unit norm and the gate
// Everything is float32 arithmetic from the projection's values to y (also the products inside a chunk); angles are
// formed and reduced in float64.  Powers of g are 2^(n log2 g).
#include "common.cuh"

__device__ __forceinline__ void rotation_of(double pos, double inv_freq, float* c, float* s) {
  const double two_pi = 6.283185307179586476925286766559;
  const double ang = pos * inv_freq;
  const float r = (float)(ang - two_pi * rint(ang * (1.0 / two_pi)));
  sincosf(r, s, c);
}

#define RET_HEADS 8          // heads (of q, k or v) a block of the element-wise rows kernel takes

__device__ __forceinline__ float4 ret_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ret_load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}

__device__ __forceinline__ void ret_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ret_store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}

// grid T, 256 threads: a token's whole row, four neighbouring values (of both halves of the rotated pairs) a thread.
// d, dv and the row stride multiples of 4, rot a multiple of 8, half-split pairs, aligned rows.
template <typename TA>
__global__ void __launch_bounds__(256)
retention_rows_vec_kernel(const TA* __restrict__ x, long long x_stride, const int* __restrict__ positions,
                          const double* __restrict__ inv_freq, int H, int d, int dv, int rot, float kscale, float* __restrict__ out) {
  extern __shared__ float cs[];                    // cos [rot/2], sin [rot/2]
  pdl_trigger();
  const size_t t = blockIdx.x;
  const int half = rot >> 1;
  for (int p = threadIdx.x; p < half; p += 256) rotation_of((double)positions[t], inv_freq[p], &cs[p], &cs[half + p]);
  __syncthreads();
  pdl_wait();
  const TA* xr = x + t * x_stride;
  float* o = out + t * (size_t)H * (2 * d + dv);
  const int pairs = half >> 2, per = pairs + ((d - rot) >> 2);     // groups of a q or k head: turned pairs, then what passes
  for (int e = threadIdx.x; e < 2 * H * per; e += 256) {
    const int h = (unsigned)e / (unsigned)per, g = e - h * per;
    const int base = h * d;
    const float sc = h >= H ? kscale : 1.f;
    if (g < pairs) {
      const int c = g << 2;
      const float4 a = ret_load4(xr + base + c), b = ret_load4(xr + base + half + c);
      const float4 co = *reinterpret_cast<const float4*>(cs + c), si = *reinterpret_cast<const float4*>(cs + half + c);
      *reinterpret_cast<float4*>(o + base + c) =
          make_float4((a.x * co.x - b.x * si.x) * sc, (a.y * co.y - b.y * si.y) * sc, (a.z * co.z - b.z * si.z) * sc, (a.w * co.w - b.w * si.w) * sc);
      *reinterpret_cast<float4*>(o + base + half + c) =
          make_float4((b.x * co.x + a.x * si.x) * sc, (b.y * co.y + a.y * si.y) * sc, (b.z * co.z + a.z * si.z) * sc, (b.w * co.w + a.w * si.w) * sc);
    } else {
      const int c = rot + ((g - pairs) << 2);
      const float4 a = ret_load4(xr + base + c);
      *reinterpret_cast<float4*>(o + base + c) = make_float4(a.x * sc, a.y * sc, a.z * sc, a.w * sc);
    }
  }
  const int v0 = 2 * H * d, nv = (H * dv) >> 2;
  for (int e = threadIdx.x; e < nv; e += 256) *reinterpret_cast<float4*>(o + v0 + 4 * e) = ret_load4(xr + v0 + 4 * e);
}

// grid (T, ceil(3H / 8)), 256 threads, any sizes and either layout of the pairs
template <typename TA>
__global__ void __launch_bounds__(256)
retention_rows_kernel(const TA* __restrict__ x, long long x_stride, const int* __restrict__ positions,
                      const double* __restrict__ inv_freq, int H, int d, int dv, int rot, int interleaved, float kscale,
                      float* __restrict__ out) {
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
  GG_REQUIRE(dtype == GG_F32 || dtype == GG_BF16, "retention_rows: unknown dtype %d", dtype);
  const size_t smem = (size_t)rot * sizeof(float);
  if (!interleaved && d % 4 == 0 && dv % 4 == 0 && rot % 8 == 0 && x_stride % 4 == 0 && ((size_t)out % 16) == 0 && ((size_t)x % 16) == 0) {
    if (dtype == GG_F32)
      gg_launch(retention_rows_vec_kernel<float>, dim3(T), dim3(256), smem, stream, (const float*)x, x_stride, positions, inv_freq, H, d, dv, rot, kscale, out);
    else
      gg_launch(retention_rows_vec_kernel<__nv_bfloat16>, dim3(T), dim3(256), smem, stream, (const __nv_bfloat16*)x, x_stride, positions, inv_freq, H, d, dv, rot, kscale, out);
    return gg_check_launch("retention_rows");
  }
  const dim3 grid(T, (3 * H + RET_HEADS - 1) / RET_HEADS);
  if (dtype == GG_F32)
    gg_launch(retention_rows_kernel<float>, grid, dim3(256), smem, stream, (const float*)x, x_stride, positions, inv_freq, H, d, dv, rot, interleaved, kscale, out);
  else
    gg_launch(retention_rows_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, (const __nv_bfloat16*)x, x_stride, positions, inv_freq, H, d, dv, rot, interleaved, kscale, out);
  return gg_check_launch("retention_rows");
}

// ---------------------------------------------------------------- prompt portions, chunk by chunk
#define RET_C 64               // tokens of a chunk
#define RET_ST 64              // rows and columns of a state tile of the states kernel
#define RET_SLICE 16           // rows of S or of v staged at a time by the chunks kernel
#define RET_PT 68              // pitch of the transposed scores

// Chunk c of sequence b has this place in the scratch of states: unique, since a sequence's chunks start 64 tokens
// apart and the next sequence's first index is at least one higher.  Places needed: T / 64 + B + 1.
__device__ __forceinline__ size_t chunk_place(int first_token, int b) { return (size_t)(first_token / RET_C + b); }

__device__ __forceinline__ void ret_cp16(float* dst, const float* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ret_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void ret_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// two float32 multiply-adds in one instruction (each half rounded as the scalar one)
__device__ __forceinline__ float2 ret_fma2(float2 a, float2 b, float2 c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)),
        "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&d);
}
__device__ __forceinline__ float2 ret_mul2(float2 a, float2 b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)));
  return *reinterpret_cast<float2*>(&d);
}

// grid (B, H, tiles of d x tiles of dv), 256 threads: a thread holds 4 rows (of d) x 4 columns (of dv) of the state.
// scratch [place][H][d][dv]; state [slots, H, dv, d].
__global__ void __launch_bounds__(256)
retention_states_kernel(const float* __restrict__ rows, const float* __restrict__ log2_decay, float* __restrict__ state,
                        float* __restrict__ scratch, const int* __restrict__ cu_q_lens, const int* __restrict__ context_lens,
                        const int* __restrict__ state_slots, int H, int d, int dv, int vec) {
  extern __shared__ __align__(16) float sm[];        // two stages of k [64][64], v [64][64]
  __shared__ float wj[2][RET_C];
  const int b = blockIdx.x, h = blockIdx.y;
  const int slot = state_slots[b];
  const int t0 = cu_q_lens[b], qlen = cu_q_lens[b + 1] - t0;
  if (slot < 0 || qlen <= 1) return;                 // single tokens go through the decode kernel
  const int vt = (dv + RET_ST - 1) / RET_ST;
  const int r0 = (blockIdx.z / vt) * RET_ST, c0 = (blockIdx.z % vt) * RET_ST;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int start = context_lens[b] - qlen;
  const float l2 = log2_decay[h];
  const size_t C = (size_t)H * (2 * d + dv);
  float* shead = state + ((size_t)slot * H + h) * dv * d;
  float2 S[4][2];                                    // rows r0 + 4 ty + i, columns c0 + 4 tx + (0,1), (2,3)
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = r0 + 4 * ty + i, col = c0 + 4 * tx + j;
      const float v = (start > 0 && row < d && col < dv) ? shead[(size_t)col * d + row] : 0.f;
      if (j & 1) S[i][j >> 1].y = v; else S[i][j >> 1].x = v;
    }
  pdl_wait();
  const float* kb = rows + (size_t)t0 * C + (size_t)(H + h) * d + r0;
  const float* vb = rows + (size_t)t0 * C + (size_t)2 * H * d + (size_t)h * dv + c0;
  auto stage = [&](int q0, int buf) {
    const int n = min(RET_C, qlen - q0);
    float* ks = sm + buf * 2 * RET_C * RET_ST;
    float* vs = ks + RET_C * RET_ST;
    if (vec) {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int e = tid + u * 256, j = e >> 4, c = (e & 15) << 2;
        const bool live = j < n;
        const size_t at = (size_t)(q0 + (live ? j : 0)) * C;
        const bool kok = live && r0 + c < d, vok = live && c0 + c < dv;
        ret_cp16(ks + j * RET_ST + c, kb + (kok ? at + c : 0), kok);
        ret_cp16(vs + j * RET_ST + c, vb + (vok ? at + c : 0), vok);
      }
    } else {
      for (int e = tid; e < RET_C * RET_ST; e += 256) {
        const int j = e >> 6, c = e & 63;
        const size_t at = (size_t)(q0 + j) * C;
        ks[e] = (j < n && r0 + c < d) ? kb[at + c] : 0.f;
        vs[e] = (j < n && c0 + c < dv) ? vb[at + c] : 0.f;
      }
    }
    if (tid < RET_C) wj[buf][tid] = tid < n ? exp2f(l2 * (float)(n - 1 - tid)) : 0.f;
  };
  stage(0, 0);
  ret_commit();
  for (int q0 = 0, buf = 0; q0 < qlen; q0 += RET_C, buf ^= 1) {
    const int n = min(RET_C, qlen - q0);
    if (q0 + RET_C < qlen) stage(q0 + RET_C, buf ^ 1);
    ret_commit();
    if (start + q0 > 0) {                            // the state before this chunk (the very first one is zeros: not written)
      float* out = scratch + (chunk_place(t0 + q0, b) * H + h) * d * dv;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int row = r0 + 4 * ty + i, col = c0 + 4 * tx;
        if (row < d) {
          if (vec) {
            if (col < dv) *reinterpret_cast<float4*>(out + (size_t)row * dv + col) = make_float4(S[i][0].x, S[i][0].y, S[i][1].x, S[i][1].y);
          } else {
            const float v4[4] = {S[i][0].x, S[i][0].y, S[i][1].x, S[i][1].y};
#pragma unroll
            for (int j = 0; j < 4; ++j) if (col + j < dv) out[(size_t)row * dv + col + j] = v4[j];
          }
        }
      }
    }
    ret_wait<1>();
    __syncthreads();
    const float* ks = sm + buf * 2 * RET_C * RET_ST + 4 * ty;
    const float* vs = sm + buf * 2 * RET_C * RET_ST + RET_C * RET_ST + 4 * tx;
    const float gn = exp2f(l2 * (float)n);
    const float2 gn2 = make_float2(gn, gn);
#pragma unroll
    for (int i = 0; i < 4; ++i) { S[i][0] = ret_mul2(S[i][0], gn2); S[i][1] = ret_mul2(S[i][1], gn2); }
    // four tokens at a time, the next four read while these are worked on: there are few warps to hide the reads behind
    float4 kn[4], vn[4];
    float wn[4];
    auto fetch = [&](int j0) {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        kn[u] = *reinterpret_cast<const float4*>(ks + (j0 + u) * RET_ST);
        vn[u] = *reinterpret_cast<const float4*>(vs + (j0 + u) * RET_ST);
        wn[u] = wj[buf][j0 + u];
      }
    };
    fetch(0);
#pragma unroll 2
    for (int j0 = 0; j0 < n; j0 += 4) {                // (tokens past n hold zeros)
      float4 k4[4], v4[4];
      float w[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) { k4[u] = kn[u]; v4[u] = vn[u]; w[u] = wn[u]; }
      fetch(min(j0 + 4, RET_C - 4));
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float2 w2 = make_float2(w[u], w[u]);
        const float2 va = ret_mul2(make_float2(v4[u].x, v4[u].y), w2), vc = ret_mul2(make_float2(v4[u].z, v4[u].w), w2);
        const float kk[4] = {k4[u].x, k4[u].y, k4[u].z, k4[u].w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 k2 = make_float2(kk[i], kk[i]);
          S[i][0] = ret_fma2(k2, va, S[i][0]);
          S[i][1] = ret_fma2(k2, vc, S[i][1]);
        }
      }
    }
    __syncthreads();                                 // the other buffer is refilled at the top of the next round
  }
  ret_wait<0>();
  pdl_trigger();
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int col = c0 + 4 * tx + j, row = r0 + 4 * ty;
    if (col >= dv) continue;
    float s4[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) s4[i] = (j & 1) ? S[i][j >> 1].y : S[i][j >> 1].x;
    if (vec) {
      if (row < d) *reinterpret_cast<float4*>(shead + (size_t)col * d + row) = make_float4(s4[0], s4[1], s4[2], s4[3]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) if (row + i < d) shead[(size_t)col * d + row + i] = s4[i];
    }
  }
}

// grid (tiles, H), 256 threads: a warp owns 8 rows of the chunk, a lane the columns lane * 4 + 128 j of them.
template <typename TA, int NV>
__global__ void __launch_bounds__(256, NV <= 2 ? 2 : 1)
retention_chunks_kernel(const float* __restrict__ rows, const float* __restrict__ log2_decay, const float* __restrict__ scratch,
                        const int* __restrict__ tile_seq, const int* __restrict__ tile_q0, const int* __restrict__ cu_q_lens,
                        const int* __restrict__ context_lens, const TA* __restrict__ gate, long long gate_stride, float eps,
                        int H, int d, int dv, int vec, int vec_io, TA* __restrict__ out) {
  constexpr int VP = NV * 128;
  extern __shared__ __align__(16) float sm[];
  float* Qt = sm;                                    // [d][64]: q transposed
  float* Kt = Qt + d * RET_C;                        // [d][64]: k transposed; then the weighted scores, transposed [64][RET_PT]
  float* ring = Kt + max(d * RET_C, RET_C * RET_PT); // two slices [16][VP] of S, then of v
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = tile_seq[blockIdx.x], q0 = tile_q0[blockIdx.x], h = blockIdx.y;
  const int t0 = cu_q_lens[b], qlen = cu_q_lens[b + 1] - t0;
  const int n = min(RET_C, qlen - q0);
  const bool carry = context_lens[b] - qlen + q0 > 0;
  const float l2 = log2_decay[h];
  const size_t C = (size_t)H * (2 * d + dv);
  const float* rq = rows + (size_t)(t0 + q0) * C + (size_t)h * d;
  const float* rk = rq + (size_t)H * d;
  const float* rv = rows + (size_t)(t0 + q0) * C + (size_t)2 * H * d + (size_t)h * dv;
  const float* S = scratch + (chunk_place(t0 + q0, b) * H + h) * d * dv;
  const int ns = carry ? (d + RET_SLICE - 1) / RET_SLICE : 0, nsl = ns + (n + RET_SLICE - 1) / RET_SLICE;
  pdl_wait();
  auto stage = [&](int s, int buf) {                 // slice s: 16 rows of S (s < ns) or of v
    const bool of_s = s < ns;
    const int row0 = (of_s ? s : s - ns) * RET_SLICE, have = of_s ? d : n;
    const float* src = of_s ? S : rv;
    const size_t pitch = of_s ? (size_t)dv : C;
    float* dst = ring + buf * RET_SLICE * VP;
    if (vec) {
      for (int e = tid; e < RET_SLICE * (VP / 4); e += 256) {
        const int r = e / (VP / 4), c = (e % (VP / 4)) << 2;
        const bool ok = row0 + r < have && c < dv;
        ret_cp16(dst + r * VP + c, ok ? src + (size_t)(row0 + r) * pitch + c : src, ok);
      }
    } else {
      for (int e = tid; e < RET_SLICE * VP; e += 256) {
        const int r = e / VP, c = e % VP;
        dst[e] = (row0 + r < have && c < dv) ? src[(size_t)(row0 + r) * pitch + c] : 0.f;
      }
    }
  };
  stage(0, 0);
  ret_commit();
  if (vec) {
#pragma unroll 4
    for (int e = tid; e < RET_C * (d >> 2); e += 256) {
      const int r = e & (RET_C - 1), c = (e >> 6) << 2;
      const float4 q4 = r < n ? *reinterpret_cast<const float4*>(rq + (size_t)r * C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 k4 = r < n ? *reinterpret_cast<const float4*>(rk + (size_t)r * C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      Qt[(c + 0) * RET_C + r] = q4.x; Qt[(c + 1) * RET_C + r] = q4.y; Qt[(c + 2) * RET_C + r] = q4.z; Qt[(c + 3) * RET_C + r] = q4.w;
      Kt[(c + 0) * RET_C + r] = k4.x; Kt[(c + 1) * RET_C + r] = k4.y; Kt[(c + 2) * RET_C + r] = k4.z; Kt[(c + 3) * RET_C + r] = k4.w;
    }
  } else {
    for (int e = tid; e < RET_C * d; e += 256) {
      const int r = e & (RET_C - 1), c = e >> 6;
      Qt[c * RET_C + r] = r < n ? rq[(size_t)r * C + c] : 0.f;
      Kt[c * RET_C + r] = r < n ? rk[(size_t)r * C + c] : 0.f;
    }
  }
  __syncthreads();
  const int i0 = warp * 8;
  {                                                  // the chunk's scores: 8 rows x columns lane and lane + 32
    float2 p[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) p[i][0] = p[i][1] = make_float2(0.f, 0.f);
    const int last = min(i0 + 7, n - 1);
    if (i0 < n) {
#pragma unroll 4
      for (int c = 0; c < d; ++c) {
        const float4 a = *reinterpret_cast<const float4*>(Qt + c * RET_C + i0), a2 = *reinterpret_cast<const float4*>(Qt + c * RET_C + i0 + 4);
        const float x = Kt[c * RET_C + lane];
        const float2 x2 = make_float2(x, x);
        p[0][0] = ret_fma2(make_float2(a.x, a.y), x2, p[0][0]);
        p[1][0] = ret_fma2(make_float2(a.z, a.w), x2, p[1][0]);
        p[2][0] = ret_fma2(make_float2(a2.x, a2.y), x2, p[2][0]);
        p[3][0] = ret_fma2(make_float2(a2.z, a2.w), x2, p[3][0]);
        if (last >= 32) {                            // rows of the first half see no key of the second
          const float y = Kt[c * RET_C + lane + 32];
          const float2 y2 = make_float2(y, y);
          p[0][1] = ret_fma2(make_float2(a.x, a.y), y2, p[0][1]);
          p[1][1] = ret_fma2(make_float2(a.z, a.w), y2, p[1][1]);
          p[2][1] = ret_fma2(make_float2(a2.x, a2.y), y2, p[2][1]);
          p[3][1] = ret_fma2(make_float2(a2.z, a2.w), y2, p[3][1]);
        }
      }
    }
    __syncthreads();                                 // every warp has read k: its place takes the scores
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int j = lane + 32 * half;
      float w[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float v = (i & 1) ? p[i >> 1][half].y : p[i >> 1][half].x;
        w[i] = j <= i0 + i ? v * exp2f(l2 * (float)(i0 + i - j)) : 0.f;
      }
      *reinterpret_cast<float4*>(Kt + j * RET_PT + i0) = make_float4(w[0], w[1], w[2], w[3]);
      *reinterpret_cast<float4*>(Kt + j * RET_PT + i0 + 4) = make_float4(w[4], w[5], w[6], w[7]);
    }
    __syncthreads();
  }
  float2 acc[4][4 * NV];                             // row pairs x columns
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < 4 * NV; ++c) acc[i][c] = make_float2(0.f, 0.f);
  for (int s = 0; s < nsl; ++s) {
    if (s + 1 < nsl) stage(s + 1, (s + 1) & 1);
    ret_commit();
    ret_wait<1>();
    __syncthreads();
    if (s == ns && carry) {                          // through with the state: row i of it is worth g^(i+1)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = make_float2(exp2f(l2 * (float)(i0 + 2 * i + 1)), exp2f(l2 * (float)(i0 + 2 * i + 2)));
#pragma unroll
        for (int c = 0; c < 4 * NV; ++c) acc[i][c] = ret_mul2(acc[i][c], f);
      }
    }
    const bool of_s = s < ns;
    const int row0 = (of_s ? s : s - ns) * RET_SLICE;
    if (i0 < n && (of_s || row0 <= i0 + 7)) {
      const float* A = of_s ? Qt + row0 * RET_C + i0 : Kt + row0 * RET_PT + i0;
      const int pitch = of_s ? RET_C : RET_PT, live = of_s ? min(RET_SLICE, d - row0) : RET_SLICE;
      const float* B = ring + (s & 1) * RET_SLICE * VP + lane * 4;
#pragma unroll (NV == 1 ? 4 : 2)
      for (int kk = 0; kk < live; ++kk) {
        const float4 a = *reinterpret_cast<const float4*>(A + kk * pitch), a2 = *reinterpret_cast<const float4*>(A + kk * pitch + 4);
        const float2 ap[4] = {make_float2(a.x, a.y), make_float2(a.z, a.w), make_float2(a2.x, a2.y), make_float2(a2.z, a2.w)};
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const float4 bv = *reinterpret_cast<const float4*>(B + kk * VP + j * 128);
          const float bs[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float2 b2 = make_float2(bs[c], bs[c]);
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i][4 * j + c] = ret_fma2(ap[i], b2, acc[i][4 * j + c]);
          }
        }
      }
    }
    __syncthreads();
  }
  ret_wait<0>();
  pdl_trigger();
  if (i0 >= n) return;
  float ss[8];                                       // (columns past dv hold zeros)
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 q = make_float2(0.f, 0.f);
#pragma unroll
    for (int c = 0; c < 4 * NV; ++c) q = ret_fma2(acc[i][c], acc[i][c], q);
    ss[2 * i] = q.x; ss[2 * i + 1] = q.y;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int i = 0; i < 8; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (i0 + i >= n) break;
    const float f = rsqrtf(ss[i] / (float)dv + eps);
    const size_t t = (size_t)(t0 + q0 + i0 + i);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int col = j * 128 + lane * 4;
      const TA* gr = gate + t * gate_stride + (size_t)h * dv + col;
      TA* y = out + (t * H + h) * dv + col;
      float o[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) o[c] = ((i & 1) ? acc[i >> 1][4 * j + c].y : acc[i >> 1][4 * j + c].x) * f;
      if (vec_io) {
        if (col < dv) {
          const float4 z = ret_load4(gr);
          ret_store4(y, make_float4(o[0] * (z.x / (1.f + expf(-z.x))), o[1] * (z.y / (1.f + expf(-z.y))),
                                    o[2] * (z.z / (1.f + expf(-z.z))), o[3] * (z.w / (1.f + expf(-z.w)))));
        }
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (col + c < dv) {
            const float z = to_f32(gr[c]);
            y[c] = from_f32<TA>(o[c] * (z / (1.f + expf(-z))));
          }
      }
    }
  }
}

// ---------------------------------------------------------------- single decoded tokens
// grid (n_dec, H, CTAs of a head), 128 threads, the CTAs of a head one cluster: each takes `cols` columns of the state.
// A lane holds NI rows of a column (VEC: four neighbouring ones at a time), a warp a column at a time.
#define RET_DEC_COLS 4         // columns a warp has in flight
__device__ __forceinline__ unsigned ret_map(unsigned addr, int rank) {
  unsigned r;
  asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}

template <typename TA, int NI, bool VEC>
__global__ void __launch_bounds__(128)
retention_decode_kernel(const TA* __restrict__ x, long long x_stride, int gate_col, const int* __restrict__ positions,
                        const double* __restrict__ inv_freq, const float* __restrict__ decay, float* __restrict__ state,
                        const int* __restrict__ dec_seqs, const int* __restrict__ cu_q_lens, const int* __restrict__ context_lens,
                        const int* __restrict__ state_slots, int H, int d, int dv, int rot, int interleaved, float kscale, float eps,
                        int cols, TA* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float sums[8], wsum[4];                 // sums of squares by CTA of the cluster, and by warp
  float* cs = sm;                                    // cos [rot/2], sin [rot/2]
  float* qs = cs + rot;                              // [d]
  float* ks = qs + d;                                // [d]
  float* os = ks + d;                                // [cols]
  const int b = dec_seqs[blockIdx.x];
  if (b < 0) { pdl_trigger(); pdl_wait(); return; }  // padding of a captured batch (the whole cluster is)
  const int h = blockIdx.y, rank = blockIdx.z, nz = gridDim.z;
  const int slot = state_slots[b], t = cu_q_lens[b];
  if (slot < 0) { pdl_trigger(); pdl_wait(); return; }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const bool carry = context_lens[b] > 1;
  const int half = rot >> 1, c_lo = rank * cols, c_hi = min(dv, c_lo + cols);
  const float g = decay[h];
  float* shead = state + ((size_t)slot * H + h) * dv * d;
  auto row_of = [&](int i) { return VEC ? (i >> 2) * 128 + lane * 4 + (i & 3) : lane + 32 * i; };
  float S[RET_DEC_COLS][NI];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int j = 0; j < RET_DEC_COLS; ++j) {
      const int col = c0 + 4 * j;
      const bool ok = carry && col < c_hi;
      if (VEC) {
#pragma unroll
        for (int i = 0; i < NI / 4; ++i) {
          const int row = row_of(4 * i);
          const float4 v = ok && row < d ? *reinterpret_cast<const float4*>(shead + (size_t)col * d + row) : make_float4(0.f, 0.f, 0.f, 0.f);
          S[j][4 * i] = v.x; S[j][4 * i + 1] = v.y; S[j][4 * i + 2] = v.z; S[j][4 * i + 3] = v.w;
        }
      } else {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int row = row_of(i);
          S[j][i] = ok && row < d ? shead[(size_t)col * d + row] : 0.f;
        }
      }
    }
  };
  // The state was last written by this request's step before, behind a copy from the host: it is read, like the
  // position, before the projection ahead has finished.
  fetch(c_lo + warp);
  if (nz > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // waited for before another CTA's memory is written
  for (int p = tid; p < half; p += 128) rotation_of((double)positions[t], inv_freq[p], &cs[p], &cs[half + p]);
  __syncthreads();
  pdl_trigger();
  pdl_wait();
  const TA* xr = x + (size_t)t * x_stride;
  const TA* xv = xr + (size_t)2 * H * d + (size_t)h * dv;
  for (int e = tid; e < 2 * d; e += 128) {
    const bool is_k = e >= d;
    const int c = is_k ? e - d : e;
    const TA* src = xr + (size_t)(is_k ? H + h : h) * d;
    float y = to_f32(src[c]);
    if (c < rot) {
      const int p = interleaved ? c >> 1 : (c < half ? c : c - half);
      const bool second = interleaved ? (c & 1) : c >= half;
      const float z = to_f32(src[interleaved ? (c ^ 1) : (second ? c - half : c + half)]);
      y = second ? y * cs[p] + z * cs[half + p] : y * cs[p] - z * cs[half + p];
    }
    if (is_k) ks[c] = y * kscale; else qs[c] = y;
  }
  __syncthreads();
  float q[NI], k[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int row = row_of(i);
    q[i] = row < d ? qs[row] : 0.f;
    k[i] = row < d ? ks[row] : 0.f;
  }
  float ss = 0.f;                                    // the lanes of a warp all hold the same sums
  for (int c0 = c_lo + warp; c0 < c_hi; c0 += 4 * RET_DEC_COLS) {
    if (c0 != c_lo + warp) fetch(c0);
    float o[RET_DEC_COLS];
#pragma unroll
    for (int j = 0; j < RET_DEC_COLS; ++j) {
      const int col = c0 + 4 * j;
      const float v = col < c_hi ? to_f32(xv[col]) : 0.f;
      o[j] = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        S[j][i] = fmaf(k[i], v, g * S[j][i]);
        o[j] = fmaf(q[i], S[j][i], o[j]);
      }
      if (col < c_hi) {
        if (VEC) {
#pragma unroll
          for (int i = 0; i < NI / 4; ++i) {
            const int row = row_of(4 * i);
            if (row < d) *reinterpret_cast<float4*>(shead + (size_t)col * d + row) = make_float4(S[j][4 * i], S[j][4 * i + 1], S[j][4 * i + 2], S[j][4 * i + 3]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < NI; ++i) {
            const int row = row_of(i);
            if (row < d) shead[(size_t)col * d + row] = S[j][i];
          }
        }
      }
    }
#pragma unroll
    for (int s = 16; s > 0; s >>= 1)
#pragma unroll
      for (int j = 0; j < RET_DEC_COLS; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], s);
#pragma unroll
    for (int j = 0; j < RET_DEC_COLS; ++j) {
      const int col = c0 + 4 * j;
      if (col < c_hi) {
        ss += o[j] * o[j];
        if (lane == 0) os[col - c_lo] = o[j];
      }
    }
  }
  if (lane == 0) wsum[warp] = ss;
  __syncthreads();
  float total = (wsum[0] + wsum[1]) + (wsum[2] + wsum[3]);
  if (nz > 1) {
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (tid < nz) {
      const unsigned dst = ret_map((unsigned)__cvta_generic_to_shared(&sums[rank]), tid);
      asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(total) : "memory");
    }
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    total = 0.f;
    for (int r = 0; r < nz; ++r) total += sums[r];
  }
  const float f = rsqrtf(total / (float)dv + eps);
  for (int c = c_lo + tid; c < c_hi; c += 128) {
    const float z = to_f32(xr[gate_col + (size_t)h * dv + c]);
    out[((size_t)t * H + h) * dv + c] = from_f32<TA>(os[c - c_lo] * f * (z / (1.f + expf(-z))));
  }
}

// ---------------------------------------------------------------- launchers
// Scratch the caller provides: float[(T / 64 + B + 1) * H * d * dv].  rows: gg_retention_rows' output.
extern "C" int gg_retention_states(const float* rows, const float* log2_decay, float* state, float* scratch,
                                   long long scratch_floats, const int* cu_q_lens, const int* context_lens,
                                   const int* state_slots, int T, int B, int H, int d, int dv, cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && B > 0 && H > 0 && d > 0 && dv > 0, "retention_states: bad sizes T=%d B=%d H=%d d=%d dv=%d", T, B, H, d, dv);
  GG_REQUIRE(rows && log2_decay && state && scratch, "retention_states: a pointer is null");
  GG_REQUIRE(scratch_floats >= (long long)(T / RET_C + B + 1) * H * d * dv, "retention_states: scratch of %lld values is too small", scratch_floats);
  const int tiles = ((d + RET_ST - 1) / RET_ST) * ((dv + RET_ST - 1) / RET_ST);
  GG_REQUIRE(H <= 65535 && tiles <= 65535, "retention_states: too many heads or tiles");
  if (T == 0) return GG_OK;
  const size_t smem = (size_t)4 * RET_C * RET_ST * sizeof(float);
  cudaError_t e = cudaFuncSetAttribute(retention_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "retention_states: %s", cudaGetErrorString(e));
  const int vec = d % 4 == 0 && dv % 4 == 0 && ((size_t)rows % 16) == 0 && ((size_t)scratch % 16) == 0 && ((size_t)state % 16) == 0;
  gg_launch_after(retention_states_kernel, dim3(B, H, tiles), dim3(256), smem, stream, rows, log2_decay, state, scratch, cu_q_lens,
                  context_lens, state_slots, H, d, dv, vec);
  return gg_check_launch("retention_states");
}

extern "C" int gg_retention_chunks(const float* rows, const float* log2_decay, const float* scratch, const int* tile_seq,
                                   const int* tile_q0, int num_tiles, const int* cu_q_lens, const int* context_lens,
                                   const void* gate, long long gate_stride, float eps, int H, int d, int dv, int dtype,
                                   void* out, cudaStream_t stream) {
  GG_REQUIRE(num_tiles >= 0 && H > 0 && H <= 65535 && d > 0 && d <= 256 && dv > 0 && dv <= 512,
             "retention_chunks: bad sizes tiles=%d H=%d d=%d (at most 256) dv=%d (at most 512)", num_tiles, H, d, dv);
  GG_REQUIRE(rows && log2_decay && scratch && gate && out && gate_stride >= (long long)H * dv, "retention_chunks: bad arguments");
  if (num_tiles == 0) return GG_OK;
  const int vec = d % 4 == 0 && dv % 4 == 0 && ((size_t)rows % 16) == 0 && ((size_t)scratch % 16) == 0;
  const int vec_io = dv % 4 == 0 && gate_stride % 4 == 0 && ((size_t)gate % 16) == 0 && ((size_t)out % 16) == 0;
  const int NVv = dv <= 128 ? 1 : dv <= 256 ? 2 : 4;
  const int kt = d * RET_C > RET_C * RET_PT ? d * RET_C : RET_C * RET_PT;
  const size_t smem = (size_t)(d * RET_C + kt + 2 * RET_SLICE * NVv * 128) * sizeof(float);
#define RET_GO(TA, NV)                                                                                                        \
  do {                                                                                                                        \
    cudaError_t e = cudaFuncSetAttribute(retention_chunks_kernel<TA, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "retention_chunks: %s", cudaGetErrorString(e));                         \
    gg_launch(retention_chunks_kernel<TA, NV>, dim3(num_tiles, H), dim3(256), smem, stream, rows, log2_decay, scratch, tile_seq, \
              tile_q0, cu_q_lens, context_lens, (const TA*)gate, gate_stride, eps, H, d, dv, vec, vec_io, (TA*)out);                  \
  } while (0)
#define RET_GO_NV(TA) do { if (NVv == 1) RET_GO(TA, 1); else if (NVv == 2) RET_GO(TA, 2); else RET_GO(TA, 4); } while (0)
  if (dtype == GG_F32) RET_GO_NV(float);
  else if (dtype == GG_BF16) RET_GO_NV(__nv_bfloat16);
  else return gg_fail(GG_ERR_INVALID, "retention_chunks: unknown dtype %d", dtype);
#undef RET_GO_NV
#undef RET_GO
  return gg_check_launch("retention_chunks");
}

template <typename TA, int NI, bool VEC, typename... Args>
static int retention_decode_go(dim3 grid, size_t smem, cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(128);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = grid.z;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = gg_pdl_enabled() ? 2 : 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, retention_decode_kernel<TA, NI, VEC>, args...);
  if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "retention_decode: %s", cudaGetErrorString(e));
  return gg_check_launch("retention_decode");
}

// x: the projection's rows [q: H*d | k: H*d | v: H*dv | .. | gate: H*dv at gate_col]; tokens: the sequences dec_seqs
// (-1: padding), one token each.  The state is read before the kernel ahead has finished: it must not be that kernel's
// output.
extern "C" int gg_retention_decode(const void* x, long long x_stride, int gate_col, int dtype, const int* positions,
                                   const double* inv_freq, const float* decay, float* state, const int* dec_seqs, int n_dec,
                                   const int* cu_q_lens, const int* context_lens, const int* state_slots, int H, int d, int dv,
                                   int rot, int interleaved, float kscale, float eps, void* out, cudaStream_t stream) {
  GG_REQUIRE(n_dec >= 0 && H > 0 && H <= 65535 && d > 0 && d <= 256 && dv > 0, "retention_decode: bad sizes n=%d H=%d d=%d dv=%d", n_dec, H, d, dv);
  GG_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d && (rot == 0 || inv_freq), "retention_decode: %d rotated values of %d", rot, d);
  GG_REQUIRE(x && positions && decay && state && dec_seqs && out && gate_col >= H * (2 * d + dv) && x_stride >= (long long)gate_col + H * dv,
             "retention_decode: bad arguments");
  if (n_dec == 0) return GG_OK;
  // CTAs of a head: as many as fill the machine about four times over, each with 16 columns or more
  int nz = 1;
  while (nz < 8 && (long long)n_dec * H * nz < 4 * 148 && (dv + 2 * nz - 1) / (2 * nz) >= 16) nz *= 2;
  const int cols = (dv + nz - 1) / nz;
  const size_t smem = (size_t)(rot + 2 * d + cols) * sizeof(float);
  GG_REQUIRE(smem <= 40 * 1024, "retention_decode: values of %d columns do not fit", dv);
  const dim3 grid(n_dec, H, nz);
  const bool vec = d % 4 == 0 && ((size_t)state % 16) == 0;
#define RET_DEC(TA, NI, VEC)                                                                                                    \
  return retention_decode_go<TA, NI, VEC>(grid, smem, stream, (const TA*)x, x_stride, gate_col, positions, inv_freq, decay, state, \
                                          dec_seqs, cu_q_lens, context_lens, state_slots, H, d, dv, rot, interleaved, kscale, eps, cols, (TA*)out)
  if (dtype == GG_F32) {
    if (vec && d <= 128) RET_DEC(float, 4, true);
    if (vec) RET_DEC(float, 8, true);
    RET_DEC(float, 8, false);
  }
  if (dtype == GG_BF16) {
    if (vec && d <= 128) RET_DEC(__nv_bfloat16, 4, true);
    if (vec) RET_DEC(__nv_bfloat16, 8, true);
    RET_DEC(__nv_bfloat16, 8, false);
  }
#undef RET_DEC
  return gg_fail(GG_ERR_INVALID, "retention_decode: unknown dtype %d", dtype);
}
