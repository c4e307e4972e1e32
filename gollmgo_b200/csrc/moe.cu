// Routing of a mixture of experts, on the device from start to end (a step never asks the host
// how many tokens an expert got, so a step of decoded tokens can be captured and replayed).
//
// gg_moe_route:   z[t, e] = h[t] . Wr[e] + b[e] in float32; the `top` largest logits of a token
//                 (ties: the lower index) are its experts, weights = softmax over those alone, or
//                 the softmax over all experts renormalised over the chosen, or each chosen logit's
//                 sigmoid as it is; optionally only experts of the best groups can be chosen (moe_pick);
//                 optionally one more row of Wr, whose product with h[t] is left in gate[t] (the logit of a
//                 shared expert's gate); optionally the choice goes by softmax score + a correction per expert, and
//                 the weights are multiplied by a factor
// gg_moe_align:   the (token, choice) pairs sorted by expert: offsets[e] .. offsets[e+1] are the
//                 places of expert e in `sorted` (values t * top + j), `place` is the inverse; choices
//                 past the last expert (router outputs that stand for no tensors) get the place -1
// gg_moe_combine: out[t] = sum_j weight[t, j] * y[place[t * top + j]] (+ shared[t], times the sigmoid
//                 of its gate where there is one), float32 sums in the order of j; no weights: plain sum; a
//                 place of -1 reads same[t] (the experts' input) instead of a row of y
// gg_parallel_join: what a block that runs a mixer and a feed-forward side by side does at its end, a CTA a token:
//                 resid[t] += mult * (mixer[t] + bias + the sum gg_moe_combine makes), and, where the next norm is
//                 given, h[t] = resid[t] / sqrt(mean(resid[t]^2) + eps) * w; with no experts (top = 0) `shared` is a
//                 dense feed-forward's result
// The products between them are gg_grouped_gemm's (grouped_gemm.cu).
#include "common.cuh"

#define MOE_MAX_EXPERTS 1024
#define MOE_MAX_TOP 32

// A block routes ROUTE_TOK tokens: their rows are staged in shared memory as float32, and a warp
// that takes an expert reads that expert's router row once (16 bytes a lane at a time) for all of
// them, so the router's weights cross from L2 once per ROUTE_TOK tokens and not once per token.
#define ROUTE_TOK 4      // for steps of many tokens; steps of a few tokens take one token a block, for more blocks

__device__ __forceinline__ void route_load(const float* w, float (&v)[8], int n) {
  const float4 a = *reinterpret_cast<const float4*>(w);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  (void)n;
}
__device__ __forceinline__ void route_load(const __nv_bfloat16* w, float (&v)[8], int n) {
  const uint4 r = *reinterpret_cast<const uint4*>(w);
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
  for (int j = 0; j < 4; ++j) { const float2 b = __bfloat1622float2(p[j]); v[2 * j] = b.x; v[2 * j + 1] = b.y; }
  (void)n;
}

// One warp picks a token's experts from its logits zr[E] (shared memory, overwritten) and weighs them.
// weigh = 0: weights = softmax over the chosen logits alone.  weigh = 1: scores = softmax over all
// experts, weights = the chosen scores divided by their sum (+ 1e-20).  weigh = 2: weights = the sigmoid
// of each chosen logit, not normalised (the largest sigmoids are the largest logits').  groups > 1: the experts form
// that many equal groups of neighbours, a group's score is its best expert's, and only experts of the
// `keep` best groups can be chosen.  corr (weigh = 1, one group): the choice goes by score + corr[e], the
// weights are the scores alone.  The weights are multiplied by `scale`.  Ties: the lower index.
__device__ __forceinline__ void moe_pick(float* zr, int E, int top, int weigh, int groups, int keep,
                                         const float* __restrict__ corr, float scale, int lane,
                                         int* __restrict__ idx, float* __restrict__ wgt) {
  float zmax = 0.f, zsum = 1.f;
  if (weigh == 1) {
    float m = -INFINITY;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, zr[e]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float sm = 0.f;
    for (int e = lane; e < E; e += 32) sm += expf(zr[e] - m);
    zmax = m; zsum = warp_sum(sm);
  }
  if (groups > 1 && keep < groups) {
    const int per = E / groups;
    unsigned kept = 0;                             // bit i: group lane + 32 i is kept
    for (int k = 0; k < keep; ++k) {
      float best = -INFINITY;
      int bg = 0x7fffffff;
      for (int g = lane, i = 0; g < groups; g += 32, ++i) {
        if (kept >> i & 1u) continue;
        float gm = -INFINITY;
        for (int e = g * per; e < (g + 1) * per; ++e) gm = fmaxf(gm, zr[e]);
        if (gm > best || (gm == best && g < bg)) { best = gm; bg = g; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int og = __shfl_xor_sync(0xffffffffu, bg, o);
        if (ov > best || (ov == best && og < bg)) { best = ov; bg = og; }
      }
      if (bg == 0x7fffffff) break;                 // nothing but NaN left
      if ((bg & 31) == lane) kept |= 1u << (bg >> 5);
    }
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane, g = e < E ? e / per : 0;
      const unsigned owner = __shfl_sync(0xffffffffu, kept, g & 31);
      if (e < E && !(owner >> (g >> 5) & 1u)) zr[e] = -INFINITY;
    }
    __syncwarp();
  }
  float val[MOE_MAX_TOP];
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      float v = zr[e];
      if (corr && v != -INFINITY) v = expf(v - zmax) / zsum + corr[e];     // -inf: chosen already
      if (v > best || (v == best && e < bi)) { best = v; bi = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (bi == 0x7fffffff) bi = 0;                    // every logit left is -inf or NaN
    val[j] = corr ? zr[bi] : best;
    __syncwarp();
    if (lane == 0) { idx[j] = bi; zr[bi] = -INFINITY; }
    __syncwarp();
  }
  if (lane == 0) {
    if (weigh == 1) {
      float sum = 0.f;
      for (int j = 0; j < top; ++j) { val[j] = expf(val[j] - zmax) / zsum; sum += val[j]; }
      for (int j = 0; j < top; ++j) wgt[j] = val[j] / (sum + 1e-20f) * scale;
    } else if (weigh == 2) {
      for (int j = 0; j < top; ++j) wgt[j] = scale / (1.f + expf(-val[j]));
    } else {
      const float m = val[0];                        // the largest comes first
      float sum = 0.f;
      for (int j = 0; j < top; ++j) { val[j] = expf(val[j] - m); sum += val[j]; }
      for (int j = 0; j < top; ++j) wgt[j] = val[j] / sum * scale;
    }
  }
}

template <typename TA, int TOK>
__global__ void moe_route_kernel(const TA* __restrict__ h, const TA* __restrict__ wr, const float* __restrict__ bias,
                                 int T, int D, int E, int top, int weigh, int groups, int keep,
                                 const float* __restrict__ corr, float scale,
                                 int* __restrict__ idx, float* __restrict__ wgt, float* __restrict__ gate, int vec) {
  __shared__ float z[TOK][MOE_MAX_EXPERTS];
  extern __shared__ __align__(16) float xs[];              // TOK rows of D floats
  constexpr int VPT = 16 / (int)sizeof(TA);
  pdl_trigger();
  pdl_wait();
  const int t0 = blockIdx.x * TOK, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const int nt = min(TOK, T - t0);
  for (int e = threadIdx.x; e < TOK * D; e += blockDim.x) {
    const int r = e / D;
    xs[e] = r < nt ? to_f32(h[(size_t)(t0 + r) * D + (e - r * D)]) : 0.f;
  }
  __syncthreads();
  const int rows = E + (gate ? 1 : 0);
  for (int e = warp; e < rows; e += nw) {
    const TA* w = wr + (size_t)e * D;
    float s[TOK];
#pragma unroll
    for (int r = 0; r < TOK; ++r) s[r] = 0.f;
    if (vec) {
      for (int c = lane * VPT; c < D; c += 32 * VPT) {
        float v[8];
        route_load(w + c, v, VPT);
#pragma unroll
        for (int r = 0; r < TOK; ++r) {
#pragma unroll
          for (int j = 0; j < VPT; j += 4) {                // the staged rows four values at a time
            const float4 x = *reinterpret_cast<const float4*>(xs + r * D + c + j);
            s[r] = fmaf(x.x, v[j], s[r]); s[r] = fmaf(x.y, v[j + 1], s[r]);
            s[r] = fmaf(x.z, v[j + 2], s[r]); s[r] = fmaf(x.w, v[j + 3], s[r]);
          }
        }
      }
    } else {
      for (int c = lane; c < D; c += 32) {
        const float v = to_f32(w[c]);
#pragma unroll
        for (int r = 0; r < TOK; ++r) s[r] = fmaf(xs[r * D + c], v, s[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < TOK; ++r) {
      const float tot = warp_sum(s[r]);
      if (lane == 0) {
        if (e < E) z[r][e] = tot + (bias ? bias[e] : 0.f);
        else if (r < nt) gate[t0 + r] = tot;
      }
    }
  }
  __syncthreads();
  if (warp < nt)                                           // warp r picks for token t0 + r (the block has TOK warps or more)
    moe_pick(z[warp], E, top, weigh, groups, keep, corr, scale, lane, idx + (size_t)(t0 + warp) * top, wgt + (size_t)(t0 + warp) * top);
}

// The choice alone, from logits a product has already made (long steps: z = h Wr^T in float32 by the
// vendor library from the bfloat16 rows): one warp a token adds the bias, picks and weighs.
__global__ void moe_topk_kernel(const float* __restrict__ z, long long z_stride, const float* __restrict__ bias, int T, int E, int top,
                                int weigh, int groups, int keep, const float* __restrict__ corr, float scale,
                                int* __restrict__ idx, float* __restrict__ wgt) {
  extern __shared__ float zs[];                            // warps x E
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= T) return;
  float* zr = zs + warp * E;
  for (int e = lane; e < E; e += 32) zr[e] = z[t * z_stride + e] + (bias ? bias[e] : 0.f);
  __syncwarp();
  moe_pick(zr, E, top, weigh, groups, keep, corr, scale, lane, idx + (size_t)t * top, wgt + (size_t)t * top);
}

// One CTA.  counts and cursors in shared memory; the order of the rows inside an expert's range
// is whatever the atomics give, which no result depends on.  pad > 1: every expert's range
// starts at a multiple of pad (the places between its last row and the next range hold -1 in
// `sorted`), `slots` is the length of `sorted`, and tile_group[i] is the expert that places
// pad * i .. pad * i + pad - 1 belong to, or -1 past the last range (n_tiles entries).
__global__ void moe_align_kernel(const int* __restrict__ idx, int n, int E, int pad, int slots, int* __restrict__ offsets,
                                 int* __restrict__ sorted, int* __restrict__ place, int* __restrict__ tile_group,
                                 int n_tiles) {
  __shared__ int cnt[MOE_MAX_EXPERTS + 1];
  __shared__ int start[MOE_MAX_EXPERTS + 1];
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) cnt[e] = 0;
  if (pad > 1)
    for (int i = threadIdx.x; i < slots; i += blockDim.x) sorted[i] = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x)
    if (idx[i] < E) atomicAdd(&cnt[idx[i]], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0;
    for (int e = 0; e < E; ++e) {
      const int c = cnt[e];
      cnt[e] = run; start[e] = run; offsets[e] = run;
      run += (c + pad - 1) / pad * pad;
    }
    start[E] = run; offsets[E] = run;
  }
  __syncthreads();
  if (tile_group)
    for (int i = threadIdx.x; i < n_tiles; i += blockDim.x) {
      const int p = i * pad;
      int g = -1;
      if (p < start[E]) {
        int lo = 0, hi = E;                          // the last expert whose range starts at or before p
        while (hi - lo > 1) { const int mid = (lo + hi) >> 1; if (start[mid] <= p) lo = mid; else hi = mid; }
        g = lo;
      }
      tile_group[i] = g;
    }
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    if (idx[i] >= E) { place[i] = -1; continue; }
    const int p = atomicAdd(&cnt[idx[i]], 1);
    sorted[p] = i;
    place[i] = p;
  }
}

// xs[p] = x[sorted[p] / top] for the places that hold a pair, zeros for the others: the rows of
// every expert gathered into one block that starts at a multiple of the product's tile height.
template <typename TA>
__global__ void moe_gather_kernel(const TA* __restrict__ x, const int* __restrict__ sorted, int top, int D,
                                  TA* __restrict__ xs, int vec) {
  pdl_trigger();
  pdl_wait();
  const size_t p = blockIdx.x;
  const int src = sorted[p];
  TA* o = xs + p * D;
  if (vec) {
    constexpr int VPT = 16 / (int)sizeof(TA);
    const uint4* in = src >= 0 ? reinterpret_cast<const uint4*>(x + (size_t)(src / top) * D) : nullptr;
    for (int c = threadIdx.x; c < D / VPT; c += blockDim.x)
      reinterpret_cast<uint4*>(o)[c] = in ? in[c] : make_uint4(0, 0, 0, 0);
  } else {
    const TA* in = src >= 0 ? x + (size_t)(src / top) * D : nullptr;
    for (int c = threadIdx.x; c < D; c += blockDim.x) o[c] = in ? in[c] : from_f32<TA>(0.f);
  }
}

// The row that choice i of token t adds.
template <typename TA>
__device__ __forceinline__ const TA* moe_row(const TA* y, const int* place, const TA* same, size_t t, size_t i, int D) {
  const int p = place[i];
  return p >= 0 ? y + (size_t)p * D : same + t * D;
}

template <typename TA>
__global__ void moe_combine_kernel(const TA* __restrict__ y, const int* __restrict__ place, const float* __restrict__ wgt,
                                   const TA* __restrict__ shared_out, const float* __restrict__ gate, long long gate_stride,
                                   const TA* __restrict__ same, TA* __restrict__ out, int D, int top) {
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const float sg = gate ? 1.f / (1.f + expf(-gate[t * gate_stride])) : 1.f;      // on the shared expert
  if (D % 4 == 0) {                              // rows of every buffer are then 8-byte aligned at least
    for (int c = threadIdx.x * 4; c < D; c += blockDim.x * 4) {
      float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
      for (int j = 0; j < top; ++j) {
        const float w = wgt ? wgt[t * top + j] : 1.f;
        const TA* r = moe_row(y, place, same, t, t * top + j, D) + c;
        s0 = fmaf(w, to_f32(r[0]), s0); s1 = fmaf(w, to_f32(r[1]), s1);
        s2 = fmaf(w, to_f32(r[2]), s2); s3 = fmaf(w, to_f32(r[3]), s3);
      }
      if (shared_out) {
        const TA* r = shared_out + t * D + c;
        s0 = fmaf(sg, to_f32(r[0]), s0); s1 = fmaf(sg, to_f32(r[1]), s1);
        s2 = fmaf(sg, to_f32(r[2]), s2); s3 = fmaf(sg, to_f32(r[3]), s3);
      }
      TA* o = out + t * D + c;
      o[0] = from_f32<TA>(s0); o[1] = from_f32<TA>(s1); o[2] = from_f32<TA>(s2); o[3] = from_f32<TA>(s3);
    }
    return;
  }
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    float s = 0.f;
    for (int j = 0; j < top; ++j)
      s = fmaf(wgt ? wgt[t * top + j] : 1.f, to_f32(moe_row(y, place, same, t, t * top + j, D)[c]), s);
    if (shared_out) s = fmaf(sg, to_f32(shared_out[t * D + c]), s);
    out[t * D + c] = from_f32<TA>(s);
  }
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}
__device__ __forceinline__ void axpy4(float4& s, float w, float4 v) {
  s.x = fmaf(w, v.x, s.x); s.y = fmaf(w, v.y, s.y); s.z = fmaf(w, v.z, s.z); s.w = fmaf(w, v.w, s.w);
}

template <typename TA>
__global__ void parallel_join_kernel(float* __restrict__ resid, const TA* __restrict__ mixer, const TA* __restrict__ y,
                                     const int* __restrict__ place, const float* __restrict__ wgt, int top,
                                     const TA* __restrict__ shared_out, const float* __restrict__ gate, long long gate_stride,
                                     const TA* __restrict__ same, const float* __restrict__ bias, float mult, const float* __restrict__ norm_w, float eps,
                                     TA* __restrict__ h, int D, int vec) {
  extern __shared__ __align__(16) float row[];       // [D]
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const float sg = gate ? 1.f / (1.f + expf(-gate[t * gate_stride])) : 1.f;
  float* x = resid + t * D;
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < D; c += blockDim.x * 4) {
      float4 s = load4(mixer + t * D + c), r = load4(x + c);
      for (int j = 0; j < top; ++j)
        axpy4(s, wgt ? wgt[t * top + j] : 1.f, load4(moe_row(y, place, same, t, t * top + j, D) + c));
      if (shared_out) axpy4(s, sg, load4(shared_out + t * D + c));
      if (bias) axpy4(s, 1.f, load4(bias + c));
      axpy4(r, mult, s);
      store4(x + c, r);
      if (norm_w) { store4(row + c, r); ss += r.x * r.x + r.y * r.y + r.z * r.z + r.w * r.w; }
    }
  } else {
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
      float s = to_f32(mixer[t * D + c]);
      for (int j = 0; j < top; ++j)
        s = fmaf(wgt ? wgt[t * top + j] : 1.f, to_f32(moe_row(y, place, same, t, t * top + j, D)[c]), s);
      if (shared_out) s = fmaf(sg, to_f32(shared_out[t * D + c]), s);
      if (bias) s += bias[c];
      const float r = fmaf(mult, s, x[c]);
      x[c] = r;
      if (norm_w) { row[c] = r; ss += r * r; }
    }
  }
  if (!norm_w) return;
  const float f = rsqrtf(block_sum(ss, red) / (float)D + eps);
  if (vec) {
    for (int c = threadIdx.x * 4; c < D; c += blockDim.x * 4) {
      const float4 r = load4(row + c), w = load4(norm_w + c);
      store4(h + t * D + c, make_float4(r.x * f * w.x, r.y * f * w.y, r.z * f * w.z, r.w * f * w.w));
    }
  } else {
    for (int c = threadIdx.x; c < D; c += blockDim.x) h[t * D + c] = from_f32<TA>(row[c] * f * norm_w[c]);
  }
}

static int check_pick(const char* who, int E, int top, int weigh, int groups, int keep, const float* corr) {
  GG_REQUIRE(!corr || (weigh == 1 && groups == 1), "%s: a correction of the choice goes with softmax scores over all experts in one group", who);
  GG_REQUIRE(weigh >= 0 && weigh <= 2, "%s: unknown way %d of weighing the chosen experts", who, weigh);
  GG_REQUIRE(groups >= 1 && keep >= 1 && keep <= groups && E % groups == 0, "%s: %d experts in %d groups of which %d are kept", who, E, groups, keep);
  GG_REQUIRE(top <= keep * (E / groups), "%s: %d choices from %d groups of %d experts", who, top, keep, E / groups);
  return GG_OK;
}

extern "C" int gg_moe_route(const void* h, const void* wr, const float* bias, int T, int D, int E, int top,
                            int weigh, int groups, int keep, const float* corr, float scale, int* idx, float* wgt, float* gate, int act_dtype,
                            cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && D > 0 && E > 0 && top > 0 && top <= E, "moe_route: bad sizes T=%d D=%d E=%d top=%d", T, D, E, top);
  GG_REQUIRE(E <= MOE_MAX_EXPERTS && top <= MOE_MAX_TOP, "moe_route: at most %d experts and %d choices a token (got %d, %d)",
             MOE_MAX_EXPERTS, MOE_MAX_TOP, E, top);
  GG_REQUIRE(h && wr && idx && wgt, "moe_route: a pointer is null");
  if (int rc = check_pick("moe_route", E, top, weigh, groups, keep, corr)) return rc;
  if (T == 0) return GG_OK;
  const int tok = T > 256 ? ROUTE_TOK : 1;
  const size_t smem = (size_t)tok * D * sizeof(float);
  GG_REQUIRE(smem <= 200 * 1024, "moe_route: rows of %d values do not fit in shared memory", D);
  const int vec = (act_dtype == GG_F32 ? D % 4 == 0 : D % 8 == 0) && ((size_t)wr % 16) == 0;
  // at least ROUTE_TOK warps; steps of a few tokens: a warp for every row of Wr where there are up to 32
  const int wr_rows = E + (gate ? 1 : 0);
  const int threads = tok == 1 && wr_rows > 8 ? (wr_rows < 32 ? wr_rows * 32 : 1024) : E >= 8 ? 256 : 128;
  const int blocks = (T + tok - 1) / tok;
#define ROUTE_LAUNCH(T_, N_)                                                                                     \
  do {                                                                                                           \
    if (smem > 28 * 1024) cudaFuncSetAttribute(moe_route_kernel<T_, N_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    gg_launch(moe_route_kernel<T_, N_>, dim3(blocks), dim3(threads), smem, stream, (const T_*)h, (const T_*)wr, bias, T, D, E, top, weigh, groups, keep, corr, scale, idx, wgt, gate, vec); \
  } while (0)
  if (act_dtype == GG_F32) {
    if (tok == 1) ROUTE_LAUNCH(float, 1); else ROUTE_LAUNCH(float, ROUTE_TOK);
  } else if (act_dtype == GG_BF16) {
    if (tok == 1) ROUTE_LAUNCH(__nv_bfloat16, 1); else ROUTE_LAUNCH(__nv_bfloat16, ROUTE_TOK);
  } else
    return gg_fail(GG_ERR_INVALID, "moe_route: unknown dtype %d", act_dtype);
  return gg_check_launch("moe_route");
}

extern "C" int gg_moe_topk(const float* z, long long z_stride, const float* bias, int T, int E, int top, int weigh, int groups, int keep,
                           const float* corr, float scale, int* idx, float* wgt, cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && E > 0 && top > 0 && top <= E && E <= MOE_MAX_EXPERTS && top <= MOE_MAX_TOP,
             "moe_topk: bad sizes T=%d E=%d top=%d", T, E, top);
  GG_REQUIRE(z && idx && wgt && z_stride >= E, "moe_topk: a pointer is null or the rows are too short");
  if (int rc = check_pick("moe_topk", E, top, weigh, groups, keep, corr)) return rc;
  if (T == 0) return GG_OK;
  const int warps = 4;
  gg_launch(moe_topk_kernel, dim3((T + warps - 1) / warps), dim3(32 * warps), (size_t)warps * E * sizeof(float), stream,
            z, z_stride, bias, T, E, top, weigh, groups, keep, corr, scale, idx, wgt);
  return gg_check_launch("moe_topk");
}

extern "C" int gg_moe_align(const int* idx, int n, int E, int pad, int slots, int* offsets, int* sorted, int* place,
                            int* tile_group, int n_tiles, cudaStream_t stream) {
  GG_REQUIRE(n >= 0 && E > 0 && E <= MOE_MAX_EXPERTS && pad >= 1, "moe_align: bad sizes n=%d E=%d pad=%d", n, E, pad);
  GG_REQUIRE(idx && offsets && sorted && place, "moe_align: a pointer is null");
  GG_REQUIRE(pad == 1 || (long long)slots >= (long long)n + (long long)E * (pad - 1),
             "moe_align: %d places do not hold %d rows of %d experts padded to %d", slots, n, E, pad);
  GG_REQUIRE(!tile_group || (long long)n_tiles * pad >= slots, "moe_align: %d tile entries for %d places", n_tiles, slots);
  gg_launch(moe_align_kernel, dim3(1), dim3(1024), 0, stream, idx, n, E, pad, slots, offsets, sorted, place, tile_group, n_tiles);
  return gg_check_launch("moe_align");
}

extern "C" int gg_moe_gather(const void* x, const int* sorted, int slots, int top, int D, void* xs, int act_dtype,
                             cudaStream_t stream) {
  GG_REQUIRE(slots >= 0 && top > 0 && D > 0 && x && sorted && xs, "moe_gather: bad arguments");
  if (slots == 0) return GG_OK;
  const int vpt = act_dtype == GG_F32 ? 4 : 8;
  const int vec = D % vpt == 0 && ((size_t)x % 16) == 0 && ((size_t)xs % 16) == 0;
  if (act_dtype == GG_F32)
    gg_launch(moe_gather_kernel<float>, dim3(slots), dim3(128), 0, stream, (const float*)x, sorted, top, D, (float*)xs, vec);
  else if (act_dtype == GG_BF16)
    gg_launch(moe_gather_kernel<__nv_bfloat16>, dim3(slots), dim3(128), 0, stream, (const __nv_bfloat16*)x, sorted, top, D,
              (__nv_bfloat16*)xs, vec);
  else
    return gg_fail(GG_ERR_INVALID, "moe_gather: unknown dtype %d", act_dtype);
  return gg_check_launch("moe_gather");
}

extern "C" int gg_moe_combine(const void* y, const int* place, const float* wgt, const void* shared_out,
                              const float* gate, long long gate_stride, const void* same, void* out, int T, int D, int top, int act_dtype, cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && D > 0 && top > 0, "moe_combine: bad sizes T=%d D=%d top=%d", T, D, top);
  GG_REQUIRE(y && place && out && (shared_out || !gate), "moe_combine: a pointer is null");
  if (T == 0) return GG_OK;
  const int threads = D >= 1024 ? 256 : 128;
  if (act_dtype == GG_F32)
    gg_launch(moe_combine_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)y, place, wgt, (const float*)shared_out,
              gate, gate_stride, (const float*)same, (float*)out, D, top);
  else if (act_dtype == GG_BF16)
    gg_launch(moe_combine_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const __nv_bfloat16*)y, place, wgt,
              (const __nv_bfloat16*)shared_out, gate, gate_stride, (const __nv_bfloat16*)same, (__nv_bfloat16*)out, D, top);
  else
    return gg_fail(GG_ERR_INVALID, "moe_combine: unknown dtype %d", act_dtype);
  return gg_check_launch("moe_combine");
}

extern "C" int gg_parallel_join(float* resid, const void* mixer, const void* y, const int* place, const float* wgt, int top,
                                const void* shared_out, const float* gate, long long gate_stride, const void* same, const float* bias, float mult,
                                const float* norm_w, float eps, void* h, int T, int D, int act_dtype, cudaStream_t stream) {
  GG_REQUIRE(T >= 0 && D > 0 && top >= 0, "parallel_join: bad sizes T=%d D=%d top=%d", T, D, top);
  GG_REQUIRE(resid && mixer && (top == 0 || (y && place)) && (shared_out || !gate) && (h || !norm_w), "parallel_join: a pointer is null");
  const size_t smem = norm_w ? (size_t)D * sizeof(float) : 0;
  GG_REQUIRE(smem <= 200 * 1024, "parallel_join: rows of %d values do not fit in shared memory", D);
  if (T == 0) return GG_OK;
  const size_t at = (size_t)resid | (size_t)mixer | (size_t)y | (size_t)shared_out | (size_t)same | (size_t)bias | (size_t)norm_w | (size_t)h;
  const int vec = D % 4 == 0 && at % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((D + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
#define JOIN_LAUNCH(T_)                                                                                                          \
  do {                                                                                                                           \
    if (smem > 40 * 1024) cudaFuncSetAttribute(parallel_join_kernel<T_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    gg_launch(parallel_join_kernel<T_>, dim3(T), dim3(threads), smem, stream, resid, (const T_*)mixer, (const T_*)y, place, wgt, top, \
              (const T_*)shared_out, gate, gate_stride, (const T_*)same, bias, mult, norm_w, eps, (T_*)h, D, vec);                                 \
  } while (0)
  if (act_dtype == GG_F32) JOIN_LAUNCH(float);
  else if (act_dtype == GG_BF16) JOIN_LAUNCH(__nv_bfloat16);
  else return gg_fail(GG_ERR_INVALID, "parallel_join: unknown dtype %d", act_dtype);
#undef JOIN_LAUNCH
  return gg_check_launch("parallel_join");
}
