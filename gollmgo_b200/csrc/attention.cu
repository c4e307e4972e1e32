// Attention over the paged cache: the general kernels (any head size up to 256,
// any number of heads and groups, float32 or bfloat16 cache, optional window).
//
// One tile routine serves both shapes of work:
//   * a prompt portion: up to 16 consecutive query tokens of one sequence, one head;
//   * a decoded token:  up to 16 query heads that share one kv head, one token,
//     optionally over one slice of the context (split-KV), merged afterwards.
// It streams the keys and values of [lo, hi) through shared memory 64 tokens at a
// time and keeps a running maximum, sum and output per row (online softmax), all
// in float32.  Keys come only from the cache, found through the sequence's block
// table, so a portion sees every earlier portion and never another sequence.
//
// Formulas: kernels/gollmgo_paged_attn.cu:149-223 (scores, softmax, sum of p*V;
// kv head = head / (nh/nkv); scale = 1/sqrt(d)) and :234-384 (partition + merge).
// The reference's prompt kernel (kernels/gollmgo_ops.cu:377-446) reads only the
// current call's keys and masks by position alone; this one does not share those
// two properties.
#include "attention_common.cuh"
#include <stdlib.h>

#define ATT_BQ 16
#define ATT_BK 64
#define ATT_THREADS 128

template <typename TA, int DMAX>
__device__ __forceinline__ void attn_tile(const AttnArgs& a, int nrows, const TA* const* qptr_s,
                                          const int* pos_s, const int* head_s, const float* scale_s, int kvh, const int* bt, int lo_main,
                                          int hi_main, int first_hi, float* smem, float* acc) {
  constexpr int NACC = ATT_BQ * DMAX / ATT_THREADS;
  const int d = a.d, dv = a.dv > 0 ? a.dv : a.d, ps = a.page_size;
  const int vsh = a.v_share > 1 ? a.v_share : 1, nv = a.nkv / vsh, vh = kvh / vsh;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* Qs = smem;                                  // [16][d]
  float* Ks = Qs + ATT_BQ * d;                       // [64][d+1]
  float* Vs = Ks + ATT_BK * (d + 1);                 // [64][dv]
  float* Ss = Vs + ATT_BK * dv;                      // [16][64]
  float* m_s = Ss + ATT_BQ * ATT_BK;                 // [16]
  float* l_s = m_s + ATT_BQ;                         // [16]
  float* al_s = l_s + ATT_BQ;                        // [16]
  const TA* kc = (const TA*)a.kcache;
  const TA* vc = (const TA*)a.vcache;

  for (int e = tid; e < ATT_BQ * d; e += ATT_THREADS) {
    const int r = e / d, c = e - r * d;
    Qs[e] = r < nrows ? to_f32(qptr_s[r][c]) : 0.f;
  }
  if (tid < ATT_BQ) { m_s[tid] = -INFINITY; l_s[tid] = 0.f; al_s[tid] = 1.f; }
#pragma unroll
  for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
  __syncthreads();

  // two runs of keys: the first tokens that stay visible behind the window, [0, first_hi), where
  // there are any (first_hi <= lo), then [lo, hi)
  for (int run = first_hi > 0 ? 0 : 1; run < 2; ++run) {
  const int lo = run ? lo_main : 0, hi = run ? hi_main : first_hi;
  const int kstart = (lo / ATT_BK) * ATT_BK;
  for (int kb = kstart; kb < hi; kb += ATT_BK) {
    // ---- stage keys and values of tokens [kb, kb+64)
    for (int j = warp; j < ATT_BK; j += ATT_THREADS / 32) {
      const int tok = kb + j;
      int page = -1;
      if (tok >= lo && tok < hi) page = bt[tok / ps];
      if (page >= 0) {
        const size_t base = (((size_t)page * a.nkv + kvh) * ps + (tok % ps)) * d;
        const size_t vbase = (((size_t)page * nv + vh) * ps + (tok % ps)) * dv;
        for (int c = lane; c < d; c += 32) Ks[j * (d + 1) + c] = to_f32(kc[base + c]);
        for (int c = lane; c < dv; c += 32) Vs[j * dv + c] = to_f32(vc[vbase + c]);
      } else {
        for (int c = lane; c < d; c += 32) Ks[j * (d + 1) + c] = 0.f;
        for (int c = lane; c < dv; c += 32) Vs[j * dv + c] = 0.f;
      }
    }
    __syncthreads();
    // ---- scores: thread (j = tid%64, rows tid/64 + 2i)
    {
      const int j = tid & 63, rb = tid >> 6;
      float s[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) s[i] = 0.f;
      const float* kr = Ks + j * (d + 1);
      for (int c = 0; c < d; ++c) {
        const float kv = kr[c];
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i] = fmaf(Qs[(rb + 2 * i) * d + c], kv, s[i]);
      }
      const int tok = kb + j;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = rb + 2 * i;
        const int p = pos_s[r];
        const bool ok = tok >= lo && tok < hi && tok <= p && (a.window <= 0 || tok > p - a.window || tok < a.keep_first) &&
                        (a.chunk <= 0 || tok >= (p / a.chunk) * a.chunk);
        float sc = s[i] * scale_s[r];
        if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
        if (ok && a.slopes) sc -= a.slopes[head_s[r]] * (float)(p - tok);
        if (ok && a.dist_bias) sc += a.dist_bias[(size_t)a.dist_bucket[min(p - tok, a.dist_max)] * a.nh + head_s[r]];
        if (ok && a.head_bias) sc += a.head_bias[head_s[r]];
        Ss[r * ATT_BK + j] = ok ? sc : -INFINITY;
      }
    }
    __syncthreads();
    // ---- running softmax: warp w owns rows 4w .. 4w+3
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = warp * 4 + i;
      const float s0 = Ss[r * ATT_BK + lane], s1 = Ss[r * ATT_BK + lane + 32];
      if (a.weights == 1) {                        // a weight per key on its own: no maximum, no sum, nothing to rescale
        Ss[r * ATT_BK + lane] = 1.f / (1.f + expf(-s0));
        Ss[r * ATT_BK + lane + 32] = 1.f / (1.f + expf(-s1));
        if (lane == 0) { m_s[r] = 0.f; l_s[r] = 1.f; }
        continue;
      }
      const float mx = warp_max(fmaxf(s0, s1));
      const float m_old = m_s[r];
      const float m_new = fmaxf(m_old, mx);
      float p0 = 0.f, p1 = 0.f, alpha = 1.f;
      if (m_new != -INFINITY) {
        alpha = expf(m_old - m_new);
        p0 = expf(s0 - m_new);
        p1 = expf(s1 - m_new);
      }
      const float sum = warp_sum(p0 + p1);
      Ss[r * ATT_BK + lane] = p0;
      Ss[r * ATT_BK + lane + 32] = p1;
      if (lane == 0) { m_s[r] = m_new; l_s[r] = l_s[r] * alpha + sum; al_s[r] = alpha; }
    }
    __syncthreads();
    // ---- output: thread owns elements e = tid + 128*i of the [16][d] tile
#pragma unroll
    for (int i = 0; i < NACC; ++i) {
      const int e = tid + ATT_THREADS * i;
      if (e < ATT_BQ * dv) {
        const int r = e / dv, c = e - r * dv;
        float o = acc[i] * al_s[r];
        const float* pr = Ss + r * ATT_BK;
        const float* vcol = Vs + c;
#pragma unroll 8
        for (int j = 0; j < ATT_BK; ++j) o = fmaf(pr[j], vcol[j * dv], o);
        acc[i] = o;
      }
    }
    __syncthreads();
  }
  }
}

__host__ __device__ constexpr int attn_smem_floats(int d, int dv) {
  return ATT_BQ * d + ATT_BK * (d + 1) + ATT_BK * dv + ATT_BQ * ATT_BK + 3 * ATT_BQ;
}
// where the running maximum of the rows lies in the tile's shared memory (the sums follow it)
__device__ __forceinline__ const float* attn_tile_max(const AttnArgs& a, const float* smem) {
  const int dv = a.dv > 0 ? a.dv : a.d;
  return smem + ATT_BQ * a.d + ATT_BK * (a.d + 1) + ATT_BK * dv + ATT_BQ * ATT_BK;
}

// ---------------------------------------------------------------- prompt portions
template <typename TA, int DMAX>
__global__ void __launch_bounds__(ATT_THREADS) attn_prefill_kernel(AttnArgs a) {
  constexpr int NACC = ATT_BQ * DMAX / ATT_THREADS;
  extern __shared__ float smem[];
  __shared__ const TA* qptr_s[ATT_BQ];
  __shared__ int pos_s[ATT_BQ];
  __shared__ int head_s[ATT_BQ];
  __shared__ float scale_s[ATT_BQ];
  pdl_wait();
  const int b = a.tile_seq[blockIdx.x], q0 = a.tile_q0[blockIdx.x];
  const int h = blockIdx.y, kvh = h / (a.nh / a.nkv);
  const int t0 = a.cu_q_lens[b], qlen = a.cu_q_lens[b + 1] - t0;
  const int ctx = a.context_lens[b];
  const int qstart = ctx - qlen;                 // tokens cached before this step
  const int nrows = min(ATT_BQ, qlen - q0);
  if (threadIdx.x < ATT_BQ) {
    const int r = threadIdx.x;
    qptr_s[r] = r < nrows ? (const TA*)a.q + (size_t)(t0 + q0 + r) * a.q_stride + (size_t)h * a.d : nullptr;
    pos_s[r] = r < nrows ? qstart + q0 + r : -1;
    head_s[r] = h;
    scale_s[r] = a.scale * query_temperature(a, qstart + q0 + r);
  }
  __syncthreads();
  const int first = qstart + q0, last = first + nrows - 1;
  int lo = a.window > 0 ? max(0, first - a.window + 1) : 0;
  if (a.chunk > 0) lo = max(lo, (first / a.chunk) * a.chunk);       // the chunk of the tile's first row starts earliest
  float acc[NACC];
  attn_tile<TA, DMAX>(a, nrows, qptr_s, pos_s, head_s, scale_s, kvh, a.block_tables + (size_t)b * a.bt_stride, lo, last + 1,
                      min(a.keep_first, lo), smem, acc);
  pdl_trigger();
  float* m_s = const_cast<float*>(attn_tile_max(a, smem));
  float* l_s = m_s + ATT_BQ;
  if (a.sink) {                                  // one more term of the denominator: rows rescaled to max(m, sink)
    __shared__ float sink_f[ATT_BQ];
    if (threadIdx.x < ATT_BQ) {
      const int r = threadIdx.x;
      const float sk = a.sink[h], m = m_s[r], M = fmaxf(m, sk);
      const float f = m == -INFINITY ? 0.f : expf(m - M);
      sink_f[r] = f;
      l_s[r] = l_s[r] * f + expf(sk - M);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NACC; ++i) {
      const int e = threadIdx.x + ATT_THREADS * i;
      if (e < ATT_BQ * (a.dv > 0 ? a.dv : a.d)) acc[i] *= sink_f[e / (a.dv > 0 ? a.dv : a.d)];
    }
  }
  const int dv = a.dv > 0 ? a.dv : a.d;
#pragma unroll
  for (int i = 0; i < NACC; ++i) {
    const int e = threadIdx.x + ATT_THREADS * i;
    if (e < ATT_BQ * dv) {
      const int r = e / dv, c = e - r * dv;
      if (r < nrows) {
        const size_t at = (size_t)(t0 + q0 + r) * a.nh * dv + (size_t)h * dv + c;
        if (a.out_f32) ((float*)a.out)[at] = acc[i] / l_s[r];
        else ((TA*)a.out)[at] = from_f32<TA>(acc[i] / l_s[r]);
      }
    }
  }
}

// ---------------------------------------------------------------- decoded tokens, split-KV
// grid (n_dec, nkv * ceil(G/16), num_splits).  Slice s of a context of n visible
// keys covers ceil(n/S) keys rounded up to 64.  Writes un-normalised partial
// outputs with their (max, sum); a slice without keys writes (-inf, 0).
template <typename TA, int DMAX>
__global__ void __launch_bounds__(ATT_THREADS) attn_decode_kernel(AttnArgs a) {
  constexpr int NACC = ATT_BQ * DMAX / ATT_THREADS;
  extern __shared__ float smem[];
  __shared__ const TA* qptr_s[ATT_BQ];
  __shared__ int pos_s[ATT_BQ];
  __shared__ int head_s[ATT_BQ];
  __shared__ float scale_s[ATT_BQ];
  pdl_wait();
  const int G = a.nh / a.nkv, gchunks = (G + ATT_BQ - 1) / ATT_BQ;
  const int b = a.dec_seqs[blockIdx.x];
  const int kvh = blockIdx.y / gchunks, g0 = (blockIdx.y % gchunks) * ATT_BQ;
  const int split = blockIdx.z, S = a.num_splits;
  const int nrows = min(ATT_BQ, G - g0);
  const int ctx = b >= 0 ? a.context_lens[b] : 0;      // b < 0: padding of a captured batch
  const int t = b >= 0 ? a.cu_q_lens[b] : 0;
  int lo0 = a.window > 0 ? max(0, ctx - a.window) : 0;
  if (a.chunk > 0 && ctx > 0) lo0 = max(lo0, ((ctx - 1) / a.chunk) * a.chunk);
  const int n = ctx - lo0;
  int chunk = (n + S - 1) / S;
  chunk = ((chunk + ATT_BK - 1) / ATT_BK) * ATT_BK;
  const int lo = lo0 + split * chunk, hi = min(ctx, lo + chunk);
  if (threadIdx.x < ATT_BQ) {
    const int r = threadIdx.x;
    qptr_s[r] = r < nrows ? (const TA*)a.q + (size_t)t * a.q_stride + (size_t)(kvh * G + g0 + r) * a.d : nullptr;
    pos_s[r] = r < nrows ? ctx - 1 : -1;
    head_s[r] = kvh * G + g0 + (r < nrows ? r : 0);
    scale_s[r] = a.scale * query_temperature(a, max(ctx - 1, 0));
  }
  __syncthreads();
  float acc[NACC];
  if (lo < hi) {
    // the first slice also takes the first tokens that stay visible behind the window
    attn_tile<TA, DMAX>(a, nrows, qptr_s, pos_s, head_s, scale_s, kvh, a.block_tables + (size_t)b * a.bt_stride, lo, hi,
                        split == 0 ? min(a.keep_first, lo0) : 0, smem, acc);
  } else {
#pragma unroll
    for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
  }
  pdl_trigger();
  const float* m_s = attn_tile_max(a, smem);
  const float* l_s = m_s + ATT_BQ;
  const int dv = a.dv > 0 ? a.dv : a.d;
#pragma unroll
  for (int i = 0; i < NACC; ++i) {
    const int e = threadIdx.x + ATT_THREADS * i;
    if (e < ATT_BQ * dv) {
      const int r = e / dv, c = e - r * dv;
      if (r < nrows) {
        const size_t row = ((size_t)blockIdx.x * a.nh + kvh * G + g0 + r) * S + split;
        a.part_o[row * dv + c] = acc[i];
        if (c == 0) {
          a.part_ml[row * 2] = lo < hi ? m_s[r] : -INFINITY;
          a.part_ml[row * 2 + 1] = lo < hi ? l_s[r] : 0.f;
        }
      }
    }
  }
}

// Merge of the slices: M = max m_s; o = sum_s e^{m_s-M} acc_s / sum_s e^{m_s-M} l_s
// (kernels/gollmgo_paged_attn.cu:331-384).  grid (n_dec, nh), one thread per column.
template <typename TA>
__global__ void attn_merge_kernel(AttnArgs a) {
  pdl_trigger();
  pdl_wait();
  const int b = a.dec_seqs[blockIdx.x];
  if (b < 0) return;
  const int h = blockIdx.y, S = a.num_splits, d = a.dv > 0 ? a.dv : a.d;
  const int t = a.cu_q_lens[b];
  const size_t row0 = ((size_t)blockIdx.x * a.nh + h) * S;
  float M = -INFINITY;
  for (int s = 0; s < S; ++s) M = fmaxf(M, a.part_ml[(row0 + s) * 2]);
  if (a.sink) M = fmaxf(M, a.sink[h]);
  float L = a.sink ? expf(a.sink[h] - M) : 0.f;
  for (int s = 0; s < S; ++s) {
    const float m = a.part_ml[(row0 + s) * 2];
    if (m != -INFINITY) L += expf(m - M) * a.part_ml[(row0 + s) * 2 + 1];
  }
  const size_t at = (size_t)t * a.nh * d + (size_t)h * d;
  if (a.weights == 1) {                            // weights that are not normalised: the slices' sums add up
    for (int c = threadIdx.x; c < d; c += blockDim.x) {
      float o = 0.f;
      for (int s = 0; s < S; ++s)
        if (a.part_ml[(row0 + s) * 2] != -INFINITY) o += a.part_o[(row0 + s) * d + c];
      if (a.out_f32) ((float*)a.out)[at + c] = o;
      else ((TA*)a.out)[at + c] = from_f32<TA>(o);
    }
    return;
  }
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < S; ++s) {
      const float m = a.part_ml[(row0 + s) * 2];
      if (m != -INFINITY) o += expf(m - M) * a.part_o[(row0 + s) * d + c];
    }
    o = L > 0.f ? o / L : 0.f;
    if (a.out_f32) ((float*)a.out)[at + c] = o;
    else ((TA*)a.out)[at + c] = from_f32<TA>(o);
  }
}

// ---------------------------------------------------------------- launchers
static int check_common(const AttnArgs& a, const char* who) {
  GG_REQUIRE(a.nh > 0 && a.nkv > 0 && a.nh % a.nkv == 0, "%s: %d heads are not a multiple of %d kv heads", who, a.nh, a.nkv);
  GG_REQUIRE(a.d > 0 && a.d <= 256, "%s: head size %d is outside 1..256", who, a.d);
  GG_REQUIRE(a.dv >= 0 && a.dv <= 256, "%s: value head size %d is outside 1..256", who, a.dv);
  GG_REQUIRE(a.v_share <= 1 || a.nkv % a.v_share == 0, "%s: %d key heads cannot share values %d by %d", who, a.nkv, a.v_share, a.v_share);
  GG_REQUIRE(a.page_size > 0 && a.bt_stride > 0, "%s: bad page size %d or block table width %d", who, a.page_size, a.bt_stride);
  return GG_OK;
}

template <typename K> static int set_smem(K kernel, size_t bytes, const char* who) {
  if (bytes > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "%s: %s", who, cudaGetErrorString(e));
  }
  return GG_OK;
}

#define ATT_DISPATCH(KERNEL, grid, who)                                                        \
  do {                                                                                         \
    const int dvv = a.dv > 0 ? a.dv : a.d;                                                     \
    const size_t smem = (size_t)attn_smem_floats(a.d, dvv) * sizeof(float);                    \
    int rc = GG_OK;                                                                            \
    if (dtype == GG_F32) {                                                                     \
      if (dvv <= 64) { rc = set_smem(KERNEL<float, 64>, smem, who); if (rc) return rc; gg_launch(KERNEL<float, 64>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
      else if (dvv <= 128) { rc = set_smem(KERNEL<float, 128>, smem, who); if (rc) return rc; gg_launch(KERNEL<float, 128>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
      else { rc = set_smem(KERNEL<float, 256>, smem, who); if (rc) return rc; gg_launch(KERNEL<float, 256>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
    } else if (dtype == GG_BF16) {                                                             \
      if (dvv <= 64) { rc = set_smem(KERNEL<__nv_bfloat16, 64>, smem, who); if (rc) return rc; gg_launch(KERNEL<__nv_bfloat16, 64>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
      else if (dvv <= 128) { rc = set_smem(KERNEL<__nv_bfloat16, 128>, smem, who); if (rc) return rc; gg_launch(KERNEL<__nv_bfloat16, 128>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
      else { rc = set_smem(KERNEL<__nv_bfloat16, 256>, smem, who); if (rc) return rc; gg_launch(KERNEL<__nv_bfloat16, 256>, dim3(grid), dim3(ATT_THREADS), smem, stream, a); } \
    } else {                                                                                   \
      return gg_fail(GG_ERR_INVALID, "%s: unknown dtype %d", who, dtype);                      \
    }                                                                                          \
  } while (0)

int attn_prefill_general(const AttnArgs& a, int dtype, int num_tiles, cudaStream_t stream) {
  GG_REQUIRE(num_tiles >= 0 && a.nh <= 65535, "attn_prefill: bad grid %d x %d", num_tiles, a.nh);
  if (num_tiles == 0) return GG_OK;
  dim3 grid(num_tiles, a.nh);
  ATT_DISPATCH(attn_prefill_kernel, grid, "attn_prefill");
  return gg_check_launch("attn_prefill");
}

int attn_decode_general(const AttnArgs& a, int dtype, int n_dec, cudaStream_t stream) {
  const int G = a.nh / a.nkv, gchunks = (G + ATT_BQ - 1) / ATT_BQ;
  GG_REQUIRE(a.nkv * gchunks <= 65535 && a.nh <= 65535, "attn_decode: too many heads");
  dim3 grid(n_dec, a.nkv * gchunks, a.num_splits);
  ATT_DISPATCH(attn_decode_kernel, grid, "attn_decode");
  return gg_check_launch("attn_decode");
}

int attn_merge_launch(const AttnArgs& a, int dtype, int n_dec, cudaStream_t stream) {
  dim3 mgrid(n_dec, a.nh);
  const int md = a.dv > 0 ? a.dv : a.d;
  const int mthreads = md >= 128 ? 128 : (md >= 64 ? 64 : 32);
  if (dtype == GG_F32) gg_launch(attn_merge_kernel<float>, dim3(mgrid), dim3(mthreads), 0, stream, a);
  else gg_launch(attn_merge_kernel<__nv_bfloat16>, dim3(mgrid), dim3(mthreads), 0, stream, a);
  return gg_check_launch("attn_merge");
}

// Which tcgen05 prompt kernel a launch with allow_tc = 1 runs for a shape on this build and
// device: 3 = two heads per CTA in steps of 128 keys, 2 = the same in steps of 64, 1 = one head
// per CTA, 0 = none (the mma.sync or the general kernel).
extern "C" int gg_attn_prefill_choice(int dtype, int d, int page_size, int nh, int nkv) {
  static const bool wide = !(getenv("GOLLMGO_B200_ATTN_STEP") && atoi(getenv("GOLLMGO_B200_ATTN_STEP")) == 64);
  if (wide && attn_tc3_supported(dtype, d, page_size, nh, nkv)) return 3;
  if (attn_tc2_supported(dtype, d, page_size, nh, nkv)) return 2;
  return attn_tc_supported(dtype, d, page_size) ? 1 : 0;
}

// Three tile lists describe the same portions cut into 16, 64 and 128 query rows, for the
// general kernel, the mma.sync kernel and the tcgen05 kernel; the launcher picks the kernel
// from dtype, head size and what the caller allows.  T = rows of the q buffer, num_pages =
// pages of the cache, status = the word the tcgen05 kernel reports a timed-out wait in.
extern "C" int gg_attn_prefill(const void* q, long long q_stride, const void* kcache,
                               const void* vcache, int dtype, const int* block_tables,
                               int bt_stride, const int* cu_q_lens, const int* context_lens,
                               const int* tile_seq, const int* tile_q0, int num_tiles,
                               const int* tile64_seq, const int* tile64_q0, int num_tiles64,
                               const int* tile128_seq, const int* tile128_q0, int num_tiles128,
                               void* out, int T, int num_pages, int nh, int nkv, int d, int page_size,
                               int window, float scale, int allow_mma, int allow_tc, int* status,
                               cudaStream_t stream) {
  AttnArgs a = {};
  a.q = q; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  int rc = check_common(a, "attn_prefill");
  if (rc) return rc;
  if (allow_tc && tile128_seq && status && q_stride % 8 == 0) {
    a.tile_seq = tile128_seq; a.tile_q0 = tile128_q0;
    // allow_tc: 1 = the best tcgen05 kernel for the shape, 2 = the one-head-per-CTA kernel only,
    // 3 = two heads per CTA in steps of 64 keys (what 1 gave before there were steps of 128)
    static const bool wide = !(getenv("GOLLMGO_B200_ATTN_STEP") && atoi(getenv("GOLLMGO_B200_ATTN_STEP")) == 64);
    if (allow_tc == 1 && wide && attn_tc3_supported(dtype, d, page_size, nh, nkv))
      return attn_prefill_tc3(a, num_tiles128, T, num_pages, status, stream);
    if (allow_tc != 2 && attn_tc2_supported(dtype, d, page_size, nh, nkv))
      return attn_prefill_tc2(a, num_tiles128, T, num_pages, status, stream);
    if (attn_tc_supported(dtype, d, page_size))
      return attn_prefill_tc(a, num_tiles128, T, num_pages, status, stream);
  }
  if (allow_mma && tile64_seq && attn_mma_supported(dtype, d) && q_stride % 8 == 0) {
    a.tile_seq = tile64_seq; a.tile_q0 = tile64_q0;
    return attn_prefill_mma(a, num_tiles64, stream);
  }
  a.tile_seq = tile_seq; a.tile_q0 = tile_q0;
  return attn_prefill_general(a, dtype, num_tiles, stream);
}

// Scratch the caller provides: part_o float[n_dec * nh * num_splits * d],
// part_ml float[n_dec * nh * num_splits * 2].
extern "C" int gg_attn_decode(const void* q, long long q_stride, const void* kcache,
                              const void* vcache, int dtype, const int* block_tables,
                              int bt_stride, const int* cu_q_lens, const int* context_lens,
                              const int* dec_seqs, int n_dec, int num_splits, float* part_o,
                              float* part_ml, void* out, int nh, int nkv, int d, int page_size,
                              int window, float scale, int allow_mma, cudaStream_t stream) {
  AttnArgs a = {};
  a.q = q; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  a.dec_seqs = dec_seqs; a.num_splits = num_splits; a.part_o = part_o; a.part_ml = part_ml;
  int rc = check_common(a, "attn_decode");
  if (rc) return rc;
  GG_REQUIRE(n_dec >= 0 && num_splits >= 1 && num_splits <= 65535, "attn_decode: bad n_dec %d or splits %d", n_dec, num_splits);
  GG_REQUIRE(part_o && part_ml, "attn_decode: no scratch given");
  if (n_dec == 0) return GG_OK;
  bool merged = false;
  if (allow_mma && attn_mma_supported(dtype, d) && q_stride % 2 == 0)
    rc = attn_decode_mma(a, n_dec, stream, &merged);
  else
    rc = attn_decode_general(a, dtype, n_dec, stream);
  if (rc || merged) return rc;
  return attn_merge_launch(a, dtype, n_dec, stream);
}

// gg_attn_decode with the work of gg_rope_kv_write for the same tokens folded in: q is the raw
// projection output [T, (nh + 2 nkv) * d] (left as it is), the kernel rotates q and k with
// half-split pairs over the whole head and writes k and v into the cache at slot_mapping[t]
// (write_cache = 0: rotates q only).  Frequencies of zero turn nothing (a cosine of exactly 1): an attention
// without rotation.  sink, slopes and the query temperature as in gg_attn_decode_x.  bfloat16, head sizes 64 and 128, at most 16 heads per
// kv head; anything else is refused.
extern "C" int gg_attn_decode_rope(const void* qkv, long long q_stride, void* kcache, void* vcache, int dtype,
                                   const int* block_tables, int bt_stride, const int* cu_q_lens,
                                   const int* context_lens, const int* dec_seqs, int n_dec, int num_splits,
                                   float* part_o, float* part_ml, void* out, int nh, int nkv, int d,
                                   int page_size, int window, float scale, const int* positions,
                                   const int* slot_mapping, const double* inv_freq, int write_cache,
                                   const float* sink, const float* slopes, float temp_coef, float temp_every,
                                   cudaStream_t stream) {
  AttnArgs a = {};
  a.q = qkv; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  a.dec_seqs = dec_seqs; a.num_splits = num_splits; a.part_o = part_o; a.part_ml = part_ml;
  a.rope_inv_freq = inv_freq; a.rope_positions = positions; a.slot_mapping = slot_mapping;
  a.rope_write_cache = write_cache;
  a.sink = sink; a.slopes = slopes; a.temp_coef = temp_coef; a.temp_every = temp_every;
  int rc = check_common(a, "attn_decode_rope");
  if (rc) return rc;
  GG_REQUIRE(n_dec >= 0 && num_splits >= 1 && num_splits <= 65535, "attn_decode_rope: bad n_dec %d or splits %d", n_dec, num_splits);
  GG_REQUIRE(part_o && part_ml, "attn_decode_rope: no scratch given");
  GG_REQUIRE(inv_freq != nullptr, "attn_decode_rope: no inverse frequencies given");
  GG_REQUIRE(attn_mma_supported(dtype, d), "attn_decode_rope: only bfloat16 with head size 64 or 128 (got dtype %d, head size %d)", dtype, d);
  if (n_dec == 0) return GG_OK;
  bool merged = false;
  rc = attn_decode_mma(a, n_dec, stream, &merged);
  if (rc || merged) return rc;
  return attn_merge_launch(a, dtype, n_dec, stream);
}

// Decode attention for large batches (bfloat16, head size 64 or 128): the work is cut into
// equal ranges of tiles instead of whole slices (attention_mma.cu).  Scratch the caller
// provides: pieces = n_dec * nkv * ceil((nh / nkv) / 16) + gg_attn_decode_flat_ctas(d);
// part_o float[pieces * 16 * d], part_ml float[pieces * 16 * 2], prefix int[prefix_ints] with
// prefix_ints >= n_dec + 1 + 2 * n_dec * nkv * ceil((nh / nkv) / 16).
extern "C" int gg_attn_decode_flat(const void* q, long long q_stride, const void* kcache, const void* vcache,
                                   int dtype, const int* block_tables, int bt_stride, const int* cu_q_lens,
                                   const int* context_lens, const int* dec_seqs, int n_dec, float* part_o,
                                   float* part_ml, int* prefix, int prefix_ints, void* out, int nh, int nkv, int d,
                                   int page_size, int window, float scale, cudaStream_t stream) {
  AttnArgs a = {};
  a.q = q; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  a.dec_seqs = dec_seqs; a.num_splits = 0; a.part_o = part_o; a.part_ml = part_ml;
  int rc = check_common(a, "attn_decode_flat");
  if (rc) return rc;
  GG_REQUIRE(n_dec >= 0, "attn_decode_flat: bad n_dec %d", n_dec);
  GG_REQUIRE(part_o && part_ml && prefix, "attn_decode_flat: no scratch given");
  GG_REQUIRE(nkv > 0 && nh >= nkv && (long long)prefix_ints >= (long long)n_dec + 1 + 2LL * n_dec * nkv * ((nh / nkv + 15) / 16),
             "attn_decode_flat: prefix scratch of %d ints is too small for %d tokens", prefix_ints, n_dec);
  GG_REQUIRE(attn_mma_supported(dtype, d) && q_stride % 2 == 0,
             "attn_decode_flat: only bfloat16 with head size 64 or 128 (got dtype %d, head size %d)", dtype, d);
  if (n_dec == 0) return GG_OK;
  return attn_decode_flat(a, n_dec, prefix, stream);
}

extern "C" int gg_attn_decode_flat_ctas(int d) { return attn_decode_flat_ctas(d); }

// Clusters of `splits` decode CTAs that the device holds at once for head size d in
// bfloat16 with `group` query heads to a kv head; 0 where gg_attn_decode would not use
// clusters for that count.
extern "C" int gg_attn_decode_cluster_capacity(int dtype, int d, int splits, int group) {
  if (!attn_mma_supported(dtype, d)) return 0;
  return attn_decode_cluster_capacity(d, splits, group);
}

extern "C" int gg_attn_mma_x_chunk_sink() { return attn_mma_x_chunk_sink_supported() ? 1 : 0; }

// The general kernels with everything they take: keys of size d and values of size dv, `v_share`
// consecutive key heads reading one value head (vcache [num_pages, nkv / v_share, page_size, dv]),
// scores capped by softcap * tanh(score / softcap) where softcap > 0, the result in float32 where
// out_f32.  Float32 arithmetic whatever the cache's type.  part_o float[n_dec * nh * num_splits * dv].
extern "C" int gg_attn_prefill_x(const void* q, long long q_stride, const void* kcache, const void* vcache,
                                 int dtype, const int* block_tables, int bt_stride, const int* cu_q_lens,
                                 const int* context_lens, const int* tile_seq, const int* tile_q0, int num_tiles,
                                 const int* tile64_seq, const int* tile64_q0, int num_tiles64, int allow_mma,
                                 void* out, int out_f32, int nh, int nkv, int d, int dv, int v_share,
                                 int page_size, int window, float scale, float softcap, int keep_first, int weights,
                                 const float* head_bias, const float* dist_bias, const int* dist_bucket, int dist_max, int chunk, const float* sink,
                                 const float* slopes, float temp_coef, float temp_every, cudaStream_t stream) {
  AttnArgs a = {};
  a.q = q; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  a.dv = dv; a.v_share = v_share; a.softcap = softcap; a.out_f32 = out_f32;
  a.tile_seq = tile_seq; a.tile_q0 = tile_q0;
  a.keep_first = window > 0 ? keep_first : 0; a.weights = weights; a.head_bias = head_bias;
  a.dist_bias = dist_bias; a.dist_bucket = dist_bucket; a.dist_max = dist_max;
  a.chunk = chunk > 0 ? chunk : 0; a.sink = sink;
  a.slopes = slopes; a.temp_coef = temp_coef; a.temp_every = temp_every;
  int rc = check_common(a, "attn_prefill_x");
  if (rc) return rc;
  GG_REQUIRE(weights == 0 || weights == 1, "attn_prefill_x: unknown kind of weights %d", weights);
  GG_REQUIRE(!dist_bias || (dist_bucket && dist_max >= 0), "attn_prefill_x: a distance bias needs its bucket table");
  GG_REQUIRE(!(weights && (a.chunk || sink || slopes || temp_every > 0.f)), "attn_prefill_x: chunks, a sink, slopes and a query temperature go with softmax weights");
  // what the mma.sync kernels compute: softmax without these extras, or sigmoid weights with all of them
  const bool plain = (!a.keep_first && !weights && !head_bias && !dist_bias) || attn_mma_x_sigmoid_supported(a);
  if (a.chunk || a.sink) allow_mma = allow_mma && attn_mma_x_chunk_sink_supported();
  // bfloat16 with sizes of 64 or 128: the mma.sync kernel over tiles of 64 queries
  if (plain && allow_mma && tile64_seq && attn_mma_x_supported(dtype, d, dv > 0 ? dv : d, page_size) && q_stride % 8 == 0) {
    a.tile_seq = tile64_seq; a.tile_q0 = tile64_q0;
    return attn_prefill_mma_x(a, num_tiles64, stream);
  }
  return attn_prefill_general(a, dtype, num_tiles, stream);
}

extern "C" int gg_attn_decode_x(const void* q, long long q_stride, const void* kcache, const void* vcache,
                                int dtype, const int* block_tables, int bt_stride, const int* cu_q_lens,
                                const int* context_lens, const int* dec_seqs, int n_dec, int num_splits,
                                float* part_o, float* part_ml, void* out, int out_f32, int nh, int nkv, int d,
                                int dv, int v_share, int page_size, int window, float scale, float softcap,
                                int allow_mma, int keep_first, int weights, const float* head_bias,
                                const float* dist_bias, const int* dist_bucket, int dist_max, int chunk, const float* sink,
                                const float* slopes, float temp_coef, float temp_every, cudaStream_t stream) {
  AttnArgs a = {};
  a.q = q; a.q_stride = q_stride; a.kcache = kcache; a.vcache = vcache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_q_lens = cu_q_lens;
  a.context_lens = context_lens; a.out = out; a.nh = nh; a.nkv = nkv; a.d = d;
  a.page_size = page_size; a.window = window; a.scale = scale;
  a.dv = dv; a.v_share = v_share; a.softcap = softcap; a.out_f32 = out_f32;
  a.dec_seqs = dec_seqs; a.num_splits = num_splits; a.part_o = part_o; a.part_ml = part_ml;
  a.keep_first = window > 0 ? keep_first : 0; a.weights = weights; a.head_bias = head_bias;
  a.dist_bias = dist_bias; a.dist_bucket = dist_bucket; a.dist_max = dist_max;
  a.chunk = chunk > 0 ? chunk : 0; a.sink = sink;
  a.slopes = slopes; a.temp_coef = temp_coef; a.temp_every = temp_every;
  int rc = check_common(a, "attn_decode_x");
  if (rc) return rc;
  GG_REQUIRE(weights == 0 || weights == 1, "attn_decode_x: unknown kind of weights %d", weights);
  GG_REQUIRE(!dist_bias || (dist_bucket && dist_max >= 0), "attn_decode_x: a distance bias needs its bucket table");
  GG_REQUIRE(!(weights && (a.chunk || sink || slopes || temp_every > 0.f)), "attn_decode_x: chunks, a sink, slopes and a query temperature go with softmax weights");
  if ((a.keep_first || weights || head_bias || dist_bias) && !attn_mma_x_sigmoid_supported(a))
    allow_mma = 0;                                                            // only the general kernel has these with softmax
  if (a.chunk) allow_mma = allow_mma && attn_mma_x_chunk_sink_supported();     // (the sink is the merge kernel's)
  GG_REQUIRE(n_dec >= 0 && num_splits >= 1 && num_splits <= 65535, "attn_decode_x: bad n_dec %d or splits %d", n_dec, num_splits);
  GG_REQUIRE(part_o && part_ml, "attn_decode_x: no scratch given");
  if (n_dec == 0) return GG_OK;
  if (allow_mma && attn_mma_x_supported(dtype, d, dv > 0 ? dv : d, page_size) && q_stride % 8 == 0)
    rc = attn_decode_mma_x(a, n_dec, stream);
  else
    rc = attn_decode_general(a, dtype, n_dec, stream);
  if (rc) return rc;
  return attn_merge_launch(a, dtype, n_dec, stream);
}
