// Many small products with one launch: out_g = A_g @ W_g^T for groups g = 0 .. G-1, where a
// group is an expert of a mixture (its rows are the tokens routed to it, found through an
// offsets table and a row list made on the device) or a head of an attention layer (every group
// has all rows, and reads and writes its own columns of A and out).
//
//   rows of group g:  [offsets[g], offsets[g+1])   (offsets given)   or   [0, M)   (no offsets)
//   A row of row r:   row_index ? row_index[r] / row_div : r;   group g reads columns
//                     [g * a_group_cols, g * a_group_cols + K) of it
//   W_g:              [N, K] row-major ([2N, K] if gated: gate rows, then up rows) at W + g * rows * K
//   out row r, columns [g * o_group_cols, g * o_group_cols + Np): the N results, then zeros
//   epilogue:         gated = 1: silu(x Wg^T) * (x Wu^T);   gated = 2: the square of relu(x W^T);   gate given: the row is multiplied by
//                     sigmoid(gate[A row, gate_col0 + g])   (an output gate per head);
//                     row_scale given: row r's products are multiplied by row_scale[row_index ? row_index[r] : r]
//                     before the activation (a factor on the input row, without rounding the row again)
//
// No host code learns how many rows a group has: the grid is sized for the worst case and a CTA
// whose tile lies past its group's rows returns.  A row's result depends on that row and on W_g
// alone (fixed order over K), so it is the same wherever the row lands in its group's list.
// bfloat16: tensor cores through wmma 16x16x16 with float32 accumulators; float32: FMA.  Tiles
// of 32 rows x 64 columns, K in steps through shared memory, any N and K.  This is the kernel for
// few rows per group (decoded tokens, heads of short steps) and for float32; long prompt steps
// of a mixture of experts in bfloat16 go through the tcgen05 product instead (gemm_tc.cu,
// gg_gemm_tc_grouped).
#include <mma.h>

#include <stdlib.h>

#include <type_traits>

#include "attention_common.cuh"

#define GGM_BM 32
#define GGM_BN 64
#define GGM_LDC (GGM_BN + 8)
#define GGM_THREADS 256

struct GroupedArgs {
  const void* A; long long lda; long long a_group_cols;
  const int* row_index; int row_div;
  const void* W;
  void* out; long long ldo; long long o_group_cols;
  const int* offsets;
  int M, G, N, K, Np, relu2;
  const void* gate; long long ldg; int gate_col0;
  const float* row_scale;
};

template <typename TA> struct GgmZero;
template <> struct GgmZero<float> { static __device__ __forceinline__ float v() { return 0.f; } };
template <> struct GgmZero<__nv_bfloat16> { static __device__ __forceinline__ __nv_bfloat16 v() { return __float2bfloat16_rn(0.f); } };

// K is walked in steps of BK (128 for bfloat16, 32 for float32).  VEC: every row of A and W
// starts on a 16-byte boundary and K is a multiple of the 16-byte chunk, so tiles are fetched
// in chunks of 16 bytes, and the chunks of the next step are asked for (into registers) before
// the products of this one, which hides most of a trip to memory when a group has only a few
// rows and the kernel streams its weights (decoded tokens).
template <typename TA, bool GATED, int BK, bool VEC>
__global__ void __launch_bounds__(GGM_THREADS, (sizeof(TA) == 2 ? (GATED ? 2 : 4) : 1)) grouped_gemm_kernel(GroupedArgs a) {
  constexpr int LD = BK + 8;
  constexpr int NB = GATED ? 2 : 1;
  constexpr int VPT = 16 / (int)sizeof(TA);                     // values in a 16-byte chunk
  constexpr int CPR = BK / VPT;                                 // chunks in a tile row
  constexpr int A_CH = GGM_BM * CPR / GGM_THREADS, B_CH = GGM_BN * CPR / GGM_THREADS;
  static_assert(GGM_BM * CPR % GGM_THREADS == 0 && GGM_BN * CPR % GGM_THREADS == 0, "tile chunks must divide over the threads");
  constexpr int AB_BYTES = (GGM_BM + NB * GGM_BN) * LD * (int)sizeof(TA);
  constexpr int C_BYTES = NB * GGM_BM * GGM_LDC * (int)sizeof(float);
  __shared__ __align__(32) unsigned char raw[AB_BYTES > C_BYTES ? AB_BYTES : C_BYTES];
  __shared__ int arow_s[GGM_BM];
  __shared__ float scale_s[GGM_BM];
  TA* As = reinterpret_cast<TA*>(raw);
  TA* Bs = As + GGM_BM * LD;                                    // [NB][GGM_BN * LD]
  float* Cs = reinterpret_cast<float*>(raw);                    // [NB][GGM_BM * GGM_LDC], over the tiles once they are used up
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  int g = -1, r0 = 0, r_end = 0;
  if (a.offsets) {
    int tile = blockIdx.y;
    for (int e = 0; e < a.G; ++e) {
      const int lo = a.offsets[e], hi = a.offsets[e + 1];
      const int nt = (hi - lo + GGM_BM - 1) / GGM_BM;
      if (tile < nt) { g = e; r0 = lo + tile * GGM_BM; r_end = hi; break; }
      tile -= nt;
    }
    if (g < 0) return;
  } else {
    g = blockIdx.z; r0 = blockIdx.y * GGM_BM; r_end = a.M;
    if (r0 >= r_end) return;
  }
  const int n0 = blockIdx.x * GGM_BN;
  const int nrows = min(GGM_BM, r_end - r0);
  if (tid < GGM_BM) {
    const int entry = tid < nrows ? (a.row_index ? a.row_index[r0 + tid] : r0 + tid) : -1;
    arow_s[tid] = entry < 0 ? -1 : (a.row_index ? entry / a.row_div : entry);
    scale_s[tid] = entry >= 0 && a.row_scale ? a.row_scale[entry] : 1.f;
  }
  __syncthreads();
  const int N = a.N, K = a.K;
  const TA* A = (const TA*)a.A + (size_t)g * a.a_group_cols;
  const TA* W = (const TA*)a.W + (size_t)g * NB * N * K;
  const TA zero = GgmZero<TA>::v();

  constexpr bool TC = !std::is_same<TA, float>::value;
  const int warp = tid >> 5;
  const int rt = warp >> 2, ct = warp & 3;                 // tensor cores: the warp's 16 x 16 tile
  const int frow = tid >> 3, fcg = tid & 7;                // FMA: row, and columns fcg + 8 j
  nvcuda::wmma::fragment<nvcuda::wmma::accumulator, 16, 16, 16, float> acc0, acc1;
  float f0[8], f1[8];
  if (TC) {
    nvcuda::wmma::fill_fragment(acc0, 0.f);
    nvcuda::wmma::fill_fragment(acc1, 0.f);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) { f0[j] = 0.f; f1[j] = 0.f; }
  }

  uint4 ra[A_CH], rb[NB][B_CH];
  auto fetch = [&](int k0) {                               // VEC: this step's chunks into registers
#pragma unroll
    for (int u = 0; u < A_CH; ++u) {
      const int e = tid + u * GGM_THREADS, r = e / CPR, k = k0 + (e - r * CPR) * VPT;
      const int row = arow_s[r];
      ra[u] = (row >= 0 && k < K) ? *reinterpret_cast<const uint4*>(A + (size_t)row * a.lda + k) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int u = 0; u < B_CH; ++u) {
      const int e = tid + u * GGM_THREADS, n = e / CPR, k = k0 + (e - n * CPR) * VPT;
      const bool ok = n0 + n < N && k < K;
      rb[0][u] = ok ? *reinterpret_cast<const uint4*>(W + (size_t)(n0 + n) * K + k) : make_uint4(0, 0, 0, 0);
      if (GATED) rb[NB - 1][u] = ok ? *reinterpret_cast<const uint4*>(W + (size_t)(N + n0 + n) * K + k) : make_uint4(0, 0, 0, 0);
    }
  };
  auto stash = [&]() {                                     // VEC: the registers into the shared tiles
#pragma unroll
    for (int u = 0; u < A_CH; ++u) {
      const int e = tid + u * GGM_THREADS, r = e / CPR, c = (e - r * CPR) * VPT;
      *reinterpret_cast<uint4*>(As + r * LD + c) = ra[u];
    }
#pragma unroll
    for (int u = 0; u < B_CH; ++u) {
      const int e = tid + u * GGM_THREADS, n = e / CPR, c = (e - n * CPR) * VPT;
      *reinterpret_cast<uint4*>(Bs + n * LD + c) = rb[0][u];
      if (GATED) *reinterpret_cast<uint4*>(Bs + (NB - 1) * GGM_BN * LD + n * LD + c) = rb[NB - 1][u];
    }
  };
  if (VEC) fetch(0);
  for (int k0 = 0; k0 < K; k0 += BK) {
    if (VEC) {
      stash();
    } else {
      for (int e = tid; e < GGM_BM * BK; e += GGM_THREADS) {
        const int r = e / BK, c = e - r * BK;
        const int row = arow_s[r], k = k0 + c;
        As[r * LD + c] = (row >= 0 && k < K) ? A[(size_t)row * a.lda + k] : zero;
      }
      for (int e = tid; e < GGM_BN * BK; e += GGM_THREADS) {
        const int n = e / BK, c = e - n * BK;
        const int col = n0 + n, k = k0 + c;
        const bool ok = col < N && k < K;
        Bs[n * LD + c] = ok ? W[(size_t)col * K + k] : zero;
        if (GATED) Bs[(NB - 1) * GGM_BN * LD + n * LD + c] = ok ? W[(size_t)(N + col) * K + k] : zero;
      }
    }
    __syncthreads();
    if (VEC && k0 + BK < K) fetch(k0 + BK);
    if constexpr (TC) {
      using namespace nvcuda;
      wmma::fragment<wmma::matrix_a, 16, 16, 16, __nv_bfloat16, wmma::row_major> fa;
      wmma::fragment<wmma::matrix_b, 16, 16, 16, __nv_bfloat16, wmma::col_major> fb;
#pragma unroll
      for (int kk = 0; kk < BK; kk += 16) {
        wmma::load_matrix_sync(fa, As + rt * 16 * LD + kk, LD);
        wmma::load_matrix_sync(fb, Bs + ct * 16 * LD + kk, LD);
        wmma::mma_sync(acc0, fa, fb, acc0);
        if (GATED) {
          wmma::load_matrix_sync(fb, Bs + (NB - 1) * GGM_BN * LD + ct * 16 * LD + kk, LD);
          wmma::mma_sync(acc1, fa, fb, acc1);
        }
      }
    } else {
#pragma unroll 8
      for (int k = 0; k < BK; ++k) {
        const float av = As[frow * LD + k];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          f0[j] = fmaf(av, Bs[(fcg + 8 * j) * LD + k], f0[j]);
          if (GATED) f1[j] = fmaf(av, Bs[(NB - 1) * GGM_BN * LD + (fcg + 8 * j) * LD + k], f1[j]);
        }
      }
    }
    __syncthreads();
  }
  float* Cs1 = Cs + (NB - 1) * GGM_BM * GGM_LDC;
  if constexpr (TC) {
    nvcuda::wmma::store_matrix_sync(Cs + rt * 16 * GGM_LDC + ct * 16, acc0, GGM_LDC, nvcuda::wmma::mem_row_major);
    if (GATED) nvcuda::wmma::store_matrix_sync(Cs1 + rt * 16 * GGM_LDC + ct * 16, acc1, GGM_LDC, nvcuda::wmma::mem_row_major);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      Cs[frow * GGM_LDC + fcg + 8 * j] = f0[j];
      if (GATED) Cs1[frow * GGM_LDC + fcg + 8 * j] = f1[j];
    }
  }
  __syncthreads();
  TA* out = (TA*)a.out + (size_t)g * a.o_group_cols;
  for (int e = tid; e < GGM_BM * GGM_BN; e += GGM_THREADS) {
    const int r = e / GGM_BN, c = e - r * GGM_BN;
    const int col = n0 + c;
    if (r >= nrows || col >= a.Np) continue;
    float v = 0.f;
    if (col < N) {
      v = Cs[r * GGM_LDC + c] * scale_s[r];
      if (GATED) {
        const float u = Cs1[r * GGM_LDC + c] * scale_s[r];
        v = v / (1.f + expf(-v)) * u;
      } else if (a.relu2) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      if (a.gate) {
        const float z = to_f32(((const TA*)a.gate)[(size_t)arow_s[r] * a.ldg + a.gate_col0 + g]);
        v *= 1.f / (1.f + expf(-z));
      }
    }
    out[(size_t)(r0 + r) * a.ldo + col] = from_f32<TA>(v);
  }
}

// The same product for bfloat16 with long K (the experts' products of decoded tokens, where a CTA
// streams its slab of W and the rows are few): K in steps of 64 through a ring of four shared-memory
// stages filled by cp.async, so that three steps of a CTA are in flight while it multiplies the
// fourth; two CTAs per SM.  Rows past a group's end and columns past N or K arrive as zeros
// (cp.async with a source size of 0).  Needs what VEC needs.
#define GGR_BK 64
#define GGR_LD (GGR_BK + 8)
#define GGR_STAGES 4

template <bool GATED>
__global__ void __launch_bounds__(GGM_THREADS, 2) grouped_gemm_ring_kernel(GroupedArgs a) {
  using TA = __nv_bfloat16;
  constexpr int NB = GATED ? 2 : 1;
  constexpr int CPR = GGR_BK / 8;                                // 16-byte chunks in a tile row
  constexpr int A_ELEMS = GGM_BM * GGR_LD, B_ELEMS = GGM_BN * GGR_LD;
  constexpr int STAGE_ELEMS = A_ELEMS + NB * B_ELEMS;
  extern __shared__ __align__(128) unsigned char ring_raw[];
  __shared__ int arow_s[GGM_BM];
  __shared__ float scale_s[GGM_BM];
  TA* stages = reinterpret_cast<TA*>(ring_raw);
  float* Cs = reinterpret_cast<float*>(ring_raw);                // over the ring once it has drained
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  int g = -1, r0 = 0, r_end = 0;
  if (a.offsets) {
    int tile = blockIdx.y;
    for (int e = 0; e < a.G; ++e) {
      const int lo = a.offsets[e], hi = a.offsets[e + 1];
      const int nt = (hi - lo + GGM_BM - 1) / GGM_BM;
      if (tile < nt) { g = e; r0 = lo + tile * GGM_BM; r_end = hi; break; }
      tile -= nt;
    }
    if (g < 0) return;
  } else {
    g = blockIdx.z; r0 = blockIdx.y * GGM_BM; r_end = a.M;
    if (r0 >= r_end) return;
  }
  const int n0 = blockIdx.x * GGM_BN;
  const int nrows = min(GGM_BM, r_end - r0);
  if (tid < GGM_BM) {
    const int entry = tid < nrows ? (a.row_index ? a.row_index[r0 + tid] : r0 + tid) : -1;
    arow_s[tid] = entry < 0 ? -1 : (a.row_index ? entry / a.row_div : entry);
    scale_s[tid] = entry >= 0 && a.row_scale ? a.row_scale[entry] : 1.f;
  }
  __syncthreads();
  const int N = a.N, K = a.K;
  const TA* A = (const TA*)a.A + (size_t)g * a.a_group_cols;
  const TA* W = (const TA*)a.W + (size_t)g * NB * N * K;

  // what this thread fetches in every step: one chunk of A, two of each W tile
  const int ar = tid / CPR, ac = (tid % CPR) * 8;
  const int arow = arow_s[ar];
  const TA* a_src = A + (size_t)(arow >= 0 ? arow : 0) * a.lda + ac;
  const TA* b_src[2];
  bool b_ok[2];
  int b_off[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int e = tid + u * GGM_THREADS, n = e / CPR, c = (e % CPR) * 8;
    b_ok[u] = n0 + n < N;
    b_src[u] = W + (size_t)(b_ok[u] ? n0 + n : 0) * K + c;
    b_off[u] = n * GGR_LD + c;
  }
  auto issue = [&](int stage, int k0) {
    TA* As = stages + stage * STAGE_ELEMS;
    TA* Bs = As + A_ELEMS;
    const bool kin = k0 + ac < K;
    cp_async16(smem_u32(As + ar * GGR_LD + ac), kin ? a_src + k0 : A, (arow >= 0 && kin) ? 16 : 0);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int c = (tid + u * GGM_THREADS) % CPR * 8;
      const bool ok = b_ok[u] && k0 + c < K;
      cp_async16(smem_u32(Bs + b_off[u]), ok ? b_src[u] + k0 : W, ok ? 16 : 0);
      if (GATED) cp_async16(smem_u32(Bs + B_ELEMS + b_off[u]), ok ? b_src[u] + (size_t)N * K + k0 : W, ok ? 16 : 0);
    }
  };

  const int warp = tid >> 5, rt = warp >> 2, ct = warp & 3;
  nvcuda::wmma::fragment<nvcuda::wmma::accumulator, 16, 16, 16, float> acc0, acc1;
  nvcuda::wmma::fill_fragment(acc0, 0.f);
  nvcuda::wmma::fill_fragment(acc1, 0.f);
  const int nk = (K + GGR_BK - 1) / GGR_BK;
#pragma unroll
  for (int s = 0; s < GGR_STAGES - 1; ++s) {
    if (s < nk) issue(s, s * GGR_BK);
    cp_async_commit();
  }
  for (int it = 0; it < nk; ++it) {
    cp_async_wait<GGR_STAGES - 2>();                             // this step's stage has landed
    __syncthreads();                                             // ... for every thread; and the stage refilled below is used up
    const int nxt = it + GGR_STAGES - 1;
    if (nxt < nk) issue(nxt % GGR_STAGES, nxt * GGR_BK);
    cp_async_commit();
    const TA* As = stages + (it % GGR_STAGES) * STAGE_ELEMS;
    const TA* Bs = As + A_ELEMS;
    using namespace nvcuda;
    wmma::fragment<wmma::matrix_a, 16, 16, 16, __nv_bfloat16, wmma::row_major> fa;
    wmma::fragment<wmma::matrix_b, 16, 16, 16, __nv_bfloat16, wmma::col_major> fb;
#pragma unroll
    for (int kk = 0; kk < GGR_BK; kk += 16) {
      wmma::load_matrix_sync(fa, As + rt * 16 * GGR_LD + kk, GGR_LD);
      wmma::load_matrix_sync(fb, Bs + ct * 16 * GGR_LD + kk, GGR_LD);
      wmma::mma_sync(acc0, fa, fb, acc0);
      if (GATED) {
        wmma::load_matrix_sync(fb, Bs + B_ELEMS + ct * 16 * GGR_LD + kk, GGR_LD);
        wmma::mma_sync(acc1, fa, fb, acc1);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  float* Cs1 = Cs + (NB - 1) * GGM_BM * GGM_LDC;
  nvcuda::wmma::store_matrix_sync(Cs + rt * 16 * GGM_LDC + ct * 16, acc0, GGM_LDC, nvcuda::wmma::mem_row_major);
  if (GATED) nvcuda::wmma::store_matrix_sync(Cs1 + rt * 16 * GGM_LDC + ct * 16, acc1, GGM_LDC, nvcuda::wmma::mem_row_major);
  __syncthreads();
  TA* out = (TA*)a.out + (size_t)g * a.o_group_cols;
  for (int e = tid; e < GGM_BM * GGM_BN; e += GGM_THREADS) {
    const int r = e / GGM_BN, c = e - r * GGM_BN;
    const int col = n0 + c;
    if (r >= nrows || col >= a.Np) continue;
    float v = 0.f;
    if (col < N) {
      v = Cs[r * GGM_LDC + c] * scale_s[r];
      if (GATED) {
        const float u = Cs1[r * GGM_LDC + c] * scale_s[r];
        v = v / (1.f + expf(-v)) * u;
      } else if (a.relu2) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      if (a.gate) {
        const float z = to_f32(((const TA*)a.gate)[(size_t)arow_s[r] * a.ldg + a.gate_col0 + g]);
        v *= 1.f / (1.f + expf(-z));
      }
    }
    out[(size_t)(r0 + r) * a.ldo + col] = from_f32<TA>(v);
  }
}

// ---------------------------------------------------------------- few rows per group: streaming the weights
// The experts' products of decoded tokens once more, as gemm_small_m.cu does a product of a few tokens: rows of W are
// the M side of mma.sync m16n8k16 and a group's rows the N side (8 NT of them at a time), a lane copies 16-byte chunks
// of its two rows of W into a private ring of shared memory several steps ahead and feeds each to the instruction, the
// eight warps of a CTA take interleaved spans of K and are summed in a fixed order.  A CTA walks over units of GROUP
// tiles of 16 rows of W (8 gate and 8 up rows if gated) of the groups that have rows, in steps of the grid, its ring
// running across their borders; a group with more than 8 NT rows is walked once for every 8 NT of them.  Which groups
// have rows is known on the device alone: every CTA makes the list from the offsets.
#define GGS_WARPS 8
#define GGS_THREADS (GGS_WARPS * 32)
#define GGS_SPAN 64
#define GGS_STAGES 5
#define GGS_MAX_ENTRIES 256            // (group, first row) pairs with rows
#define GGS_MAX_ROWS 1024

template <bool GATED, int NT, int GROUP, int XB>
__global__ void __launch_bounds__(GGS_THREADS, 2) grouped_stream_kernel(GroupedArgs a) {
  constexpr int PASS = 8 * NT;
  extern __shared__ __align__(16) unsigned char ggs_smem[];
  uint4* ring = reinterpret_cast<uint4*>(ggs_smem);                                   // [warps][stages][4][32]
  float (*red)[16][PASS + 1] = reinterpret_cast<float (*)[16][PASS + 1]>(ggs_smem + (size_t)GGS_WARPS * GGS_STAGES * 4 * 32 * 16);
  int* arow_s = reinterpret_cast<int*>(red + GGS_WARPS);                              // [M]
  float* scale_s = reinterpret_cast<float*>(arow_s + a.M);                            // [M]
  __shared__ int ent_g[GGS_MAX_ENTRIES], ent_r[GGS_MAX_ENTRIES], ent_n[GGS_MAX_ENTRIES];
  __shared__ int entries_s;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const int N = a.N, K = a.K;
  const int iters = K > warp * GGS_SPAN ? (K - warp * GGS_SPAN + GGS_WARPS * GGS_SPAN - 1) / (GGS_WARPS * GGS_SPAN) : 0;
  const int tiles = GATED ? (N + 7) / 8 : (N + 15) / 16;                              // of one group
  const int upe = (tiles + GROUP - 1) / GROUP;                                        // units of one list entry
  const unsigned ring_base = smem_u32(ring) + (unsigned)((warp * GGS_STAGES * 4 * 32 + lane) * 16);
  const __nv_bfloat16* A = (const __nv_bfloat16*)a.A;
  const __nv_bfloat16* W = (const __nv_bfloat16*)a.W;
  pdl_trigger();
  pdl_wait();
  if (warp == 0) {
    int run = 0;
    for (int e0 = 0; e0 < a.G; e0 += 32) {
      const int e = e0 + lane;
      const int lo = e < a.G ? a.offsets[e] : 0, hi = e < a.G ? a.offsets[e + 1] : 0;
      const int cnt = (hi - lo + PASS - 1) / PASS;
      int at = cnt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, at, o); if (lane >= o) at += v; }
      const int total = __shfl_sync(0xffffffffu, at, 31);
      at += run - cnt;
      for (int i = 0; i < cnt; ++i)
        if (at + i < GGS_MAX_ENTRIES) { ent_g[at + i] = e; ent_r[at + i] = lo + i * PASS; ent_n[at + i] = min(PASS, hi - lo - i * PASS); }
      run += total;
    }
    if (lane == 0) entries_s = min(run, GGS_MAX_ENTRIES);
  }
  for (int r = threadIdx.x; r < a.M; r += GGS_THREADS) {
    const int entry = a.row_index ? a.row_index[r] : r;
    arow_s[r] = a.row_index ? entry / a.row_div : entry;
    scale_s[r] = a.row_scale ? a.row_scale[entry] : 1.f;
  }
  __syncthreads();
  const int units = entries_s * upe;
  // CTAs start at different places of K and wrap around, so that they do not all ask for the same lines of A at once
  const int rot = iters > 0 ? (int)(blockIdx.x % (unsigned)iters) : 0;
  int p_unit = blockIdx.x, p_ki = 0, p_tj = 0, p_stage = 0, p_tile = 0, p_size = 0;
  const __nv_bfloat16* p_w = W;
  auto p_enter = [&]() {
    if (p_unit < units) {
      const int e = p_unit / upe;
      p_tile = (p_unit - e * upe) * GROUP;
      p_size = min(GROUP, tiles - p_tile);
      p_w = W + (size_t)ent_g[e] * (GATED ? 2 : 1) * N * K;
    }
  };
  p_enter();
  auto issue = [&]() {
    if (iters > 0 && p_unit < units) {
      int n_a, n_b;
      if (GATED) { n_a = (p_tile + p_tj) * 8 + g; n_b = n_a < N ? N + n_a : -1; if (n_a >= N) n_a = -1; }
      else { n_a = (p_tile + p_tj) * 16 + g; n_b = n_a + 8; if (n_a >= N) n_a = -1; if (n_b >= N) n_b = -1; }
      const int kk = p_ki + rot < iters ? p_ki + rot : p_ki + rot - iters;
      const int k0 = (kk * GGS_WARPS + warp) * GGS_SPAN + c * 8, k1 = k0 + 32;
      const unsigned dst = ring_base + (unsigned)(p_stage * 4 * 32 * 16);
      const __nv_bfloat16* wa = p_w + (size_t)max(n_a, 0) * K;
      const __nv_bfloat16* wb = p_w + (size_t)max(n_b, 0) * K;
      cp_async16(dst, wa + min(k0, K - 8), (n_a >= 0 && k0 < K) ? 16 : 0);
      cp_async16(dst + 512, wb + min(k0, K - 8), (n_b >= 0 && k0 < K) ? 16 : 0);
      cp_async16(dst + 1024, wa + min(k1, K - 8), (n_a >= 0 && k1 < K) ? 16 : 0);
      cp_async16(dst + 1536, wb + min(k1, K - 8), (n_b >= 0 && k1 < K) ? 16 : 0);
      if (++p_tj == p_size) {
        p_tj = 0;
        if (++p_ki == iters) { p_ki = 0; p_unit += gridDim.x; p_enter(); }
      }
      p_stage = p_stage + 1 == GGS_STAGES ? 0 : p_stage + 1;
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < GGS_STAGES - 1; ++s) issue();
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  int c_stage = 0;
  for (int unit = blockIdx.x; unit < units; unit += gridDim.x) {
    const int e = unit / upe, tile0 = (unit - e * upe) * GROUP, gsize = min(GROUP, tiles - tile0);
    const int r0 = ent_r[e], nrows = ent_n[e];
    const __nv_bfloat16* xr[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) xr[j] = g + 8 * j < nrows ? A + (size_t)arow_s[r0 + g + 8 * j] * a.lda : nullptr;
    const int nt = (nrows + 7) >> 3;                   // how many of the NT column groups hold rows
    float acc[GROUP][NT][4];
#pragma unroll
    for (int t = 0; t < GROUP; ++t)
#pragma unroll
      for (int j = 0; j < NT; ++j) { acc[t][j][0] = acc[t][j][1] = acc[t][j][2] = acc[t][j][3] = 0.f; }
    for (int kb = 0; kb < iters; kb += XB) {
      uint4 xb[XB][2 * NT];
#pragma unroll
      for (int u = 0; u < XB; ++u) {
        const int ki = kb + u;
        const int kk = ki + rot < iters ? ki + rot : ki + rot - iters;
        const int k0 = (kk * GGS_WARPS + warp) * GGS_SPAN + c * 8, k1 = k0 + 32;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          xb[u][2 * j] = (xr[j] && ki < iters && k0 < K) ? __ldg(reinterpret_cast<const uint4*>(xr[j] + k0)) : zero;
          xb[u][2 * j + 1] = (xr[j] && ki < iters && k1 < K) ? __ldg(reinterpret_cast<const uint4*>(xr[j] + k1)) : zero;
        }
      }
#pragma unroll
      for (int u = 0; u < XB; ++u) {
        if (kb + u < iters) {
#pragma unroll
          for (int t = 0; t < GROUP; ++t) {
            if (t < gsize) {
              issue();
              cp_async_wait<GGS_STAGES - 1>();
              const uint4* st = ring + ((size_t)(warp * GGS_STAGES + c_stage) * 4) * 32 + lane;
              const uint4 w0 = st[0], w1 = st[32], w2 = st[64], w3 = st[96];
              c_stage = c_stage + 1 == GGS_STAGES ? 0 : c_stage + 1;
#pragma unroll
              for (int j = 0; j < NT; ++j) {
                if (j < nt) {
                  const uint4 x0 = xb[u][2 * j], x1 = xb[u][2 * j + 1];
                  unsigned f[4];
                  f[0] = w0.x; f[1] = w1.x; f[2] = w0.y; f[3] = w1.y;
                  mma_bf16(acc[t][j], f, x0.x, x0.y);
                  f[0] = w0.z; f[1] = w1.z; f[2] = w0.w; f[3] = w1.w;
                  mma_bf16(acc[t][j], f, x0.z, x0.w);
                  f[0] = w2.x; f[1] = w3.x; f[2] = w2.y; f[3] = w3.y;
                  mma_bf16(acc[t][j], f, x1.x, x1.y);
                  f[0] = w2.z; f[1] = w3.z; f[2] = w2.w; f[3] = w3.w;
                  mma_bf16(acc[t][j], f, x1.z, x1.w);
                }
              }
            }
          }
        }
      }
    }
    // per tile: the warps' shares through shared memory, then the epilogue
#pragma unroll
    for (int t = 0; t < GROUP; ++t) {
      if (t < gsize) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          if (j < nt) {
            red[warp][g][8 * j + 2 * c] = acc[t][j][0];
            red[warp][g][8 * j + 2 * c + 1] = acc[t][j][1];
            red[warp][g + 8][8 * j + 2 * c] = acc[t][j][2];
            red[warp][g + 8][8 * j + 2 * c + 1] = acc[t][j][3];
          }
        }
        __syncthreads();
        __nv_bfloat16* out = (__nv_bfloat16*)a.out;
        if (GATED) {
          for (int i = threadIdx.x; i < nrows * 8; i += GGS_THREADS) {
            const int tok = i >> 3, r = i & 7, f = (tile0 + t) * 8 + r;
            if (f < N) {
              float gate = 0.f, up = 0.f;
#pragma unroll
              for (int w = 0; w < GGS_WARPS; ++w) { gate += red[w][r][tok]; up += red[w][r + 8][tok]; }
              const float sc = scale_s[r0 + tok];
              gate *= sc; up *= sc;
              out[(size_t)(r0 + tok) * a.ldo + f] = __float2bfloat16_rn(gate / (1.f + expf(-gate)) * up);
            }
          }
        } else {
          for (int i = threadIdx.x; i < nrows * 16; i += GGS_THREADS) {
            const int tok = i >> 4, r = i & 15, n = (tile0 + t) * 16 + r;
            if (n < N) {
              float v = 0.f;
#pragma unroll
              for (int w = 0; w < GGS_WARPS; ++w) v += red[w][r][tok];
              v *= scale_s[r0 + tok];
              if (a.relu2) { v = fmaxf(v, 0.f); v *= v; }
              out[(size_t)(r0 + tok) * a.ldo + n] = __float2bfloat16_rn(v);
            }
          }
        }
        __syncthreads();
      }
    }
  }
  cp_async_wait<0>();
}

template <bool GATED, int NT, int GROUP, int XB>
static int grouped_stream_go(const GroupedArgs& a, cudaStream_t stream) {
  const size_t smem = (size_t)GGS_WARPS * GGS_STAGES * 4 * 32 * 16 + sizeof(float) * GGS_WARPS * 16 * (8 * NT + 1) + (size_t)a.M * 8;
  static int num_sms = 0;
  if (!num_sms) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess ||
        cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || num_sms <= 0)
      num_sms = 148;
  }
  cudaError_t e = cudaFuncSetAttribute(grouped_stream_kernel<GATED, NT, GROUP, XB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "grouped_gemm: %s", cudaGetErrorString(e));
  gg_launch(grouped_stream_kernel<GATED, NT, GROUP, XB>, dim3(2 * num_sms), dim3(GGS_THREADS), smem, stream, a);
  return gg_check_launch("grouped_gemm");
}

// max_rows: no group has more rows than this (0: not known).  It only chooses between kernels.
extern "C" int gg_grouped_gemm(const void* A, long long lda, long long a_group_cols, const int* row_index,
                               int row_div, const void* W, void* out, long long ldo, long long o_group_cols,
                               const int* offsets, int M, int G, int N, int K, int Np, int act,
                               const void* gate, long long ldg, int gate_col0, const float* row_scale, int max_rows, int act_dtype,
                               cudaStream_t stream) {
  GG_REQUIRE(M >= 0 && G > 0 && N > 0 && K > 0 && Np >= N, "grouped_gemm: bad sizes M=%d G=%d N=%d K=%d Np=%d", M, G, N, K, Np);
  GG_REQUIRE(A && W && out, "grouped_gemm: a pointer is null");
  GG_REQUIRE(!row_index || row_div > 0, "grouped_gemm: a row list needs its divisor");
  GG_REQUIRE(act >= 0 && act <= 2, "grouped_gemm: unknown activation %d", act);
  if (M == 0) return GG_OK;
  const bool gated = act == 1;
  GroupedArgs a;
  a.A = A; a.lda = lda; a.a_group_cols = a_group_cols; a.row_index = row_index; a.row_div = row_div;
  a.W = W; a.out = out; a.ldo = ldo; a.o_group_cols = o_group_cols; a.offsets = offsets;
  a.M = M; a.G = G; a.N = N; a.K = K; a.Np = Np; a.relu2 = act == 2;
  a.gate = gate; a.ldg = ldg; a.gate_col0 = gate_col0; a.row_scale = row_scale;
  const int row_tiles = offsets ? (M + GGM_BM - 1) / GGM_BM + G : (M + GGM_BM - 1) / GGM_BM;
  GG_REQUIRE(row_tiles <= 65535 && G <= 65535, "grouped_gemm: %d row tiles or %d groups are too many for one launch", row_tiles, G);
  dim3 grid((Np + GGM_BN - 1) / GGM_BN, row_tiles, offsets ? 1 : G);
  const int esize = act_dtype == GG_F32 ? 4 : 2, vpt = 16 / esize;
  const bool vec = K % vpt == 0 && lda % vpt == 0 && a_group_cols % vpt == 0 && ((size_t)A % 16) == 0 && ((size_t)W % 16) == 0;
#define GGM_LAUNCH(T, BK)                                                                                      \
  do {                                                                                                         \
    if (gated && vec) gg_launch(grouped_gemm_kernel<T, true, BK, true>, grid, dim3(GGM_THREADS), 0, stream, a);        \
    else if (gated) gg_launch(grouped_gemm_kernel<T, true, BK, false>, grid, dim3(GGM_THREADS), 0, stream, a);         \
    else if (vec) gg_launch(grouped_gemm_kernel<T, false, BK, true>, grid, dim3(GGM_THREADS), 0, stream, a);           \
    else gg_launch(grouped_gemm_kernel<T, false, BK, false>, grid, dim3(GGM_THREADS), 0, stream, a);                   \
  } while (0)
  static const bool stream_on = !(getenv("GOLLMGO_B200_GROUPED_STREAM") && getenv("GOLLMGO_B200_GROUPED_STREAM")[0] == '0');
  if (act_dtype == GG_BF16 && vec && stream_on && offsets && !gate && a_group_cols == 0 && o_group_cols == 0 && Np == N &&
      K >= 64 && M <= GGS_MAX_ROWS && M <= 20 * G && max_rows > 0) {
    // rows a walk over a group's weights takes: enough for most groups of a step whose choices are spread by chance
    // (8 experts of 4096 x 2048, gate and up: 24 tokens with two each 53 us in walks of 16 rows and 59 in walks of 24, 64
    // tokens 77 and 66; beyond 20 rows a group on average the kernel with tiles of 32 rows is level)
    const int pass = max_rows <= 8 ? 8 : M <= 10 * G ? 16 : 24;
    if (G + M / pass <= GGS_MAX_ENTRIES) {
      const bool many = (long long)G * (gated ? (N + 7) / 8 : (N + 15) / 16) >= 2048;     // enough tiles for units of two
      if (gated) {
        if (pass == 8) return many ? grouped_stream_go<true, 1, 2, 4>(a, stream) : grouped_stream_go<true, 1, 1, 4>(a, stream);
        if (pass == 16) return many ? grouped_stream_go<true, 2, 2, 2>(a, stream) : grouped_stream_go<true, 2, 1, 4>(a, stream);
        return many ? grouped_stream_go<true, 3, 2, 2>(a, stream) : grouped_stream_go<true, 3, 1, 2>(a, stream);
      }
      if (pass == 8) return many ? grouped_stream_go<false, 1, 2, 4>(a, stream) : grouped_stream_go<false, 1, 1, 4>(a, stream);
      if (pass == 16) return many ? grouped_stream_go<false, 2, 2, 2>(a, stream) : grouped_stream_go<false, 2, 1, 4>(a, stream);
      return many ? grouped_stream_go<false, 3, 2, 2>(a, stream) : grouped_stream_go<false, 3, 1, 2>(a, stream);
    }
  }
  static const bool ring_on = !(getenv("GOLLMGO_B200_GROUPED_RING") && getenv("GOLLMGO_B200_GROUPED_RING")[0] == '0');
  if (act_dtype == GG_BF16 && vec && K >= 4 * GGR_BK && ring_on) {
    const size_t smem = (size_t)GGR_STAGES * (GGM_BM + (gated ? 2 : 1) * GGM_BN) * GGR_LD * sizeof(__nv_bfloat16);
    cudaError_t e = gated ? cudaFuncSetAttribute(grouped_gemm_ring_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
                          : cudaFuncSetAttribute(grouped_gemm_ring_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return gg_fail(GG_ERR_CUDA, "grouped_gemm: %s", cudaGetErrorString(e));
    if (gated) gg_launch(grouped_gemm_ring_kernel<true>, grid, dim3(GGM_THREADS), smem, stream, a);
    else gg_launch(grouped_gemm_ring_kernel<false>, grid, dim3(GGM_THREADS), smem, stream, a);
    return gg_check_launch("grouped_gemm");
  }
  if (act_dtype == GG_F32) {
    GGM_LAUNCH(float, 32);
  } else if (act_dtype == GG_BF16) {
    GGM_LAUNCH(__nv_bfloat16, 128);
  } else {
    return gg_fail(GG_ERR_INVALID, "grouped_gemm: unknown dtype %d", act_dtype);
  }
  return gg_check_launch("grouped_gemm");
}
