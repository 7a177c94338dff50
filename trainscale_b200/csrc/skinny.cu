// Products of a few token rows with (groups of) weight matrices: out[r, n] = act(sum_k A[r, k] W_g[n, k]).
//
// Decode multiplies a handful of rows with every weight of the layer, so the cost is reading the weights once.  A
// tcgen05 tile would be 128 rows high with almost all of them empty and gives too few CTAs to pull from every memory
// channel; here the WEIGHTS are the 16-row operand of a warp MMA, tokens are its 8 columns, and the eight warps of a CTA
// split the reduction of one 16-row tile (or of several, when it is short), so a projection of N rows spreads over up to
// N / 16 CTAs.  Both operands are read
// straight from global memory as 16-byte vectors: the reduction index is permuted the same way on both sides (a lane's
// eight consecutive values feed two MMA steps), so no shared-memory staging or transposition is needed.
//
// Groups (grid.y) are the experts of a mixture (slots sorted by expert: order / start / count), the heads of a per-head
// projection (every group takes all rows; A, W and out advance by a stride per group) or one dense matrix.
//
// Gated products (glu_act): the 16 weight rows of a tile are eight gate rows and the up rows of the same eight outputs, so
// both halves of an output meet in the CTA that reduced them.  A result may be multiplied by the sigmoid of a gate operand.
// `grouped_simt_kernel` computes the same for fp32 operands and for sizes the vector loads cannot take.
#include "common.cuh"
#include "host_common.h"

namespace ts {

struct SkinnyParams {
  const void* A;               // rows of K values
  const void* W;               // [N][ldw] per group
  void* out;
  long long lda, ldw, ldo;     // row strides in elements
  long long a_group, w_group, o_group;   // group strides in elements
  const int* order;            // slots in group order (nullptr: slot = row)
  const int* start;            // [groups] first entry of the group in `order` (nullptr: 0)
  const int* count;            // [groups] rows of the group (nullptr: M)
  int a_div;                   // row of A = slot / a_div
  int M, N, K;
  int act;                     // of common.cuh product_act or glu_act (0: none)
  float act_a, act_b;          // its constants
  int act_cols;                // outputs it applies to, from the first
  int out_fp32;
  const void* gate;            // result *= sigmoid(gate[slot * gate_ld + g * gate_group + n * gate_col]) (nullptr: none)
  long long gate_ld, gate_group;
  int gate_col;
};

__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                               uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

constexpr int SK_WARPS = 8;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ void skinny_store(const SkinnyParams& p, int g, int slot, int n, float v) {
  if (p.gate) v *= sigmoid(to_f32(reinterpret_cast<const T*>(p.gate)[slot * p.gate_ld + g * p.gate_group + n * p.gate_col]));
  const long long at = g * p.o_group + static_cast<long long>(slot) * p.ldo + n;
  if (p.out_fp32) reinterpret_cast<float*>(p.out)[at] = v;
  else reinterpret_cast<__nv_bfloat16*>(p.out)[at] = __float2bfloat16(v);
}
// weight row of the gate of output n (its up row is GLU_BLOCK below)
__device__ __forceinline__ int glu_row(int n) { return n / GLU_BLOCK * (2 * GLU_BLOCK) + n % GLU_BLOCK; }

__device__ __forceinline__ uint4 ld_stream(const void* p) {   // weights: read once, keep them out of L1
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p));
  return v;
}

// 32-wide reduction steps a warp has in flight
__host__ __device__ constexpr int skinny_unroll(int nt) { return nt == 1 ? 8 : (nt <= 4 ? 4 : 2); }

// NT: token tiles of 8 per pass; grid.z shares the passes.  KW: warps that share a row tile and split its reduction; the CTA's 8 / KW row tiles are
// neighbours.  grid (ceil(N / (16 * 8 / KW)), groups, passes side by side).
template <int NT, int KW>
__global__ void __launch_bounds__(SK_WARPS * 32)
skinny_gemm_kernel(SkinnyParams p) {
  constexpr int UN = skinny_unroll(NT);
  __shared__ float red[SK_WARPS][16][NT * 8 + 1];
  constexpr int TILES = SK_WARPS / KW;
  const int g = blockIdx.y;
  const int m_total = p.count ? p.count[g] : p.M;
  const int first = p.start ? p.start[g] : 0;
  if (m_total == 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gid = lane >> 2, tig = lane & 3;
  const bool glu = p.act >= ACT_FIRST_GLU;
  const int tile0 = blockIdx.x * TILES + warp / KW, wk = warp % KW;
  const int n0 = glu ? glu_row(tile0 * 8) : tile0 * 16, up = glu ? GLU_BLOCK : 8;      // first weight row, distance of the other half
  const __nv_bfloat16* A = reinterpret_cast<const __nv_bfloat16*>(p.A) + g * p.a_group;
  const __nv_bfloat16* W = reinterpret_cast<const __nv_bfloat16*>(p.W) + g * p.w_group;
  const bool row0 = n0 + gid < p.N, row1 = n0 + gid + up < p.N;
  const __nv_bfloat16* w0 = W + (row0 ? n0 + gid : 0) * p.ldw + tig * 8;
  const __nv_bfloat16* w1 = W + (row1 ? n0 + gid + up : 0) * p.ldw + tig * 8;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);

  for (int base = blockIdx.z * NT * 8; base < m_total; base += gridDim.z * NT * 8) {
    const int m = min(NT * 8, m_total - base);
    const __nv_bfloat16* x[NT];
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      const int i = t * 8 + gid;
      int slot = -1;
      if (i < m) slot = p.order ? p.order[first + base + i] : base + i;
      x[t] = slot < 0 ? nullptr : A + static_cast<long long>(slot / p.a_div) * p.lda + tig * 8;
    }
    float acc[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[t][q] = 0.f;

    const int steps = (p.K + 31) / 32;
    for (int s = wk * UN; s < steps; s += KW * UN) {       // UN steps in a row: 64 * UN bytes of a weight row at once
      uint4 a0[UN], a1[UN], b[UN][NT];
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const int k = (s + u) * 32;
        const bool in = k + tig * 8 < p.K;
        a0[u] = in && row0 ? ld_stream(w0 + k) : zero;
        a1[u] = in && row1 ? ld_stream(w1 + k) : zero;
#pragma unroll
        for (int t = 0; t < NT; ++t)
          b[u][t] = in && x[t] ? *reinterpret_cast<const uint4*>(x[t] + k) : zero;
      }
#pragma unroll
      for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int t = 0; t < NT; ++t)
          if (t * 8 < m) {
            mma_bf16_16816(acc[t], a0[u].x, a1[u].x, a0[u].y, a1[u].y, b[u][t].x, b[u][t].y);
            mma_bf16_16816(acc[t], a0[u].z, a1[u].z, a0[u].w, a1[u].w, b[u][t].z, b[u][t].w);
          }
    }
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      red[warp][gid][t * 8 + tig * 2] = acc[t][0];
      red[warp][gid][t * 8 + tig * 2 + 1] = acc[t][1];
      red[warp][gid + 8][t * 8 + tig * 2] = acc[t][2];
      red[warp][gid + 8][t * 8 + tig * 2 + 1] = acc[t][3];
    }
    __syncthreads();
    const int lg = glu ? 3 : 4, n_out = glu ? p.N / 2 : p.N;       // outputs of a tile: 8 or 16
    for (int i = threadIdx.x; i < TILES * m << lg; i += SK_WARPS * 32) {
      const int tile = TILES == 1 ? 0 : i / (m << lg), r = i - tile * (m << lg);
      const int tk = r >> lg, n = r & ((1 << lg) - 1), nn = ((blockIdx.x * TILES + tile) << lg) + n;
      if (nn < n_out) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < KW; ++w) v += red[tile * KW + w][n][tk];
        if (glu) {
          float f = 0.f;
#pragma unroll
          for (int w = 0; w < KW; ++w) f += red[tile * KW + w][n + 8][tk];
          v = glu_act<true>(v, f, p.act);
        } else {
          if (nn < p.act_cols) v = product_act(v, p.act, p.act_a, p.act_b);
        }
        skinny_store<__nv_bfloat16>(p, g, p.order ? p.order[first + base + tk] : base + tk, nn, v);
      }
    }
    __syncthreads();
  }
}

// One warp per weight row (gated: per pair of rows), four token rows at a time, lanes split the reduction.  Any size, fp32 or bf16 operands.
template <typename T>
__global__ void __launch_bounds__(256) grouped_simt_kernel(SkinnyParams p) {
  constexpr int TM = 4;
  const int g = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + warp;
  const int m_total = p.count ? p.count[g] : p.M;
  const int first = p.start ? p.start[g] : 0;
  const bool glu = p.act >= ACT_FIRST_GLU;
  if (n >= (glu ? p.N / 2 : p.N)) return;
  const T* A = reinterpret_cast<const T*>(p.A) + g * p.a_group;
  const T* w = reinterpret_cast<const T*>(p.W) + g * p.w_group + (glu ? glu_row(n) : n) * p.ldw;
  const T* w_up = w + GLU_BLOCK * p.ldw;
  for (int base = blockIdx.z * TM; base < m_total; base += gridDim.z * TM) {
    const T* x[TM];
    int slot[TM];
#pragma unroll
    for (int t = 0; t < TM; ++t) {
      const int i = min(base + t, m_total - 1);
      slot[t] = p.order ? p.order[first + i] : i;
      x[t] = A + static_cast<long long>(slot[t] / p.a_div) * p.lda;
    }
    float acc[TM] = {0.f, 0.f, 0.f, 0.f}, fac[TM] = {0.f, 0.f, 0.f, 0.f};
    for (int k = lane; k < p.K; k += 32) {
      const float wk = to_f32(w[k]);
#pragma unroll
      for (int t = 0; t < TM; ++t) acc[t] += wk * to_f32(x[t][k]);
      if (glu) {
        const float uk = to_f32(w_up[k]);
#pragma unroll
        for (int t = 0; t < TM; ++t) fac[t] += uk * to_f32(x[t][k]);
      }
    }
#pragma unroll
    for (int t = 0; t < TM; ++t) {
      float v = warp_sum(acc[t]);
      if (glu) v = glu_act<false>(v, warp_sum(fac[t]), p.act);
      else if (n < p.act_cols) v = product_act(v, p.act, p.act_a, p.act_b);
      if (lane == 0 && base + t < m_total) skinny_store<T>(p, g, slot[t], n, v);
    }
  }
}

template <int NT>
static void launch_skinny(int kw, dim3 grid, cudaStream_t st, const SkinnyParams& p) {
  if (kw == 8) skinny_gemm_kernel<NT, 8><<<grid, SK_WARPS * 32, 0, st>>>(p);
  else if (kw == 4) skinny_gemm_kernel<NT, 4><<<grid, SK_WARPS * 32, 0, st>>>(p);
  else if (kw == 2) skinny_gemm_kernel<NT, 2><<<grid, SK_WARPS * 32, 0, st>>>(p);
  else skinny_gemm_kernel<NT, 1><<<grid, SK_WARPS * 32, 0, st>>>(p);
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace ts

TS_DEFINE_ERROR_API(ts_skinny)
using namespace ts;

// M: rows of every group, or an upper bound of them when `count` is given (`typical`: how many a group usually has; more
// take further passes over the weights, which then come from L2).  fp32: A and W are fp32 (else bf16).  Gated activations:
// W has N rows in alternating blocks of GLU_BLOCK gate and up rows, the result N / 2 columns.  `act` (with act_a, act_b)
// applies to the first act_cols outputs.  gate (of the type of A): nullptr or a factor sigmoid(gate) of every result; gate_col 0:
// one for all outputs of a row and group.
extern "C" int ts_skinny_gemm(const void* A, const void* W, void* out, long long lda, long long ldw, long long ldo,
                              long long a_group, long long w_group, long long o_group, const int* order,
                              const int* start, const int* count, int a_div, int groups, int M, int N, int K, int act,
                              float act_a, float act_b, int act_cols, int fp32, int out_fp32, int typical, const void* gate,
                              long long gate_ld, long long gate_group, int gate_col, int row_tiles, void* stream) {
  if (M <= 0 || groups <= 0) return 0;
  if (N <= 0 || K <= 0 || a_div <= 0 || act < 0 || act > ACT_LAST_GLU || (act == 3 && !(act_a > 0.f)) || act_cols < 0 || groups > 65535)
    return -10;
  if (act >= ACT_FIRST_GLU && N % (2 * GLU_BLOCK)) return -12;
  if (fp32 && !out_fp32) return -11;
  SkinnyParams p;
  p.A = A; p.W = W; p.out = out; p.lda = lda; p.ldw = ldw; p.ldo = ldo; p.a_group = a_group; p.w_group = w_group;
  p.o_group = o_group; p.order = order; p.start = start; p.count = count; p.a_div = a_div; p.M = M; p.N = N; p.K = K;
  p.act = act; p.act_a = act_a; p.act_b = act_b; p.act_cols = act_cols; p.out_fp32 = out_fp32; p.gate = gate; p.gate_ld = gate_ld;
  p.gate_group = gate_group; p.gate_col = gate_col;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = !fp32 && K % 8 == 0 && lda % 8 == 0 && ldw % 8 == 0 && a_group % 8 == 0 && w_group % 8 == 0 &&
                   aligned16(A) && aligned16(W);
  if (!vec) {
    int z = (M + 3) / 4;
    if (z > 64) z = 64;
    const int n_out = act >= ACT_FIRST_GLU ? N / 2 : N;
    const dim3 grid((n_out + 7) / 8, groups, z);
    if (fp32) grouped_simt_kernel<float><<<grid, 256, 0, st>>>(p);
    else grouped_simt_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(p);
    return (int)cudaGetLastError();
  }
  const int per_pass = count && typical > 0 && typical < M ? typical : M;
  int nt = per_pass <= 8 ? 1 : (per_pass <= 16 ? 2 : (per_pass <= 32 ? 4 : 8)), z = 1;
  if (row_tiles > 0) {
    while (nt > row_tiles) nt /= 2;
    z = (M + nt * 8 - 1) / (nt * 8);
  }
  int kw = 1;
  while (kw < SK_WARPS && kw * skinny_unroll(nt) * 32 < K) kw *= 2;
  const int rows = 16 * SK_WARPS / kw;
  const dim3 grid((N + rows - 1) / rows, groups, z);
  if (nt == 1) launch_skinny<1>(kw, grid, st, p);
  else if (nt == 2) launch_skinny<2>(kw, grid, st, p);
  else if (nt == 4) launch_skinny<4>(kw, grid, st, p);
  else launch_skinny<8>(kw, grid, st, p);
  return (int)cudaGetLastError();
}
