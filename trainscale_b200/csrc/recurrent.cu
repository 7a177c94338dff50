// Recurrent mixers with a matrix state per head, S [dim keys x vdim values], carried in fp32 from step to step:
//
//   gated delta rule   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q        (g, beta one number per head)
//   WKV                o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T                (w per key channel)
//   retention          S <- g S + k v^T;  o = S^T q, q and k rotated by their position     (g one constant per head)
//
// Rows are tokens of a flattened batch.  A portion of a prompt runs as: inputs (short convolution, unit norms, gates), a
// scan over its tokens, the gated norm of the result.  A single decoded row is one launch from projection to gated norm.
// A state row of a sequence holds [convolution inputs (taps - 1) x C | S per head] or [token-shift row | S per head];
// a step reads one row and writes another, so nothing of a launch is overwritten while it is still read.
//
// Two scans.  bf16 models (`block_scan_kernel`): blocks of eight tokens as warp MMAs with operands split into two TF32 parts.
// fp32 models and head sizes that are not multiples of eight (`delta_scan_kernel`, `wkv_scan_kernel`): fp32 arithmetic on the
// FMA pipe in packed pairs, S in registers, 8 key rows x 4 value columns per thread.  The latter walks blocks too: for four
// tokens of the delta rule all products S^T k and S^T q with the state before the block are formed at once (eight vectors, one
// reduction over the lanes that share a column), the four-step triangular recurrence that is left is solved per column with
// the block's small Gram matrices, and the state is updated with all four writes; the latency of a reduction is paid once
// per block, not per token.
#include "common.cuh"
#include "host_common.h"

namespace ts {

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
// activations of 16-bit models: fp32 arithmetic with the approximate exponential and quotient
template <typename T> __device__ __forceinline__ float act_silu(float x) {
  return sizeof(T) == 2 ? __fdividef(x, 1.f + __expf(-x)) : silu(x);
}
__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
  return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
template <int VEC> __device__ __forceinline__ void load_vec(const float* p, float (&v)[VEC]) {
  if (VEC == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[VEC > 1 ? 1 : 0] = a.y; v[VEC > 2 ? 2 : 0] = a.z; v[VEC > 3 ? 3 : 0] = a.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC> __device__ __forceinline__ void store_vec(float* p, const float (&v)[VEC]) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[VEC > 1 ? 1 : 0], v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]);
  else *p = v[0];
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 4 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// ---------------------------------------------------------------------------------------------------------
// gated delta rule
// ---------------------------------------------------------------------------------------------------------
struct DeltaParams {
  const void* proj;            // rows [q G x D | k G x D | v H x V | gate H x V | b H | a H]
  long long ld;
  const float* conv_w;         // [C][taps], C = 2 G D + H V
  const float* A_log;          // [H]
  const float* dt_bias;        // [H]
  const float* norm_w;         // [V]
  float eps, q_scale;
  float* state;
  long long state_ld;
  int s_off;                   // first value of S in a state row
  const int* row_prev;         // [rows] state row a sequence continues from (>= 0), else zeros / the row before
  const int* row_next;         // [rows] state row to leave, -1: not a last row
  const int* cu;               // portions: [n + 1] first rows
  int portions, max_rows;      // portions: count, rows of the longest
  float* qkv;                  // portions: [rows][C] convolved inputs
  float* gates;                // portions: [rows][2 H] log g | beta
  float* o;                    // portions: [rows][H V]
  void* out;                   // decoding: [rows][out_ld]
  long long out_ld;
  float out_scale;
  int rows, H, G, D, V, taps;
};

// input of channel c at row `src` of a sequence whose portion starts at row `start`; rows before it come from the state
template <typename T>
__device__ __forceinline__ float conv_input(const DeltaParams& p, int src, int start, int prev, int c, int C) {
  if (src >= start) return to_f32(reinterpret_cast<const T*>(p.proj)[src * p.ld + c]);
  const int i = src - start + p.taps - 1;
  return prev >= 0 && i >= 0 ? p.state[prev * p.state_ld + static_cast<long long>(i) * C + c] : 0.f;
}

constexpr int DI_TOKENS = 8;

// A warp takes DI_TOKENS rows of a portion, one head of q, k or v (or the gates); lanes hold VEC neighbouring channels, NI
// times.  FAST: at most four taps, inputs of the rows before stay in registers.  grid (runs of the longest portion, units / 4,
// portions).
template <typename T, int VEC, int NI, bool FAST>
__global__ void __launch_bounds__(128) delta_inputs_kernel(DeltaParams p) {
  const int lane = threadIdx.x & 31, units = 2 * p.G + p.H + 1;
  const int unit = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int start = p.cu[blockIdx.z], end = p.cu[blockIdx.z + 1];
  const int t0 = start + blockIdx.x * DI_TOKENS, t1 = min(end, t0 + DI_TOKENS);
  if (t0 >= t1) return;
  const int C = 2 * p.G * p.D + p.H * p.V;
  const T* proj = reinterpret_cast<const T*>(p.proj);
  if (unit == units - 1) {
    const int b0 = C + p.H * p.V;
    for (int i = lane; i < (t1 - t0) * p.H; i += 32) {
      const int t = t0 + i / p.H, h = i % p.H;
      const float b = to_f32(proj[t * p.ld + b0 + h]), a = to_f32(proj[t * p.ld + b0 + p.H + h]);
      p.gates[static_cast<long long>(t) * 2 * p.H + h] = -expf(p.A_log[h]) * softplus(a + p.dt_bias[h]);
      p.gates[static_cast<long long>(t) * 2 * p.H + p.H + h] = sigmoid(b);
    }
    return;
  }
  const int n = unit < 2 * p.G ? p.D : p.V;                       // channels of this head
  const int c0 = unit < 2 * p.G ? unit * p.D : 2 * p.G * p.D + (unit - 2 * p.G) * p.V;
  const int taps = p.taps;
  float w[4][NI * VEC], hist[3][NI * VEC];
  if (FAST) {
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const int c = i * 32 * VEC + lane * VEC + e;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int k = j - (4 - taps);                           // fewer taps: leading zeros
          w[j][i * VEC + e] = c < n && k >= 0 ? p.conv_w[static_cast<long long>(c0 + c) * taps + k] : 0.f;
        }
      }
  }
  float in[DI_TOKENS][NI * VEC];           // the run's own inputs, all loads issued at once
#pragma unroll
  for (int k = 0; k < DI_TOKENS; ++k) {
    const T* x = proj + min(t0 + k, t1 - 1) * p.ld + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = min(i * 32 * VEC + lane * VEC, n - VEC);
      if (VEC == 2 && sizeof(T) == 2) {
        const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x + c));
        in[k][i * VEC] = f.x;
        in[k][i * VEC + VEC - 1] = f.y;
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) in[k][i * VEC + e] = to_f32(x[c + e]);
      }
    }
  }
  const int prev = p.row_prev[start];
  if (FAST) {
#pragma unroll
    for (int i = 0; i < NI * VEC; ++i) {
      const int c = (i / VEC) * 32 * VEC + lane * VEC + i % VEC;
#pragma unroll
      for (int j = 0; j < 3; ++j) hist[j][i] = c < n ? conv_input<T>(p, t0 - 3 + j, start, prev, c0 + c, C) : 0.f;
    }
  }
#pragma unroll
  for (int k = 0; k < DI_TOKENS; ++k) {
    const int t = t0 + k;
    if (t >= t1) break;
    float y[NI * VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const int q = i * VEC + e, c = i * 32 * VEC + lane * VEC + e;
        float v = 0.f;
        if (FAST) {
          v = w[0][q] * hist[0][q] + w[1][q] * hist[1][q] + w[2][q] * hist[2][q] + w[3][q] * in[k][q];
          hist[0][q] = hist[1][q];
          hist[1][q] = hist[2][q];
          hist[2][q] = in[k][q];
        } else if (c < n) {
          for (int j = 0; j < taps; ++j)
            v += p.conv_w[static_cast<long long>(c0 + c) * taps + j] *
                 conv_input<T>(p, t - (taps - 1) + j, start, prev, c0 + c, C);
        }
        y[q] = c < n ? act_silu<T>(v) : 0.f;
        ss += y[q] * y[q];
      }
    }
    float f = 1.f;
    if (unit < 2 * p.G) f = (unit < p.G ? p.q_scale : 1.f) / sqrtf(warp_sum(ss) + 1e-6f);
    float* dst = p.qkv + static_cast<long long>(t) * C + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int cb = i * 32 * VEC + lane * VEC;
      if (cb < n) {
        if (VEC == 2) *reinterpret_cast<float2*>(dst + cb) = make_float2(y[i * VEC] * f, y[i * VEC + VEC - 1] * f);
        else dst[cb] = y[i] * f;
      }
    }
  }
  const int next = t1 == end ? p.row_next[end - 1] : -1;
  if (next >= 0)
    for (int c = lane; c < n; c += 32)
      for (int j = 0; j < taps - 1; ++j)
        p.state[next * p.state_ld + static_cast<long long>(j) * C + c0 + c] =
            conv_input<T>(p, end - (taps - 1) + j, start, prev, c0 + c, C);
}

constexpr int SC_TILE = 32;                // tokens staged at a time
constexpr int SC_WARPS = 4;

// sum of v[32] over the LANES lanes of a column group; afterwards lane rl holds sums rl * 32 / LANES, ... in v[0 ..]
template <int LANES> __device__ __forceinline__ void reduce_scatter(float (&v)[32], int rl) {
#pragma unroll
  for (int m = LANES / 2, n = 16; m > 0; m >>= 1, n >>= 1) {
    const bool up = (rl & m) != 0;
#pragma unroll
    for (int j = 0; j < 16; ++j)
      if (j < n) {
        const float send = up ? v[j] : v[j + n], keep = up ? v[j + n] : v[j];
        v[j] = keep + __shfl_xor_sync(0xffffffffu, send, m);
      }
  }
}

template <int LANES> struct DeltaScan {
  static constexpr int DP = LANES * 8;                 // key rows, padded
  static constexpr int KS = DP + 4;                    // row stride of a staged vector
  static constexpr int NCW = 4 * (32 / LANES);         // columns per warp
  static constexpr int NC = NCW * SC_WARPS;            // columns per CTA
  static constexpr int STAGE = SC_TILE * (2 * KS + NC + 2);   // floats: q, k | v | log g, beta
  static constexpr int COEF = 32;                      // per block: 6 L, 10 A, 4 beta g, 4 g, 4 r, 4 beta
  static constexpr int XS = 16 * NCW;                  // per warp: 8 sums, 4 u, 4 r u per column
  static constexpr size_t SMEM = (2 * STAGE + SC_TILE / 4 * COEF + SC_WARPS * XS) * sizeof(float);
};

// grid (column tiles, H, portions)
template <int LANES>
__global__ void __launch_bounds__(SC_WARPS * 32, LANES <= 16 ? 2 : 1) delta_scan_kernel(DeltaParams p) {
  using Z = DeltaScan<LANES>;
  extern __shared__ __align__(16) float smf[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane / LANES, rl = lane % LANES;
  const int h = blockIdx.y, g = h / (p.H / p.G), col_cta = blockIdx.x * Z::NC;
  const int row0 = p.cu[blockIdx.z], n = p.cu[blockIdx.z + 1] - row0;
  if (n <= 0) return;
  const int C = 2 * p.G * p.D + p.H * p.V;
  const int wc = warp * Z::NCW, col0 = col_cta + wc + cg * 4;      // this lane's four columns
  float* coef = smf + 2 * Z::STAGE;
  float* xs = coef + SC_TILE / 4 * Z::COEF + warp * Z::XS;         // [8][NCW]
  float* us = xs + 8 * Z::NCW;                                     // [4][NCW]
  float* ur = us + 4 * Z::NCW;                                     // [4][NCW]
  const bool vec = p.D % 4 == 0 && p.V % 4 == 0;                   // then every staged piece is 16-byte aligned

  auto stage_tile = [&](int s, int t) {
    float* base = smf + s * Z::STAGE;
    const float* src = p.qkv + static_cast<long long>(row0 + t) * C;
    if (vec) {
      constexpr int U = Z::DP / 4;
      for (int i = threadIdx.x; i < SC_TILE * 2 * U; i += SC_WARPS * 32) {
        const int tk = i / (2 * U), r = i - tk * 2 * U, w = r / U, c = (r - w * U) * 4;
        const bool ok = t + tk < n && c < p.D;
        cp_async16(base + (tk * 2 + w) * Z::KS + c, ok ? src + static_cast<long long>(tk) * C + (w * p.G + g) * p.D + c : p.qkv, ok);
      }
      for (int i = threadIdx.x; i < SC_TILE * Z::NC / 4; i += SC_WARPS * 32) {
        const int tk = i / (Z::NC / 4), c = (i - tk * (Z::NC / 4)) * 4;
        const bool ok = t + tk < n && col_cta + c < p.V;
        cp_async16(base + SC_TILE * 2 * Z::KS + tk * Z::NC + c,
                   ok ? src + static_cast<long long>(tk) * C + 2 * p.G * p.D + h * p.V + col_cta + c : p.qkv, ok);
      }
    } else {
      for (int i = threadIdx.x; i < SC_TILE * 2 * Z::DP; i += SC_WARPS * 32) {
        const int tk = i / (2 * Z::DP), r = i - tk * 2 * Z::DP, w = r / Z::DP, c = r - w * Z::DP;
        const bool ok = t + tk < n && c < p.D;
        cp_async4(base + (tk * 2 + w) * Z::KS + c, ok ? src + static_cast<long long>(tk) * C + (w * p.G + g) * p.D + c : p.qkv, ok);
      }
      for (int i = threadIdx.x; i < SC_TILE * Z::NC; i += SC_WARPS * 32) {
        const int tk = i / Z::NC, c = i - tk * Z::NC;
        const bool ok = t + tk < n && col_cta + c < p.V;
        cp_async4(base + SC_TILE * 2 * Z::KS + tk * Z::NC + c,
                  ok ? src + static_cast<long long>(tk) * C + 2 * p.G * p.D + h * p.V + col_cta + c : p.qkv, ok);
      }
    }
    float* gt = base + SC_TILE * (2 * Z::KS + Z::NC);
    for (int i = threadIdx.x; i < SC_TILE * 2; i += SC_WARPS * 32) {
      const int tk = i >> 1;
      const bool ok = t + tk < n;
      cp_async4(gt + i, ok ? p.gates + static_cast<long long>(row0 + t + tk) * 2 * p.H + (i & 1) * p.H + h : p.gates, ok);
    }
    cp_commit();
  };

  // state: pairs of key rows r, r + 1 of column c; the lane's rows are 4 LANES j + 4 rl + {0, 1, 2, 3}
  uint64_t S[4][4];
  const int prev = p.row_prev[row0];
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = (j >> 1) * LANES * 4 + rl * 4 + (j & 1) * 2;
      float a = 0.f, b = 0.f;
      if (prev >= 0 && col0 + c < p.V) {
        const float* src = p.state + prev * p.state_ld + p.s_off + static_cast<long long>(h) * p.D * p.V + col0 + c;
        if (r < p.D) a = src[static_cast<long long>(r) * p.V];
        if (r + 1 < p.D) b = src[static_cast<long long>(r + 1) * p.V];
      }
      S[c][j] = pack2(a, b);
    }

  stage_tile(0, 0);
  int s = 0;
  for (int t = 0; t < n; t += SC_TILE, s ^= 1) {
    if (t + SC_TILE < n) {
      stage_tile(s ^ 1, t + SC_TILE);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const float* base = smf + s * Z::STAGE;
    const float* vt = base + SC_TILE * 2 * Z::KS;
    const float* gt = vt + SC_TILE * Z::NC;
    {   // Gram matrices and decays of the tile's blocks: 16 threads per block of four tokens
      const int blk = threadIdx.x >> 4, e = threadIdx.x & 15;
      int i, j, q = 0;                                   // pair (i, j): k_i . k_j for e < 6, q_i . k_j after that
      if (e < 6) {
        i = e < 1 ? 1 : (e < 3 ? 2 : 3);
        j = e - i * (i - 1) / 2;
        q = 1;
      } else {
        const int f = e - 6;
        i = f < 1 ? 0 : (f < 3 ? 1 : (f < 6 ? 2 : 3));
        j = f - i * (i + 1) / 2;
      }
      const float* x = base + ((blk * 4 + i) * 2 + q) * Z::KS;
      const float* y = base + ((blk * 4 + j) * 2 + 1) * Z::KS;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll 8
      for (int c = 0; c < Z::DP; c += 4) {
        const float4 a = *reinterpret_cast<const float4*>(x + c), b = *reinterpret_cast<const float4*>(y + c);
        d0 += a.x * b.x; d1 += a.y * b.y; d2 += a.z * b.z; d3 += a.w * b.w;
      }
      const float* lg = gt + blk * 8;                    // log g, beta alternate
      float decay = 0.f;
      for (int z = j + 1; z <= i; ++z) decay += lg[2 * z];
      const float v = expf(decay) * ((d0 + d1) + (d2 + d3));
      float* co = coef + blk * Z::COEF;
      co[e] = e < 6 ? lg[2 * i + 1] * v : v;
      if (e < 4) {
        float head = 0.f, tail = 0.f;
        for (int z = 0; z <= e; ++z) head += lg[2 * z];
        for (int z = e + 1; z < 4; ++z) tail += lg[2 * z];
        const float gh = expf(head), beta = lg[2 * e + 1];
        co[16 + e] = beta * gh;
        co[20 + e] = gh;
        co[24 + e] = expf(tail);
        co[28 + e] = beta;
      }
    }
    __syncthreads();
    const int blocks = (min(n - t, SC_TILE) + 3) / 4;
    for (int blk = 0; blk < blocks; ++blk) {
      const float* tok = base + blk * 4 * 2 * Z::KS;
      const float* co = coef + blk * Z::COEF;
      float v[32];                                       // [vector: k of four tokens, q of four tokens][column]
      uint64_t kk[4][4];
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const float* src = tok + ((x & 3) * 2 + (x < 4 ? 1 : 0)) * Z::KS + rl * 4;
        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(src);
        const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(src + LANES * 4);
        if (x < 4) {
          kk[x][0] = a.x; kk[x][1] = a.y; kk[x][2] = b.x; kk[x][3] = b.y;
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float2 d = unpack2(fma2(S[c][3], b.y, fma2(S[c][2], b.x, fma2(S[c][1], a.y, mul2(S[c][0], a.x)))));
          v[x * 4 + c] = d.x + d.y;
        }
      }
      reduce_scatter<LANES>(v, rl);
#pragma unroll
      for (int e = 0; e < 32 / LANES; ++e) {
        const int idx = rl * (32 / LANES) + e;
        xs[(idx >> 2) * Z::NCW + cg * 4 + (idx & 3)] = v[e];
      }
      __syncwarp();
      if (lane < Z::NCW) {                               // u of the four tokens, one column per lane
        const float* vv = vt + blk * 4 * Z::NC + wc + lane;
        const float4 bg = *reinterpret_cast<const float4*>(co + 16), rr = *reinterpret_cast<const float4*>(co + 24);
        const float4 be = *reinterpret_cast<const float4*>(co + 28);
        const float u0 = be.x * vv[0] - bg.x * xs[lane];
        float u1 = be.y * vv[Z::NC] - bg.y * xs[Z::NCW + lane];
        float u2 = be.z * vv[2 * Z::NC] - bg.z * xs[2 * Z::NCW + lane];
        float u3 = be.w * vv[3 * Z::NC] - bg.w * xs[3 * Z::NCW + lane];
        u1 -= co[0] * u0;
        u2 -= co[1] * u0;
        u3 -= co[3] * u0;
        u2 -= co[2] * u1;
        u3 -= co[4] * u1;
        u3 -= co[5] * u2;
        us[lane] = u0; us[Z::NCW + lane] = u1; us[2 * Z::NCW + lane] = u2; us[3 * Z::NCW + lane] = u3;
        ur[lane] = rr.x * u0; ur[Z::NCW + lane] = rr.y * u1; ur[2 * Z::NCW + lane] = rr.z * u2; ur[3 * Z::NCW + lane] = rr.w * u3;
      }
      __syncwarp();
      const uint64_t g4 = pack2(co[23], co[23]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 f = *reinterpret_cast<const float4*>(ur + i * Z::NCW + cg * 4);
        const uint64_t w[4] = {pack2(f.x, f.x), pack2(f.y, f.y), pack2(f.z, f.z), pack2(f.w, f.w)};
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int j = 0; j < 4; ++j) S[c][j] = fma2(kk[i][j], w[c], i == 0 ? mul2(S[c][j], g4) : S[c][j]);
      }
#pragma unroll
      for (int x = 0; x < (4 * Z::NCW + 31) / 32; ++x) {
        const int idx = x * 32 + lane, i = idx / Z::NCW, c = idx % Z::NCW;
        if (idx < 4 * Z::NCW && t + blk * 4 + i < n && col_cta + wc + c < p.V) {
          const float* A = co + 6 + i * (i + 1) / 2;
          float o = co[20 + i] * xs[(4 + i) * Z::NCW + c];
          for (int j = 0; j <= i; ++j) o += A[j] * us[j * Z::NCW + c];
          p.o[static_cast<long long>(row0 + t + blk * 4 + i) * p.H * p.V + h * p.V + col_cta + wc + c] = o;
        }
      }
      __syncwarp();
    }
    __syncthreads();
  }
  const int next = p.row_next[row0 + n - 1];
  if (next >= 0) {
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = (j >> 1) * LANES * 4 + rl * 4 + (j & 1) * 2;
        const float2 d = unpack2(S[c][j]);
        if (col0 + c < p.V) {
          float* dst = p.state + next * p.state_ld + p.s_off + static_cast<long long>(h) * p.D * p.V + col0 + c;
          if (r < p.D) dst[static_cast<long long>(r) * p.V] = d.x;
          if (r + 1 < p.D) dst[static_cast<long long>(r + 1) * p.V] = d.y;
        }
      }
  }
}

// ---------------------------------------------------------------------------------------------------------
// WKV
// ---------------------------------------------------------------------------------------------------------
struct WkvParams {
  const void* rkvg;            // rows [r | k | v | gate], each H x D
  long long ld;
  const float* w_raw;          // [rows][H D]: exponent of the decay before '+ w0'
  const float* w0;             // [H D]
  const float* u;              // [H D]
  const float* norm_w;         // [H D]
  float eps;
  float* state;
  long long state_ld;
  int s_off;
  const int* row_prev;
  const int* row_next;
  const int* cu;               // portions
  float* o;                    // portions: [rows][H D]
  void* out;                   // decoding: [rows][out_ld]
  long long out_ld;
  int rows, H, D;
};

template <int LANES, typename T> struct WkvScan {
  static constexpr int TT = LANES == 32 ? 16 : SC_TILE;            // tokens staged at a time
  static constexpr int DP = LANES * 8;
  static constexpr int NCW = 4 * (32 / LANES);
  static constexpr int NC = NCW * SC_WARPS;
  static constexpr int RAW = TT * ((2 * DP + NC) * static_cast<int>(sizeof(T)) + DP * 4);   // bytes: r | k | v | w
  static constexpr int TILE = TT * (3 * DP + NC + 1);         // floats: r, k, decay | v | r . (u k)
  static constexpr int XS = 8 * NCW;
  static constexpr size_t SMEM = 2 * RAW + (TILE + SC_WARPS * XS + 2 * DP) * sizeof(float);
};

// grid (column tiles, H, portions)
template <int LANES, typename T>
__global__ void __launch_bounds__(SC_WARPS * 32) wkv_scan_kernel(WkvParams p) {
  using Z = WkvScan<LANES, T>;
  extern __shared__ __align__(16) uint8_t smb[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane / LANES, rl = lane % LANES;
  const int h = blockIdx.y, col_cta = blockIdx.x * Z::NC;
  const int row0 = p.cu[blockIdx.z], n = p.cu[blockIdx.z + 1] - row0;
  if (n <= 0) return;
  const int HD = p.H * p.D, D = p.D;
  const int wc = warp * Z::NCW, col0 = col_cta + wc + cg * 4;
  float* tile = reinterpret_cast<float*>(smb + 2 * Z::RAW);        // [Z::TT][3][DP]
  float* vt = tile + Z::TT * 3 * Z::DP;                          // [Z::TT][NC]
  float* rk = vt + Z::TT * Z::NC;                                // [Z::TT]
  float* xs = rk + Z::TT + warp * Z::XS;                         // [8][NCW]
  float* w0s = rk + Z::TT + SC_WARPS * Z::XS;                    // [DP]
  float* uss = w0s + Z::DP;                                        // [DP]
  for (int c = threadIdx.x; c < Z::DP; c += SC_WARPS * 32) {
    w0s[c] = c < D ? p.w0[h * D + c] : 0.f;
    uss[c] = c < D ? p.u[h * D + c] : 0.f;
  }
  constexpr int E = 16 / sizeof(T);
  const bool vec = D % 8 == 0 && p.ld % 8 == 0;
  auto stage_tile = [&](int s, int t) {
    T* raw = reinterpret_cast<T*>(smb + s * Z::RAW);
    float* wr = reinterpret_cast<float*>(raw + Z::TT * (2 * Z::DP + Z::NC));
    const T* src = reinterpret_cast<const T*>(p.rkvg) + (row0 + t) * p.ld + h * D;
    const float* wsrc = p.w_raw + static_cast<long long>(row0 + t) * HD + h * D;
    if (vec) {
      for (int i = threadIdx.x; i < Z::TT * 2 * (Z::DP / E); i += SC_WARPS * 32) {
        const int tk = i / (2 * (Z::DP / E)), r = i - tk * 2 * (Z::DP / E), w = r / (Z::DP / E), c = (r - w * (Z::DP / E)) * E;
        const bool ok = t + tk < n && c < D;
        cp_async16(raw + (tk * 2 + w) * Z::DP + c, ok ? src + tk * p.ld + w * HD + c : p.rkvg, ok);
      }
      for (int i = threadIdx.x; i < Z::TT * (Z::NC / E); i += SC_WARPS * 32) {
        const int tk = i / (Z::NC / E), c = (i - tk * (Z::NC / E)) * E;
        const bool ok = t + tk < n && col_cta + c < D;
        cp_async16(raw + Z::TT * 2 * Z::DP + tk * Z::NC + c, ok ? src + tk * p.ld + 2 * HD + col_cta + c : p.rkvg, ok);
      }
      for (int i = threadIdx.x; i < Z::TT * (Z::DP / 4); i += SC_WARPS * 32) {
        const int tk = i / (Z::DP / 4), c = (i - tk * (Z::DP / 4)) * 4;
        const bool ok = t + tk < n && c < D;
        cp_async16(wr + tk * Z::DP + c, ok ? wsrc + static_cast<long long>(tk) * HD + c : p.w_raw, ok);
      }
    } else {
      const T zero = from_f32<T>(0.f);
      for (int i = threadIdx.x; i < Z::TT * 2 * Z::DP; i += SC_WARPS * 32) {
        const int tk = i / (2 * Z::DP), r = i - tk * 2 * Z::DP, w = r / Z::DP, c = r - w * Z::DP;
        raw[i] = t + tk < n && c < D ? src[tk * p.ld + w * HD + c] : zero;
      }
      for (int i = threadIdx.x; i < Z::TT * Z::NC; i += SC_WARPS * 32) {
        const int tk = i / Z::NC, c = i - tk * Z::NC;
        raw[Z::TT * 2 * Z::DP + i] = t + tk < n && col_cta + c < D ? src[tk * p.ld + 2 * HD + col_cta + c] : zero;
      }
      for (int i = threadIdx.x; i < Z::TT * Z::DP; i += SC_WARPS * 32) {
        const int tk = i / Z::DP, c = i - tk * Z::DP;
        wr[i] = t + tk < n && c < D ? wsrc[static_cast<long long>(tk) * HD + c] : 0.f;
      }
    }
    cp_commit();
  };

  uint64_t S[4][4];
  const int prev = p.row_prev[row0];
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = (j >> 1) * LANES * 4 + rl * 4 + (j & 1) * 2;
      float a = 0.f, b = 0.f;
      if (prev >= 0 && col0 + c < D) {
        const float* src = p.state + prev * p.state_ld + p.s_off + static_cast<long long>(h) * D * D + col0 + c;
        if (r < D) a = src[static_cast<long long>(r) * D];
        if (r + 1 < D) b = src[static_cast<long long>(r + 1) * D];
      }
      S[c][j] = pack2(a, b);
    }

  stage_tile(0, 0);
  int s = 0;
  for (int t = 0; t < n; t += Z::TT, s ^= 1) {
    if (t + Z::TT < n) {
      stage_tile(s ^ 1, t + Z::TT);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    {
      const T* raw = reinterpret_cast<const T*>(smb + s * Z::RAW);
      const float* wr = reinterpret_cast<const float*>(raw + Z::TT * (2 * Z::DP + Z::NC));
      for (int tk = warp; tk < Z::TT; tk += SC_WARPS) {
        float dot = 0.f;
        for (int c = lane; c < Z::DP; c += 32) {
          const float r = to_f32(raw[tk * 2 * Z::DP + c]), k = to_f32(raw[(tk * 2 + 1) * Z::DP + c]);
          tile[tk * 3 * Z::DP + c] = r;
          tile[(tk * 3 + 1) * Z::DP + c] = k;
          tile[(tk * 3 + 2) * Z::DP + c] = expf(-expf(wr[tk * Z::DP + c] + w0s[c]));
          dot += r * uss[c] * k;
        }
        dot = warp_sum(dot);
        if (lane == 0) rk[tk] = dot;
        for (int c = lane; c < Z::NC; c += 32) vt[tk * Z::NC + c] = to_f32(raw[Z::TT * 2 * Z::DP + tk * Z::NC + c]);
      }
    }
    __syncthreads();
    const int m = min(n - t, Z::TT);
    for (int b0 = 0; b0 < m; b0 += 8) {
      float v[32];                                       // [token of the block][column]
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (b0 + i < m) {
          const float* src = tile + (b0 + i) * 3 * Z::DP + rl * 4;
          const ulonglong2 ra = *reinterpret_cast<const ulonglong2*>(src), rb = *reinterpret_cast<const ulonglong2*>(src + LANES * 4);
          const ulonglong2 ka = *reinterpret_cast<const ulonglong2*>(src + Z::DP), kb = *reinterpret_cast<const ulonglong2*>(src + Z::DP + LANES * 4);
          const ulonglong2 da = *reinterpret_cast<const ulonglong2*>(src + 2 * Z::DP), db = *reinterpret_cast<const ulonglong2*>(src + 2 * Z::DP + LANES * 4);
          const float4 f = *reinterpret_cast<const float4*>(vt + (b0 + i) * Z::NC + wc + cg * 4);
          const uint64_t w[4] = {pack2(f.x, f.x), pack2(f.y, f.y), pack2(f.z, f.z), pack2(f.w, f.w)};
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float2 d = unpack2(fma2(S[c][3], rb.y, fma2(S[c][2], rb.x, fma2(S[c][1], ra.y, mul2(S[c][0], ra.x)))));
            v[i * 4 + c] = d.x + d.y;
            S[c][0] = fma2(S[c][0], da.x, mul2(ka.x, w[c]));
            S[c][1] = fma2(S[c][1], da.y, mul2(ka.y, w[c]));
            S[c][2] = fma2(S[c][2], db.x, mul2(kb.x, w[c]));
            S[c][3] = fma2(S[c][3], db.y, mul2(kb.y, w[c]));
          }
        } else {
#pragma unroll
          for (int c = 0; c < 4; ++c) v[i * 4 + c] = 0.f;
        }
      }
      reduce_scatter<LANES>(v, rl);
#pragma unroll
      for (int e = 0; e < 32 / LANES; ++e) {
        const int idx = rl * (32 / LANES) + e;
        xs[(idx >> 2) * Z::NCW + cg * 4 + (idx & 3)] = v[e];
      }
      __syncwarp();
#pragma unroll
      for (int x = 0; x < (8 * Z::NCW + 31) / 32; ++x) {
        const int idx = x * 32 + lane, i = idx / Z::NCW, c = idx % Z::NCW;
        if (idx < 8 * Z::NCW && b0 + i < m && col_cta + wc + c < D)
          p.o[static_cast<long long>(row0 + t + b0 + i) * HD + h * D + col_cta + wc + c] =
              xs[i * Z::NCW + c] + rk[b0 + i] * vt[(b0 + i) * Z::NC + wc + c];
      }
      __syncwarp();
    }
    __syncthreads();
  }
  const int next = p.row_next[row0 + n - 1];
  if (next >= 0) {
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = (j >> 1) * LANES * 4 + rl * 4 + (j & 1) * 2;
        const float2 d = unpack2(S[c][j]);
        if (col0 + c < D) {
          float* dst = p.state + next * p.state_ld + p.s_off + static_cast<long long>(h) * D * D + col0 + c;
          if (r < D) dst[static_cast<long long>(r) * D] = d.x;
          if (r + 1 < D) dst[static_cast<long long>(r + 1) * D] = d.y;
        }
      }
  }
}

// ---------------------------------------------------------------------------------------------------------
// scan of portions in bf16 models: blocks of eight tokens on the tensor cores, operands split into two TF32 parts (three
// products), which keeps fp32 accuracy
//
// Within a block (states S0 -> S8, gamma_i the decay from the block's start to token i, inclusive):
//   delta rule   U = T (V - gamma S0^T K),  T = (I + L)^-1 diag(beta),  L_ij = beta_i gamma_i / gamma_j (k_i . k_j)  (j < i)
//                O = gamma S0^T Q + A U,    A_ij = gamma_i / gamma_j (q_i . k_j)                               (j <= i)
//                S8 = gamma_8 S0 + K^T diag(gamma_8 / gamma_j) U
//   WKV          O = S0^T R~ + A V,         R~_i = r_i gamma_(i-1),  A_ij = sum_d r_id k_jd gamma_(i-1)d / gamma_jd  (j < i)
//                S8 = diag(gamma_8) S0 + K~^T V,  K~_j = k_j gamma_8 / gamma_j;  A_ii = sum_d r_id u_d k_id
//   retention    as WKV with R~_i = q_i g^(i+1), A_ij = g^(i-j) (q_i . k_j)  (j <= i), one decay g^8 for all key rows
// T, A and (WKV, retention) R~, K~ depend on the inputs alone and come from a launch over all blocks at once.  Every decay above is a
// product of factors <= 1 formed directly, never a quotient.
//
// A warp owns 16 value columns x 8 NT key rows of S^T as MMA accumulators.  The accumulator layout (column g, rows 2t and
// 2t + 1) IS the layout of an A operand if the reduction index is renumbered (t -> 2t, t + 4 -> 2t + 1), the same way for
// the B operand; so S, the products with it and U go from one MMA to the next in registers, without a shuffle.
// WR warps share the key rows of 16 columns and add their partial products through shared memory.
// ---------------------------------------------------------------------------------------------------------
constexpr int BS_BLOCK = 8;                // tokens of a block
constexpr int BS_TILE = 32;                // tokens staged at a time
constexpr int BS_COEF = 144;               // delta rule, per block and head: T [8][8], A [8][8], gamma [8], gamma_8 / gamma_j [8]
constexpr int BS_COEF_WKV = 64;            // WKV: A [8][8] (the decay of the key rows is kept beside it)
constexpr int BS_COEF_RET = 68;            // retention: A [8][8], decay of the block, padding
enum { SCAN_WKV = 0, SCAN_DELTA = 1, SCAN_RETENTION = 2 };

struct BlockScanParams {
  const float* q;              // first row, head 0; row stride below
  const float* k;
  const void* v;
  long long qk_ld, v_ld;
  int rep;                     // heads per query / key head
  const float* coef;           // [blocks][H][BS_COEF, BS_COEF_WKV or BS_COEF_RET]
  const float* row_decay;      // WKV: [blocks][H][D]
  float* state;
  long long state_ld;
  int s_off;
  const int* row_prev;
  const int* row_next;
  const int* cu;
  float* o;                    // [rows][H V]
  int H, D, V;
};

// block 0 of portion z; the portions' ranges do not overlap
__device__ __forceinline__ long long first_block(const int* cu, int z) { return cu[z] / BS_BLOCK + z; }

// x = hi + lo exactly: hi keeps the 11 leading bits (a TF32 number), lo the other 13, of which the product uses 11
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// A operand of an accumulator tile
__device__ __forceinline__ void split_tile(const float (&c)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split_tf32(c[0], hi[0], lo[0]);
  split_tf32(c[2], hi[1], lo[1]);
  split_tf32(c[1], hi[2], lo[2]);
  split_tf32(c[3], hi[3], lo[3]);
}
// B operand of two values, split
struct SplitB {
  uint32_t h0, h1, l0, l1;
  __device__ __forceinline__ SplitB() {}
  __device__ __forceinline__ SplitB(float b0, float b1) {
    split_tf32(b0, h0, l0);
    split_tf32(b1, h1, l1);
  }
};
// the three products of a split A operand with a split B operand, each into an accumulator of its own: no product waits for
// the one before
__device__ __forceinline__ void mma_split(float (&c)[3][4], const uint32_t (&hi)[4], const uint32_t (&lo)[4], const SplitB& b) {
  mma_tf32(c[0], hi, b.h0, b.h1);
  mma_tf32(c[1], hi, b.l0, b.l1);
  mma_tf32(c[2], lo, b.h0, b.h1);
}
__device__ __forceinline__ void zero_acc(float (&c)[3][4]) {
#pragma unroll
  for (int i = 0; i < 3; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) c[i][e] = 0.f;
}

template <int KIND, int NT, int WR, typename TV> struct BlockScan {
  static constexpr int WC = 4 / WR;                    // column groups of a CTA
  static constexpr int NC = 16 * WC;
  static constexpr int DP = 8 * NT * WR;               // key rows, padded
  static constexpr int KS = DP + 4;
  static constexpr int VS = NC + 8;
  static constexpr int CO = KIND == SCAN_DELTA ? BS_COEF : (KIND == SCAN_WKV ? BS_COEF_WKV + DP : BS_COEF_RET);
  static constexpr int QK = BS_TILE * 2 * KS * 4, VB = BS_TILE * VS * static_cast<int>(sizeof(TV));     // bytes
  static constexpr int STAGE = QK + VB + BS_TILE / BS_BLOCK * CO * 4;
  static constexpr int EX = WR > 1 ? 2 * 4 * 32 * 8 * 4 : 0;      // two blocks' partial products of the four warps
  static constexpr size_t SMEM = 2 * STAGE + EX;
};

// grid (column tiles, H, portions)
template <int KIND, int NT, int WR, typename TV>
__global__ void __launch_bounds__(128, 2) block_scan_kernel(BlockScanParams p) {
  using Z = BlockScan<KIND, NT, WR, TV>;
  constexpr bool DELTA = KIND == SCAN_DELTA;
  constexpr int XT = NT < 4 ? NT : 4;
  extern __shared__ __align__(16) uint8_t smb[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int wr = warp % WR, wc = warp / WR;
  const int h = blockIdx.y, g = h / p.rep, col_cta = blockIdx.x * Z::NC;
  const int row0 = p.cu[blockIdx.z], n = p.cu[blockIdx.z + 1] - row0;
  if (n <= 0) return;
  const long long block0 = first_block(p.cu, blockIdx.z);
  const int r_first = wr * NT * 8;                       // this warp's key rows
  const int c0 = col_cta + wc * 16 + gid;                // and value columns c0, c0 + 8
  const TV* vsrc = reinterpret_cast<const TV*>(p.v);

  auto stage_tile = [&](int s, int t) {
    float* qk = reinterpret_cast<float*>(smb + s * Z::STAGE);
    TV* vt = reinterpret_cast<TV*>(smb + s * Z::STAGE + Z::QK);
    float* co = reinterpret_cast<float*>(smb + s * Z::STAGE + Z::QK + Z::VB);
    constexpr int U = Z::DP / 4;
    for (int i = threadIdx.x; i < BS_TILE * 2 * U; i += 128) {
      const int tk = i / (2 * U), r = i - tk * 2 * U, w = r / U, c = (r - w * U) * 4;
      const bool ok = t + tk < n && c < p.D;
      const float* src = (w ? p.k : p.q) + (row0 + t + tk) * p.qk_ld + g * p.D + c;
      cp_async16(qk + (tk * 2 + w) * Z::KS + c, ok ? src : p.q, ok);
    }
    constexpr int E = 16 / sizeof(TV);
    for (int i = threadIdx.x; i < BS_TILE * (Z::NC / E); i += 128) {
      const int tk = i / (Z::NC / E), c = (i - tk * (Z::NC / E)) * E;
      const bool ok = t + tk < n && col_cta + c < p.V;
      cp_async16(vt + tk * Z::VS + c, ok ? vsrc + (row0 + t + tk) * p.v_ld + h * p.V + col_cta + c : vsrc, ok);
    }
    constexpr int CU = Z::CO / 4;
    for (int i = threadIdx.x; i < BS_TILE / BS_BLOCK * CU; i += 128) {
      const int b = i / CU, c = (i - b * CU) * 4;
      const bool in = t + b * BS_BLOCK < n;
      const long long at = (block0 + t / BS_BLOCK + b) * p.H + h;
      if (DELTA) {
        cp_async16(co + b * Z::CO + c, in ? p.coef + at * BS_COEF + c : p.coef, in);
      } else if (KIND == SCAN_RETENTION) {
        cp_async16(co + b * Z::CO + c, in ? p.coef + at * BS_COEF_RET + c : p.coef, in);
      } else {
        const bool mat = c < BS_COEF_WKV, ok = in && (mat || c - BS_COEF_WKV < p.D);
        cp_async16(co + b * Z::CO + c,
                   !ok ? p.coef : (mat ? p.coef + at * BS_COEF_WKV + c : p.row_decay + at * p.D + c - BS_COEF_WKV), ok);
      }
    }
    cp_commit();
  };

  float S[NT][4];
  const int prev = p.row_prev[row0];
  const float* s_in = p.state + (prev >= 0 ? prev * p.state_ld : 0) + p.s_off + static_cast<long long>(h) * p.D * p.V;
#pragma unroll
  for (int x = 0; x < NT; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r_first + x * 8 + tig * 2 + (e & 1), c = c0 + (e >> 1) * 8;
      S[x][e] = prev >= 0 && r < p.D && c < p.V ? s_in[static_cast<long long>(r) * p.V + c] : 0.f;
    }

  stage_tile(0, 0);
  int s = 0, parity = 0;
  for (int t = 0; t < n; t += BS_TILE, s ^= 1) {
    cp_wait<0>();
    __syncthreads();                                     // the tile is here; nobody reads the other stage any more
    if (t + BS_TILE < n) stage_tile(s ^ 1, t + BS_TILE);
    const float* qk = reinterpret_cast<const float*>(smb + s * Z::STAGE);
    const TV* vt = reinterpret_cast<const TV*>(smb + s * Z::STAGE + Z::QK);
    const float* cof = reinterpret_cast<const float*>(smb + s * Z::STAGE + Z::QK + Z::VB);
    const int blocks = (min(n - t, BS_TILE) + BS_BLOCK - 1) / BS_BLOCK;
    for (int b = 0; b < blocks; ++b) {
      const float* tok = qk + b * BS_BLOCK * 2 * Z::KS + r_first;            // [token][q, k][row]
      const float* co = cof + b * Z::CO;
      const float* A = co + (DELTA ? 64 : 0);
      const float2 av = *reinterpret_cast<const float2*>(A + gid * 8 + tig * 2);
      float2 tv, gm, rt;
      float g8 = 1.f;
      if (DELTA) {
        tv = *reinterpret_cast<const float2*>(co + gid * 8 + tig * 2);
        gm = *reinterpret_cast<const float2*>(co + 128 + tig * 2);
        rt = *reinterpret_cast<const float2*>(co + 136 + tig * 2);
        g8 = co[128 + 7];
      }
      if (KIND == SCAN_RETENTION) g8 = co[64];
      float u[4];                                        // v, then U: column g (g + 8), tokens 2t, 2t + 1
      {
        const TV* vv = vt + (b * BS_BLOCK + tig * 2) * Z::VS + wc * 16 + gid;
        u[0] = to_f32(vv[0]);
        u[1] = to_f32(vv[Z::VS]);
        u[2] = to_f32(vv[8]);
        u[3] = to_f32(vv[Z::VS + 8]);
      }
      // products with the state before the block
      float xk[4], xq[4];
      {
        float ck[3][4], cq[3][4];
        zero_acc(ck);
        zero_acc(cq);
#pragma unroll
        for (int x = 0; x < NT; ++x) {
          uint32_t hi[4], lo[4];
          split_tile(S[x], hi, lo);
          const float* src = tok + gid * 2 * Z::KS + x * 8 + tig * 2;
          if (DELTA) {
            const float2 kv = *reinterpret_cast<const float2*>(src + Z::KS);
            mma_split(ck, hi, lo, SplitB(kv.x, kv.y));
          }
          const float2 qv = *reinterpret_cast<const float2*>(src);
          mma_split(cq, hi, lo, SplitB(qv.x, qv.y));
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          xk[e] = ck[0][e] + (ck[1][e] + ck[2][e]);
          xq[e] = cq[0][e] + (cq[1][e] + cq[2][e]);
        }
      }
      if (WR > 1) {                                      // sum over the warps that share the columns, in a fixed order
        float4* ex = reinterpret_cast<float4*>(smb + 2 * Z::STAGE) + parity * 4 * 64;
        if (DELTA) ex[warp * 64 + lane] = make_float4(xk[0], xk[1], xk[2], xk[3]);
        ex[warp * 64 + 32 + lane] = make_float4(xq[0], xq[1], xq[2], xq[3]);
        if (wc == 0) asm volatile("bar.sync 1, %0;" ::"n"(WR * 32) : "memory");
        else asm volatile("bar.sync 2, %0;" ::"n"(WR * 32) : "memory");
#pragma unroll
        for (int w = 0; w < WR; ++w) {
          const float4 a = ex[(wc * WR + w) * 64 + 32 + lane];
          xq[0] = w ? xq[0] + a.x : a.x; xq[1] = w ? xq[1] + a.y : a.y;
          xq[2] = w ? xq[2] + a.z : a.z; xq[3] = w ? xq[3] + a.w : a.w;
          if (DELTA) {
            const float4 k4 = ex[(wc * WR + w) * 64 + lane];
            xk[0] = w ? xk[0] + k4.x : k4.x; xk[1] = w ? xk[1] + k4.y : k4.y;
            xk[2] = w ? xk[2] + k4.z : k4.z; xk[3] = w ? xk[3] + k4.w : k4.w;
          }
        }
        parity ^= 1;
      }
      uint32_t uh[4], ul[4], wh[4], wl[4];               // U; U with the decay to the block's end
      if (DELTA) {
        u[0] -= gm.x * xk[0]; u[1] -= gm.y * xk[1]; u[2] -= gm.x * xk[2]; u[3] -= gm.y * xk[3];
        split_tile(u, uh, ul);
        float c[3][4];
        zero_acc(c);
        mma_split(c, uh, ul, SplitB(tv.x, tv.y));
#pragma unroll
        for (int e = 0; e < 4; ++e) u[e] = c[0][e] + (c[1][e] + c[2][e]);
        split_tile(u, uh, ul);
        u[0] *= rt.x; u[1] *= rt.y; u[2] *= rt.x; u[3] *= rt.y;
        split_tile(u, wh, wl);
      } else {
        split_tile(u, uh, ul);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          wh[e] = uh[e];
          wl[e] = ul[e];
        }
      }
      const float* kt = tok + Z::KS;
#pragma unroll
      for (int x0 = 0; x0 < NT; x0 += XT) {              // XT row tiles at a time: their products interleave
        SplitB kb[XT];
#pragma unroll
        for (int x = 0; x < XT; ++x) {
          const float* src = kt + tig * 4 * Z::KS + (x0 + x) * 8 + gid;
          kb[x] = SplitB(src[0], src[2 * Z::KS]);
          float (&s4)[4] = S[x0 + x];
          if (KIND != SCAN_WKV) {
#pragma unroll
            for (int e = 0; e < 4; ++e) s4[e] *= g8;
          } else {
            const float2 pd = *reinterpret_cast<const float2*>(co + BS_COEF_WKV + r_first + (x0 + x) * 8 + tig * 2);
            s4[0] *= pd.x; s4[1] *= pd.y; s4[2] *= pd.x; s4[3] *= pd.y;
          }
        }
#pragma unroll
        for (int x = 0; x < XT; ++x) mma_tf32(S[x0 + x], wh, kb[x].l0, kb[x].l1);
#pragma unroll
        for (int x = 0; x < XT; ++x) mma_tf32(S[x0 + x], wl, kb[x].h0, kb[x].h1);
#pragma unroll
        for (int x = 0; x < XT; ++x) mma_tf32(S[x0 + x], wh, kb[x].h0, kb[x].h1);
      }
      if (wr == 0) {
        float c[3][4];
        zero_acc(c);
        mma_split(c, uh, ul, SplitB(av.x, av.y));
        if (DELTA) {
          xq[0] *= gm.x; xq[1] *= gm.y; xq[2] *= gm.x; xq[3] *= gm.y;
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int tt = t + b * BS_BLOCK + tig * 2 + (e & 1), cc = c0 + (e >> 1) * 8;
          if (tt < n && cc < p.V)
            p.o[static_cast<long long>(row0 + tt) * p.H * p.V + h * p.V + cc] = (xq[e] + c[0][e]) + (c[1][e] + c[2][e]);
        }
      }
    }
  }
  const int next = p.row_next[row0 + n - 1];
  if (next >= 0) {
    float* s_out = p.state + next * p.state_ld + p.s_off + static_cast<long long>(h) * p.D * p.V;
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = r_first + x * 8 + tig * 2 + (e & 1), c = c0 + (e >> 1) * 8;
        if (r < p.D && c < p.V) s_out[static_cast<long long>(r) * p.V + c] = S[x][e];
      }
  }
}

// T, A, gamma of every block of the delta rule, one warp per (block, query / key head): k_i . k_j and q_i . k_j are one MMA
// with the rows [K; Q] and the columns K, whose operands are read once, straight from global memory.
// grid (blocks of the longest portion, ceil(G / 4), portions)
__global__ void __launch_bounds__(128) delta_blocks_kernel(const float* __restrict__ qkv, const float* __restrict__ gates,
                                                           const int* __restrict__ cu, float* __restrict__ coef, int H, int G,
                                                           int D, int V) {
  __shared__ float lower[4][8][9];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int z = blockIdx.z, g = blockIdx.y * 4 + warp, rep = H / G, C = 2 * G * D + H * V;
  const int row0 = cu[z] + blockIdx.x * BS_BLOCK, n = min(BS_BLOCK, cu[z + 1] - row0);
  if (n <= 0 || g >= G) return;
  const long long block = first_block(cu, z) + blockIdx.x;
  float (&Lm)[8][9] = lower[warp];
  float dots[3][4];                                      // k_i . k_j (0, 1) and q_i . k_j (2, 3): i = gid, j = 2 tig, 2 tig + 1
  zero_acc(dots);
  {
    const bool in = gid < n;
    const float* q = qkv + static_cast<long long>(row0 + (in ? gid : 0)) * C + g * D + tig * 2;
    const float* k = q + G * D;
    for (int c0 = 0; c0 < D; c0 += 64) {
      float2 qv[8], kv[8];
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const bool ok = in && c0 + x * 8 < D;
        qv[x] = ok ? *reinterpret_cast<const float2*>(q + c0 + x * 8) : make_float2(0.f, 0.f);
        kv[x] = ok ? *reinterpret_cast<const float2*>(k + c0 + x * 8) : make_float2(0.f, 0.f);
      }
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const SplitB b(kv[x].x, kv[x].y);
        uint32_t hi[4] = {b.h0, 0, b.h1, 0}, lo[4] = {b.l0, 0, b.l1, 0};
        split_tf32(qv[x].x, hi[1], lo[1]);
        split_tf32(qv[x].y, hi[3], lo[3]);
        mma_split(dots, hi, lo, b);
      }
    }
  }
  float d[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) d[e] = dots[0][e] + (dots[1][e] + dots[2][e]);
  const int j0 = tig * 2;
  for (int hh = 0; hh < rep; ++hh) {
    const int h = g * rep + hh;
    float lg = 0.f, bt = 0.f;                            // of token `lane`
    if (lane < n) {
      lg = gates[static_cast<long long>(row0 + lane) * 2 * H + h];
      bt = gates[static_cast<long long>(row0 + lane) * 2 * H + H + h];
    }
    float e0 = 0.f, e1 = 0.f, head = 0.f, tail = 0.f;    // sums of log decays: j + 1 .. i; start .. lane; lane + 1 .. end
#pragma unroll
    for (int l = 0; l < 8; ++l) {
      const float v = __shfl_sync(0xffffffffu, lg, l);
      if (l > j0 && l <= gid) e0 += v;
      if (l > j0 + 1 && l <= gid) e1 += v;
      if (l <= lane) head += v;
      else tail += v;
    }
    e0 = expf(e0);
    e1 = expf(e1);
    const float bi = __shfl_sync(0xffffffffu, bt, gid);
    float* out = coef + (block * H + h) * BS_COEF;
    Lm[gid][j0] = bi * e0 * d[0];
    Lm[gid][j0 + 1] = bi * e1 * d[1];
    *reinterpret_cast<float2*>(out + 64 + gid * 8 + j0) = make_float2(j0 <= gid ? e0 * d[2] : 0.f, j0 + 1 <= gid ? e1 * d[3] : 0.f);
    if (lane < 8) {
      out[128 + lane] = expf(head);
      out[136 + lane] = expf(tail);
    }
    __syncwarp();
    if (lane < 8) {                                      // column `lane` of (I + L)^-1, times beta
      float col[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float v = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int l = 0; l < 8; ++l)
          if (l < i) v -= Lm[i][l] * col[l];
        col[i] = i < lane ? 0.f : v;
        out[i * 8 + lane] = col[i] * bt;
      }
    }
    __syncwarp();
  }
}

// R~, K~, A and the decay of every block of the WKV recurrence: one warp per (block, head).  grid (blocks of the longest
// portion, ceil(H / 4), portions).
template <typename T>
__global__ void __launch_bounds__(128, 3) wkv_blocks_kernel(WkvParams p, float* __restrict__ rt, float* __restrict__ kt,
                                                         float* __restrict__ coef, float* __restrict__ row_decay) {
  const int z = blockIdx.z, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = p.D, HD = p.H * D;
  const int row0 = p.cu[z] + blockIdx.x * BS_BLOCK, n = min(BS_BLOCK, p.cu[z + 1] - row0);
  if (n <= 0 || h >= p.H) return;
  const long long at = (first_block(p.cu, z) + blockIdx.x) * p.H + h;
  float low[32], diag[8];                                // A below the diagonal (28 values) and on it
#pragma unroll
  for (int i = 0; i < 32; ++i) low[i] = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) diag[i] = 0.f;
  const T* x = reinterpret_cast<const T*>(p.rkvg) + row0 * p.ld + h * D;
  const float* raw = p.w_raw + static_cast<long long>(row0) * HD + h * D;
  for (int c = lane * 2; c < D; c += 64) {               // two neighbouring channels per lane
    float r[8][2], k[8][2], w[8][2];
#pragma unroll
    for (int i = 0; i < 8; ++i) {                        // all loads of the block at once
      const int ii = min(i, n - 1);
      const float2 rr = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x + ii * p.ld + c));
      const float2 kk = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x + ii * p.ld + HD + c));
      const float2 ww = *reinterpret_cast<const float2*>(raw + static_cast<long long>(ii) * HD + c);
      r[i][0] = rr.x; r[i][1] = rr.y; k[i][0] = kk.x; k[i][1] = kk.y; w[i][0] = ww.x; w[i][1] = ww.y;
    }
    const float2 w0 = *reinterpret_cast<const float2*>(p.w0 + h * D + c), uu = *reinterpret_cast<const float2*>(p.u + h * D + c);
    float head[2] = {1.f, 1.f}, tail[2] = {1.f, 1.f};
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool in = i < n;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        r[i][e] = in ? r[i][e] : 0.f;
        k[i][e] = in ? k[i][e] : 0.f;
        w[i][e] = in ? __expf(-__expf(w[i][e] + (e ? w0.y : w0.x))) : 1.f;
        diag[i] += r[i][e] * (e ? uu.y : uu.x) * k[i][e];
      }
      if (in) *reinterpret_cast<float2*>(rt + static_cast<long long>(row0 + i) * HD + h * D + c) = make_float2(r[i][0] * head[0], r[i][1] * head[1]);
      head[0] *= w[i][0];
      head[1] *= w[i][1];
    }
    *reinterpret_cast<float2*>(row_decay + at * D + c) = make_float2(head[0], head[1]);
#pragma unroll
    for (int j = 7; j >= 0; --j) {
      if (j < n) *reinterpret_cast<float2*>(kt + static_cast<long long>(row0 + j) * HD + h * D + c) = make_float2(k[j][0] * tail[0], k[j][1] * tail[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        tail[e] *= w[j][e];
        float f = k[j][e];
#pragma unroll
        for (int i = j + 1; i < 8; ++i) {
          low[i * (i - 1) / 2 + j] += r[i][e] * f;
          f *= w[i][e];
        }
      }
    }
  }
  reduce_scatter<32>(low, lane);                         // lane l holds entry l
#pragma unroll
  for (int i = 0; i < 8; ++i) diag[i] = warp_sum(diag[i]);
  float* A = coef + at * BS_COEF_WKV;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (lane >= i * (i - 1) / 2 && lane < i * (i + 1) / 2) A[i * 8 + lane - i * (i - 1) / 2] = low[0];
    if (lane >= i && lane < 8) A[i * 8 + lane] = lane == i ? diag[i] : 0.f;
  }
}

// ---------------------------------------------------------------------------------------------------------
// retention
// ---------------------------------------------------------------------------------------------------------
struct RetentionParams {
  const void* proj;            // rows [q H x D | k H x D | v H x V | gate H x V]
  long long ld;
  const float* angles;         // [rows][cos (rot / 2) | sin (rot / 2)]
  const float* powers;         // [H][powers_ld] g^0, g^1, ... (BS_BLOCK + 1 of them at least)
  int powers_ld;
  float k_scale, eps;
  float* state;
  long long state_ld;
  const int* row_prev;
  const int* row_next;
  const int* cu;               // portions
  float* o;                    // portions: [rows][H V]
  void* out;                   // decoding: [rows][out_ld]
  long long out_ld;
  int rows, H, D, V, rot;
};
// coordinate c of a head whose projected row is x, rotated (halves) and scaled
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int c, int rot, const float* cs, float scale) {
  const int half = rot / 2;
  float v = to_f32(x[c]);
  if (c < half) v = v * cs[c] - to_f32(x[c + half]) * cs[half + c];
  else if (c < rot) v = v * cs[c - half] + to_f32(x[c - half]) * cs[c];
  return v * scale;
}

// Plain fp32 scan.  grid (ceil(V / 32), H, portions); a warp owns NR key rows of 32 value columns, a lane one column.
constexpr int RT_TILE = 8;                 // tokens staged at a time
template <typename T, int NR>
__global__ void __launch_bounds__(256) retention_scan_kernel(RetentionParams p) {
  constexpr int DP = NR * 8;
  __shared__ __align__(16) float qs[RT_TILE][DP], ks[RT_TILE][DP];
  __shared__ float vs[RT_TILE][32], part[RT_TILE][8][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, col = blockIdx.x * 32 + lane;
  const int row0 = p.cu[blockIdx.z], n = p.cu[blockIdx.z + 1] - row0, D = p.D, V = p.V;
  if (n <= 0) return;
  const int prev = p.row_prev[row0], next = p.row_next[row0 + n - 1];
  const float g = p.powers[h * p.powers_ld + 1];
  const long long head = static_cast<long long>(h) * D * V;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = warp * NR + i;
    S[i] = prev >= 0 && r < D && col < V ? p.state[prev * p.state_ld + head + static_cast<long long>(r) * V + col] : 0.f;
  }
  for (int t = 0; t < n; t += RT_TILE) {
    const int m = min(RT_TILE, n - t);
    for (int i = threadIdx.x; i < RT_TILE * DP; i += 256) {
      const int tk = i / DP, c = i - tk * DP;
      const long long row = row0 + t + min(tk, m - 1);
      const T* x = reinterpret_cast<const T*>(p.proj) + row * p.ld + h * D;
      const float* cs = p.angles + row * p.rot;
      qs[tk][c] = c < D ? rotated(x, c, p.rot, cs, 1.f) : 0.f;
      ks[tk][c] = c < D ? rotated(x + p.H * D, c, p.rot, cs, p.k_scale) : 0.f;
    }
    {
      const T* x = reinterpret_cast<const T*>(p.proj) + (row0 + t + min(warp, m - 1)) * p.ld + 2 * p.H * D + h * V;
      vs[warp][lane] = col < V ? to_f32(x[col]) : 0.f;
    }
    __syncthreads();
    for (int tk = 0; tk < m; ++tk) {
      const float v = vs[tk][lane];
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < NR; i += 4) {
        const float4 q = *reinterpret_cast<const float4*>(&qs[tk][warp * NR + i]);
        const float4 k = *reinterpret_cast<const float4*>(&ks[tk][warp * NR + i]);
        S[i] = g * S[i] + k.x * v;
        S[i + 1] = g * S[i + 1] + k.y * v;
        S[i + 2] = g * S[i + 2] + k.z * v;
        S[i + 3] = g * S[i + 3] + k.w * v;
        acc += (S[i] * q.x + S[i + 1] * q.y) + (S[i + 2] * q.z + S[i + 3] * q.w);
      }
      part[tk][warp][lane] = acc;
    }
    __syncthreads();
    if (warp < m && col < V) {             // warp: token
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += part[warp][w][lane];
      p.o[static_cast<long long>(row0 + t + warp) * p.H * V + h * V + col] = s;
    }
  }
  if (next >= 0) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = warp * NR + i;
      if (r < D && col < V) p.state[next * p.state_ld + head + static_cast<long long>(r) * V + col] = S[i];
    }
  }
}

// R~, K~, A and decay of every block, one warp per (block, head); a lane holds key channels lane, lane + 32, ...
// grid (blocks of the longest portion, ceil(H / 4), portions); dynamic shared memory [4 warps][q, k][8][D + 1].
__global__ void __launch_bounds__(128) retention_blocks_kernel(RetentionParams p, float* __restrict__ rt, float* __restrict__ kt,
                                                               float* __restrict__ coef) {
  extern __shared__ __align__(16) float smf[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, z = blockIdx.z, h = blockIdx.y * 4 + warp;
  const int row0 = p.cu[z] + blockIdx.x * BS_BLOCK, n = min(BS_BLOCK, p.cu[z + 1] - row0);
  if (n <= 0 || h >= p.H) return;
  const int D = p.D, ds = D + 1;
  float* qs = smf + warp * 2 * BS_BLOCK * ds;
  float* ks = qs + BS_BLOCK * ds;
  const float* pw = p.powers + h * p.powers_ld;
  const long long at = (first_block(p.cu, z) + blockIdx.x) * p.H + h;
  for (int c = lane; c < D; c += 32) {
#pragma unroll
    for (int i = 0; i < BS_BLOCK; ++i) {
      float q = 0.f, k = 0.f;
      if (i < n) {
        const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.proj) + (row0 + i) * p.ld + h * D;
        const float* cs = p.angles + static_cast<long long>(row0 + i) * p.rot;
        q = rotated(x, c, p.rot, cs, 1.f);
        k = rotated(x + p.H * D, c, p.rot, cs, p.k_scale);
        const long long to = static_cast<long long>(row0 + i) * p.H * D + h * D + c;
        rt[to] = q * pw[i + 1];
        kt[to] = k * pw[n - 1 - i];
      }
      qs[i * ds + c] = q;
      ks[i * ds + c] = k;
    }
  }
  __syncwarp();
  const int i = lane >> 2, j = (lane & 3) * 2;           // A[i][j], A[i][j + 1]
  float d0 = 0.f, d1 = 0.f;
#pragma unroll 8
  for (int c = 0; c < D; ++c) {
    const float q = qs[i * ds + c];
    d0 += q * ks[j * ds + c];
    d1 += q * ks[(j + 1) * ds + c];
  }
  float* out = coef + at * BS_COEF_RET;
  *reinterpret_cast<float2*>(out + i * 8 + j) = make_float2(j <= i ? d0 * pw[max(i - j, 0)] : 0.f, j + 1 <= i ? d1 * pw[max(i - j - 1, 0)] : 0.f);
  if (lane == 0) out[64] = pw[n];
}

// Single rows: projection -> gated norm, state advanced.  A cluster of CTAs per (row, head), each with its share of the value
// columns; their sums of squares meet in every CTA's shared memory.  grid (rows, H, shares), cluster (1, 1, shares).
constexpr int RTS_THREADS = 256;
constexpr int RTS_SHARES = 8;
template <typename T, int VEC>
__global__ void __launch_bounds__(RTS_THREADS) retention_step_kernel(RetentionParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float scratch[32], sums[RTS_SHARES];
  const int row = blockIdx.x, h = blockIdx.y, shares = gridDim.z, D = p.D, V = p.V / shares, v0 = blockIdx.z * V, tid = threadIdx.x;
  const int nvec = V / VEC, span = min(nvec, RTS_THREADS), groups = RTS_THREADS / span;
  float* vs = smf;                               // [V] this CTA's columns
  float* part = vs + (V + 3) / 4 * 4;            // [groups][V]
  float* qs = part + (groups * V + 3) / 4 * 4;   // [D]
  float* ks = qs + D;                            // [D]
  const int prev = p.row_prev[row], next = p.row_next[row];
  const T* x = reinterpret_cast<const T*>(p.proj) + row * p.ld;
  const float* cs = p.angles + static_cast<long long>(row) * p.rot;
  const long long head = static_cast<long long>(h) * D * p.V + v0;
  const float* S = prev >= 0 ? p.state + prev * p.state_ld + head : nullptr;
  float* N = next >= 0 ? p.state + next * p.state_ld + head : nullptr;
  const float g = p.powers[h * p.powers_ld + 1];
  for (int c = tid; c < D; c += RTS_THREADS) {
    qs[c] = rotated(x + h * D, c, p.rot, cs, 1.f);
    ks[c] = rotated(x + (p.H + h) * D, c, p.rot, cs, p.k_scale);
  }
  for (int c = tid; c < V; c += RTS_THREADS) vs[c] = to_f32(x[2 * p.H * D + h * p.V + v0 + c]);
  __syncthreads();
  const int grp = tid / span;
  for (int base = 0; base < nvec; base += span) {
    const int cv = (base + tid - grp * span) * VEC;
    if (grp >= groups || cv >= V) continue;
    float acc[VEC], v[VEC];
    load_vec<VEC>(vs + cv, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll 8
    for (int r = grp; r < D; r += groups) {
      float st[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[e] = 0.f;
      if (S) load_vec<VEC>(S + static_cast<long long>(r) * p.V + cv, st);
      const float k = ks[r], q = qs[r];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        st[e] = g * st[e] + k * v[e];
        acc[e] += st[e] * q;
      }
      if (N) store_vec<VEC>(N + static_cast<long long>(r) * p.V + cv, st);
    }
    store_vec<VEC>(part + grp * V + cv, acc);
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < V; c += RTS_THREADS) {
    float s = 0.f;
    for (int i = 0; i < groups; ++i) s += part[i * V + c];
    vs[c] = s;
    ss += s * s;
  }
  ss = block_sum(ss, scratch);
  if (shares > 1) {
    if (tid < shares) st_shared_cluster(&sums[blockIdx.z], tid, ss);
    cluster_sync_all();
    ss = 0.f;
    for (int i = 0; i < shares; ++i) ss += sums[i];
  }
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.V) + p.eps);
  const T* gate = x + 2 * p.H * D + (p.H + h) * p.V + v0;
  T* out = reinterpret_cast<T*>(p.out) + row * p.out_ld + h * p.V + v0;
  for (int c = tid; c < V; c += RTS_THREADS) out[c] = from_f32<T>(vs[c] * inv * silu(to_f32(gate[c])));
}

// ---------------------------------------------------------------------------------------------------------
// norm and gate of a scan's result: out = o / rms_head(o) * w * silu(gate) * scale, one warp per (row, head)
// ---------------------------------------------------------------------------------------------------------
template <typename T, int VEC> __device__ __forceinline__ void load_act(const T* p, float (&v)[VEC]) {
  if (VEC == 4 && sizeof(T) == 2) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 x = unpack_bf16x2(r.x), y = unpack_bf16x2(r.y);
    v[0] = x.x; v[VEC > 1 ? 1 : 0] = x.y; v[VEC > 2 ? 2 : 0] = y.x; v[VEC > 3 ? 3 : 0] = y.y;
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = to_f32(p[e]);
  }
}

constexpr int GN_ROWS = 4;       // rows of a warp, their loads in flight together

// grid (ceil(rows / GN_ROWS), ceil(H / heads of a CTA)); LPH lanes per head of up to LPH * VEC * NI values
template <typename T, int VEC, int NI, int LPH>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, int w_head, const T* __restrict__ gate,
                  long long gate_ld, T* __restrict__ out, long long out_ld, int rows, int H, int V, float eps, float scale) {
  constexpr int HPW = 32 / LPH;
  const int lane = threadIdx.x & 31, sub = lane % LPH, t0 = blockIdx.x * GN_ROWS;
  const int h = (blockIdx.y * 8 + (threadIdx.x >> 5)) * HPW + lane / LPH;
  const bool on = h < H;
  float a[GN_ROWS][NI][VEC], b[GN_ROWS][NI][VEC];
#pragma unroll
  for (int k = 0; k < GN_ROWS; ++k) {
    const long long t = min(t0 + k, rows - 1);
    const float* src = o + (t * H + h) * V;
    const T* g = gate + t * gate_ld + h * V;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * LPH + sub) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[k][i][e] = b[k][i][e] = 0.f;
      if (on && c < V) {
        if (VEC == 4) {
          const float4 f = *reinterpret_cast<const float4*>(src + c);
          a[k][i][0] = f.x; a[k][i][VEC > 1 ? 1 : 0] = f.y; a[k][i][VEC > 2 ? 2 : 0] = f.z; a[k][i][VEC > 3 ? 3 : 0] = f.w;
        } else {
          a[k][i][0] = src[c];
        }
        load_act<T, VEC>(g + c, b[k][i]);
      }
    }
  }
#pragma unroll
  for (int k = 0; k < GN_ROWS; ++k) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += a[k][i][e] * a[k][i][e];
#pragma unroll
    for (int m = LPH / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    const float inv = scale / sqrtf(ss / static_cast<float>(V) + eps);
    T* dst = out + (t0 + k) * out_ld + h * V;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * LPH + sub) * VEC;
      if (on && c < V && t0 + k < rows) {
        float r[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) r[e] = a[k][i][e] * inv * (w ? w[h * w_head + c + e] : 1.f) * act_silu<T>(b[k][i][e]);
        if (VEC == 4 && sizeof(T) == 2) {
          *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16x2(r[0], r[VEC > 1 ? 1 : 0]), pack_bf16x2(r[VEC > 2 ? 2 : 0], r[VEC > 3 ? 3 : 0]));
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) dst[c + e] = from_f32<T>(r[e]);
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// single rows: projection -> gated result in one launch, one CTA per (row, head)
// ---------------------------------------------------------------------------------------------------------
constexpr int RS_THREADS = 256;

// NR: key rows of the state a thread keeps in registers between the two passes (0: it reads them twice)
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(RS_THREADS) delta_step_kernel(DeltaParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float scratch[32];
  const int row = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G), D = p.D, V = p.V, taps = p.taps, tid = threadIdx.x;
  const int C = 2 * p.G * D + p.H * V, nvec = V / VEC, groups = RS_THREADS / nvec;
  float* qs = smf;                         // [D]
  float* ks = qs + D;                      // [D]
  float* vs = ks + D;                      // [V], later u
  float* part = smf + (2 * D + V + 3) / 4 * 4;   // [groups][V]
  const int prev = p.row_prev[row], next = p.row_next[row];
  const T* proj = reinterpret_cast<const T*>(p.proj) + row * p.ld;
  const float* S = prev >= 0 ? p.state + prev * p.state_ld + p.s_off + static_cast<long long>(h) * D * V : nullptr;
  float* N = next >= 0 ? p.state + next * p.state_ld + p.s_off + static_cast<long long>(h) * D * V : nullptr;
  const int grp = tid / nvec, cv = (tid - grp * nvec) * VEC;
  const bool on = grp < groups;
  float st[NR > 0 ? NR : 1][VEC];
  if (NR > 0) {                            // the state is on its way while the inputs are formed
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = grp + i * groups;
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[i][e] = 0.f;
      if (on && S && r < D) load_vec<VEC>(S + static_cast<long long>(r) * V + cv, st[i]);
    }
  }
  const bool owner = h % (p.H / p.G) == 0; // of the group's query / key convolution inputs
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < 2 * D + V; i += RS_THREADS) {
    const int c = i < D ? g * D + i : (i < 2 * D ? p.G * D + g * D + i - D : 2 * p.G * D + h * V + i - 2 * D);
    const float x = to_f32(proj[c]);
    float y = p.conv_w[static_cast<long long>(c) * taps + taps - 1] * x;
    const float* tail = prev >= 0 ? p.state + prev * p.state_ld + c : nullptr;
    float* keep = next >= 0 && (i >= 2 * D || owner) ? p.state + next * p.state_ld + c : nullptr;
    for (int j = 0; j < taps - 1; ++j) {
      const float in = tail ? tail[static_cast<long long>(j) * C] : 0.f;
      y += p.conv_w[static_cast<long long>(c) * taps + j] * in;
      if (keep && j > 0) keep[static_cast<long long>(j - 1) * C] = in;
    }
    if (keep && taps > 1) keep[static_cast<long long>(taps - 2) * C] = x;
    y = silu(y);
    smf[i] = y;
    if (i < D) sq += y * y;
    else if (i < 2 * D) sk += y * y;
  }
  sq = block_sum(sq, scratch);
  sk = block_sum(sk, scratch);             // also orders the inputs
  const float fq = p.q_scale / sqrtf(sq + 1e-6f), fk = 1.f / sqrtf(sk + 1e-6f);
  const int b0 = C + p.H * V;
  const float beta = sigmoid(to_f32(proj[b0 + h]));
  const float dec = expf(-expf(p.A_log[h]) * softplus(to_f32(proj[b0 + p.H + h]) + p.dt_bias[h]));
  float acc[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
  if (on && S) {
    if (NR > 0) {
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = grp + i * groups;
        if (r < D) {
          const float k = ks[r] * fk;
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[e] += st[i][e] * k;
        }
      }
    } else {
      for (int r = grp; r < D; r += groups) {
        float x[VEC];
        load_vec<VEC>(S + static_cast<long long>(r) * V + cv, x);
        const float k = ks[r] * fk;
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += x[e] * k;
      }
    }
  }
  if (on) store_vec<VEC>(part + grp * V + cv, acc);
  __syncthreads();
  for (int c = tid; c < V; c += RS_THREADS) {
    float s = 0.f;
    for (int i = 0; i < groups; ++i) s += part[i * V + c];
    vs[c] = beta * (vs[c] - dec * s);
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
  if (on) {
    float u[VEC];
    load_vec<VEC>(vs + cv, u);
    auto advance = [&](int r, float (&x)[VEC]) {
      const float k = ks[r] * fk, q = qs[r] * fq;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        x[e] = dec * x[e] + k * u[e];
        acc[e] += x[e] * q;
      }
      if (N) store_vec<VEC>(N + static_cast<long long>(r) * V + cv, x);
    };
    if (NR > 0) {
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = grp + i * groups;
        if (r < D) advance(r, st[i]);
      }
    } else {
      for (int r = grp; r < D; r += groups) {
        float x[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] = 0.f;
        if (S) load_vec<VEC>(S + static_cast<long long>(r) * V + cv, x);
        advance(r, x);
      }
    }
    store_vec<VEC>(part + grp * V + cv, acc);
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < V; c += RS_THREADS) {
    float s = 0.f;
    for (int i = 0; i < groups; ++i) s += part[i * V + c];
    vs[c] = s;
    ss += s * s;
  }
  ss = block_sum(ss, scratch);
  const float inv = p.out_scale / sqrtf(ss / static_cast<float>(V) + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + row * p.out_ld + h * V;
  for (int c = tid; c < V; c += RS_THREADS)
    out[c] = from_f32<T>(vs[c] * inv * p.norm_w[c] * silu(to_f32(proj[C + h * V + c])));
}

template <typename T, int VEC>
__global__ void __launch_bounds__(RS_THREADS) wkv_step_kernel(WkvParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float scratch[32];
  const int row = blockIdx.x, h = blockIdx.y, D = p.D, HD = p.H * D, tid = threadIdx.x;
  const int nvec = D / VEC, groups = RS_THREADS / nvec;
  float* rs = smf;
  float* ks = rs + D;
  float* ws = ks + D;
  float* vs = ws + D;
  float* part = smf + (4 * D + 3) / 4 * 4;       // [groups][D]
  const int prev = p.row_prev[row], next = p.row_next[row];
  const T* x = reinterpret_cast<const T*>(p.rkvg) + row * p.ld + h * D;
  float bonus = 0.f;
  for (int c = tid; c < D; c += RS_THREADS) {
    const float r = to_f32(x[c]), k = to_f32(x[HD + c]);
    rs[c] = r;
    ks[c] = k;
    vs[c] = to_f32(x[2 * HD + c]);
    ws[c] = expf(-expf(p.w_raw[static_cast<long long>(row) * HD + h * D + c] + p.w0[h * D + c]));
    bonus += r * p.u[h * D + c] * k;
  }
  bonus = block_sum(bonus, scratch);
  const int grp = tid / nvec, cv = (tid - grp * nvec) * VEC;
  const float* S = prev >= 0 ? p.state + prev * p.state_ld + p.s_off + static_cast<long long>(h) * D * D : nullptr;
  float* N = next >= 0 ? p.state + next * p.state_ld + p.s_off + static_cast<long long>(h) * D * D : nullptr;
  if (grp < groups) {
    float acc[VEC], v[VEC];
    load_vec<VEC>(vs + cv, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll 4
    for (int r = grp; r < D; r += groups) {
      float st[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[e] = 0.f;
      if (S) load_vec<VEC>(S + static_cast<long long>(r) * D + cv, st);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        acc[e] += st[e] * rs[r];
        st[e] = ws[r] * st[e] + ks[r] * v[e];
      }
      if (N) store_vec<VEC>(N + static_cast<long long>(r) * D + cv, st);
    }
    store_vec<VEC>(part + grp * D + cv, acc);
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < D; c += RS_THREADS) {
    float s = bonus * vs[c];
    for (int i = 0; i < groups; ++i) s += part[i * D + c];
    rs[c] = s;                             // the row's r is no longer needed
    ss += s * s;
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(D) + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + row * p.out_ld + h * D;
  for (int c = tid; c < D; c += RS_THREADS)
    out[c] = from_f32<T>(rs[c] * inv * p.norm_w[h * D + c] * silu(to_f32(x[3 * HD + c])));
}

// ---------------------------------------------------------------------------------------------------------
// launchers
// ---------------------------------------------------------------------------------------------------------
template <typename K> static int allow_smem(K kernel, size_t bytes) {
  return bytes <= 48 * 1024 ? 0 : (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <typename T, int VEC, int NI>
static int launch_inputs(const DeltaParams& p, cudaStream_t st) {
  const int units = 2 * p.G + p.H + 1;
  const dim3 grid((p.max_rows + DI_TOKENS - 1) / DI_TOKENS, (units + 3) / 4, p.portions);
  if (p.taps <= 4) delta_inputs_kernel<T, VEC, NI, true><<<grid, 128, 0, st>>>(p);
  else delta_inputs_kernel<T, VEC, NI, false><<<grid, 128, 0, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T> static int dispatch_inputs(const DeltaParams& p, cudaStream_t st) {
  const int most = p.D > p.V ? p.D : p.V;
  if (p.D % 2 == 0 && p.V % 2 == 0 && p.ld % 2 == 0 && (reinterpret_cast<uintptr_t>(p.proj) & 3u) == 0) {
    if (most <= 64) return launch_inputs<T, 2, 1>(p, st);
    if (most <= 128) return launch_inputs<T, 2, 2>(p, st);
    return launch_inputs<T, 2, 4>(p, st);
  }
  return most <= 64 ? launch_inputs<T, 1, 2>(p, st) : launch_inputs<T, 1, 8>(p, st);
}

template <int LANES> static int launch_delta_scan(const DeltaParams& p, int portions, cudaStream_t st) {
  using Z = DeltaScan<LANES>;
  if (int e = allow_smem(delta_scan_kernel<LANES>, Z::SMEM)) return e;
  delta_scan_kernel<LANES><<<dim3((p.V + Z::NC - 1) / Z::NC, p.H, portions), SC_WARPS * 32, Z::SMEM, st>>>(p);
  return (int)cudaGetLastError();
}

template <int LANES, typename T> static int launch_wkv_scan(const WkvParams& p, int portions, cudaStream_t st) {
  using Z = WkvScan<LANES, T>;
  if (int e = allow_smem(wkv_scan_kernel<LANES, T>, Z::SMEM)) return e;
  wkv_scan_kernel<LANES, T><<<dim3((p.D + Z::NC - 1) / Z::NC, p.H, portions), SC_WARPS * 32, Z::SMEM, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T> static int dispatch_wkv_scan(const WkvParams& p, int portions, cudaStream_t st) {
  if (p.D <= 32) return launch_wkv_scan<4, T>(p, portions, st);
  if (p.D <= 64) return launch_wkv_scan<8, T>(p, portions, st);
  if (p.D <= 128) return launch_wkv_scan<16, T>(p, portions, st);
  return launch_wkv_scan<32, T>(p, portions, st);
}

template <typename T, int VEC> static int launch_delta_step(const DeltaParams& p, cudaStream_t st) {
  const int nvec = p.V / VEC, groups = RS_THREADS / nvec, per = (p.D + groups - 1) / groups;
  const size_t smem = ((2 * p.D + p.V + 3) / 4 * 4 + static_cast<size_t>(groups) * p.V) * sizeof(float);
  const dim3 grid(p.rows, p.H);
  if (per <= 4) delta_step_kernel<T, VEC, 4><<<grid, RS_THREADS, smem, st>>>(p);
  else if (per <= 8) delta_step_kernel<T, VEC, 8><<<grid, RS_THREADS, smem, st>>>(p);
  else if (per <= 16) delta_step_kernel<T, VEC, 16><<<grid, RS_THREADS, smem, st>>>(p);
  else delta_step_kernel<T, VEC, 0><<<grid, RS_THREADS, smem, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T> static int launch_gated_norm(const float* o, const float* w, int w_head, const void* gate, long long gate_ld,
                                                   void* out, long long out_ld, int rows, int H, int V, float eps, float scale,
                                                   cudaStream_t st) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out);
  const bool vec = V % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && bits % (4 * sizeof(T)) == 0;
  const T* g = reinterpret_cast<const T*>(gate);
  T* d = reinterpret_cast<T*>(out);
  auto grid = [&](int heads_per_warp) { return dim3((rows + GN_ROWS - 1) / GN_ROWS, (H + 8 * heads_per_warp - 1) / (8 * heads_per_warp)); };
  if (vec && V <= 64) gated_norm_kernel<T, 4, 1, 16><<<grid(2), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  else if (vec && V <= 128) gated_norm_kernel<T, 4, 1, 32><<<grid(1), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  else if (vec && V <= 256) gated_norm_kernel<T, 4, 2, 32><<<grid(1), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  else if (vec) gated_norm_kernel<T, 4, 4, 32><<<grid(1), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  else if (V > 256) gated_norm_kernel<T, 1, 16, 32><<<grid(1), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  else gated_norm_kernel<T, 1, 8, 32><<<grid(1), 256, 0, st>>>(o, w, w_head, g, gate_ld, d, out_ld, rows, H, V, eps, scale);
  return (int)cudaGetLastError();
}

template <int KIND, int NT, int WR, typename TV>
static int launch_block_scan(const BlockScanParams& p, int portions, cudaStream_t st) {
  using Z = BlockScan<KIND, NT, WR, TV>;
  if (int e = allow_smem(block_scan_kernel<KIND, NT, WR, TV>, Z::SMEM)) return e;
  block_scan_kernel<KIND, NT, WR, TV><<<dim3((p.V + Z::NC - 1) / Z::NC, p.H, portions), 128, Z::SMEM, st>>>(p);
  return (int)cudaGetLastError();
}

// The key rows of a head stay with one warp when there are (head, portion) pairs for every SM, else they are split over two or
// four: half the latency of a block for a third more work.
template <int KIND, typename TV> static int dispatch_block_scan(const BlockScanParams& p, int portions, cudaStream_t st) {
  const long long groups = static_cast<long long>((p.V + 15) / 16) * p.H * portions;       // of 16 value columns
  const int wr = groups >= 4 * sm_count() ? 1 : (groups > sm_count() ? 2 : 4);
  if (p.D <= 32) return launch_block_scan<KIND, 4, 1, TV>(p, portions, st);
  if (p.D <= 64)
    return wr == 1 ? launch_block_scan<KIND, 8, 1, TV>(p, portions, st)
                   : (wr == 2 ? launch_block_scan<KIND, 4, 2, TV>(p, portions, st) : launch_block_scan<KIND, 2, 4, TV>(p, portions, st));
  if (p.D <= 128)
    return wr == 1 ? launch_block_scan<KIND, 16, 1, TV>(p, portions, st)
                   : (wr == 2 ? launch_block_scan<KIND, 8, 2, TV>(p, portions, st) : launch_block_scan<KIND, 4, 4, TV>(p, portions, st));
  return launch_block_scan<KIND, 8, 4, TV>(p, portions, st);
}

static bool blocked_ok(int D, int V) { return D % 8 == 0 && V % 8 == 0; }

static bool delta_sizes_ok(int H, int G, int D, int V, int taps) {
  return H > 0 && G > 0 && H % G == 0 && D > 0 && V > 0 && D <= 256 && V <= 256 && taps >= 1 && H <= 65535;
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_recurrent)
using namespace ts;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

// Portions of prompts, step 1: convolved inputs [rows][C] and gates [rows][2 H]; leaves the convolution state.
extern "C" int ts_delta_inputs(const void* proj, long long ld, const float* conv_w, const float* A_log, const float* dt_bias,
                               float q_scale, float* state, long long state_ld, const int* row_prev, const int* row_next,
                               const int* cu, int portions, int max_rows, float* qkv, float* gates, int H, int G, int D, int V,
                               int taps, int fp32, void* stream) {
  if (portions <= 0) return 0;
  if (!delta_sizes_ok(H, G, D, V, taps) || portions > 65535 || max_rows <= 0) return -10;
  DeltaParams p = {};
  p.proj = proj; p.ld = ld; p.conv_w = conv_w; p.A_log = A_log; p.dt_bias = dt_bias; p.q_scale = q_scale; p.state = state;
  p.state_ld = state_ld; p.row_prev = row_prev; p.row_next = row_next; p.cu = cu; p.portions = portions;
  p.max_rows = max_rows; p.qkv = qkv; p.gates = gates; p.H = H; p.G = G; p.D = D; p.V = V; p.taps = taps;
  return fp32 ? dispatch_inputs<float>(p, ST(stream)) : dispatch_inputs<__nv_bfloat16>(p, ST(stream));
}

// Portions, step 2: o [rows][H V] of the recurrence, the last state of every portion to its state row.
extern "C" int ts_delta_scan(const float* qkv, const float* gates, float* state, long long state_ld, int s_off,
                             const int* row_prev, const int* row_next, const int* cu, int portions, float* o, int H, int G,
                             int D, int V, void* stream) {
  if (portions <= 0) return 0;
  if (!delta_sizes_ok(H, G, D, V, 1) || portions > 65535) return -10;
  DeltaParams p = {};
  p.qkv = const_cast<float*>(qkv); p.gates = const_cast<float*>(gates); p.state = state; p.state_ld = state_ld;
  p.s_off = s_off; p.row_prev = row_prev; p.row_next = row_next; p.cu = cu; p.o = o; p.H = H; p.G = G; p.D = D; p.V = V;
  if (D <= 32) return launch_delta_scan<4>(p, portions, ST(stream));
  if (D <= 64) return launch_delta_scan<8>(p, portions, ST(stream));
  if (D <= 128) return launch_delta_scan<16>(p, portions, ST(stream));
  return launch_delta_scan<32>(p, portions, ST(stream));
}

// 1 when the block scans take these head sizes.
extern "C" int ts_block_scan_supported(int D, int V) { return blocked_ok(D, V) ? 1 : 0; }
// Blocks of `rows` rows in `portions` portions (upper bound) and the floats a block and head needs.
extern "C" int ts_block_scan_blocks(int rows, int portions) { return rows / BS_BLOCK + portions + 1; }
extern "C" int ts_block_scan_coef(int kind) {
  return kind == SCAN_DELTA ? BS_COEF : (kind == SCAN_WKV ? BS_COEF_WKV : BS_COEF_RET);
}

// Portions, step 2 of bf16 models: as ts_delta_scan, on the tensor cores.  coef: [blocks][H][BS_COEF] workspace.
extern "C" int ts_delta_block_scan(const float* qkv, const float* gates, float* coef, float* state, long long state_ld, int s_off,
                                   const int* row_prev, const int* row_next, const int* cu, int portions, int max_rows, float* o,
                                   int H, int G, int D, int V, void* stream) {
  if (portions <= 0) return 0;
  if (!delta_sizes_ok(H, G, D, V, 1) || !blocked_ok(D, V) || portions > 65535) return -10;
  const dim3 grid((max_rows + BS_BLOCK - 1) / BS_BLOCK, (G + 3) / 4, portions);
  delta_blocks_kernel<<<grid, 128, 0, ST(stream)>>>(qkv, gates, cu, coef, H, G, D, V);
  if (int e = (int)cudaGetLastError()) return e;
  BlockScanParams p = {};
  p.q = qkv; p.k = qkv + G * D; p.v = qkv + 2 * G * D; p.qk_ld = p.v_ld = 2 * G * D + H * V; p.rep = H / G; p.coef = coef;
  p.state = state; p.state_ld = state_ld; p.s_off = s_off; p.row_prev = row_prev; p.row_next = row_next; p.cu = cu; p.o = o;
  p.H = H; p.D = D; p.V = V;
  return dispatch_block_scan<SCAN_DELTA, float>(p, portions, ST(stream));
}

// Portions of the WKV recurrence of bf16 models.  Workspaces: rt, kt [rows][H D], coef [blocks][H][BS_COEF_WKV], row_decay
// [blocks][H][D].
extern "C" int ts_wkv_block_scan(const void* rkvg, long long ld, const float* w_raw, const float* w0, const float* u, float* rt,
                                 float* kt, float* coef, float* row_decay, float* state, long long state_ld, int s_off,
                                 const int* row_prev, const int* row_next, const int* cu, int portions, int max_rows, float* o,
                                 int H, int D, void* stream) {
  if (portions <= 0) return 0;
  if (!delta_sizes_ok(H, H, D, D, 1) || !blocked_ok(D, D) || portions > 65535 || ld % 8 ||
      (reinterpret_cast<uintptr_t>(rkvg) & 15u))
    return -10;
  WkvParams w = {};
  w.rkvg = rkvg; w.ld = ld; w.w_raw = w_raw; w.w0 = w0; w.u = u; w.cu = cu; w.H = H; w.D = D;
  const dim3 grid((max_rows + BS_BLOCK - 1) / BS_BLOCK, (H + 3) / 4, portions);
  wkv_blocks_kernel<__nv_bfloat16><<<grid, 128, 0, ST(stream)>>>(w, rt, kt, coef, row_decay);
  if (int e = (int)cudaGetLastError()) return e;
  BlockScanParams p = {};
  p.q = rt; p.k = kt; p.v = reinterpret_cast<const __nv_bfloat16*>(rkvg) + 2 * H * D; p.qk_ld = H * D; p.v_ld = ld; p.rep = 1;
  p.coef = coef; p.row_decay = row_decay; p.state = state; p.state_ld = state_ld; p.s_off = s_off; p.row_prev = row_prev;
  p.row_next = row_next; p.cu = cu; p.o = o; p.H = H; p.D = D; p.V = D;
  return dispatch_block_scan<SCAN_WKV, __nv_bfloat16>(p, portions, ST(stream));
}

// Portions, last step (either recurrence): o [rows][H V] fp32; w per channel (w_head = V), shared by heads (w_head = 0) or
// absent (nullptr).
extern "C" int ts_gated_norm(const float* o, const float* w, int w_head, const void* gate, long long gate_ld, void* out,
                             long long out_ld, int rows, int H, int V, float eps, float scale, int fp32, void* stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || V <= 0 || V > 512) return -10;
  return fp32 ? launch_gated_norm<float>(o, w, w_head, gate, gate_ld, out, out_ld, rows, H, V, eps, scale, ST(stream))
              : launch_gated_norm<__nv_bfloat16>(o, w, w_head, gate, gate_ld, out, out_ld, rows, H, V, eps, scale, ST(stream));
}

// Single rows: projection -> out [rows][out_ld] = out_scale * gated norm, state and convolution state advanced.
extern "C" int ts_delta_step(const void* proj, long long ld, const float* conv_w, const float* A_log, const float* dt_bias,
                             const float* norm_w, float eps, float q_scale, float* state, long long state_ld, int s_off,
                             const int* row_prev, const int* row_next, void* out, long long out_ld, float out_scale,
                             int rows, int H, int G, int D, int V, int taps, int fp32, void* stream) {
  if (rows <= 0) return 0;
  if (!delta_sizes_ok(H, G, D, V, taps)) return -10;
  DeltaParams p = {};
  p.proj = proj; p.ld = ld; p.conv_w = conv_w; p.A_log = A_log; p.dt_bias = dt_bias; p.norm_w = norm_w; p.eps = eps;
  p.q_scale = q_scale; p.state = state; p.state_ld = state_ld; p.s_off = s_off; p.row_prev = row_prev;
  p.row_next = row_next; p.out = out; p.out_ld = out_ld; p.out_scale = out_scale; p.rows = rows; p.H = H; p.G = G;
  p.D = D; p.V = V; p.taps = taps;
  const bool vec = V % 4 == 0 && D % 2 == 0 && s_off % 4 == 0 && state_ld % 4 == 0;
  if (fp32) return vec ? launch_delta_step<float, 4>(p, ST(stream)) : launch_delta_step<float, 1>(p, ST(stream));
  return vec ? launch_delta_step<__nv_bfloat16, 4>(p, ST(stream)) : launch_delta_step<__nv_bfloat16, 1>(p, ST(stream));
}

// Portions: o [rows][H D] of the WKV recurrence.  rkvg rows: r | k | v | gate.
extern "C" int ts_wkv_scan(const void* rkvg, long long ld, const float* w_raw, const float* w0, const float* u, float* state,
                           long long state_ld, int s_off, const int* row_prev, const int* row_next, const int* cu,
                           int portions, float* o, int H, int D, int fp32, void* stream) {
  if (portions <= 0) return 0;
  if (!delta_sizes_ok(H, H, D, D, 1) || portions > 65535) return -10;
  WkvParams p = {};
  p.rkvg = rkvg; p.ld = ld; p.w_raw = w_raw; p.w0 = w0; p.u = u; p.state = state; p.state_ld = state_ld; p.s_off = s_off;
  p.row_prev = row_prev; p.row_next = row_next; p.cu = cu; p.o = o; p.H = H; p.D = D;
  return fp32 ? dispatch_wkv_scan<float>(p, portions, ST(stream)) : dispatch_wkv_scan<__nv_bfloat16>(p, portions, ST(stream));
}

// Single rows of the WKV recurrence: projections -> out = gated norm, state advanced.
extern "C" int ts_wkv_step(const void* rkvg, long long ld, const float* w_raw, const float* w0, const float* u,
                           const float* norm_w, float eps, float* state, long long state_ld, int s_off, const int* row_prev,
                           const int* row_next, void* out, long long out_ld, int rows, int H, int D, int fp32, void* stream) {
  if (rows <= 0) return 0;
  if (!delta_sizes_ok(H, H, D, D, 1)) return -10;
  WkvParams p = {};
  p.rkvg = rkvg; p.ld = ld; p.w_raw = w_raw; p.w0 = w0; p.u = u; p.norm_w = norm_w; p.eps = eps; p.state = state;
  p.state_ld = state_ld; p.s_off = s_off; p.row_prev = row_prev; p.row_next = row_next; p.out = out; p.out_ld = out_ld;
  p.rows = rows; p.H = H; p.D = D;
  const bool vec = D % 4 == 0 && s_off % 4 == 0 && state_ld % 4 == 0;
  const int groups = RS_THREADS / (vec ? D / 4 : D);
  const size_t smem = ((4 * D + 3) / 4 * 4 + static_cast<size_t>(groups) * D) * sizeof(float);
  const dim3 grid(rows, H);
  if (fp32) {
    if (vec) wkv_step_kernel<float, 4><<<grid, RS_THREADS, smem, ST(stream)>>>(p);
    else wkv_step_kernel<float, 1><<<grid, RS_THREADS, smem, ST(stream)>>>(p);
  } else {
    if (vec) wkv_step_kernel<__nv_bfloat16, 4><<<grid, RS_THREADS, smem, ST(stream)>>>(p);
    else wkv_step_kernel<__nv_bfloat16, 1><<<grid, RS_THREADS, smem, ST(stream)>>>(p);
  }
  return (int)cudaGetLastError();
}

static int retention_params(RetentionParams& p, const void* proj, long long ld, const float* angles, const float* powers, int powers_ld,
                            float k_scale, float* state, long long state_ld, const int* row_prev, const int* row_next, int H, int D,
                            int V, int rot) {
  if (H <= 0 || H > 65535 || D <= 0 || D > 256 || V <= 0 || V > 512 || rot < 0 || rot > D || rot % 2 ||
      powers_ld <= BS_BLOCK || state_ld < static_cast<long long>(H) * D * V)
    return -10;
  p = {};
  p.proj = proj; p.ld = ld; p.angles = angles; p.powers = powers; p.powers_ld = powers_ld; p.k_scale = k_scale; p.state = state; p.state_ld = state_ld;
  p.row_prev = row_prev; p.row_next = row_next; p.H = H; p.D = D; p.V = V; p.rot = rot;
  return 0;
}

// Shares of the value columns: enough CTAs for two per SM, at least 32 columns each.
template <typename T, int VEC> static int launch_retention_step(const RetentionParams& p, cudaStream_t st) {
  int shares = 1;
  while (VEC == 4 && shares < RTS_SHARES && p.V % (shares * 2 * 4) == 0 && p.V / (shares * 2) >= 32 &&
         static_cast<long long>(p.rows) * p.H * shares < 2 * sm_count())
    shares *= 2;
  const int V = p.V / shares, nvec = V / VEC, groups = RTS_THREADS / (nvec < RTS_THREADS ? nvec : RTS_THREADS);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.rows, p.H, shares);
  cfg.blockDim = dim3(RTS_THREADS);
  cfg.dynamicSmemBytes = ((V + 3) / 4 * 4 + (groups * V + 3) / 4 * 4 + 2 * p.D) * sizeof(float);
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = 1;
  at[0].val.clusterDim.y = 1;
  at[0].val.clusterDim.z = shares;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  return (int)cudaLaunchKernelEx(&cfg, retention_step_kernel<T, VEC>, p);
}

// Single rows of retention: projection -> out [rows][out_ld] = norm * silu(gate), state advanced.
extern "C" int ts_retention_step(const void* proj, long long ld, const float* angles, const float* powers, int powers_ld, float k_scale, float eps,
                                 float* state, long long state_ld, const int* row_prev, const int* row_next, void* out,
                                 long long out_ld, int rows, int H, int D, int V, int rot, int fp32, void* stream) {
  if (rows <= 0) return 0;
  RetentionParams p;
  if (int e = retention_params(p, proj, ld, angles, powers, powers_ld, k_scale, state, state_ld, row_prev, row_next, H, D, V, rot)) return e;
  p.eps = eps; p.out = out; p.out_ld = out_ld; p.rows = rows;
  const bool vec = V % 4 == 0 && state_ld % 4 == 0;
  if (fp32) return vec ? launch_retention_step<float, 4>(p, ST(stream)) : launch_retention_step<float, 1>(p, ST(stream));
  return vec ? launch_retention_step<__nv_bfloat16, 4>(p, ST(stream)) : launch_retention_step<__nv_bfloat16, 1>(p, ST(stream));
}

template <typename T> static int dispatch_retention_scan(const RetentionParams& p, int portions, cudaStream_t st) {
  const dim3 grid((p.V + 31) / 32, p.H, portions);
  if (p.D <= 32) retention_scan_kernel<T, 4><<<grid, 256, 0, st>>>(p);
  else if (p.D <= 64) retention_scan_kernel<T, 8><<<grid, 256, 0, st>>>(p);
  else if (p.D <= 128) retention_scan_kernel<T, 16><<<grid, 256, 0, st>>>(p);
  else retention_scan_kernel<T, 32><<<grid, 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}

// Portions of retention: o [rows][H V] of the recurrence, the last state of every portion to its state row.  fp32 arithmetic.
extern "C" int ts_retention_scan(const void* proj, long long ld, const float* angles, const float* powers, int powers_ld, float k_scale,
                                 float* state, long long state_ld, const int* row_prev, const int* row_next, const int* cu,
                                 int portions, float* o, int H, int D, int V, int rot, int fp32, void* stream) {
  if (portions <= 0) return 0;
  RetentionParams p;
  if (int e = retention_params(p, proj, ld, angles, powers, powers_ld, k_scale, state, state_ld, row_prev, row_next, H, D, V, rot)) return e;
  if (portions > 65535) return -10;
  p.cu = cu; p.o = o;
  return fp32 ? dispatch_retention_scan<float>(p, portions, ST(stream)) : dispatch_retention_scan<__nv_bfloat16>(p, portions, ST(stream));
}

// Portions of retention in bf16 models: as ts_retention_scan, on the tensor cores.  Workspaces: rt, kt [rows][H D], coef
// [blocks][H][BS_COEF_RET].
extern "C" int ts_retention_block_scan(const void* proj, long long ld, const float* angles, const float* powers, int powers_ld, float k_scale,
                                       float* rt, float* kt, float* coef, float* state, long long state_ld, const int* row_prev,
                                       const int* row_next, const int* cu, int portions, int max_rows, float* o, int H, int D,
                                       int V, int rot, void* stream) {
  if (portions <= 0) return 0;
  RetentionParams r;
  if (int e = retention_params(r, proj, ld, angles, powers, powers_ld, k_scale, state, state_ld, row_prev, row_next, H, D, V, rot)) return e;
  if (!blocked_ok(D, V) || portions > 65535 || max_rows <= 0 || ld % 8 || (reinterpret_cast<uintptr_t>(proj) & 15u)) return -10;
  r.cu = cu;
  const size_t smem = 4 * 2 * BS_BLOCK * (D + 1) * sizeof(float);
  if (int e = allow_smem(retention_blocks_kernel, smem)) return e;
  retention_blocks_kernel<<<dim3((max_rows + BS_BLOCK - 1) / BS_BLOCK, (H + 3) / 4, portions), 128, smem, ST(stream)>>>(r, rt, kt, coef);
  if (int e = (int)cudaGetLastError()) return e;
  BlockScanParams p = {};
  p.q = rt; p.k = kt; p.v = reinterpret_cast<const __nv_bfloat16*>(proj) + 2 * H * D; p.qk_ld = H * D; p.v_ld = ld; p.rep = 1;
  p.coef = coef; p.state = state; p.state_ld = state_ld; p.row_prev = row_prev; p.row_next = row_next; p.cu = cu; p.o = o;
  p.H = H; p.D = D; p.V = V;
  return dispatch_block_scan<SCAN_RETENTION, __nv_bfloat16>(p, portions, ST(stream));
}
