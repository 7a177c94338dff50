// Sliding-window attention with grouped queries over a paged cache whose rows hold a token's keys and values side by side:
// row = [G key heads x dim | G value heads x vdim | padding].
//
// Keys a position sees: itself and the `window` - 1 before it, or the part of its chunk of `window` positions up to itself
// (chunks count from position 0); besides, the first `keep` positions of the sequence.
//
//   ts_window_angles  cosines and sines of a step's positions, shared by all layers with the same frequencies
//   ts_window_prep    bias, per-head RMS norm of queries and keys, a factor of the queries that grows with the position, rotary
//                     embedding of the first `rot` dimensions of a head (in place in the projection), cache write of keys and
//                     values - one launch.  Each step but the last
//                     is optional; values can be the projected keys themselves
//   ts_window_attend  single query rows (decoding, fp32, and head sizes the prefill kernel does not take) against the paged
//                     cache; the result may be multiplied by the sigmoid of a gate per head or per element
//
// Scores are (q . k) * scale, plus a number per head, minus a slope per head times the distance of query and key (either may be
// absent).  Weights are their softmax over the visible keys or, without any normalization, their sigmoids.  With a bound of the
// products and a slope, sigmoids fade below 2^-48 at a distance that is known beforehand; keys beyond it are not read.
// Portions of prompts: ts_window_prefill (latent_prefill.cu).
//
// Decoding reads every cached key and value in the window once per key/value head.  `window_attend_mma_kernel` (bf16): the
// query heads of a group are the 16 rows of warp MMAs; every warp walks its own 16-key tiles through its own ring of
// shared-memory stages (cp.async), with its own running softmax, so nothing in the loop waits for another warp.  Long
// windows are split over CTAs and merged by log-sum-exp.  `window_attend_simt_kernel`: fp32 and sizes the tiles do not fit.
#include "common.cuh"
#include "host_common.h"

namespace ts {

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

// ---------------------------------------------------------------------------------------------------------
// norm, rotation, cache write
// ---------------------------------------------------------------------------------------------------------
struct WindowPrepParams {
  void* proj;                  // rows [H x dim | G x dim | G x vdim | ...]
  long long ld;
  const float* bias;           // [(H + G) x dim] or nullptr
  const float* q_norm;         // [dim] or nullptr (no norms)
  const float* k_norm;
  float eps;
  const float* angles;         // [T][cos (rot / 2) | sin (rot / 2)]
  const long long* slots;
  void* cache;
  int T, H, G, dim, vdim, rot, row_width;
  int h0;                      // first head that changes (H: queries stay as projected)
  int pairs;                   // rotation partners: 0 coordinates i and i + rot / 2, 1 coordinates 2 i and 2 i + 1
  int values_are_keys;         // values: the keys before norm and rotation, also written behind them in the projection
  const int* pos;              // [T] (for the queries' factor)
  float temp_coef;             // queries *= 1 + temp_coef * log(floor((pos + 1) / temp_every) + 1); temp_every 0: no factor
  int temp_every;
};

__device__ __forceinline__ float query_factor(const WindowPrepParams& p, int t) {
  return p.temp_every > 0 ? 1.f + p.temp_coef * logf(static_cast<float>((p.pos[t] + 1) / p.temp_every) + 1.f) : 1.f;
}

__global__ void window_angles_kernel(const float* __restrict__ inv_freq, const int* __restrict__ pos, float* __restrict__ out, int T,
                                     int half, float magnitude) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= T * half) return;
  const int t = i / half, f = i - t * half;
  float s, c;
  sincosf(static_cast<float>(pos[t]) * inv_freq[f], &s, &c);
  out[static_cast<long long>(t) * 2 * half + f] = c * magnitude;
  out[static_cast<long long>(t) * 2 * half + half + f] = s * magnitude;
}

constexpr int WP_WARPS = 8;

// Any sizes: one CTA per token, a warp takes heads in turn.
template <typename T>
__global__ void __launch_bounds__(WP_WARPS * 32) window_prep_kernel(WindowPrepParams p) {
  const int t = blockIdx.x, half = p.rot / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* cs = p.angles + static_cast<long long>(t) * p.rot;
  T* row = reinterpret_cast<T*>(p.proj) + t * p.ld;
  T* crow = reinterpret_cast<T*>(p.cache) + p.slots[t] * p.row_width;
  T* v = row + (p.H + p.G) * p.dim;
  const float qf = query_factor(p, t);
  for (int c = threadIdx.x; c < p.row_width - p.G * p.dim; c += blockDim.x) {
    if (c >= p.G * p.vdim) crow[p.G * p.dim + c] = from_f32<T>(0.f);
    else if (!p.values_are_keys) crow[p.G * p.dim + c] = v[c];
  }
  for (int h = p.h0 + warp; h < p.H + p.G; h += WP_WARPS) {
    T* x = row + h * p.dim;
    const float* bias = p.bias ? p.bias + h * p.dim : nullptr;
    auto value = [&](int c) { return to_f32(x[c]) + (bias ? bias[c] : 0.f); };
    const float* w = h < p.H ? p.q_norm : p.k_norm;
    float inv = 1.f;
    if (w) {
      float ss = 0.f;
      for (int c = lane; c < p.dim; c += 32) {
        const float a = value(c);
        ss += a * a;
      }
      ss = warp_sum(ss);
      inv = 1.f / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
    }
    const float factor = h < p.H ? qf : 1.f;
    auto normed = [&](int c) { return (w ? value(c) * inv * w[c] : value(c)) * factor; };
    T* out2 = h < p.H ? nullptr : crow + (h - p.H) * p.dim;
    if (p.values_are_keys && h >= p.H)
      for (int c = lane; c < p.dim; c += 32) {
        const T y = from_f32<T>(value(c));
        v[(h - p.H) * p.dim + c] = y;
        crow[p.G * p.dim + (h - p.H) * p.dim + c] = y;
      }
    for (int i = lane; i < half; i += 32) {
      const int c0 = p.pairs ? 2 * i : i, c1 = p.pairs ? 2 * i + 1 : i + half;
      const float a = normed(c0), b = normed(c1);
      const T lo = from_f32<T>(a * cs[i] - b * cs[half + i]), hi = from_f32<T>(b * cs[i] + a * cs[half + i]);
      x[c0] = lo;
      x[c1] = hi;
      if (out2) {
        out2[c0] = lo;
        out2[c1] = hi;
      }
    }
    for (int c = p.rot + lane; c < p.dim; c += 32) {
      const T y = from_f32<T>(normed(c));
      x[c] = y;
      if (out2) out2[c] = y;
    }
  }
}

// bf16, head sizes multiples of eight.  A warp takes 32 / LPH heads of a token, LPH lanes hold one head as 16-byte vectors;
// or it copies 32 vectors of the token's values.  The halves of a rotated pair meet by shuffles when they are whole vectors
// apart, else through shared memory.
template <int LPH>
__global__ void __launch_bounds__(WP_WARPS * 32) window_prep_vec_kernel(WindowPrepParams p) {
  constexpr int HPW = 32 / LPH;
  __shared__ float swap[WP_WARPS][HPW][LPH * 8];
  const int half = p.rot / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head_items = (p.H + p.G - p.h0 + HPW - 1) / HPW;
  const int per_token = head_items + (p.values_are_keys ? 0 : (p.G * p.vdim / 8 + 31) / 32);
  const unsigned item = blockIdx.x * WP_WARPS + warp;
  const int t = item / per_token, part = item - t * per_token;
  if (t >= p.T) return;
  __nv_bfloat16* row = reinterpret_cast<__nv_bfloat16*>(p.proj) + t * p.ld;
  __nv_bfloat16* crow = reinterpret_cast<__nv_bfloat16*>(p.cache) + p.slots[t] * p.row_width;
  if (part >= head_items) {
    const int c = (part - head_items) * 32 + lane;
    if (c < p.G * p.vdim / 8)
      reinterpret_cast<uint4*>(crow + p.G * p.dim)[c] = reinterpret_cast<const uint4*>(row + (p.H + p.G) * p.dim)[c];
    return;
  }
  const int sub = lane % LPH, slot = lane / LPH, h = p.h0 + part * HPW + slot, c0 = sub * 8;
  const bool on = c0 < p.dim && h < p.H + p.G;
  __nv_bfloat16* x = row + h * p.dim + c0;
  float a[8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] = 0.f;
  if (on) {
    const uint4 raw = *reinterpret_cast<const uint4*>(x);
    const uint32_t r[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(r[j]);
      a[2 * j] = f.x;
      a[2 * j + 1] = f.y;
    }
    if (p.bias) {
      const float* b = p.bias + h * p.dim + c0;
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] += b[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += a[j] * a[j];
    if (p.values_are_keys && h >= p.H) {
      const uint4 o = make_uint4(pack_bf16x2(a[0], a[1]), pack_bf16x2(a[2], a[3]), pack_bf16x2(a[4], a[5]), pack_bf16x2(a[6], a[7]));
      const int at = (h - p.H) * p.dim + c0;
      *reinterpret_cast<uint4*>(row + (p.H + p.G) * p.dim + at) = o;
      *reinterpret_cast<uint4*>(crow + p.G * p.dim + at) = o;
    }
  }
  const float* cs = p.angles + static_cast<long long>(t) * p.rot;
  if (p.q_norm) {
    const float* w = (h < p.H ? p.q_norm : p.k_norm) + c0;
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.f / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
    if (on) {
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= inv * w[j];
    }
  }
  if (p.temp_every > 0 && h < p.H) {
    const float f = query_factor(p, t);
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] *= f;
  }
  if (p.pairs) {
    if (on) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int f = c0 / 2 + j;
        if (f < half) {
          const float c = cs[f], s = cs[half + f], u = a[2 * j], v = a[2 * j + 1];
          a[2 * j] = u * c - v * s;
          a[2 * j + 1] = v * c + u * s;
        }
      }
    }
  } else if (half % 8 == 0 && p.rot > 0) {
    const bool first = c0 < half, rotated = c0 < p.rot;
    const int other = slot * LPH + (first ? sub + half / 8 : (rotated ? sub - half / 8 : sub)), f0 = first ? c0 : c0 - half;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float b = __shfl_sync(0xffffffffu, a[j], other);
      if (on && rotated) {
        const float c = cs[f0 + j], s = cs[half + f0 + j];
        a[j] = first ? a[j] * c - b * s : a[j] * c + b * s;
      }
    }
  } else if (p.rot > 0) {
    float* buf = swap[warp][slot];
#pragma unroll
    for (int j = 0; j < 8; ++j) buf[c0 + j] = a[j];
    __syncwarp();
    if (on) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int c = c0 + j;
        if (c < half) a[j] = a[j] * cs[c] - buf[c + half] * cs[half + c];
        else if (c < p.rot) a[j] = a[j] * cs[c - half] + buf[c - half] * cs[c];
      }
    }
  }
  if (on) {
    const uint4 o = make_uint4(pack_bf16x2(a[0], a[1]), pack_bf16x2(a[2], a[3]), pack_bf16x2(a[4], a[5]), pack_bf16x2(a[6], a[7]));
    *reinterpret_cast<uint4*>(x) = o;
    if (h >= p.H) *reinterpret_cast<uint4*>(crow + (h - p.H) * p.dim + c0) = o;
  }
}

// ---------------------------------------------------------------------------------------------------------
// attention of single rows
// ---------------------------------------------------------------------------------------------------------
struct WindowAttendParams {
  const void* q;               // rows [H x dim | ...]
  long long q_ld;
  const void* cache;           // [slots][row_width]
  const int* block_table;      // [sequences][max_blocks]
  const int* row_seq;          // [rows]
  const int* row_len;          // [rows] keys visible before the window is applied (position + 1)
  void* out;                   // [rows][out_ld], head h at column h * vdim
  long long out_ld;
  float* part_out;             // [rows][H][splits][vdim]
  float* part_lse;             // [rows][H][splits]
  const void* gate;            // result *= sigmoid(gate), type of q: rows [gate_ld], see gate_mode (nullptr: none)
  long long gate_ld;
  int gate_mode;               // GATE_HEAD: column h, GATE_ELEMENT: column h * vdim + c
  const float* slopes;         // [H] subtracted from a score per position of distance (nullptr: none)
  const float* add;            // [H] added to every score (nullptr: none)
  int sigmoid;                 // weights: sigmoid(score), not normalized
  float limit;                 // no (q . k) * scale exceeds it: sigmoid weights that fade with the distance end at some key
  int rows, H, G, dim, vdim, row_width, max_blocks, block_size, window, keep, chunked, chunk, splits;
  float scale, o_scale;
};

// A row's visible keys, numbered 0 .. count - 1 in key order: the kept first positions, then those from `lo` on.
struct VisibleKeys {
  int lo, kept, count;
  __device__ VisibleKeys(const WindowAttendParams& p, int len, int reach) {
    lo = p.chunked ? (len - 1) / p.window * p.window : max(0, len - min(p.window, reach));
    kept = min(p.keep, lo);
    count = len - lo + kept;
  }
  __device__ int position(int i) const { return i < kept ? i : i - kept + lo; }
};

template <typename T> __device__ __forceinline__ float gate_factor(const WindowAttendParams& p, int row, int h, int c) {
  if (!p.gate) return 1.f;
  const int col = p.gate_mode == GATE_HEAD ? h : h * p.vdim + c;
  return sigmoid(to_f32(reinterpret_cast<const T*>(p.gate)[row * p.gate_ld + col]));
}

__device__ __forceinline__ float sigmoid_ex2(float x) {      // 1 / (1 + 2^-x)
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + fast_ex2(-x)));
  return y;
}

constexpr int WS_CHUNK = 512;

// grid (rows, H).  Scores of WS_CHUNK keys at a time in shared memory, then threads own value columns.
template <typename T>
__global__ void __launch_bounds__(128) window_attend_simt_kernel(WindowAttendParams p) {
  extern __shared__ float sm[];
  __shared__ float scratch[32];
  float* qs = sm;                          // [dim]
  float* acc = sm + p.dim;                 // [vdim]
  float* sc = acc + p.vdim;                // [WS_CHUNK]
  const int row = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int len = p.row_len[row];
  const int* bt = p.block_table + static_cast<long long>(p.row_seq[row]) * p.max_blocks;
  const T* cache = reinterpret_cast<const T*>(p.cache);
  const T* q = reinterpret_cast<const T*>(p.q) + row * p.q_ld + h * p.dim;
  for (int i = threadIdx.x; i < p.dim; i += blockDim.x) qs[i] = to_f32(q[i]);
  for (int i = threadIdx.x; i < p.vdim; i += blockDim.x) acc[i] = 0.f;
  float m = p.sigmoid ? 0.f : -INFINITY, l = 0.f;
  const float slope = p.slopes ? p.slopes[h] : 0.f, add = p.add ? p.add[h] : 0.f;
  const VisibleKeys vis(p, len, p.sigmoid ? sigmoid_reach(p.limit, add, slope) : 1 << 30);
  auto key_row = [&](int i) {
    const int j = vis.position(i);
    return cache + (static_cast<long long>(bt[j / p.block_size]) * p.block_size + j % p.block_size) * p.row_width;
  };
  for (int j0 = 0; j0 < vis.count; j0 += WS_CHUNK) {
    const int j1 = min(vis.count, j0 + WS_CHUNK);
    __syncthreads();
    float mx = -INFINITY;
    for (int j = j0 + warp; j < j1; j += nw) {
      const T* c = key_row(j) + g * p.dim;
      float s = 0.f;
      for (int i = lane; i < p.dim; i += 32) s += qs[i] * to_f32(c[i]);
      s = warp_sum(s) * p.scale - slope * static_cast<float>(len - 1 - vis.position(j)) + add;
      if (lane == 0) sc[j - j0] = s;
      mx = fmaxf(mx, s);
    }
    const float top = block_max(mx, scratch), m_new = p.sigmoid ? 0.f : fmaxf(m, top);
    const float alpha = expf(m - m_new);   // m = -inf at first: 0
    float part = 0.f;
    for (int j = j0 + threadIdx.x; j < j1; j += blockDim.x) {
      const float w = p.sigmoid ? sigmoid(sc[j - j0]) : expf(sc[j - j0] - m_new);
      sc[j - j0] = w;
      part += w;
    }
    l = l * alpha + block_sum(part, scratch);    // also orders the weights
    m = m_new;
    for (int r = threadIdx.x; r < p.vdim; r += blockDim.x) {
      float a = acc[r] * alpha;
      for (int j = j0; j < j1; ++j) a += sc[j - j0] * to_f32(key_row(j)[p.G * p.dim + g * p.vdim + r]);
      acc[r] = a;
    }
  }
  const float inv = p.sigmoid ? p.o_scale : (l > 0.f ? p.o_scale / l : 0.f);
  T* out = reinterpret_cast<T*>(p.out) + row * p.out_ld + h * p.vdim;
  for (int r = threadIdx.x; r < p.vdim; r += blockDim.x) out[r] = from_f32<T>(acc[r] * inv * gate_factor<T>(p, row, h, r));
}

constexpr int WA_WARPS = 4;
constexpr int WA_STAGES = 3;
constexpr int WA_KT = 16;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// shared-memory row stride in elements for `cols` columns (rounded up to 16): an odd number of 16-byte units
__host__ __device__ inline int window_stride(int cols) { return (cols + 15) / 16 * 16 + 8; }
static size_t window_smem(int dim, int vdim) {
  const size_t ring = static_cast<size_t>(WA_WARPS) * WA_STAGES * WA_KT * (window_stride(dim) + window_stride(vdim)) * 2;
  const size_t merge = static_cast<size_t>(WA_WARPS) * 16 * (vdim + 2) * 4;
  return (ring > merge ? ring : merge) + 16 * window_stride(dim) * 2;
}

// grid (rows, G * ceil(group / 16), splits).  DC: head sizes up to DC columns.  SIG: sigmoid weights.
template <int DC, bool SIG>
__global__ void __launch_bounds__(WA_WARPS * 32) window_attend_mma_kernel(WindowAttendParams p) {
  constexpr int KS = DC / 16, NV = DC / 8;
  extern __shared__ __align__(16) uint8_t raw[];
  const int kst = window_stride(p.dim), vst = window_stride(p.vdim);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(raw);                       // [16][kst]
  __nv_bfloat16* ring = qs + 16 * kst;
  const int row = blockIdx.x, split = blockIdx.z;
  const int group = p.H / p.G, tiles_h = (group + 15) / 16;
  const int g = blockIdx.y / tiles_h, h0 = g * group + (blockIdx.y % tiles_h) * 16;
  const int nh = min(16, (g + 1) * group - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int len = p.row_len[row];
  int reach = 1 << 30;                     // of the farthest-reaching head
  if (SIG && p.slopes) {
    reach = 0;
    for (int i = 0; i < nh; ++i) reach = max(reach, sigmoid_reach(p.limit, p.add ? p.add[h0 + i] : 0.f, p.slopes[h0 + i]));
  }
  const VisibleKeys vis(p, len, reach);
  const int chunk = SIG ? ((vis.count + p.splits - 1) / p.splits + WA_KT - 1) / WA_KT * WA_KT : p.chunk;
  const int j0 = split * chunk, j1 = min(vis.count, j0 + chunk);           // this CTA's share of them
  const int* bt = p.block_table + static_cast<long long>(p.row_seq[row]) * p.max_blocks;
  const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(p.cache) + g * p.dim;
  const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(p.cache) + p.G * p.dim + g * p.vdim;
  const int ku = (p.dim + 15) / 16 * 2, vu = (p.vdim + 15) / 16 * 2;               // 16-byte units of a staged row
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + row * p.q_ld + h0 * p.dim;
    for (int i = threadIdx.x; i < 16 * ku; i += blockDim.x) {
      const int r = i / ku, c = i - r * ku;
      *reinterpret_cast<uint4*>(qs + r * kst + c * 8) =
          r < nh && c * 8 < p.dim ? *reinterpret_cast<const uint4*>(q + r * p.dim + c * 8) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  __nv_bfloat16* mine = ring + warp * WA_STAGES * WA_KT * (kst + vst);
  // this warp's tiles: visible keys t * 16 .. + 15 for t = t_first + warp, + 4, ... (a chunk is whole tiles)
  const int t_first = j0 / WA_KT, t_end = j1 > j0 ? (j1 + WA_KT - 1) / WA_KT : t_first;
  auto slot_of = [&](int tile) {         // cache row of key tile * 16 + lane % 16 (-1: outside the range)
    const int i = tile * WA_KT + (lane & 15), j = vis.position(i);
    return tile < t_end && i < j1 ? bt[j / p.block_size] * p.block_size + j % p.block_size : -1;
  };
  auto load = [&](int stage, int slot) {
    const uint32_t kd = smem_u32(mine + stage * WA_KT * (kst + vst)), vd = kd + WA_KT * kst * 2;
    for (int i = lane; i < WA_KT * ku + (32 - WA_KT * ku % 32) % 32; i += 32) {
      const int r = min(i / ku, WA_KT - 1), c = i - r * ku;
      const int s = __shfl_sync(0xffffffffu, slot, r);
      if (i < WA_KT * ku) {
        const bool ok = s >= 0 && c * 8 < p.dim;
        cp_async16(kd + (r * kst + c * 8) * 2, ok ? kc + static_cast<long long>(s) * p.row_width + c * 8 : kc, ok);
      }
    }
    for (int i = lane; i < WA_KT * vu + (32 - WA_KT * vu % 32) % 32; i += 32) {
      const int r = min(i / vu, WA_KT - 1), c = i - r * vu;
      const int s = __shfl_sync(0xffffffffu, slot, r);
      if (i < WA_KT * vu) {
        const bool ok = s >= 0 && c * 8 < p.vdim;
        cp_async16(vd + (r * vst + c * 8) * 2, ok ? vc + static_cast<long long>(s) * p.row_width + c * 8 : vc, ok);
      }
    }
  };
  int next = t_first + warp;
  int slot = slot_of(next);
#pragma unroll
  for (int s = 0; s < WA_STAGES - 1; ++s) {
    if (next < t_end) load(s, slot);
    cp_commit();
    next += WA_WARPS;
    slot = slot_of(next);
  }
  __syncthreads();                         // queries staged
  uint32_t qf[KS][4];
#pragma unroll
  for (int k = 0; k < KS; ++k)
    if (k * 16 < p.dim) ldsm_x4(qf[k], smem_u32(qs + (lane & 15) * kst + k * 16 + (lane >> 4) * 8));
  float o[NV][4];
#pragma unroll
  for (int n = 0; n < NV; ++n)
#pragma unroll
    for (int q = 0; q < 4; ++q) o[n][q] = 0.f;
  constexpr float LOG2E = 1.4426950408889634f;
  float m0 = SIG ? 0.f : -INFINITY, m1 = m0, l0 = 0.f, l1 = 0.f;
  const float sl = p.scale * LOG2E;
  // slope and addend of this thread's two heads, in powers of two
  const bool biased = p.slopes || p.add;
  const int ha = h0 + min(gid, nh - 1), hb = h0 + min(gid + 8, nh - 1);
  const float slope0 = p.slopes ? p.slopes[ha] * LOG2E : 0.f, slope1 = p.slopes ? p.slopes[hb] * LOG2E : 0.f;
  const float add0 = p.add ? p.add[ha] * LOG2E : 0.f, add1 = p.add ? p.add[hb] * LOG2E : 0.f;
  int stage = 0;
  for (int t = t_first + warp; t < t_end; t += WA_WARPS) {
    cp_wait<WA_STAGES - 2>();
    __syncwarp();
    const __nv_bfloat16* kt = mine + stage * WA_KT * (kst + vst);
    const __nv_bfloat16* vt = kt + WA_KT * kst;
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t ka = smem_u32(kt + ((lane & 7) + (lane >> 4) * 8) * kst + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int k = 0; k < KS; ++k)
      if (k * 16 < p.dim) {
        uint32_t b[4];                     // keys 0-7: b[0], b[1]; keys 8-15: b[2], b[3]
        ldsm_x4(b, ka + k * 32);
        mma_16816(s0, qf[k], b[0], b[1]);
        mma_16816(s1, qf[k], b[2], b[3]);
      }
    const int j = t * WA_KT + tig * 2;
    auto keep = [&](float v, int key) { return key < j1 ? v * sl : -INFINITY; };
    s0[0] = keep(s0[0], j); s0[1] = keep(s0[1], j + 1); s0[2] = keep(s0[2], j); s0[3] = keep(s0[3], j + 1);
    s1[0] = keep(s1[0], j + 8); s1[1] = keep(s1[1], j + 9); s1[2] = keep(s1[2], j + 8); s1[3] = keep(s1[3], j + 9);
    if (biased) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float da = static_cast<float>(len - 1 - vis.position(j + e)), db = static_cast<float>(len - 1 - vis.position(j + 8 + e));
        s0[e] += add0 - slope0 * da;
        s1[e] += add0 - slope0 * db;
        s0[2 + e] += add1 - slope1 * da;
        s1[2 + e] += add1 - slope1 * db;
      }
    }
    float f0 = 1.f, f1 = 1.f;
    if (SIG) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s0[e] = sigmoid_ex2(s0[e]);
        s1[e] = sigmoid_ex2(s1[e]);
      }
    } else {
      float a = fmaxf(fmaxf(s0[0], s0[1]), fmaxf(s1[0], s1[1])), b = fmaxf(fmaxf(s0[2], s0[3]), fmaxf(s1[2], s1[3]));
      a = fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 1));
      b = fmaxf(b, __shfl_xor_sync(0xffffffffu, b, 1));
      a = fmaxf(m0, fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 2)));   // finite: every tile has a key in the range
      b = fmaxf(m1, fmaxf(b, __shfl_xor_sync(0xffffffffu, b, 2)));
      f0 = fast_ex2(m0 - a);
      f1 = fast_ex2(m1 - b);
      m0 = a;
      m1 = b;
      s0[0] = fast_ex2(s0[0] - a); s0[1] = fast_ex2(s0[1] - a); s1[0] = fast_ex2(s1[0] - a); s1[1] = fast_ex2(s1[1] - a);
      s0[2] = fast_ex2(s0[2] - b); s0[3] = fast_ex2(s0[3] - b); s1[2] = fast_ex2(s1[2] - b); s1[3] = fast_ex2(s1[3] - b);
      l0 = l0 * f0 + ((s0[0] + s0[1]) + (s1[0] + s1[1]));
      l1 = l1 * f1 + ((s0[2] + s0[3]) + (s1[2] + s1[3]));
    }
    const uint32_t pf[4] = {pack_bf16x2(s0[0], s0[1]), pack_bf16x2(s0[2], s0[3]), pack_bf16x2(s1[0], s1[1]),
                            pack_bf16x2(s1[2], s1[3])};
    const uint32_t va = smem_u32(vt + (lane & 15) * vst + (lane >> 4) * 8);
#pragma unroll
    for (int n = 0; n < NV; n += 2)
      if (n * 8 < p.vdim) {
        uint32_t bv[4];                    // columns 8 n: bv[0], bv[1]; the next eight: bv[2], bv[3]
        ldsm_x4_t(bv, va + n * 16);
        if (!SIG) {
          o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1;
          o[n + 1][0] *= f0; o[n + 1][1] *= f0; o[n + 1][2] *= f1; o[n + 1][3] *= f1;
        }
        mma_16816(o[n], pf, bv[0], bv[1]);
        mma_16816(o[n + 1], pf, bv[2], bv[3]);
      }
    __syncwarp();                          // all lanes are done with the stage that is filled next
    {
      const int fill = stage == 0 ? WA_STAGES - 1 : stage - 1;
      if (next < t_end) load(fill, slot);
      cp_commit();
      next += WA_WARPS;
      slot = slot_of(next);
    }
    stage = stage + 1 == WA_STAGES ? 0 : stage + 1;
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  cp_wait<0>();
  __syncthreads();
  // merge of the four warps: [warp][16][vdim + 2] = sums, maximum, weight
  float* mg = reinterpret_cast<float*>(ring);
  const int ms = p.vdim + 2;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float* d = mg + (warp * 16 + gid + half * 8) * ms;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int c = n * 8 + tig * 2;
      if (c < p.vdim) {
        d[c] = o[n][2 * half];
        d[c + 1] = o[n][2 * half + 1];
      }
    }
    if (tig == 0) {
      d[p.vdim] = half ? m1 : m0;
      d[p.vdim + 1] = half ? l1 : l0;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * p.vdim; i += blockDim.x) {
    const int r = i / p.vdim, c = i - r * p.vdim;
    float mm = -INFINITY, l = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < WA_WARPS; ++w) mm = fmaxf(mm, mg[(w * 16 + r) * ms + p.vdim]);
#pragma unroll
    for (int w = 0; w < WA_WARPS; ++w) {
      const float* d = mg + (w * 16 + r) * ms;
      const float f = d[p.vdim] == -INFINITY ? 0.f : fast_ex2(d[p.vdim] - mm);
      l += d[p.vdim + 1] * f;
      acc += d[c] * f;
    }
    if (SIG) l = 1.f;                      // the sums are the result
    const int h = h0 + r;
    if (p.splits == 1) {
      reinterpret_cast<__nv_bfloat16*>(p.out)[row * p.out_ld + h * p.vdim + c] =
          __float2bfloat16(l > 0.f ? acc * (p.o_scale / l) * gate_factor<__nv_bfloat16>(p, row, h, c) : 0.f);
    } else {
      const long long at = (static_cast<long long>(row) * p.H + h) * p.splits + split;
      p.part_out[at * p.vdim + c] = l > 0.f ? acc / l : 0.f;
      if (c == 0 && !SIG) p.part_lse[at] = l > 0.f ? mm + log2f(l) : -INFINITY;      // in powers of two
    }
  }
}

constexpr int WM_MAX_SPLITS = 64;
__global__ void __launch_bounds__(128) window_merge_kernel(WindowAttendParams p) {
  const int row = blockIdx.x, h = blockIdx.y;
  const long long base = (static_cast<long long>(row) * p.H + h) * p.splits;
  float mm = -INFINITY, l = p.sigmoid ? 1.f : 0.f;
  if (!p.sigmoid) {
    for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.part_lse[base + s]);
    for (int s = 0; s < p.splits; ++s) l += fast_ex2(p.part_lse[base + s] - mm);
  }
  for (int c = threadIdx.x; c < p.vdim; c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < p.splits; ++s)
      acc += (p.sigmoid ? 1.f : fast_ex2(p.part_lse[base + s] - mm)) * p.part_out[(base + s) * p.vdim + c];
    reinterpret_cast<__nv_bfloat16*>(p.out)[row * p.out_ld + h * p.vdim + c] =
        __float2bfloat16(acc * (p.o_scale / l) * gate_factor<__nv_bfloat16>(p, row, h, c));
  }
}

template <int DC, bool SIG> static int launch_window_mma(const WindowAttendParams& p, cudaStream_t st) {
  const size_t smem = window_smem(p.dim, p.vdim);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(window_attend_mma_kernel<DC, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int tiles_h = (p.H / p.G + 15) / 16;
  window_attend_mma_kernel<DC, SIG><<<dim3(p.rows, p.G * tiles_h, p.splits), WA_WARPS * 32, smem, st>>>(p);
  return (int)cudaGetLastError();
}

template <bool SIG> static int dispatch_window_mma(const WindowAttendParams& p, cudaStream_t st) {
  const int dc = p.dim > p.vdim ? p.dim : p.vdim;
  return dc <= 64 ? launch_window_mma<64, SIG>(p, st) : (dc <= 128 ? launch_window_mma<128, SIG>(p, st) : launch_window_mma<256, SIG>(p, st));
}

static bool window_mma_ok(int dim, int vdim, int fp32) {
  return !fp32 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && vdim <= 256 && window_smem(dim, vdim) <= 227 * 1024;
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_window)
using namespace ts;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

// out: [T][cos | sin of pos * inv_freq], both times `magnitude`, half frequencies.
extern "C" int ts_window_angles(const float* inv_freq, const int* pos, float* out, int T, int half, float magnitude,
                                void* stream) {
  if (T <= 0 || half <= 0) return 0;
  window_angles_kernel<<<(T * half + 255) / 256, 256, 0, ST(stream)>>>(inv_freq, pos, out, T, half, magnitude);
  return (int)cudaGetLastError();
}

// angles: of ts_window_angles (unused without rotated dimensions).  bias, norms: nullptr for none (both norms or neither).
// pairs: rotation partners are neighbours.  values_are_keys: the projection has no values, its columns behind the keys
// receive the keys before norm and rotation.  pos, temp_coef, temp_every: the queries' factor (temp_every 0: none).
extern "C" int ts_window_prep(void* proj, long long ld, const float* bias, const float* q_norm, const float* k_norm, float eps,
                              const float* angles, const long long* slots, void* cache, int T, int H, int G, int dim, int vdim,
                              int rot, int pairs, int values_are_keys, const int* pos, float temp_coef, int temp_every, int row_width,
                              int fp32, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || dim <= 0 || vdim <= 0 || rot < 0 || rot > dim || rot % 2 || row_width < G * (dim + vdim)) return -10;
  if ((q_norm == nullptr) != (k_norm == nullptr) || (values_are_keys && dim != vdim) || temp_every < 0 || (temp_every > 0 && !pos))
    return -10;
  WindowPrepParams p;
  p.bias = bias; p.pairs = pairs; p.values_are_keys = values_are_keys; p.h0 = bias || q_norm || rot || temp_every ? 0 : H;
  p.pos = pos; p.temp_coef = temp_coef; p.temp_every = temp_every;
  p.proj = proj; p.ld = ld; p.q_norm = q_norm; p.k_norm = k_norm; p.eps = eps; p.angles = angles; p.slots = slots;
  p.cache = cache; p.T = T; p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.rot = rot; p.row_width = row_width;
  const bool vec = !fp32 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && ld % 8 == 0 && row_width == G * (dim + vdim) &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cache)) & 15u) == 0;
  if (vec) {
    int lph = 4;
    while (lph * 8 < dim) lph *= 2;
    const int hpw = 32 / lph;
    const int per_token = (H + G - p.h0 + hpw - 1) / hpw + (values_are_keys ? 0 : (G * vdim / 8 + 31) / 32);
    const unsigned grid = (unsigned)((static_cast<long long>(T) * per_token + WP_WARPS - 1) / WP_WARPS);
    if (lph == 4) window_prep_vec_kernel<4><<<grid, WP_WARPS * 32, 0, ST(stream)>>>(p);
    else if (lph == 8) window_prep_vec_kernel<8><<<grid, WP_WARPS * 32, 0, ST(stream)>>>(p);
    else if (lph == 16) window_prep_vec_kernel<16><<<grid, WP_WARPS * 32, 0, ST(stream)>>>(p);
    else window_prep_vec_kernel<32><<<grid, WP_WARPS * 32, 0, ST(stream)>>>(p);
    return (int)cudaGetLastError();
  }
  if (fp32) window_prep_kernel<float><<<T, WP_WARPS * 32, 0, ST(stream)>>>(p);
  else window_prep_kernel<__nv_bfloat16><<<T, WP_WARPS * 32, 0, ST(stream)>>>(p);
  return (int)cudaGetLastError();
}

// Split count of ts_window_attend for `keys` visible keys: enough CTAs for two per SM, at least 128 keys each.
extern "C" int ts_window_splits(int rows, int H, int G, int dim, int vdim, int keys, int fp32) {
  if (!window_mma_ok(dim, vdim, fp32)) return 1;
  const int ctas = rows * G * ((H / G + 15) / 16);
  int s = (2 * sm_count() + ctas - 1) / ctas, most = (keys + 127) / 128;
  if (s > most) s = most;
  if (s > WM_MAX_SPLITS) s = WM_MAX_SPLITS;
  return s < 1 ? 1 : s;
}

// window, keep, chunked: which keys a row sees; slopes, add, sigmoid, limit: their weights (top of the file).  `keys`: upper bound of their number; `splits` of ts_window_splits with the workspaces it needs (splits > 1).
extern "C" int ts_window_attend(const void* q, long long q_ld, const void* cache, const int* block_table, int max_blocks,
                                const int* row_seq, const int* row_len, void* out, long long out_ld, float* part_out,
                                float* part_lse, int rows, int H, int G, int dim, int vdim, int row_width, int block_size,
                                int window, int keep, int chunked, int keys, int splits, float scale, float o_scale,
                                const float* slopes, const float* add, int sigmoid, float limit, const void* gate, long long gate_ld,
                                int gate_mode, int fp32, void* stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dim <= 0 || vdim <= 0 || window <= 0 || keep < 0 || keys <= 0 || splits < 1 ||
      splits > WM_MAX_SPLITS)
    return -10;
  WindowAttendParams p;
  p.q = q; p.q_ld = q_ld; p.cache = cache; p.block_table = block_table; p.row_seq = row_seq; p.row_len = row_len; p.out = out;
  p.out_ld = out_ld; p.part_out = part_out; p.part_lse = part_lse; p.rows = rows; p.H = H; p.G = G; p.dim = dim;
  p.vdim = vdim; p.row_width = row_width; p.max_blocks = max_blocks; p.block_size = block_size; p.window = window;
  p.keep = keep; p.chunked = chunked; p.slopes = slopes; p.add = add; p.sigmoid = sigmoid; p.limit = limit; p.gate = gate; p.gate_ld = gate_ld; p.gate_mode = gate_mode;
  p.splits = splits; p.chunk = ((keys + splits - 1) / splits + 15) / 16 * 16; p.scale = scale; p.o_scale = o_scale;
  const bool vec = window_mma_ok(dim, vdim, fp32) && scale > 0.f && q_ld % 8 == 0 && row_width % 8 == 0 &&
                   (reinterpret_cast<uintptr_t>(q) & 15u) == 0 && (reinterpret_cast<uintptr_t>(cache) & 15u) == 0;
  if (!vec) {
    const size_t smem = (dim + vdim + WS_CHUNK) * sizeof(float);
    if (smem > 48 * 1024) return -11;
    if (fp32) window_attend_simt_kernel<float><<<dim3(rows, H), 128, smem, ST(stream)>>>(p);
    else window_attend_simt_kernel<__nv_bfloat16><<<dim3(rows, H), 128, smem, ST(stream)>>>(p);
    return (int)cudaGetLastError();
  }
  int rc = sigmoid ? dispatch_window_mma<true>(p, ST(stream)) : dispatch_window_mma<false>(p, ST(stream));
  if (rc == 0 && splits > 1) {
    window_merge_kernel<<<dim3(rows, H), 128, 0, ST(stream)>>>(p);
    rc = (int)cudaGetLastError();
  }
  return rc;
}
