// Windowed causal attention for portions of prompts (tcgen05 / TMEM / TMA), two entry points:
//   ts_latent_prefill  keys come from a latent cache
//   ts_window_prefill  keys and values per key/value head (grouped queries), query / key and value sizes of their own
//
// The latents a portion needs (its own tokens and the window before them) have been expanded to per-head keys and values
// by one GEMM; the rotated key part is shared by all heads and read from the latent rows.  Scores are therefore a sum of
// two products with operands of different origin:  S = Qn Kn^T (per head) + Qr Kr^T (shared),  O = softmax(S) V.
//
// Per CTA: one 256-row query block of one head of one sequence, as two 128-row tiles that ping-pong:
//   warp 0       TMA loader: Q tiles once, then rings of 128-row key and value tiles.  Every operand is cut into
//                64-column blocks (128-byte swizzle); 3-D maps (column, head, token) zero-fill columns past the head's
//                size, so heads of any multiple of eight columns use the same code
//   warp 1       MMA issuer: S_t = Q_t K^T over the unrotated, then the rotated columns; O_t += P_t V, P_t from TMEM
//   warps 2..9   softmax: one thread per query row; scores, running max and sum in fp32.  Or (`SIG`) weights that are not
//                normalized: sigmoid(score + a number per head - a slope per head times the distance), so there is no running
//                maximum, no rescaling and no sum; with a slope the key tiles begin where a weight can reach 2^-48
// Queries are the LAST Lq of the sequence's Lk keys.  A query sees the `window` keys up to its own, or those of its chunk of
// `window` keys (the first key row then lies on a chunk's border), and besides the first `keep` key rows; these are the
// sequence's first positions, which a portion's caller may have put right in front of its window.  Key tiles that no row
// sees are never loaded.  The result may be multiplied by the sigmoid of a gate per head or per element.
#include "common.cuh"
#include "host_common.h"

namespace ts {

constexpr int LP_THREADS = 320;
constexpr int LP_BLOCK = 16384;          // 128 rows x 64 bf16 columns

__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct LatentPrefillParams {
  const int* cu_q;                       // [sequences + 1] query rows
  const int* cu_k;                       // [sequences + 1] key rows
  int H;
  int nb_n, nb_r, nb_v;                  // 64-column blocks of the unrotated part, the rotated part, the value
  int ks_n, ks_r;                        // 16-column MMA steps
  int vdim, v_cols;                      // value size; rounded up to 16
  int k_stages, v_stages;
  int window, keep, chunked;
  int kv_group;                          // query heads that share a key/value head
  const __nv_bfloat16* gate;             // [query rows][gate_ld] (nullptr: none)
  long long gate_ld;
  int gate_mode;                         // GATE_HEAD: column h, GATE_ELEMENT: column h * vdim + c
  const float* slopes;                   // SIG: [H] (nullptr: zeros)
  const float* add;                      // SIG: [H] (nullptr: zeros)
  float limit;                           // SIG: no (q . k) * scale exceeds it
  float scale_log2;
  float o_scale;                         // factor of the result
  __nv_bfloat16* o;                      // [rows][o_stride], head h at column h * vdim
  long long o_stride;
};

// first key row of the window or chunk of the query at key row c
__device__ __forceinline__ int window_first(const LatentPrefillParams& p, int window, int c) {
  return p.chunked ? c / window * window : max(0, c - window + 1);
}

template <bool SIG>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQn, const __grid_constant__ CUtensorMap tmQr,
                      const __grid_constant__ CUtensorMap tmKn, const __grid_constant__ CUtensorMap tmKr,
                      const __grid_constant__ CUtensorMap tmV, LatentPrefillParams p) {
  constexpr uint32_t TMEM_COLS = 512;
  constexpr uint32_t O_COL0 = 256;       // O_t at O_COL0 + 128 t
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nb_k = p.nb_n + p.nb_r;
  const int q_bytes = nb_k * LP_BLOCK, k_bytes = nb_k * LP_BLOCK, v_bytes = p.nb_v * LP_BLOCK;
  uint8_t* k_base = smem + 2 * q_bytes;
  uint8_t* v_base = k_base + p.k_stages * k_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_base + p.v_stages * v_bytes);
  uint64_t* q_full = bars;          // [2]
  uint64_t* k_full = bars + 2;      // [2]
  uint64_t* k_empty = bars + 4;     // [2]
  uint64_t* v_full = bars + 6;      // [2]
  uint64_t* v_empty = bars + 8;     // [2]
  uint64_t* s_full = bars + 10;     // [2]
  uint64_t* p_full = bars + 12;     // [2]
  uint64_t* o_full = bars + 14;     // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x % p.H, b = blockIdx.x / p.H;
  const int hk = h / p.kv_group;
  const int q_start = p.cu_q[b], Lq = p.cu_q[b + 1] - q_start;
  const int k_start = p.cu_k[b], Lk = p.cu_k[b + 1] - k_start;
  const int n_qblocks = (Lq + 255) / 256;
  if ((int)blockIdx.y >= n_qblocks) return;
  const int qb = n_qblocks - 1 - blockIdx.y;
  const int off = Lk - Lq;
  // sigmoid weights that fade with the distance: keys behind the last one that can count are not looked at
  const int window = SIG && !p.chunked && p.slopes
                         ? min(p.window, sigmoid_reach(p.limit, p.add ? p.add[h] : 0.f, p.slopes[h]) + 1) : p.window;
  // the block's key tiles: those of the kept rows left of its first window, then the windows' (kb_lo on).  Query tile t works
  // on [0, held[t]), which hold kept rows (also where they are among the windows'), and on [first[t], nkv[t])
  int r0[2], held[2], first[2], nkv[2];
  const int keep_tiles = (p.keep + 127) / 128;
  const int kb_lo = window_first(p, window, qb * 256 + off) / 128, kept = min(keep_tiles, kb_lo);
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    r0[t] = qb * 256 + t * 128;
    first[t] = kept + window_first(p, window, r0[t] + off) / 128 - kb_lo;
    held[t] = min(keep_tiles, first[t]);
    nkv[t] = r0[t] >= Lq ? 0 : max(0, kept + (min(Lk, r0[t] + 128 + off) + 127) / 128 - kb_lo);
  }
  const int n = max(nkv[0], nkv[1]);
  auto key_tile = [&](int i) { return i < kept ? i : kb_lo + i - kept; };
  auto works_on = [&](int t, int i) { return i < nkv[t] && (i < held[t] || i >= first[t]); };
  // how many tiles t has worked on before tile i
  auto worked = [&](int t, int i) { return i < held[t] ? i : held[t] + i - first[t]; };

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQn);
    tma_prefetch_desc(&tmKn);
    tma_prefetch_desc(&tmKr);
    tma_prefetch_desc(&tmV);
    for (int i = 0; i < 16; ++i) mbar_init(&bars[i], (i == 12 || i == 13) ? 4 : 1);
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, TMEM_COLS);
    tmem_relinquish();
    tc_fence_before_sync();
  }
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  bool alive = true;

  if (warp == 0) {
    if (elect_one_sync()) {
      for (int t = 0; t < 2; ++t) {
        if (nkv[t] == 0) continue;
        mbar_expect_tx(&q_full[t], q_bytes);
        for (int j = 0; j < p.nb_n; ++j)
          tma_load_3d(smem + t * q_bytes + j * LP_BLOCK, &tmQn, &q_full[t], j * 64, h, q_start + r0[t]);
        for (int j = 0; j < p.nb_r; ++j)
          tma_load_3d(smem + t * q_bytes + (p.nb_n + j) * LP_BLOCK, &tmQr, &q_full[t], j * 64, h, q_start + r0[t]);
      }
      uint32_t ki = 0, vi = 0;
      for (int i = 0; i < n && alive; ++i, ++ki, ++vi) {
        const int ks = ki % p.k_stages, vs = vi % p.v_stages, row = k_start + key_tile(i) * 128;
        if (!mbar_wait(&k_empty[ks], ((ki / p.k_stages) & 1u) ^ 1u, alive, 400)) break;
        mbar_expect_tx(&k_full[ks], k_bytes);
        for (int j = 0; j < p.nb_n; ++j)
          tma_load_3d(k_base + ks * k_bytes + j * LP_BLOCK, &tmKn, &k_full[ks], j * 64, hk, row);
        for (int j = 0; j < p.nb_r; ++j)
          tma_load_2d(k_base + ks * k_bytes + (p.nb_n + j) * LP_BLOCK, &tmKr, &k_full[ks], j * 64, row);
        if (!mbar_wait(&v_empty[vs], ((vi / p.v_stages) & 1u) ^ 1u, alive, 401)) break;
        mbar_expect_tx(&v_full[vs], v_bytes);
        for (int j = 0; j < p.nb_v; ++j)
          tma_load_3d(v_base + vs * v_bytes + j * LP_BLOCK, &tmV, &v_full[vs], j * 64, hk, row);
      }
    }
  } else if (warp == 1) {
    if (elect_one_sync()) {
      const uint32_t idesc_s = make_idesc(128, 128, 1, 1, 0, 0);
      const uint32_t idesc_o = make_idesc(128, p.v_cols, 1, 1, 0, 1);
      auto issue_s = [&](int t, int stage) {
        const uint32_t qa = smem_u32(smem + t * q_bytes), ka = smem_u32(k_base + stage * k_bytes);
        for (int k = 0; k < p.ks_n; ++k) {
          const uint32_t o = (k >> 2) * LP_BLOCK + (k & 3) * 32;
          umma_f16_ss(tmem_base + t * 128, make_smem_desc_sw128(qa + o, 16, 1024),
                      make_smem_desc_sw128(ka + o, 16, 1024), idesc_s, k != 0);
        }
        for (int k = 0; k < p.ks_r; ++k) {
          const uint32_t o = (p.nb_n + (k >> 2)) * LP_BLOCK + (k & 3) * 32;
          umma_f16_ss(tmem_base + t * 128, make_smem_desc_sw128(qa + o, 16, 1024),
                      make_smem_desc_sw128(ka + o, 16, 1024), idesc_s, 1u);
        }
        umma_commit(&s_full[t]);
      };
      for (int t = 0; t < 2; ++t)
        if (nkv[t] > 0) mbar_wait(&q_full[t], 0, alive, 500);
      if (n > 0 && mbar_wait(&k_full[0], 0, alive, 501)) {
        tc_fence_after_sync();
        for (int t = 0; t < 2; ++t)
          if (works_on(t, 0)) issue_s(t, 0);
        umma_commit(&k_empty[0]);
      }
      for (int i = 0; i < n && alive; ++i) {
        const int vs = i % p.v_stages, kn = (i + 1) % p.k_stages;
        if (!mbar_wait(&v_full[vs], (i / p.v_stages) & 1u, alive, 502)) break;
        bool k_waited = false;
        for (int t = 0; t < 2 && alive; ++t) {
          if (works_on(t, i)) {
            if (!mbar_wait(&p_full[t], worked(t, i) & 1u, alive, 503)) break;
            tc_fence_after_sync();
            const uint32_t va = smem_u32(v_base + vs * v_bytes);
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              umma_f16_ts(tmem_base + O_COL0 + t * 128, tmem_base + t * 128 + kk * 8,
                          make_smem_desc_sw128(va + kk * 2048, LP_BLOCK, 1024), idesc_o, worked(t, i) != 0 || kk != 0);
            if (i == nkv[t] - 1) umma_commit(&o_full[t]);
          }
          if (works_on(t, i + 1)) {
            if (!k_waited) {
              if (!mbar_wait(&k_full[kn], ((i + 1) / p.k_stages) & 1u, alive, 504)) break;
              tc_fence_after_sync();
              k_waited = true;
            }
            issue_s(t, kn);
          }
        }
        if (!alive) break;
        if (i + 1 < n) umma_commit(&k_empty[kn]);
        umma_commit(&v_empty[vs]);
      }
    }
  } else {
    const int t = (warp - 2) >> 2;
    const int q4 = warp & 3;
    const int r = q4 * 32 + lane;
    const int row = r0[t] + r;
    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(q4 * 32) << 16);
    const uint32_t t_s = t_lane + t * 128;
    const uint32_t t_o = t_lane + O_COL0 + t * 128;
    float m_used = -INFINITY, l = 0.f;
    const int nt = nkv[t];
    const float sc = p.scale_log2;
    const int limit = min(Lk - 1, row + off);          // last visible key
    const int lo = window_first(p, window, row + off);         // first key of the window
    const int lo_last = window_first(p, window, r0[t] + 127 + off);
    constexpr float LOG2E = 1.4426950408889634f;
    const float slope = SIG && p.slopes ? p.slopes[h] * LOG2E : 0.f, add = SIG && p.add ? p.add[h] * LOG2E : 0.f;
    for (int i = 0; i < nt && alive; ++i) {
      if (!works_on(t, i)) continue;
      if (!mbar_wait(&s_full[t], worked(t, i) & 1u, alive, 600)) break;
      tc_fence_after_sync();
      const int c0 = key_tile(i) * 128;
      const bool need_mask = (c0 + 127 > r0[t] + off) || (c0 + 128 > Lk) || (c0 < lo_last && c0 + 128 > p.keep);
      uint32_t v[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32b_x32(t_s + c * 32, v + c * 32);
      tc_wait_ld();
      uint32_t seen[4] = {0xffffffffu, 0xffffffffu, 0xffffffffu, 0xffffffffu};
      if (need_mask) {
        // visible columns of the tile are [lo - c0, limit - c0] and the kept ones [0, keep - c0): one bit per column, a word
        // per 32
        const int a = max(lo - c0, 0), e = min(limit - c0, 127), kc = p.keep - c0;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int s0 = a - c * 32, s1 = e - c * 32;      // first and last visible bit of this word
          uint32_t bits = s0 > 31 ? 0u : 0xffffffffu;
          if (s0 > 0) bits &= 0xffffffffu << (s0 & 31);
          if (kc > c * 32) bits |= kc >= c * 32 + 32 ? 0xffffffffu : (1u << (kc - c * 32)) - 1u;
          if (s1 < 31) bits &= s1 < 0 ? 0u : 0xffffffffu >> (31 - s1);
          if (SIG) {
            seen[c] = bits;
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (!(bits & (1u << j))) v[c * 32 + j] = 0xff800000u;
          }
        }
      }
      if (SIG) {
        // weight 1 / (1 + 2^e), e = -(score in powers of two); two columns share a reciprocal: 1 / d0 = d1 / (d0 d1), with e
        // held below 63 so that the product stays finite
        const float base = slope * static_cast<float>(row + off - c0) - add;
        const uint64_t nsc = pack_f32x2(-sc, -sc), nsl = pack_f32x2(-slope, -slope), bs = pack_f32x2(base, base);
        const uint64_t one = pack_f32x2(1.f, 1.f);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t pk[16];
#pragma unroll
          for (int j = 0; j < 32; j += 2) {
            const int col = c * 32 + j;
            const uint64_t b2 = fma_f32x2(pack_f32x2(static_cast<float>(col), static_cast<float>(col + 1)), nsl, bs);
            const float2 e = unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(v[col]), __uint_as_float(v[col + 1])), nsc, b2));
            const float2 d = unpack_f32x2(add_f32x2(pack_f32x2(fast_ex2(fminf(e.x, 63.f)), fast_ex2(fminf(e.y, 63.f))), one));
            const float r = fast_rcp(d.x * d.y);
            pk[j >> 1] = pack_bf16x2(d.y * r, d.x * r);
          }
          if (need_mask) {
#pragma unroll
            for (int j = 0; j < 32; j += 2)
              pk[j >> 1] &= ((seen[c] >> j & 1u) ? 0xffffu : 0u) | ((seen[c] >> (j + 1) & 1u) ? 0xffff0000u : 0u);
          }
          tmem_st_32x32b_x16(t_s + c * 16, pk);
        }
        tc_wait_st();
        tc_fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[t]);
        continue;
      }
      float mx0 = __uint_as_float(v[0]), mx1 = __uint_as_float(v[1]), mx2 = __uint_as_float(v[2]), mx3 = __uint_as_float(v[3]);
#pragma unroll
      for (int j = 4; j + 7 < 128; j += 8) {
        mx0 = max3(mx0, __uint_as_float(v[j]), __uint_as_float(v[j + 1]));
        mx1 = max3(mx1, __uint_as_float(v[j + 2]), __uint_as_float(v[j + 3]));
        mx2 = max3(mx2, __uint_as_float(v[j + 4]), __uint_as_float(v[j + 5]));
        mx3 = max3(mx3, __uint_as_float(v[j + 6]), __uint_as_float(v[j + 7]));
      }
      mx0 = max3(mx0, __uint_as_float(v[124]), __uint_as_float(v[125]));
      mx1 = max3(mx1, __uint_as_float(v[126]), __uint_as_float(v[127]));
      const float mx = fmaxf(max3(mx0, mx1, mx2), mx3);
      const float m_new = fmaxf(m_used, mx * sc);
      const bool grow = (m_new - m_used > 8.0f);       // also true on the first tile with a visible key
      if (__any_sync(0xffffffffu, grow)) {
        const float alpha = (m_used == -INFINITY) ? 0.f : fast_ex2(m_used - m_new);
        m_used = m_new;
        l *= alpha;
        if (worked(t, i) > 0) {
#pragma unroll 1
          for (int c = 0; c < p.v_cols / 16; ++c) {
            uint32_t o[16];
            tmem_ld_32x32b_x16(t_o + c * 16, o);
            tc_wait_ld();
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
            tmem_st_32x32b_x16(t_o + c * 16, o);
          }
        }
      }
      const float m_sub = (m_used == -INFINITY) ? 0.f : m_used;
      uint64_t sum0 = 0ull, sum1 = 0ull;
      const uint64_t sc2 = pack_f32x2(sc, sc), m2 = pack_f32x2(-m_sub, -m_sub);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
          const float2 e = unpack_f32x2(fma_f32x2(
              pack_f32x2(__uint_as_float(v[c * 32 + j]), __uint_as_float(v[c * 32 + j + 1])), sc2, m2));
          const float p0 = fast_ex2(e.x), p1 = fast_ex2(e.y);
          if (j & 2) sum1 = add_f32x2(sum1, pack_f32x2(p0, p1));
          else sum0 = add_f32x2(sum0, pack_f32x2(p0, p1));
          pk[j >> 1] = pack_bf16x2(p0, p1);
        }
        tmem_st_32x32b_x16(t_s + c * 16, pk);
      }
      const float2 sums = unpack_f32x2(add_f32x2(sum0, sum1));
      l += sums.x + sums.y;
      tc_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[t]);
    }
    if (nt > 0 && alive && mbar_wait(&o_full[t], 0, alive, 601)) {
      tc_fence_after_sync();
      float inv = SIG ? p.o_scale : (l > 0.f ? p.o_scale / l : 0.f);
      const bool valid = row < Lq;
      const __nv_bfloat16* gate = p.gate ? p.gate + (q_start + row) * p.gate_ld + (p.gate_mode == GATE_HEAD ? h : h * p.vdim) : nullptr;
      if (valid && gate && p.gate_mode == GATE_HEAD) inv *= sigmoid(__bfloat162float(*gate));
      const bool per_element = gate && p.gate_mode == GATE_ELEMENT;
      __nv_bfloat16* dst = p.o + (q_start + row) * p.o_stride + h * p.vdim;
#pragma unroll 1
      for (int c = 0; c < p.v_cols / 16; ++c) {
        uint32_t v[16];
        tmem_ld_32x32b_x16(t_o + c * 16, v);
        tc_wait_ld();
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          if (valid && c * 16 + j * 8 < p.vdim) {
            if (per_element) {
              const uint4 g4 = *reinterpret_cast<const uint4*>(gate + c * 16 + j * 8);
              const uint32_t g[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
              for (int x = 0; x < 4; ++x) {
                const float2 f = unpack_bf16x2(g[x]);
                v[8 * j + 2 * x] = __float_as_uint(__fdividef(__uint_as_float(v[8 * j + 2 * x]), 1.f + __expf(-f.x)));
                v[8 * j + 2 * x + 1] = __float_as_uint(__fdividef(__uint_as_float(v[8 * j + 2 * x + 1]), 1.f + __expf(-f.y)));
              }
            }
            uint4 o4;
            o4.x = pack_bf16x2(__uint_as_float(v[8 * j]) * inv, __uint_as_float(v[8 * j + 1]) * inv);
            o4.y = pack_bf16x2(__uint_as_float(v[8 * j + 2]) * inv, __uint_as_float(v[8 * j + 3]) * inv);
            o4.z = pack_bf16x2(__uint_as_float(v[8 * j + 4]) * inv, __uint_as_float(v[8 * j + 5]) * inv);
            o4.w = pack_bf16x2(__uint_as_float(v[8 * j + 6]) * inv, __uint_as_float(v[8 * j + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 16 + j * 8) = o4;
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

struct LatentPrefillPlan {
  int nb_n, nb_r, nb_v, k_stages, v_stages;
  size_t smem;
};

static bool plan_prefill(int dim, int rot, int vdim, LatentPrefillPlan& pl) {
  if (dim <= 0 || rot < 0 || vdim <= 0 || dim % 8 || rot % 8 || vdim % 8 || vdim > 128) return false;
  pl.nb_n = (dim + 63) / 64;
  pl.nb_r = (rot + 63) / 64;
  pl.nb_v = (vdim + 63) / 64;
  const size_t limit = 227 * 1024, fixed = 256 + 1024;
  const int nb_k = pl.nb_n + pl.nb_r;
  const int order[3][2] = {{2, 2}, {2, 1}, {1, 1}};
  for (auto& o : order) {
    pl.smem = static_cast<size_t>(2 * nb_k + o[0] * nb_k + o[1] * pl.nb_v) * LP_BLOCK + fixed;
    if (pl.smem <= limit) {
      pl.k_stages = o[0];
      pl.v_stages = o[1];
      return true;
    }
  }
  return false;
}

// The gate's rows are read as 16-byte vectors when there is one per element.
static bool gate_ok(const void* gate, long long ld, int mode, int vdim) {
  if (!gate) return true;
  if (mode == GATE_HEAD) return true;
  return mode == GATE_ELEMENT && ld % 8 == 0 && vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15u) == 0;
}

// Tensor maps are the caller's; `p` still lacks what follows from the sizes.
template <bool SIG>
static int launch_prefill(const CUtensorMap& tQn, const CUtensorMap& tQr, const CUtensorMap& tKn, const CUtensorMap& tKr,
                          const CUtensorMap& tV, const LatentPrefillPlan& pl, LatentPrefillParams p, int dim, int rot,
                          int vdim, int sequences, int max_q, void* stream) {
  p.nb_n = pl.nb_n; p.nb_r = pl.nb_r; p.nb_v = pl.nb_v;
  p.ks_n = (dim + 15) / 16; p.ks_r = (rot + 15) / 16; p.vdim = vdim; p.v_cols = (vdim + 15) / 16 * 16;
  p.k_stages = pl.k_stages; p.v_stages = pl.v_stages;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((unsigned)(p.H * sequences), (unsigned)((max_q + 255) / 256));
  latent_prefill_kernel<SIG><<<grid, LP_THREADS, pl.smem, reinterpret_cast<cudaStream_t>(stream)>>>(tQn, tQr, tKn, tKr, tV, p);
  return (int)cudaGetLastError();
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_latent_prefill)
using namespace ts;

// 1 when the head sizes fit this kernel (multiples of eight, values up to 128 wide, tiles within shared memory).
extern "C" int ts_latent_prefill_supported(int dim, int rot, int vdim) {
  LatentPrefillPlan pl;
  return plan_prefill(dim, rot, vdim, pl) ? 1 : 0;
}

// q: projection rows [q_rows][q_ld], head h at column h * (dim + rot).  kv: expanded rows [k_rows][kv_ld], unrotated key
// of head h at column h * dim, value at column v_col0 + h * vdim.  k_rot: [k_rows][kr_ld] shared rotated key part.
// cu_q / cu_k: [sequences + 1].  out: [q_rows][o_stride], times sigmoid(gate) when there is a gate [q_rows][gate_ld].
extern "C" int ts_latent_prefill(const void* q, long long q_ld, long long q_rows, const void* kv, long long kv_ld,
                                 int v_col0, const void* k_rot, long long kr_ld, long long k_rows, const int* cu_q,
                                 const int* cu_k, int sequences, int max_q, int H, int dim, int rot, int vdim, int window,
                                 float scale, const void* gate, long long gate_ld, int gate_mode, void* out,
                                 long long o_stride, void* stream) {
  if (sequences <= 0 || max_q <= 0) return 0;
  LatentPrefillPlan pl;
  if (H <= 0 || window <= 0 || !(scale > 0.f) || !plan_prefill(dim, rot, vdim, pl)) return -10;
  if (!gate_ok(gate, gate_ld, gate_mode, vdim)) return -12;
  if (q_ld % 8 || kv_ld % 8 || kr_ld % 8 || o_stride % 8 || (reinterpret_cast<uintptr_t>(out) & 15u)) return -11;
  const __nv_bfloat16* qp = reinterpret_cast<const __nv_bfloat16*>(q);
  const __nv_bfloat16* kvp = reinterpret_cast<const __nv_bfloat16*>(kv);
  CUtensorMap tQn, tQr, tKn, tKr, tV;
  const CUtensorMapDataType dt = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&tQn, qp, dt, 2, dim, H, q_rows, dim + rot, q_ld, 64, 1, 128);
  if (rc) return rc * 100 - 1;
  rc = make_tmap_3d(&tKn, kvp, dt, 2, dim, H, k_rows, dim, kv_ld, 64, 1, 128);
  if (rc) return rc * 100 - 2;
  rc = make_tmap_3d(&tV, kvp + v_col0, dt, 2, vdim, H, k_rows, vdim, kv_ld, 64, 1, 128);
  if (rc) return rc * 100 - 3;
  tQr = tQn;
  tKr = tKn;
  if (rot > 0) {
    rc = make_tmap_3d(&tQr, qp + dim, dt, 2, rot, H, q_rows, dim + rot, q_ld, 64, 1, 128);
    if (rc) return rc * 100 - 4;
    rc = make_tmap_2d(&tKr, k_rot, dt, 2, k_rows, rot, kr_ld, 128, 64);
    if (rc) return rc * 100 - 5;
  }
  LatentPrefillParams p = {};
  p.cu_q = cu_q; p.cu_k = cu_k; p.H = H; p.window = window; p.kv_group = 1; p.o_scale = 1.f;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.gate_ld = gate_ld; p.gate_mode = gate_mode;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.o = reinterpret_cast<__nv_bfloat16*>(out); p.o_stride = o_stride;
  return launch_prefill<false>(tQn, tQr, tKn, tKr, tV, pl, p, dim, rot, vdim, sequences, max_q, stream);
}

// q: rows [q_rows][q_ld], head h at column h * dim.  k / v: rows [k_rows][kv_ld], key/value head g at columns g * dim and
// g * vdim.  cu_q / cu_k: [sequences + 1].  window, keep, chunked: which keys a query sees (top of the file).
// sigmoid: weights sigmoid(score + add[h] - slopes[h] * distance), not normalized (add and slopes: nullptr for zeros; without
// sigmoid there are none); no (q . k) * scale may exceed `limit` (infinity: unknown).  out: [q_rows][o_stride] = o_scale * attention (* sigmoid(gate)).
extern "C" int ts_window_prefill(const void* q, long long q_ld, long long q_rows, const void* k, const void* v,
                                 long long kv_ld, long long k_rows, const int* cu_q, const int* cu_k, int sequences,
                                 int max_q, int H, int G, int dim, int vdim, int window, int keep, int chunked, float scale,
                                 float o_scale, const float* slopes, const float* add, int sigmoid, float limit, const void* gate,
                                 long long gate_ld, int gate_mode, void* out, long long o_stride, void* stream) {
  if (sequences <= 0 || max_q <= 0) return 0;
  LatentPrefillPlan pl;
  if (H <= 0 || G <= 0 || H % G || window <= 0 || keep < 0 || !(scale > 0.f) || !plan_prefill(dim, 0, vdim, pl)) return -10;
  if (!sigmoid && (slopes || add)) return -13;
  if (!gate_ok(gate, gate_ld, gate_mode, vdim)) return -12;
  if (q_ld % 8 || kv_ld % 8 || o_stride % 8 || (reinterpret_cast<uintptr_t>(out) & 15u)) return -11;
  CUtensorMap tQ, tK, tV;
  const CUtensorMapDataType dt = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&tQ, q, dt, 2, dim, H, q_rows, dim, q_ld, 64, 1, 128);
  if (rc) return rc * 100 - 1;
  rc = make_tmap_3d(&tK, k, dt, 2, dim, G, k_rows, dim, kv_ld, 64, 1, 128);
  if (rc) return rc * 100 - 2;
  rc = make_tmap_3d(&tV, v, dt, 2, vdim, G, k_rows, vdim, kv_ld, 64, 1, 128);
  if (rc) return rc * 100 - 3;
  LatentPrefillParams p = {};
  p.cu_q = cu_q; p.cu_k = cu_k; p.H = H; p.window = window; p.kv_group = H / G; p.o_scale = o_scale;
  p.keep = keep; p.chunked = chunked;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.gate_ld = gate_ld; p.gate_mode = gate_mode;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.o = reinterpret_cast<__nv_bfloat16*>(out); p.o_stride = o_stride;
  p.slopes = slopes; p.add = add; p.limit = limit;
  return sigmoid ? launch_prefill<true>(tQ, tQ, tK, tK, tV, pl, p, dim, 0, vdim, sequences, max_q, stream)
                 : launch_prefill<false>(tQ, tQ, tK, tK, tV, pl, p, dim, 0, vdim, sequences, max_q, stream);
}
