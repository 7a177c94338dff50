// Retention over portions of prompts, bf16 models, in chunks of 128 tokens on the tcgen05 tensor cores:
//   S <- g S + k v^T,  o = S^T q   (g one constant per head, q and k rotated by their position, S fp32),  out = o / rms(o) * silu(gate)
//
// A fixed decay makes the recurrence linear in its inputs with constants known beforehand, so all chunks work side by side:
//   ts_retention_chunks
//     retention_update_kernel  every chunk's own contribution  U_c = sum_j g^(n-1-j) k_j v_j^T            (chunk, head)
//     retention_carry_kernel   S_(c+1) = g^n S_c + U_c along a portion; U_c is replaced by S_c             (element, portion)
//     retention_out_kernel     O = diag(g^(i+1)) Q S_c + (Q K^T o G) V,  G_ij = g^(i-j) for j <= i; then norm and gate
//
// fp32 accuracy from bf16 products: a factor that is not bf16 to begin with (rotated q and k, scores with their decay, S) is cut
// into three bf16 parts that together hold its 24 bits, and the products of parts down to 2^-16 of the leading one are added up
// (six for two such factors, three against v, which is bf16); accumulation in fp32.
//
// Shared-memory tiles are [row][64 columns] with 128-byte swizzle.  The same tile is a K-major operand (rows x reduction over
// columns: Q K^T, Q S) or an MN-major one (reduction over rows: K^T V, P V, Q S's S).
#include "common.cuh"
#include "host_common.h"

namespace ts {

constexpr int RC_TOKENS = 128;             // tokens of a chunk
constexpr int RC_THREADS = 512;            // out kernel; warp w: lanes 32 (w % 4) .. of tensor memory, column share w / 4
constexpr int RC_SHARES = RC_THREADS / 128;
constexpr int RU_THREADS = 256;            // update kernel, two CTAs per SM
constexpr int RC_TILE = RC_TOKENS * 128;   // bytes of a tile of 128 rows
constexpr int RC_MAX_D = 128, RC_MAX_V = 256;

struct ChunkParams {
  const __nv_bfloat16* proj;   // rows [q H x D | k H x D | v H x V | gate H x V]
  long long ld;
  const float* angles;         // [rows][cos (rot / 2) | sin (rot / 2)]
  const float* powers;         // [H][powers_ld] g^0, g^1, ... (RC_TOKENS + 1 of them)
  int powers_ld;
  float k_scale, eps;
  float* state;
  long long state_ld;
  const int* row_prev;
  const int* row_next;
  const int* cu;               // [portions + 1]
  float* chunks;               // [chunks][H][D][V] U_c, later S_c
  __nv_bfloat16* out;          // [rows][out_ld]
  long long out_ld;
  int H, D, V, rot;
};

// chunk 0 of portion z; the portions' ranges do not overlap
__device__ __forceinline__ long long first_chunk(const int* cu, int z) { return cu[z] / RC_TOKENS + z; }

// the i-th piece of eight columns of a tile, 2^per_shift pieces per token
struct Piece {
  int t, c0;
  __device__ Piece(int i, int per_shift) : t(i >> per_shift), c0((i & ((1 << per_shift) - 1)) * 8) {}
};

// x = sum of three bf16 numbers, exactly: the upper two keep eight leading bits each (cut off, so that no conversion is needed),
// the third holds the other eight.  The parts of two neighbours, packed.
__device__ __forceinline__ uint32_t upper_halves(float x, float y) { return __byte_perm(__float_as_uint(x), __float_as_uint(y), 0x7632); }
__device__ __forceinline__ float upper(float x) { return __uint_as_float(__float_as_uint(x) & 0xffff0000u); }
__device__ __forceinline__ void split3_pair(float x, float y, uint32_t& a, uint32_t& b, uint32_t& c) {
  a = upper_halves(x, y);
  x -= upper(x);
  y -= upper(y);
  b = upper_halves(x, y);
  c = pack_bf16x2(x - upper(x), y - upper(y));
}

__device__ __forceinline__ void unpack8(const uint4& r, float (&v)[8]) {
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = unpack_bf16x2(w[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}

// Coordinates c0 .. c0 + 7 of the projected heads x[0 .. HEADS) of one token, rotated by halves that are whole vectors (rot a
// multiple of 16).  `fetch` only loads, so that several are in flight; `turned` computes.
template <int HEADS> struct Turn8 {
  uint4 x[HEADS], partner[HEADS];
  float4 cs[4];                // cosines, sines

  __device__ __forceinline__ void fetch(const __nv_bfloat16* head, int step, int c0, int rot, const float* angles) {
    const int half = rot / 2;
    const bool first = c0 < half, on = c0 < rot;
#pragma unroll
    for (int h = 0; h < HEADS; ++h) {
      x[h] = *reinterpret_cast<const uint4*>(head + h * step + c0);
      if (on) partner[h] = *reinterpret_cast<const uint4*>(head + h * step + (first ? c0 + half : c0 - half));
    }
    if (on) {
      const float4* c4 = reinterpret_cast<const float4*>(angles + (first ? c0 : c0 - half));
      const float4* s4 = reinterpret_cast<const float4*>(angles + half + (first ? c0 : c0 - half));
      cs[0] = c4[0]; cs[1] = c4[1]; cs[2] = s4[0]; cs[3] = s4[1];
    }
  }
  __device__ __forceinline__ void turned(int h, int c0, int rot, float (&v)[8]) const {
    unpack8(x[h], v);
    if (c0 >= rot) return;
    const float c[8] = {cs[0].x, cs[0].y, cs[0].z, cs[0].w, cs[1].x, cs[1].y, cs[1].z, cs[1].w};
    const float s[8] = {cs[2].x, cs[2].y, cs[2].z, cs[2].w, cs[3].x, cs[3].y, cs[3].z, cs[3].w};
    float o[8];
    unpack8(partner[h], o);
    const float sign = c0 < rot / 2 ? -1.f : 1.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = v[j] * c[j] + sign * o[j] * s[j];
  }
};
// the same for any even rot
__device__ __noinline__ void turned8(const __nv_bfloat16* head, int c0, int rot, const float* angles, float* v) {
  const int half = rot / 2;
  for (int j = 0; j < 8; ++j) {
    const int c = c0 + j;
    float x = __bfloat162float(head[c]);
    if (c < half) x = x * angles[c] - __bfloat162float(head[c + half]) * angles[half + c];
    else if (c < rot) x = x * angles[c - half] + __bfloat162float(head[c - half]) * angles[c];
    v[j] = x;
  }
}

// eight columns of a row as three parts, each in its own set of tiles (`stride` bytes apart)
__device__ __forceinline__ void store_parts(uint8_t* tiles, int stride, int row, int c0, const float (&v)[8]) {
  uint32_t p[3][4];
#pragma unroll
  for (int j = 0; j < 4; ++j) split3_pair(v[2 * j], v[2 * j + 1], p[0][j], p[1][j], p[2][j]);
  uint8_t* dst = tiles + (c0 >> 6) * RC_TILE + sw128_offset(row, (c0 & 63) >> 3);
#pragma unroll
  for (int i = 0; i < 3; ++i) *reinterpret_cast<uint4*>(dst + i * stride) = make_uint4(p[i][0], p[i][1], p[i][2], p[i][3]);
}

// Descriptors advance by bytes / 16 in their low bits.  One reduction step is 16 wide: 32 bytes along a K-major row (a tile holds
// four), 16 rows of an MN-major tile.
__device__ __forceinline__ uint64_t k_major(const uint8_t* tile) { return make_smem_desc_sw128(smem_u32(tile), 16, 1024); }
__device__ __forceinline__ uint64_t mn_major(const uint8_t* tile) { return make_smem_desc_sw128(smem_u32(tile), RC_TILE, 1024); }
__device__ __forceinline__ int k_major_step(int k) { return (k >> 2) * (RC_TILE / 16) + (k & 3) * 2; }
constexpr int MN_STEP = 2048 / 16;

// a chunk of a portion
struct Chunk {
  int row, n;                  // first row, tokens
  long long at;                // index of its matrix
  __device__ Chunk(const ChunkParams& p, int z, int c, int h) {
    const int row0 = p.cu[z];
    row = row0 + c * RC_TOKENS;
    n = min(RC_TOKENS, p.cu[z + 1] - row);
    at = ((first_chunk(p.cu, z) + c) * p.H + h) * p.D * p.V;
  }
};

__device__ __forceinline__ void store_zeros(uint8_t* tiles, int stride, int row, int c0) {
  uint8_t* dst = tiles + (c0 >> 6) * RC_TILE + sw128_offset(row, (c0 & 63) >> 3);
#pragma unroll
  for (int i = 0; i < 3; ++i) *reinterpret_cast<uint4*>(dst + i * stride) = make_uint4(0u, 0u, 0u, 0u);
}

// products of the parts of two factors, small ones first
__device__ constexpr int PART_A[6] = {2, 1, 0, 1, 0, 0}, PART_B[6] = {0, 1, 2, 0, 1, 0};

struct ChunkSizes {
  int nbd, nbv;                // 64-column blocks of a key head and of a value head
  int part;                    // bytes of one part of q or k
  __host__ __device__ ChunkSizes(int D, int V) : nbd((D + 63) / 64), nbv((V + 63) / 64), part(nbd * RC_TILE) {}
  // update kernel: parts of 64 columns of k | v
  __host__ __device__ int update_bytes() const { return (3 + nbv) * RC_TILE; }
  // out kernel: parts of q, later two blocks of S, later the gate and the result | parts of k, later v, later two blocks of S
  __host__ __device__ int first_bytes() const { return 3 * part > nbv * RC_TILE ? 3 * part : nbv * RC_TILE; }
  __host__ __device__ int out_bytes() const { return 2 * first_bytes(); }
};
constexpr int RC_EXTRA = 1024 + (RC_TOKENS + 8) * 4 + RC_SHARES * RC_TOKENS * 4 + 64;     // alignment, powers, partial sums, barriers

// grid (H * blocks of 64 key coordinates, chunks of the longest portion, portions)
__global__ void __launch_bounds__(RU_THREADS, 2) retention_update_kernel(const __grid_constant__ CUtensorMap tmV, ChunkParams p) {
  extern __shared__ __align__(1024) uint8_t smem[];     // no room for more than the tiles where two CTAs share an SM
  const ChunkSizes z(p.D, p.V);
  uint8_t* v_tiles = smem + 3 * RC_TILE;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + z.update_bytes());   // v, mma
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  const int h = blockIdx.x / z.nbd, d0 = (blockIdx.x - h * z.nbd) * 64, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (p.cu[blockIdx.z] + static_cast<int>(blockIdx.y) * RC_TOKENS >= p.cu[blockIdx.z + 1]) return;
  if (smem_u32(smem) & 1023u) {
    ts_report_error(ERR_BAD_ARGUMENT, 702, smem_u32(smem));
    return;
  }
  const Chunk ck(p, blockIdx.z, blockIdx.y, h);
  const float* pw = p.powers + h * p.powers_ld;
  if (threadIdx.x == 0) {
    mbar_init(&bars[0], 1);
    mbar_init(&bars[1], 1);
    fence_barrier_init();
    mbar_expect_tx(&bars[0], z.nbv * RC_TILE);
    for (int b = 0; b < z.nbv; ++b) tma_load_3d(v_tiles + b * RC_TILE, &tmV, &bars[0], b * 64, h, ck.row);
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
    tc_fence_before_sync();
  }
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  constexpr int AHEAD = 2, PIECES = RC_TOKENS * 8;
  const __nv_bfloat16* k_col = p.proj + (p.H + h) * p.D + d0;
  auto store_k = [&](const Piece& x, float (&v)[8]) {
    const float f = p.k_scale * pw[ck.n - 1 - x.t];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= f;
    store_parts(smem, RC_TILE, x.t, x.c0, v);
  };
  auto on = [&](const Piece& x) {
    if (x.t < ck.n && d0 + x.c0 < p.D) return true;
    if (x.t < RC_TOKENS) store_zeros(smem, RC_TILE, x.t, x.c0);
    return false;
  };
  if (p.rot % 16 == 0) {
    for (int i0 = threadIdx.x; i0 < PIECES; i0 += AHEAD * RU_THREADS) {
      Turn8<1> raw[AHEAD];
      bool has[AHEAD];
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const Piece x(i0 + u * RU_THREADS, 3);
        has[u] = on(x);
        const long long row = ck.row + x.t;
        if (has[u]) raw[u].fetch(k_col - d0 + row * p.ld, 0, d0 + x.c0, p.rot, p.angles + row * p.rot);
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const Piece x(i0 + u * RU_THREADS, 3);
        float v[8];
        if (!has[u]) continue;
        raw[u].turned(0, d0 + x.c0, p.rot, v);
        store_k(x, v);
      }
    }
  } else {
    for (int i = threadIdx.x; i < PIECES; i += RU_THREADS) {
      const Piece x(i, 3);
      if (!on(x)) continue;
      const long long row = ck.row + x.t;
      float v[8];
      turned8(k_col - d0 + row * p.ld, d0 + x.c0, p.rot, p.angles + row * p.rot, v);
      store_k(x, v);
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  bool alive = true;
  const int v_cols = (p.V + 15) / 16 * 16;
  if (warp == 0 && elect_one_sync()) {
    if (mbar_wait(&bars[0], 0, alive, 700)) {
      // the result's first 64 rows are the key coordinates; the others are made of whatever follows a part and are not read
      const uint32_t idesc = make_idesc(128, v_cols, 1, 1, 1, 1);
      const uint64_t a = mn_major(smem), b = mn_major(v_tiles);
      for (int i = 2; i >= 0; --i)
#pragma unroll
        for (int k = 0; k < RC_TOKENS / 16; ++k)
          umma_f16_ss(tmem, a + i * (RC_TILE / 16) + k * MN_STEP, b + k * MN_STEP, idesc, i != 2 || k != 0);
      umma_commit(&bars[1]);
    }
  }
  __syncthreads();                 // reconverged before the warp-wide loads; the elected thread may have given up
  mbar_wait(&bars[1], 0, alive, 701);
  tc_fence_after_sync();
  // rows of the result to shared memory (the operands are no longer needed; a row is 16 bytes longer: no bank conflicts), then
  // out as one contiguous piece.  Rows 0 .. 63 are lanes of two warps out of four
  const int pitch = p.V + 4, rows = min(64, p.D - d0);
  float* staged = reinterpret_cast<float*>(smem);
  if ((warp & 3) < 2) {
    const int d = (warp & 3) * 32 + lane;
    for (int c = (warp >> 2) * 32; c < v_cols; c += 64) {
      uint32_t r[32];
      tmem_ld_32x32b_x32(tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16) + c, r);
      tc_wait_ld();
      if (d < rows)
#pragma unroll
        for (int j = 0; j < 32; j += 4)
          if (c + j < p.V) *reinterpret_cast<uint4*>(staged + d * pitch + c + j) = make_uint4(r[j], r[j + 1], r[j + 2], r[j + 3]);
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, 256);
  }
  const int vecs = p.V / 4;
  float4* dst = reinterpret_cast<float4*>(p.chunks + ck.at + static_cast<long long>(d0) * p.V);
#pragma unroll 4
  for (int i = threadIdx.x; i < rows * vecs; i += RU_THREADS) {
    const int d = i / vecs;
    dst[i] = *reinterpret_cast<const float4*>(staged + d * pitch + (i - d * vecs) * 4);
  }
}

// grid (ceil(D V / 1024), H, portions); a thread carries four elements along its portion
__global__ void __launch_bounds__(256) retention_carry_kernel(ChunkParams p) {
  constexpr int AHEAD = 8;
  const int h = blockIdx.y, z = blockIdx.z, row0 = p.cu[z], n = p.cu[z + 1] - row0, DV = p.D * p.V;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (n <= 0 || e >= DV) return;
  const int count = (n + RC_TOKENS - 1) / RC_TOKENS;
  const float* pw = p.powers + h * p.powers_ld;
  const float g = pw[RC_TOKENS], g_last = pw[n - (count - 1) * RC_TOKENS];
  const int prev = p.row_prev[row0], next = p.row_next[row0 + n - 1];
  const long long head = static_cast<long long>(h) * DV + e, step = static_cast<long long>(p.H) * DV;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (prev >= 0) s = *reinterpret_cast<const float4*>(p.state + prev * p.state_ld + head);
  float* x = p.chunks + first_chunk(p.cu, z) * step + head;
  for (int c0 = 0; c0 < count; c0 += AHEAD) {
    float4 u[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c0 + i < count) u[i] = *reinterpret_cast<const float4*>(x + (c0 + i) * step);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c0 + i < count) {
        *reinterpret_cast<float4*>(x + (c0 + i) * step) = s;
        const float f = c0 + i == count - 1 ? g_last : g;
        s = make_float4(f * s.x + u[i].x, f * s.y + u[i].y, f * s.z + u[i].z, f * s.w + u[i].w);
      }
  }
  if (next >= 0) *reinterpret_cast<float4*>(p.state + next * p.state_ld + head) = s;
}

// grid (H, chunks of the longest portion, portions)
__global__ void __launch_bounds__(RC_THREADS + 32, 1) retention_out_kernel(const __grid_constant__ CUtensorMap tmV, ChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const ChunkSizes z(p.D, p.V);
  uint8_t* q_tiles = smem;
  uint8_t* k_tiles = smem + z.first_bytes();
  float* pw = reinterpret_cast<float*>(smem + z.out_bytes());              // [RC_TOKENS + 8]
  float* sums = pw + RC_TOKENS + 8;                                        // [RC_SHARES][RC_TOKENS]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sums + RC_SHARES * RC_TOKENS);
  uint64_t *b_qk = bars, *b_v = bars + 1, *b_pv = bars + 2, *b_s = bars + 3, *b_o = bars + 4, *b_g = bars + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 6);
  const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, share = warp >> 2;
  if (p.cu[blockIdx.z] + static_cast<int>(blockIdx.y) * RC_TOKENS >= p.cu[blockIdx.z + 1]) return;
  const Chunk ck(p, blockIdx.z, blockIdx.y, h);
  const int ks = (p.D + 15) / 16, v_cols = (p.V + 15) / 16 * 16;
  const uint32_t tmem_cols = z.nbv == 1 ? 256 : 512;
  const bool odd_block = z.nbv > 1, second_pair = z.nbv > 2;
  const int s_part = z.nbd * 64 * 128;   // bytes of one part of a block of S
  bool alive = true;

  if (warp == RC_THREADS / 32) {         // this warp only issues: copies by the tensor units, products
    if (lane == 0) {
      for (int i = 0; i < 6; ++i) mbar_init(&bars[i], 1);
      fence_barrier_init();
    }
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
    tc_fence_before_sync();
    __syncthreads();                     // (1) q and k are there
    tc_fence_after_sync();
    const uint32_t tmem = *tmem_slot, t_s = tmem + z.nbv * 64;
    const bool one = elect_one_sync();
    if (one) {
      const uint32_t idesc = make_idesc(128, 128, 1, 1, 0, 0);
      const uint64_t q = k_major(q_tiles), k = k_major(k_tiles);
#pragma unroll
      for (int i = 0; i < 6; ++i)
        for (int x = 0; x < ks; ++x)
          umma_f16_ss(t_s, q + PART_A[i] * (z.part / 16) + k_major_step(x), k + PART_B[i] * (z.part / 16) + k_major_step(x), idesc,
                      i != 0 || x != 0);
      umma_commit(b_qk);
      if (mbar_wait(b_qk, 0, alive, 710)) {          // v takes the place of k
        mbar_expect_tx(b_v, z.nbv * RC_TILE);
        for (int b = 0; b < z.nbv; ++b) tma_load_3d(k_tiles + b * RC_TILE, &tmV, b_v, b * 64, h, ck.row);
      }
    }
    __syncwarp();
    __syncthreads();                     // (2) the scores have been read
    __syncthreads();                     // (3) their parts are there
    if (one && mbar_wait(b_v, 0, alive, 711)) {
      tc_fence_after_sync();
      const uint32_t idesc = make_idesc(128, v_cols, 1, 1, 0, 1);
      const uint64_t v = mn_major(k_tiles);
      for (int i = 2; i >= 0; --i)
#pragma unroll
        for (int k = 0; k < RC_TOKENS / 16; ++k) umma_f16_ts(tmem, t_s + i * 64 + k * 8, v + k * MN_STEP, idesc, i != 2 || k != 0);
      umma_commit(b_pv);
    }
    __syncwarp();
    auto issue_s = [&](int b) {          // O += q S of a block, q from tensor memory
      const uint32_t idesc = make_idesc(128, 64, 1, 1, 0, 1);
      const uint64_t sb = mn_major((b < 2 ? q_tiles : k_tiles) + (b & 1) * 3 * s_part);
#pragma unroll
      for (int i = 0; i < 6; ++i)
        for (int k = 0; k < ks; ++k)
          umma_f16_ts(tmem + b * 64, t_s + PART_A[i] * 64 + k * 8, sb + PART_B[i] * (s_part / 16) + k * MN_STEP, idesc, 1u);
    };
    __syncthreads();                     // (4) q has been read
    __syncthreads();                     // (5) q with its decay and two blocks of S are there
    if (one) {
      tc_fence_after_sync();
      issue_s(0);
      if (odd_block) issue_s(1);
      umma_commit(b_s);
    }
    __syncwarp();
    if (second_pair) {
      __syncthreads();                   // (6) the other two
      if (one) {
        issue_s(2);
        if (z.nbv > 3) issue_s(3);
        umma_commit(b_o);
      }
      __syncwarp();
    }
    if (one && mbar_wait(b_s, 0, alive, 712)) {      // the gate takes the place of the first two
      mbar_expect_tx(b_g, z.nbv * RC_TILE);
      for (int b = 0; b < z.nbv; ++b) tma_load_3d(q_tiles + b * RC_TILE, &tmV, b_g, b * 64, p.H + h, ck.row);
    }
    __syncwarp();
    __syncthreads();                     // (7) sums of squares
    __syncthreads();                     // (8) the result is in shared memory
    tc_fence_after_sync();
    tmem_dealloc(tmem, tmem_cols);
    return;
  }

  for (int i = threadIdx.x; i <= RC_TOKENS; i += RC_THREADS) pw[i] = p.powers[h * p.powers_ld + i];
  // S of the chunk, 64 columns at a time: element (d, c) of block b in float4s, thread after thread
  const float* s_src = p.chunks + ck.at;
  constexpr int SV = RC_MAX_D * 16 / RC_THREADS;
  float4 s_reg[SV];
  auto fetch_s = [&](int b) {
#pragma unroll
    for (int u = 0; u < SV; ++u) {
      const int i = threadIdx.x + u * RC_THREADS, d = i >> 4, c = b * 64 + (i & 15) * 4;
      s_reg[u] = d < p.D && c < p.V ? *reinterpret_cast<const float4*>(s_src + static_cast<long long>(d) * p.V + c)
                                    : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  constexpr int AHEAD = 2;
  const int per = z.nbd == 2 ? 4 : 3, pieces = RC_TOKENS << per, to_k = p.H * p.D;
  const __nv_bfloat16* q_col = p.proj + h * p.D;
  auto store_k = [&](const Piece& x, float (&v)[8]) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= p.k_scale;
    store_parts(k_tiles, z.part, x.t, x.c0, v);
  };
  auto on = [&](const Piece& x) {
    if (x.t < ck.n && x.c0 < p.D) return true;
    if (x.t < RC_TOKENS) {
      store_zeros(q_tiles, z.part, x.t, x.c0);
      store_zeros(k_tiles, z.part, x.t, x.c0);
    }
    return false;
  };
  if (p.rot % 16 == 0) {
    for (int i0 = threadIdx.x; i0 < pieces; i0 += AHEAD * RC_THREADS) {
      Turn8<2> raw[AHEAD];
      bool has[AHEAD];
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const Piece x(i0 + u * RC_THREADS, per);
        has[u] = on(x);
        const long long row = ck.row + x.t;
        if (has[u]) raw[u].fetch(q_col + row * p.ld, to_k, x.c0, p.rot, p.angles + row * p.rot);
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const Piece x(i0 + u * RC_THREADS, per);
        float v[8];
        if (!has[u]) continue;
        raw[u].turned(0, x.c0, p.rot, v);
        store_parts(q_tiles, z.part, x.t, x.c0, v);
        raw[u].turned(1, x.c0, p.rot, v);
        store_k(x, v);
      }
    }
  } else {
    for (int i = threadIdx.x; i < pieces; i += RC_THREADS) {
      const Piece x(i, per);
      if (!on(x)) continue;
      const long long row = ck.row + x.t;
      float v[8];
      turned8(q_col + row * p.ld, x.c0, p.rot, p.angles + row * p.rot, v);
      store_parts(q_tiles, z.part, x.t, x.c0, v);
      turned8(q_col + row * p.ld + to_k, x.c0, p.rot, p.angles + row * p.rot, v);
      store_k(x, v);
    }
  }
  fence_proxy_async_smem();
  __syncthreads();                       // (1)
  tc_fence_after_sync();
  // tensor memory: O | scores, later their parts, later the parts of q times its decay
  const uint32_t tmem = *tmem_slot, t_s = tmem + z.nbv * 64;
  fetch_s(0);
  const int i_row = (warp & 3) * 32 + lane;
  const uint32_t t_lane = static_cast<uint32_t>((warp & 3) * 32) << 16;
  mbar_wait(b_qk, 0, alive, 720);
  // scores times their decay, in parts, back to tensor memory as the A operand of P V
  tc_fence_after_sync();
  {
    constexpr int COLS = RC_TOKENS / RC_SHARES;
    static_assert(COLS == 32, "a thread holds 32 scores");
    uint32_t s[COLS];
    tmem_ld_32x32b_x32(t_s + t_lane + share * COLS, s);
    tc_wait_ld();
    tc_fence_before_sync();
    __syncthreads();                     // (2) everybody has read the scores: the parts overwrite them
    tc_fence_after_sync();
#pragma unroll
    for (int c = 0; c < COLS; c += 16) {
      uint32_t a[8], b[8], d[8];
#pragma unroll
      for (int j = 0; j < 16; j += 2) {
        const int gap = i_row - share * COLS - c - j;
        const float x = gap >= 0 ? __uint_as_float(s[c + j]) * pw[max(gap, 0)] : 0.f;
        const float y = gap >= 1 ? __uint_as_float(s[c + j + 1]) * pw[max(gap - 1, 0)] : 0.f;
        split3_pair(x, y, a[j >> 1], b[j >> 1], d[j >> 1]);
      }
      const uint32_t at = t_s + t_lane + (share * COLS + c) / 2;
      tmem_st_32x32b_x8(at, a);
      tmem_st_32x32b_x8(at + 64, b);
      tmem_st_32x32b_x8(at + 128, d);
    }
    tc_wait_st();
    tc_fence_before_sync();
  }
  __syncthreads();                       // (3)
  // q of this thread's row and 32 columns times the decay since the chunk's start, in parts, for Q S
  const bool has_q = share < 2 * z.nbd;
  uint32_t qp[3][16];
  if (has_q) {
    const float f = pw[i_row + 1];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const uint8_t* at = q_tiles + (share >> 1) * RC_TILE + sw128_offset(i_row, (share & 1) * 4 + c);
      float v[3][8];
#pragma unroll
      for (int i = 0; i < 3; ++i) unpack8(*reinterpret_cast<const uint4*>(at + i * z.part), v[i]);
#pragma unroll
      for (int j = 0; j < 8; j += 2)
        split3_pair((v[0][j] + (v[1][j] + v[2][j])) * f, (v[0][j + 1] + (v[1][j + 1] + v[2][j + 1])) * f, qp[0][c * 4 + j / 2],
                    qp[1][c * 4 + j / 2], qp[2][c * 4 + j / 2]);
    }
  }
  __syncthreads();                       // (4) everybody has read q
  // blocks of S in parts: the first two where q was, the others where v was
  auto stage_s = [&](int b) {
    uint8_t* buf = (b < 2 ? q_tiles : k_tiles) + (b & 1) * 3 * s_part;
#pragma unroll
    for (int u = 0; u < SV; ++u) {
      const int i = threadIdx.x + u * RC_THREADS, d = i >> 4, c = (i & 15) * 4;
      if (d < z.nbd * 64) {
        uint32_t x[3], y[3];
        split3_pair(s_reg[u].x, s_reg[u].y, x[0], x[1], x[2]);
        split3_pair(s_reg[u].z, s_reg[u].w, y[0], y[1], y[2]);
        uint8_t* dst = buf + sw128_offset(d, c >> 3) + (c & 4) * 2;
#pragma unroll
        for (int j = 0; j < 3; ++j) *reinterpret_cast<uint2*>(dst + j * s_part) = make_uint2(x[j], y[j]);
      }
    }
    if (b + 1 < z.nbv) fetch_s(b + 1);
  };
  stage_s(0);
  if (odd_block) stage_s(1);
  mbar_wait(b_pv, 0, alive, 721);        // the parts of the scores and v are no longer needed
  tc_fence_after_sync();
  if (has_q) {
#pragma unroll
    for (int i = 0; i < 3; ++i) tmem_st_32x32b_x16(t_s + t_lane + i * 64 + share * 16, qp[i]);
    tc_wait_st();
  }
  tc_fence_before_sync();
  fence_proxy_async_smem();
  __syncthreads();                       // (5)
  if (second_pair) {
    stage_s(2);
    if (z.nbv > 3) stage_s(3);
    fence_proxy_async_smem();
    __syncthreads();                     // (6)
  }
  mbar_wait(second_pair ? b_o : b_s, 0, alive, 722);
  tc_fence_after_sync();
  // norm and gate; the shares of the warps take 32 columns of their row in turn
  float ss = 0.f;
  for (int c = share * 32; c < v_cols; c += RC_SHARES * 32) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem + t_lane + c, r);
    tc_wait_ld();
#pragma unroll
    for (int j = 0; j < 32; ++j)
      if (c + j < p.V) ss += __uint_as_float(r[j]) * __uint_as_float(r[j]);
  }
  sums[share * RC_TOKENS + i_row] = ss;
  mbar_wait(b_g, 0, alive, 723);
  __syncthreads();                       // (7)
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < RC_SHARES; ++i) ss += sums[i * RC_TOKENS + i_row];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.V) + p.eps);
  for (int c = share * 32; c < v_cols; c += RC_SHARES * 32) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem + t_lane + c, r);
    tc_wait_ld();
#pragma unroll
    for (int j = 0; j < 32; j += 8) {
      uint4* at = reinterpret_cast<uint4*>(q_tiles + (c >> 6) * RC_TILE + sw128_offset(i_row, ((c & 63) + j) >> 3));
      float g[8];
      unpack8(*at, g);
      uint32_t o[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float g0 = g[2 * x], g1 = g[2 * x + 1];
        o[x] = pack_bf16x2(__uint_as_float(r[j + 2 * x]) * inv * __fdividef(g0, 1.f + __expf(-g0)),
                           __uint_as_float(r[j + 2 * x + 1]) * inv * __fdividef(g1, 1.f + __expf(-g1)));
      }
      *at = make_uint4(o[0], o[1], o[2], o[3]);
    }
  }
  tc_fence_before_sync();
  __syncthreads();                       // (8)
  const int vecs = p.V / 8;
  __nv_bfloat16* dst = p.out + ck.row * p.out_ld + h * p.V;
  for (int i = threadIdx.x; i < ck.n * vecs; i += RC_THREADS) {
    const int t = i / vecs, c = i - t * vecs;
    *reinterpret_cast<uint4*>(dst + t * p.out_ld + c * 8) = *reinterpret_cast<const uint4*>(q_tiles + (c >> 3) * RC_TILE + sw128_offset(t, c & 7));
  }
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_retention)
using namespace ts;

// 1 when the chunk kernels take these head sizes.
extern "C" int ts_retention_chunks_supported(int D, int V) {
  return D > 0 && V > 0 && D % 8 == 0 && V % 8 == 0 && D <= RC_MAX_D && V <= RC_MAX_V;
}
// Matrices that `rows` rows in `portions` portions need (upper bound).
extern "C" int ts_retention_chunks_count(int rows, int portions) { return rows / RC_TOKENS + portions + 1; }

// proj: rows [q | k | v | gate], 16-byte aligned.  angles: [rows][rot] cosines | sines.  powers: [H][powers_ld], at least 129 each.
// chunks: workspace [ts_retention_chunks_count][H][D][V].  out: [rows][out_ld] = norm * silu(gate); the last state of every portion
// goes to its state row.
extern "C" int ts_retention_chunks(const void* proj, long long ld, long long rows, const float* angles, const float* powers,
                                   int powers_ld, float k_scale, float eps, float* chunks, float* state, long long state_ld,
                                   const int* row_prev, const int* row_next, const int* cu, int portions, int max_rows, void* out,
                                   long long out_ld, int H, int D, int V, int rot, void* stream) {
  if (portions <= 0) return 0;
  if (H <= 0 || !ts_retention_chunks_supported(D, V) || rot < 0 || rot > D || rot % 2 || powers_ld <= RC_TOKENS || max_rows <= 0 ||
      portions > 65535 || max_rows > 65535 * RC_TOKENS || state_ld < static_cast<long long>(H) * D * V)
    return -10;
  if (ld % 8 || out_ld % 8 || state_ld % 4 || ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(out)) & 15u) ||
      (rot % 16 == 0 && (reinterpret_cast<uintptr_t>(angles) & 15u)))
    return -11;
  ChunkParams p;
  p.proj = reinterpret_cast<const __nv_bfloat16*>(proj); p.ld = ld; p.angles = angles; p.powers = powers; p.powers_ld = powers_ld;
  p.k_scale = k_scale; p.eps = eps; p.state = state; p.state_ld = state_ld; p.row_prev = row_prev; p.row_next = row_next; p.cu = cu;
  p.chunks = chunks; p.out = reinterpret_cast<__nv_bfloat16*>(out); p.out_ld = out_ld; p.H = H; p.D = D; p.V = V; p.rot = rot;
  CUtensorMap tV;              // v heads, then gate heads
  int rc = make_tmap_3d(&tV, p.proj + 2 * H * D, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, V, 2 * H, rows, V, ld, 64, 1, RC_TOKENS);
  if (rc) return rc * 100 - 1;
  const ChunkSizes z(D, V);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(retention_update_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(H, (max_rows + RC_TOKENS - 1) / RC_TOKENS, portions);
  retention_update_kernel<<<dim3(H * z.nbd, grid.y, portions), RU_THREADS, z.update_bytes() + 32, st>>>(tV, p);
  retention_carry_kernel<<<dim3((D * V + 1023) / 1024, H, portions), 256, 0, st>>>(p);
  retention_out_kernel<<<grid, RC_THREADS + 32, z.out_bytes() + RC_EXTRA, st>>>(tV, p);
  return (int)cudaGetLastError();
}
