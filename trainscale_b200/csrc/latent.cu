// Latent attention over a paged cache: every token caches ONE row [latent c (rank) | rotated key part (rot)] that all
// heads share, instead of keys and values per head.
//
//   ts_latent_prep    split of the q | down projection: RMS norm of the latent, rotary embedding of the shared key part
//                     and of every head's rotated query part (in place), cache write - one launch
//   ts_latent_gather  cache rows of a list of slots -> contiguous rows (the keys a portion of a prompt needs again)
//   ts_latent_attend  attention in latent space for single query rows against the paged cache.  The query's unrotated
//                     part has been carried into latent space (q_lat = W_uk^T q), so scores are dot products with the
//                     cached row, and the weighted sum of latents is returned (W_uv is applied afterwards):
//                       s_j = (q_lat . c_j + q_rot . r_j) * scale,   o = sum_j softmax(s)_j c_j
//                     for the keys max(0, len - window) <= j < len of the row's sequence.  Reads each cached row once
//                     for all heads; long windows are split over CTAs and merged by log-sum-exp.
//
// Two attention kernels: `latent_attend_mma_kernel` (bf16; 16 heads are the rows of warp MMAs, the CTA's tile of cached
// rows is both K and V) and `latent_attend_simt_kernel` (fp32, or bf16 sizes the tiles do not fit).
#include "common.cuh"
#include "host_common.h"

namespace ts {

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

// One CTA per token.  proj row: [H heads x (dim | rot)] [latent rank | rot].
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(T* __restrict__ proj, long long ld, int H, int dim, int rot, int rank, const float* __restrict__ norm_w,
                   float eps, const float* __restrict__ inv_freq, float magnitude, int pairs, const int* __restrict__ pos,
                   const long long* __restrict__ slots, T* __restrict__ cache, T* __restrict__ flat, int row_width) {
  extern __shared__ float cs[];     // cos | sin of the token's rot / 2 angles
  __shared__ float scratch[32];
  const int t = blockIdx.x, half = rot / 2;
  T* q = proj + static_cast<long long>(t) * ld;
  const T* down = q + H * (dim + rot);
  const float p = static_cast<float>(pos[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(p * inv_freq[i], &s, &c);
    cs[i] = c * magnitude;
    cs[half + i] = s * magnitude;
  }
  float ss = 0.f;
  for (int r = threadIdx.x; r < rank; r += blockDim.x) {
    const float v = to_f32(down[r]);
    ss += v * v;
  }
  ss = block_sum(ss, scratch);      // also orders the angles
  const float inv = 1.f / sqrtf(ss / static_cast<float>(rank) + eps);
  T* crow = cache + slots[t] * row_width;
  T* frow = flat ? flat + static_cast<long long>(t) * row_width : nullptr;
  for (int r = threadIdx.x; r < row_width; r += blockDim.x) {
    float v = 0.f;                  // columns past rank + rot pad the row
    if (r < rank) {
      v = to_f32(down[r]) * inv * norm_w[r];
    } else if (r < rank + rot) {
      // the first of a pair turns against the second, the second with the first
      const int i = r - rank, f = pairs ? i / 2 : (i < half ? i : i - half), step = pairs ? 1 : half;
      const bool lead = pairs ? i % 2 == 0 : i < half;
      const float a = to_f32(down[r]), b = to_f32(down[lead ? r + step : r - step]);
      v = lead ? a * cs[f] - b * cs[half + f] : a * cs[f] + b * cs[half + f];
    }
    crow[r] = from_f32<T>(v);
    if (frow) frow[r] = from_f32<T>(v);
  }
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    T* a = q + h * (dim + rot) + dim + (pairs ? 2 * j : j);
    T* b = a + (pairs ? 1 : half);
    const float u = to_f32(*a), v = to_f32(*b), c = cs[j], s = cs[half + j];
    *a = from_f32<T>(u * c - v * s);
    *b = from_f32<T>(v * c + u * s);
  }
}

// The same for bf16 rows without a rotated part, rank and row_width multiples of eight: one warp per token, 16-byte vectors.
constexpr int LPV_WARPS = 4;
__global__ void __launch_bounds__(LPV_WARPS * 32)
latent_norm_vec_kernel(const __nv_bfloat16* __restrict__ down, long long ld, int rank, const float* __restrict__ norm_w, float eps,
                       const long long* __restrict__ slots, __nv_bfloat16* __restrict__ cache, __nv_bfloat16* __restrict__ flat,
                       int row_width, int rows) {
  constexpr int NV = 4;                            // vectors of a lane: rank up to 1024
  const int t = blockIdx.x * LPV_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= rows) return;
  const uint4* src = reinterpret_cast<const uint4*>(down + t * ld);
  const int vecs = rank / 8;
  uint4 raw[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) raw[i] = i * 32 + lane < vecs ? src[i * 32 + lane] : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const uint32_t r[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(r[j]);
      ss += f.x * f.x + f.y * f.y;
    }
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(rank) + eps);
  uint4* crow = reinterpret_cast<uint4*>(cache + slots[t] * row_width);
  uint4* frow = flat ? reinterpret_cast<uint4*>(flat + static_cast<long long>(t) * row_width) : nullptr;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = i * 32 + lane;
    if (c >= row_width / 8) continue;
    uint32_t o[4] = {0u, 0u, 0u, 0u};              // columns past the latent pad the row
    if (c < vecs) {
      const uint32_t r[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
      const float4 wa = reinterpret_cast<const float4*>(norm_w)[2 * c], wb = reinterpret_cast<const float4*>(norm_w)[2 * c + 1];
      const float w[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = unpack_bf16x2(r[j]);
        o[j] = pack_bf16x2(f.x * inv * w[2 * j], f.y * inv * w[2 * j + 1]);
      }
    }
    const uint4 v = make_uint4(o[0], o[1], o[2], o[3]);
    crow[c] = v;
    if (frow) frow[c] = v;
  }
}

__global__ void latent_gather_kernel(const uint4* __restrict__ cache, const long long* __restrict__ slots,
                                     uint4* __restrict__ out, long long rows, int vec) {
  const long long total = rows * vec;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / vec;
    out[i] = cache[slots[r] * vec + (i - r * vec)];
  }
}

struct LatentAttendParams {
  const void* q_lat;          // [rows][H][rank]
  const void* q;              // projection rows; rotated part of head h at column h * (dim + rot) + dim
  long long q_ld;
  const void* cache;          // [slots][row_width]
  const int* block_table;     // [sequences][max_blocks]
  const int* row_seq;         // [rows] sequence of a row (nullptr: the row itself)
  const int* row_len;         // [rows] keys visible before the window is applied (position + 1)
  void* out;                  // [rows][H][rank]
  float* part_out;            // [rows][H][splits][rank]
  float* part_lse;            // [rows][H][splits]
  int rows, H, dim, rot, rank, row_width, max_blocks, block_size, block_shift, window, chunk, splits;
  float scale;
};

__device__ __forceinline__ void attend_range(const LatentAttendParams& p, int row, int split, int& j0, int& j1) {
  const int len = p.row_len[row];
  const int lo = max(0, len - p.window);
  j0 = lo + split * p.chunk;
  j1 = min(len, j0 + p.chunk);
}

// grid (rows, H, splits).  Scores of the chunk go to shared memory, then threads own latent columns.
template <typename T>
__global__ void __launch_bounds__(128) latent_attend_simt_kernel(LatentAttendParams p) {
  extern __shared__ float sm[];
  __shared__ float scratch[32];
  const int row = blockIdx.x, h = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  float* qs = sm;                          // [rank + rot]
  float* sc = sm + p.rank + p.rot;         // [chunk]
  int j0, j1;
  attend_range(p, row, split, j0, j1);
  const int seq = p.row_seq ? p.row_seq[row] : row;
  const int* bt = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const T* cache = reinterpret_cast<const T*>(p.cache);
  const T* ql = reinterpret_cast<const T*>(p.q_lat) + (static_cast<long long>(row) * p.H + h) * p.rank;
  const T* qr = reinterpret_cast<const T*>(p.q) + row * p.q_ld + h * (p.dim + p.rot) + p.dim;
  for (int i = threadIdx.x; i < p.rank + p.rot; i += blockDim.x) qs[i] = to_f32(i < p.rank ? ql[i] : qr[i - p.rank]);
  __syncthreads();
  float mx = -INFINITY;
  for (int j = j0 + warp; j < j1; j += nw) {
    const T* c = cache + (static_cast<long long>(bt[j / p.block_size]) * p.block_size + j % p.block_size) * p.row_width;
    float s = 0.f;
    for (int i = lane; i < p.rank + p.rot; i += 32) s += qs[i] * to_f32(c[i]);
    s = warp_sum(s) * p.scale;
    if (lane == 0) sc[j - j0] = s;
    mx = fmaxf(mx, s);
  }
  mx = block_max(mx, scratch);
  float l = 0.f;
  for (int j = j0 + threadIdx.x; j < j1; j += blockDim.x) {
    const float w = expf(sc[j - j0] - mx);
    sc[j - j0] = w;
    l += w;
  }
  l = block_sum(l, scratch);               // also orders the weights
  const float inv = l > 0.f ? 1.f / l : 0.f;
  const long long o = (static_cast<long long>(row) * p.H + h);
  for (int r = threadIdx.x; r < p.rank; r += blockDim.x) {
    float acc = 0.f;
    for (int j = j0; j < j1; ++j)
      acc += sc[j - j0] *
             to_f32(cache[(static_cast<long long>(bt[j / p.block_size]) * p.block_size + j % p.block_size) * p.row_width + r]);
    if (p.splits == 1) reinterpret_cast<T*>(p.out)[o * p.rank + r] = from_f32<T>(acc * inv);
    else p.part_out[(o * p.splits + split) * p.rank + r] = acc * inv;
  }
  if (p.splits > 1 && threadIdx.x == 0) p.part_lse[o * p.splits + split] = l > 0.f ? mx + logf(l) : -INFINITY;
}

constexpr int MERGE_MAX_SPLITS = 256;
template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(LatentAttendParams p) {
  __shared__ float w[MERGE_MAX_SPLITS];
  __shared__ float scratch[32];
  const long long o = static_cast<long long>(blockIdx.x) * p.H + blockIdx.y;
  const float* lse = p.part_lse + o * p.splits;
  float mx = -INFINITY, den = 0.f;
  for (int s = threadIdx.x; s < p.splits; s += blockDim.x) mx = fmaxf(mx, lse[s]);
  mx = block_max(mx, scratch);
  for (int s = threadIdx.x; s < p.splits; s += blockDim.x) {
    w[s] = lse[s] == -INFINITY ? 0.f : expf(lse[s] - mx);
    den += w[s];
  }
  den = block_sum(den, scratch);           // also orders the weights
  const float inv = 1.f / den;
  for (int r = threadIdx.x; r < p.rank; r += blockDim.x) {
    const float* part = p.part_out + o * p.splits * p.rank + r;
    float acc = 0.f;
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) acc += w[s] * part[static_cast<long long>(s) * p.rank];
    reinterpret_cast<T*>(p.out)[o * p.rank + r] = from_f32<T>(acc * inv);
  }
}

// ---------------------------------------------------------------------------------------------------------
// bf16 decode kernel.  grid (rows, ceil(H / 16), splits), 16 compute warps and 4 loader warps.  Tiles of 32 cached rows
// stream through a ring of shared-memory stages (one bulk copy per row, full / empty mbarriers per stage); a tile serves as
// K (all row_width columns) and as V (the first rank columns).
//   scores   warp w: the 16 heads x keys [8 (w % 4), + 8) of the tile, over quarter w / 4 of the columns; the query
//            fragments of that quarter stay in registers for the whole kernel
//   softmax  warp w: head w, one key per lane (running max and sum in registers, fp32)
//   output   warp w: latent columns [8 NP w, 8 NP (w + 1)) of the 16 heads, fp32 accumulators in registers
// Two barriers among the compute warps per tile.
// ---------------------------------------------------------------------------------------------------------
constexpr int LD_WARPS = 16;
constexpr int LD_KT = 32;
constexpr int LD_STAGES = 4;
constexpr int LD_LOADERS = 4;

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
// one contiguous row, global -> shared; both 16-byte aligned, size a multiple of 16
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void compute_barrier() {
  asm volatile("bar.sync 1, %0;" ::"n"(LD_WARPS * 32) : "memory");
}

// shared-memory row stride in elements: an odd number of 16-byte units, so that ldmatrix rows hit different banks
__host__ __device__ inline int latent_stride(int width) { return (width / 8 + 1 - (width / 8) % 2) * 8; }
static size_t latent_smem_bytes(int row_width) {
  const size_t st = latent_stride(row_width);
  return (LD_STAGES * LD_KT + 16) * st * 2 + 16 * (LD_KT + 8) * 2 + 4 * 16 * (LD_KT + 4) * 4 + 16 * 4 * 2 + 2 * LD_STAGES * 8;
}

template <int NP>   // rank <= 128 NP, row_width <= 128 NP + 64
__global__ void __launch_bounds__((LD_WARPS + LD_LOADERS) * 32, 1) latent_attend_mma_kernel(LatentAttendParams p) {
  constexpr int KS = 2 * NP + 1;           // 16-column steps of a quarter of a row
  constexpr int SW = LD_KT + 4;
  extern __shared__ __align__(16) uint8_t raw[];
  const int st = latent_stride(p.row_width), cols = p.row_width;
  __nv_bfloat16* kv = reinterpret_cast<__nv_bfloat16*>(raw);             // [STAGES][KT][st]
  __nv_bfloat16* qs = kv + LD_STAGES * LD_KT * st;                       // [16][st]
  __nv_bfloat16* ps = qs + 16 * st;                                      // [16][KT + 8]
  float* ss = reinterpret_cast<float*>(ps + 16 * (LD_KT + 8));           // [4 quarters][16][SW]
  float* s_alpha = ss + 4 * 16 * SW;                                     // [16]
  float* s_l = s_alpha + 16;                                             // [16]
  uint64_t* full = reinterpret_cast<uint64_t*>(s_l + 16);                // [STAGES]
  uint64_t* empty = full + LD_STAGES;                                    // [STAGES]
  const int row = blockIdx.x, h0 = blockIdx.y * 16, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int j0, j1;
  attend_range(p, row, split, j0, j1);
  const int seq = p.row_seq ? p.row_seq[row] : row;
  const int* bt = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  const __nv_bfloat16* ql = reinterpret_cast<const __nv_bfloat16*>(p.q_lat) + static_cast<long long>(row) * p.H * p.rank;
  const __nv_bfloat16* qr = reinterpret_cast<const __nv_bfloat16*>(p.q) + row * p.q_ld;
  const int tiles = j1 > j0 ? (j1 - j0 + LD_KT - 1) / LD_KT : 0;
  bool alive = true;
  if (threadIdx.x == 0) {
    for (int i = 0; i < LD_STAGES; ++i) {
      mbar_init(&full[i], LD_LOADERS);
      mbar_init(&empty[i], LD_WARPS);
    }
    fence_barrier_init();
  }
  if (warp < LD_WARPS) {   // the 16 query rows, one per warp: [q_lat | q_rot | 0]
    const int h = h0 + warp;
    __nv_bfloat16* dst = qs + warp * st;
    const uint4* lat = reinterpret_cast<const uint4*>(ql + static_cast<long long>(h) * p.rank);
#pragma unroll
    for (int k = 0; k < (128 * NP + 255) / 256; ++k) {
      const int c = lane + k * 32;
      if (c < p.rank / 8) *reinterpret_cast<uint4*>(dst + c * 8) = h < p.H ? lat[c] : make_uint4(0u, 0u, 0u, 0u);
    }
    const __nv_bfloat16* rotated = qr + h * (p.dim + p.rot) + p.dim;
    for (int c = lane; c < cols - p.rank; c += 32)
      dst[p.rank + c] = h < p.H && c < p.rot ? rotated[c] : __float2bfloat16(0.f);
  }
  __syncthreads();

  if (warp >= LD_WARPS) {
    // loader warp w: rows 8 w .. 8 w + 7 of a tile, one per lane; the page of the lane's next row is looked up one tile ahead
    // and used no earlier, so the table's latency is off the path
    constexpr int RPW = LD_KT / LD_LOADERS;
    const int r = (warp - LD_WARPS) * RPW + lane, shift = p.block_shift;
    int page = 0;
    if (lane < RPW && j0 + r < j1) page = bt[(j0 + r) >> shift];
    for (int i = 0; i < tiles; ++i) {
      const int s = i % LD_STAGES, j = j0 + i * LD_KT + r;
      const int mine = max(0, min(RPW, j1 - (j - lane)));            // rows of this warp inside the range
      if (!__all_sync(0xffffffffu, mbar_wait(&empty[s], ((i / LD_STAGES) & 1u) ^ 1u, alive, 901))) break;
      for (int z = mine; z < RPW; ++z)                               // zero rows past the range keep 0 * x finite
        for (int c = lane; c < cols / 8; c += 32)
          *reinterpret_cast<uint4*>(kv + (s * LD_KT + r - lane + z) * st + c * 8) = make_uint4(0u, 0u, 0u, 0u);
      __syncwarp();
      if (lane == 0) mbar_expect_tx(&full[s], mine * cols * 2);
      __syncwarp();
      if (lane < mine)
        bulk_load(smem_u32(kv + (s * LD_KT + r) * st),
                  cache + ((static_cast<long long>(page) << shift) + (j & (p.block_size - 1))) * cols, cols * 2, &full[s]);
      if (lane < RPW && j + LD_KT < j1) page = bt[(j + LD_KT) >> shift];
    }
    if (!alive) {                        // a wait ran out: give the copies in flight a bounded time to land
      const long long t0 = clock64();
      while (clock64() - t0 < 2000000ll) {
      }
    }
    return;
  }
  // columns in 16-wide steps: this warp's quarter
  const int steps = cols / 16, per = (steps + 3) / 4;
  const int k_first = (warp >> 2) * per, k_count = min(per, steps - k_first);      // may be <= 0 for narrow rows
  uint32_t qf[KS][4];
#pragma unroll
  for (int k = 0; k < KS; ++k) {
    qf[k][0] = qf[k][1] = qf[k][2] = qf[k][3] = 0u;
    if (k < k_count) ldsm_x4(qf[k], smem_u32(qs + (lane & 15) * st + (lane >> 4) * 8 + (k_first + k) * 16));
  }
  float o[NP][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int q = 0; q < 4; ++q) o[i][q] = 0.f;
  float m_run = -INFINITY, l_lane = 0.f;
  const float sl = p.scale * 1.4426950408889634f;
  const int gid = lane >> 2, tig = lane & 3;

  for (int i = 0; i < tiles; ++i) {
    const int s = i % LD_STAGES;
    const __nv_bfloat16* tile = kv + s * LD_KT * st;
    const int n = min(LD_KT, j1 - (j0 + i * LD_KT));
    mbar_wait(&full[s], (i / LD_STAGES) & 1u, alive, 900);
    {
      float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t ka = smem_u32(tile + ((warp & 3) * 8 + (lane & 7)) * st + k_first * 16 + (lane >> 3) * 8);
#pragma unroll
      for (int k = 0; k < KS; k += 2) {
        if (k + 1 < KS && k + 1 < k_count) {
          uint32_t b[4];
          ldsm_x4(b, ka + k * 32);                 // 8 keys x 32 columns
          mma_16816(c0, qf[k], b[0], b[1]);
          mma_16816(c1, qf[k + 1 < KS ? k + 1 : k], b[2], b[3]);
        } else if (k < k_count) {
          uint32_t b0, b1;
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];"
                       : "=r"(b0), "=r"(b1)
                       : "r"(smem_u32(tile + ((warp & 3) * 8 + (lane & 7)) * st + (k_first + k) * 16 + ((lane >> 3) & 1) * 8)));
          mma_16816(c0, qf[k], b0, b1);
        }
      }
      float* d = ss + ((warp >> 2) * 16 + gid) * SW + (warp & 3) * 8 + tig * 2;
      *reinterpret_cast<float2*>(d) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
      *reinterpret_cast<float2*>(d + 8 * SW) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
    }
    compute_barrier();                             // scores complete
    {   // softmax of head `warp`, one key per lane
      const float* a = ss + warp * SW + lane;
      const float v = lane < n ? ((a[0] + a[16 * SW]) + (a[32 * SW] + a[48 * SW])) * sl : -INFINITY;
      const float m_new = fmaxf(m_run, warp_max(v));   // n >= 1: finite
      const float alpha = fast_ex2(m_run - m_new), w = fast_ex2(v - m_new);
      m_run = m_new;
      l_lane = l_lane * alpha + w;
      ps[warp * (LD_KT + 8) + lane] = __float2bfloat16(w);
      if (lane == 0) s_alpha[warp] = alpha;
    }
    compute_barrier();                             // weights complete
    {
      if (i > 0) {
        const float al0 = s_alpha[gid], al1 = s_alpha[gid + 8];
#pragma unroll
        for (int x = 0; x < NP; ++x) {
          o[x][0] *= al0; o[x][1] *= al0; o[x][2] *= al1; o[x][3] *= al1;
        }
      }
      const uint32_t pa = smem_u32(ps + (lane & 15) * (LD_KT + 8) + (lane >> 4) * 8);
      uint32_t a0[4], a1[4];
      ldsm_x4(a0, pa);
      ldsm_x4(a1, pa + 32);
#pragma unroll
      for (int x = 0; x < NP; ++x) {
        const int c = (warp * NP + x) * 8;
        if (c < p.rank) {
          uint32_t b[4];    // 32 keys (four 8-row matrices) x columns c .. +8, transposed
          ldsm_x4_t(b, smem_u32(tile + lane * st + c));
          mma_16816(o[x], a0, b[0], b[1]);
          mma_16816(o[x], a1, b[2], b[3]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[s]);
    }
  }
  const float l_run = warp_sum(l_lane);
  if (lane == 0) {
    s_l[warp] = l_run;
    const int h = h0 + warp;
    if (p.splits > 1 && h < p.H)
      p.part_lse[(static_cast<long long>(row) * p.H + h) * p.splits + split] =
          l_run > 0.f ? (m_run + log2f(l_run)) * 0.6931471805599453f : -INFINITY;
  }
  compute_barrier();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = gid + half * 8, h = h0 + r;
    if (h >= p.H) continue;
    const float inv = s_l[r] > 0.f ? 1.f / s_l[r] : 0.f;
    const long long base = static_cast<long long>(row) * p.H + h;
#pragma unroll
    for (int x = 0; x < NP; ++x) {
      const int c = (warp * NP + x) * 8 + tig * 2;
      if (c < p.rank) {
        const float v0 = o[x][2 * half] * inv, v1 = o[x][2 * half + 1] * inv;
        if (p.splits == 1)
          *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + base * p.rank + c) = pack_bf16x2(v0, v1);
        else
          *reinterpret_cast<float2*>(p.part_out + (base * p.splits + split) * p.rank + c) = make_float2(v0, v1);
      }
    }
  }
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_latent)
using namespace ts;
#define ST(s) reinterpret_cast<cudaStream_t>(s)

// Width of a cache row: rank + rot rounded up to whole 16-column MMA steps.
extern "C" int ts_latent_row_width(int rank, int rot) { return (rank + rot + 15) / 16 * 16; }

// cos and sin are multiplied by `magnitude`; pairs: rotation partners are coordinates 2 i and 2 i + 1 instead of i and i + rot / 2.
extern "C" int ts_latent_prep(void* proj, long long ld, int H, int dim, int rot, int rank, const float* norm_w, float eps,
                              const float* inv_freq, float magnitude, int pairs, const int* pos, const long long* slots, void* cache, void* flat,
                              int row_width, int rows, int fp32, void* stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || rank <= 0 || rot < 0 || rot % 2 || row_width < rank + rot) return -10;
  const __nv_bfloat16* down = (const __nv_bfloat16*)proj + H * dim;
  if (!fp32 && rot == 0 && rank % 8 == 0 && row_width % 8 == 0 && row_width <= 1024 && ld % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(down) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(flat) |
        reinterpret_cast<uintptr_t>(norm_w)) & 15u) == 0) {
    latent_norm_vec_kernel<<<(rows + LPV_WARPS - 1) / LPV_WARPS, LPV_WARPS * 32, 0, ST(stream)>>>(
        down, ld, rank, norm_w, eps, slots, (__nv_bfloat16*)cache, (__nv_bfloat16*)flat, row_width, rows);
    return (int)cudaGetLastError();
  }
  const size_t sm = sizeof(float) * (rot > 0 ? rot : 2);
  if (fp32)
    latent_prep_kernel<float><<<rows, 128, sm, ST(stream)>>>((float*)proj, ld, H, dim, rot, rank, norm_w, eps, inv_freq,
                                                             magnitude, pairs, pos, slots, (float*)cache, (float*)flat, row_width);
  else
    latent_prep_kernel<__nv_bfloat16><<<rows, 128, sm, ST(stream)>>>(
        (__nv_bfloat16*)proj, ld, H, dim, rot, rank, norm_w, eps, inv_freq, magnitude, pairs, pos, slots, (__nv_bfloat16*)cache,
        (__nv_bfloat16*)flat, row_width);
  return (int)cudaGetLastError();
}

extern "C" int ts_latent_gather(const void* cache, const long long* slots, void* out, long long rows, int row_bytes,
                                void* stream) {
  if (rows <= 0) return 0;
  if (row_bytes <= 0 || row_bytes % 16) return -10;
  const int vec = row_bytes / 16;
  long long blocks = (rows * vec + 255) / 256;
  const long long cap = static_cast<long long>(sm_count()) * 16;
  if (blocks > cap) blocks = cap;
  latent_gather_kernel<<<(unsigned)blocks, 256, 0, ST(stream)>>>((const uint4*)cache, slots, (uint4*)out, rows, vec);
  return (int)cudaGetLastError();
}

static int latent_mma_np(int rank, int row_width) {
  const int by_rank = (rank + 127) / 128, by_row = (row_width - 64 + 127) / 128;
  return by_rank > by_row ? by_rank : by_row;
}
static int latent_mma_fits(int rank, int row_width, int block_size, int fp32) {
  return !fp32 && (block_size & (block_size - 1)) == 0 && rank % 16 == 0 && row_width % 16 == 0 && latent_mma_np(rank, row_width) <= 4 &&
         latent_smem_bytes(row_width) <= 227 * 1024;
}

// Number of CTAs a row's window is split over.
extern "C" int ts_latent_splits(int rows, int H, int rank, int row_width, int block_size, int max_keys,
                                int fp32) {
  if (latent_mma_fits(rank, row_width, block_size, fp32)) {
    // one CTA per SM at a time: rounds x (tiles of a CTA + a start-up cost of about four tiles), and a merge
    const long long units = static_cast<long long>(rows) * ((H + 15) / 16);
    const int tiles = (max_keys + LD_KT - 1) / LD_KT;
    int best = 1;
    long long cost = -1;
    for (int s = 1; s <= tiles && s <= 64; ++s) {
      const int per = (tiles + s - 1) / s;
      if (s > 1 && (tiles + per - 1) / per != s) continue;     // some CTAs would get no tile
      const long long c = (units * s + sm_count() - 1) / sm_count() * (per + 4) + (s > 1 ? 4 : 0);
      if (cost < 0 || c < cost) {
        cost = c;
        best = s;
      }
    }
    return best;
  }
  const long long units = static_cast<long long>(rows) * H;
  const int most = (max_keys + 255) / 256;
  long long s = (2ll * sm_count() + units - 1) / units;
  if (s > most) s = most;
  if (s < (max_keys + 2047) / 2048) s = (max_keys + 2047) / 2048;   // the chunk's scores sit in shared memory
  if (s > MERGE_MAX_SPLITS) s = MERGE_MAX_SPLITS;
  return (int)(s < 1 ? 1 : s);
}

// max_keys: upper bound of the visible keys of any row (min of window and longest length).  part_out / part_lse:
// workspaces when splits > 1.
extern "C" int ts_latent_attend(const void* q_lat, const void* q, long long q_ld, const void* cache,
                                const int* block_table, int max_blocks, const int* row_seq, const int* row_len, void* out,
                                float* part_out, float* part_lse, int rows, int H, int dim, int rot, int rank,
                                int row_width, int block_size, int window, int max_keys, int splits, float scale, int fp32,
                                void* stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || rank <= 0 || block_size <= 0 || window <= 0 || splits <= 0 || splits > MERGE_MAX_SPLITS) return -10;
  LatentAttendParams p;
  p.q_lat = q_lat; p.q = q; p.q_ld = q_ld; p.cache = cache; p.block_table = block_table; p.row_seq = row_seq;
  p.row_len = row_len; p.out = out; p.part_out = part_out; p.part_lse = part_lse; p.rows = rows; p.H = H; p.dim = dim;
  p.rot = rot; p.rank = rank; p.row_width = row_width; p.max_blocks = max_blocks; p.block_size = block_size;
  p.window = window; p.splits = splits; p.scale = scale;
  p.block_shift = 0;
  while ((1 << p.block_shift) < block_size) ++p.block_shift;
  cudaStream_t st = ST(stream);
  if (latent_mma_fits(rank, row_width, block_size, fp32)) {
    const int tiles = (max_keys + LD_KT - 1) / LD_KT;
    p.chunk = (tiles + splits - 1) / splits * LD_KT;
    const size_t sm = latent_smem_bytes(row_width);
    const dim3 grid(rows, (H + 15) / 16, splits);
    const int np = latent_mma_np(rank, row_width);
#define TS_LATENT(N)                                                                                             \
  {                                                                                                              \
    static bool configured = false;                                                                              \
    if (!configured) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(latent_attend_mma_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           227 * 1024);                                                          \
      if (e != cudaSuccess) return (int)e;                                                                       \
      configured = true;                                                                                         \
    }                                                                                                            \
    latent_attend_mma_kernel<N><<<grid, (LD_WARPS + LD_LOADERS) * 32, sm, st>>>(p);                                             \
  }
    if (np <= 1) TS_LATENT(1)
    else if (np == 2) TS_LATENT(2)
    else if (np == 3) TS_LATENT(3)
    else TS_LATENT(4)
#undef TS_LATENT
  } else {
    p.chunk = (max_keys + splits - 1) / splits;
    const size_t sm = sizeof(float) * (rank + rot + p.chunk);
    if (sm > 48 * 1024) return -12;
    const dim3 grid(rows, H, splits);
    if (fp32) latent_attend_simt_kernel<float><<<grid, 128, sm, st>>>(p);
    else latent_attend_simt_kernel<__nv_bfloat16><<<grid, 128, sm, st>>>(p);
  }
  if (splits > 1) {
    const dim3 grid(rows, H);
    if (fp32) latent_merge_kernel<float><<<grid, 128, 0, st>>>(p);
    else latent_merge_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(p);
  }
  return (int)cudaGetLastError();
}
