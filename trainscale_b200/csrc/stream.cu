// Residual-stream kernels of decoders that keep the whole depth history of the stream in fp32: one launch per layer
// boundary does everything between the last GEMM of a layer and the first GEMM of the next one.
//
//   source        layer boundary: X_n = x + mixer + sum_j w_j * expert_j  (mixer and feed-forward of a parallel block)
//                 embedding:      X_0 = embed[token] + bigram[(prev * mul_prev + token * mul_cur) mod buckets]
//   depth average x = sum_{j <= n} a_j X_j
//   norm          h = x / sqrt(mean(x^2) + eps) * g, g a single number
//   token shift   hs = h + (h_prev - h) * mu, h_prev of the row before (same batch), of the sequence's state, or zero
//
// Rows are tokens of a flattened batch of sequences.  A CTA walks a run of consecutive rows and carries h of the row
// before in registers; for its first row it recomputes the row before (a halo) unless that row starts from a state
// row or from zeros.  The stream, the history, the state and all arithmetic are fp32; h and hs leave in the activation
// type.  Bandwidth-bound: every value of the history is read once per row (plus one halo row per run).
//
// `postnorm_kernel` is the boundary of decoders that norm a sublayer's OUTPUT and keep no history:
//   source        x' = x + y / sqrt(mean(y^2) + eps) * (1 + w), or x' = embed[token] * scale
//   outputs       x' (fp32); x' in the activation type, or n token-shift mixes of it, x' + (x'_prev - x') * mu_s;
//                 last boundary: x' normed once more with the final weight, only for the rows that are wanted
//
// `prenorm_kernel` is the boundary of decoders that norm a sublayer's INPUT:
//   source        x' = x + y (* sigmoid(g), one number per row, or * sigmoid(g + b), one per element) + sum_j w_j * expert_j, or
//                 x' = embed[token]
//   outputs       x' (fp32); h = x' / sqrt(mean(x'^2) + eps) * (base + w); last boundary: h only, for the wanted rows
#include "common.cuh"
#include "host_common.h"

namespace ts {

enum StreamMode { STREAM_EMBED = 0, STREAM_LAYER = 1, STREAM_FINAL = 2 };

struct StreamParams {
  // embedding source
  const long long* tok;        // [T]
  const int* prev_tok;         // [T], -1: first token of its sequence
  const void* embed;           // [vocab][W]
  const void* bigram;          // [buckets + 1][W]
  long long mul_prev, mul_cur;
  int buckets, vocab;
  // layer source
  const float* x_in;           // [T][W]
  const void* mixer;           // [T][mixer_ld] or nullptr
  int mixer_ld;
  const void* y;               // expert outputs, W wide, or nullptr
  const int* dest;             // [T * k] row of y of every routed slot (nullptr: the slot itself)
  const float* route_w;        // [T * k]
  int k;
  // depth history: X_j of row t at hist + j * hist_stride + t * W
  float* hist;
  long long hist_stride;
  const float* dwa;            // [n_hist + 1]
  int n_hist;                  // layers' results already in the history (X_0 .. X_{n_hist - 1})
  float* x_out;                // [T][W]
  // norm, shift
  const float* gain;
  float eps;
  const float* shift;          // [W] or nullptr (no hs)
  void* h;                     // [rows][W]
  void* hs;                    // [rows][W]
  const int* row_prev;         // [T] >= 0: state row, -1: zeros, -2: the row before
  const int* row_next;         // [T] >= 0: state row that receives h, -1: none
  float* state;                // [state rows][W]
  const int* rows;             // FINAL: the rows to produce
  int n_rows, W, rows_per_cta;
};

template <typename T> struct VecIO;
template <> struct VecIO<float> {
  template <int V> __device__ static void load(const float* p, float* o) {
    if (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(p);
      o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w;
    } else {
      o[0] = *p;
    }
  }
  template <int V> __device__ static void store(float* p, const float* v) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
  }
};
template <> struct VecIO<__nv_bfloat16> {
  template <int V> __device__ static void load(const __nv_bfloat16* p, float* o) {
    if (V == 4) {
      const uint2 a = *reinterpret_cast<const uint2*>(p);
      const float2 lo = unpack_bf16x2(a.x), hi = unpack_bf16x2(a.y);
      o[0] = lo.x; o[1] = lo.y; o[2] = hi.x; o[3] = hi.y;
    } else {
      o[0] = __bfloat162float(*p);
    }
  }
  template <int V> __device__ static void store(__nv_bfloat16* p, const float* v) {
    if (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
    else *p = __float2bfloat16(v[0]);
  }
};

template <typename T, int MODE, int V, int NV>
__global__ void __launch_bounds__(V == 4 ? 512 : 1024)
stream_kernel(StreamParams p) {
  __shared__ float scratch[32];
  const int W = p.W, nvec = W / V;
  const T* mixer = reinterpret_cast<const T*>(p.mixer);
  const T* y = reinterpret_cast<const T*>(p.y);
  const float gain = *p.gain;

  // value of one row of the stream after this boundary, in registers; `keep` writes it (and X_n) back
  auto row_value = [&](int t, float (&v)[NV][V], bool keep) {
    if (MODE == STREAM_EMBED) {
      long long tok = p.tok[t];
      if (tok < 0 || tok >= p.vocab) {
        if (threadIdx.x == 0) ts_report_error(ERR_BOUNDS, 8000, static_cast<unsigned int>(tok));
        tok = 0;
      }
      const int prev = p.prev_tok[t];
      const long long row = prev < 0 ? p.buckets : (prev * p.mul_prev + tok * p.mul_cur) % p.buckets;
      const T* e = reinterpret_cast<const T*>(p.embed) + static_cast<size_t>(tok) * W;
      const T* b = reinterpret_cast<const T*>(p.bigram) + static_cast<size_t>(row) * W;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < nvec) {
          float a[V], d[V];
          VecIO<T>::template load<V>(e + c * V, a);
          VecIO<T>::template load<V>(b + c * V, d);
#pragma unroll
          for (int q = 0; q < V; ++q) v[i][q] = a[q] + d[q];
          if (keep) VecIO<float>::store<V>(p.hist + static_cast<size_t>(t) * W + c * V, v[i]);
        }
      }
      return;
    }
    const size_t base = static_cast<size_t>(t) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        VecIO<float>::load<V>(p.x_in + base + c * V, v[i]);
        if (mixer) {
          float a[V];
          VecIO<T>::template load<V>(mixer + static_cast<size_t>(t) * p.mixer_ld + c * V, a);
#pragma unroll
          for (int q = 0; q < V; ++q) v[i][q] += a[q];
        }
      }
    }
    if (y) {
      for (int j = 0; j < p.k; ++j) {
        const int slot = t * p.k + j;
        const float w = p.route_w[slot];
        const T* src = y + static_cast<size_t>(p.dest ? p.dest[slot] : slot) * W;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < nvec) {
            float a[V];
            VecIO<T>::template load<V>(src + c * V, a);
#pragma unroll
            for (int q = 0; q < V; ++q) v[i][q] += w * a[q];
          }
        }
      }
    }
    // every load of the history is issued before the first store of the row
    constexpr int UN = NV == 1 ? 8 : (NV == 2 ? 4 : 2);
    float acc[NV][V];
    const float an = p.dwa[p.n_hist];
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int q = 0; q < V; ++q) acc[i][q] = an * v[i][q];
#pragma unroll UN
    for (int j = 0; j < p.n_hist; ++j) {
      const float aj = p.dwa[j];
      const float* src = p.hist + j * p.hist_stride + base;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < nvec) {
          float a[V];
          VecIO<float>::load<V>(src + c * V, a);
#pragma unroll
          for (int q = 0; q < V; ++q) acc[i][q] += aj * a[q];
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec && keep && MODE == STREAM_LAYER) {
        VecIO<float>::store<V>(p.hist + p.n_hist * p.hist_stride + base + c * V, v[i]);
        VecIO<float>::store<V>(p.x_out + base + c * V, acc[i]);
      }
#pragma unroll
      for (int q = 0; q < V; ++q) v[i][q] = acc[i][q];
    }
  };

  auto normalise = [&](float (&v)[NV][V]) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (threadIdx.x + i * blockDim.x < nvec) {
#pragma unroll
        for (int q = 0; q < V; ++q) ss += v[i][q] * v[i][q];
      }
    ss = block_sum(ss, scratch);
    const float inv = gain / sqrtf(ss / static_cast<float>(W) + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int q = 0; q < V; ++q) v[i][q] *= inv;
  };

  if (MODE == STREAM_FINAL) {
    float v[NV][V];
    row_value(p.rows[blockIdx.x], v, false);
    normalise(v);
    T* h = reinterpret_cast<T*>(p.h) + static_cast<size_t>(blockIdx.x) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) VecIO<T>::template store<V>(h + c * V, v[i]);
    }
    return;
  }

  const int r0 = blockIdx.x * p.rows_per_cta, r1 = min(p.n_rows, r0 + p.rows_per_cta);
  if (r0 >= r1) return;
  float hp[NV][V];
  if (p.row_prev[r0] == -2) {
    row_value(r0 - 1, hp, false);
    normalise(hp);
  }
  for (int t = r0; t < r1; ++t) {
    float v[NV][V];
    row_value(t, v, true);
    normalise(v);
    const int prev = p.row_prev[t], next = p.row_next[t];
    const size_t base = static_cast<size_t>(t) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        if (prev >= 0) {
          VecIO<float>::load<V>(p.state + static_cast<size_t>(prev) * W + c * V, hp[i]);
        } else if (prev == -1) {
#pragma unroll
          for (int q = 0; q < V; ++q) hp[i][q] = 0.f;
        }
        float mu[V], hs[V];
        VecIO<float>::load<V>(p.shift + c * V, mu);
#pragma unroll
        for (int q = 0; q < V; ++q) hs[q] = v[i][q] + (hp[i][q] - v[i][q]) * mu[q];
        VecIO<T>::template store<V>(reinterpret_cast<T*>(p.h) + base + c * V, v[i]);
        VecIO<T>::template store<V>(reinterpret_cast<T*>(p.hs) + base + c * V, hs);
        if (next >= 0) VecIO<float>::store<V>(p.state + static_cast<size_t>(next) * W + c * V, v[i]);
#pragma unroll
        for (int q = 0; q < V; ++q) hp[i][q] = v[i][q];
      }
    }
  }
}

template <typename T, int MODE, int V, int NV>
static int launch_stream_nv(StreamParams p, int threads, cudaStream_t st) {
  int grid = p.n_rows;
  p.rows_per_cta = 1;
  if (MODE != STREAM_FINAL) {
    // one wave: every resident CTA walks an equal run of rows (longer runs, fewer halo rows)
    static int per_sm[33] = {};
    int& occ = per_sm[threads / 32];
    if (occ == 0 && (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, stream_kernel<T, MODE, V, NV>, threads, 0) !=
                         cudaSuccess || occ < 1))
      occ = 1;
    const int slots = occ * sm_count();
    p.rows_per_cta = (p.n_rows + slots - 1) / slots;
    if (p.rows_per_cta > 32) p.rows_per_cta = 32;
    grid = (p.n_rows + p.rows_per_cta - 1) / p.rows_per_cta;
  }
  stream_kernel<T, MODE, V, NV><<<grid, threads, 0, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T, int MODE>
static int launch_stream(const StreamParams& p, cudaStream_t st) {
  const bool vec = p.W % 4 == 0 && p.mixer_ld % 4 == 0;
  const int nvec = vec ? p.W / 4 : p.W, cap = vec ? 512 : 1024;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > cap) threads = cap;
  const int nv = (nvec + threads - 1) / threads;
  if (vec) {
    if (nv <= 1) return launch_stream_nv<T, MODE, 4, 1>(p, threads, st);
    if (nv <= 2) return launch_stream_nv<T, MODE, 4, 2>(p, threads, st);
    if (nv <= 4) return launch_stream_nv<T, MODE, 4, 4>(p, threads, st);
    if (nv <= 8) return launch_stream_nv<T, MODE, 4, 8>(p, threads, st);
    return -11;
  }
  if (nv <= 1) return launch_stream_nv<T, MODE, 1, 1>(p, threads, st);
  if (nv <= 8) return launch_stream_nv<T, MODE, 1, 8>(p, threads, st);
  return -11;
}

struct PostnormParams {
  const long long* tok;        // embedding source: [T]
  const void* embed;           // [vocab][W]
  float embed_scale;
  int vocab;
  const float* x_in;           // sublayer source: [T][W]
  const void* y;               // [T][y_ld]
  long long y_ld;
  const float* w;              // [W], around zero
  float eps;
  float* x_out;                // [T][W] (not for FINAL)
  void* h;                     // [rows][W], or [rows][n_mix][W]
  const float* mu;             // [n_mix][W] or nullptr
  int n_mix;
  const int* row_prev;         // with mixes: as in StreamParams
  const int* row_next;
  float* state;                // previous x' of a sequence: first W values of a state row
  long long state_ld;
  const float* final_w;        // FINAL: [W]
  const int* rows;             // FINAL: the rows to produce
  int n_rows, W, rows_per_cta;
};

template <typename T, int MODE, int V, int NV>
__global__ void __launch_bounds__(V == 4 ? 512 : 1024)
postnorm_kernel(PostnormParams p) {
  __shared__ float scratch[32];
  const int W = p.W, nvec = W / V;

  // v / rms(v) * (1 + w), in place
  auto normed = [&](float (&v)[NV][V], const float* w) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (threadIdx.x + i * blockDim.x < nvec) {
#pragma unroll
        for (int q = 0; q < V; ++q) ss += v[i][q] * v[i][q];
      }
    ss = block_sum(ss, scratch);
    const float rms = sqrtf(ss / static_cast<float>(W) + p.eps);
    const float inv = 1.f / rms;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        float g[V];
        VecIO<float>::load<V>(w + c * V, g);
#pragma unroll
        for (int q = 0; q < V; ++q) v[i][q] = v[i][q] * inv * (1.f + g[q]);
      }
    }
  };

  auto row_value = [&](int t, float (&v)[NV][V]) {
    if (MODE == STREAM_EMBED) {
      long long tok = p.tok[t];
      if (tok < 0 || tok >= p.vocab) {
        if (threadIdx.x == 0) ts_report_error(ERR_BOUNDS, 8001, static_cast<unsigned int>(tok));
        tok = 0;
      }
      const T* e = reinterpret_cast<const T*>(p.embed) + static_cast<size_t>(tok) * W;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < nvec) {
          VecIO<T>::template load<V>(e + c * V, v[i]);
#pragma unroll
          for (int q = 0; q < V; ++q) v[i][q] *= p.embed_scale;
        }
      }
      return;
    }
    float x[NV][V];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        VecIO<T>::template load<V>(reinterpret_cast<const T*>(p.y) + t * p.y_ld + c * V, v[i]);
        VecIO<float>::load<V>(p.x_in + static_cast<size_t>(t) * W + c * V, x[i]);
      }
    }
    normed(v, p.w);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (threadIdx.x + i * blockDim.x < nvec) {
#pragma unroll
        for (int q = 0; q < V; ++q) v[i][q] += x[i][q];
      }
  };

  if (MODE == STREAM_FINAL) {
    float v[NV][V];
    row_value(p.rows[blockIdx.x], v);
    normed(v, p.final_w);
    T* h = reinterpret_cast<T*>(p.h) + static_cast<size_t>(blockIdx.x) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) VecIO<T>::template store<V>(h + c * V, v[i]);
    }
    return;
  }

  const int r0 = blockIdx.x * p.rows_per_cta, r1 = min(p.n_rows, r0 + p.rows_per_cta);
  if (r0 >= r1) return;
  float hp[NV][V];
  if (p.n_mix && p.row_prev[r0] == -2) row_value(r0 - 1, hp);
  for (int t = r0; t < r1; ++t) {
    float v[NV][V];
    row_value(t, v);
    const int prev = p.n_mix ? p.row_prev[t] : -1, next = p.n_mix ? p.row_next[t] : -1;
    const size_t base = static_cast<size_t>(t) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        VecIO<float>::store<V>(p.x_out + base + c * V, v[i]);
        if (p.n_mix == 0) {
          VecIO<T>::template store<V>(reinterpret_cast<T*>(p.h) + base + c * V, v[i]);
        } else {
          if (prev >= 0) {
            VecIO<float>::load<V>(p.state + prev * p.state_ld + c * V, hp[i]);
          } else if (prev == -1) {
#pragma unroll
            for (int q = 0; q < V; ++q) hp[i][q] = 0.f;
          }
          for (int s = 0; s < p.n_mix; ++s) {
            float mu[V], m[V];
            VecIO<float>::load<V>(p.mu + static_cast<size_t>(s) * W + c * V, mu);
#pragma unroll
            for (int q = 0; q < V; ++q) m[q] = v[i][q] + (hp[i][q] - v[i][q]) * mu[q];
            VecIO<T>::template store<V>(reinterpret_cast<T*>(p.h) + base * p.n_mix + static_cast<size_t>(s) * W + c * V, m);
          }
          if (next >= 0) VecIO<float>::store<V>(p.state + next * p.state_ld + c * V, v[i]);
#pragma unroll
          for (int q = 0; q < V; ++q) hp[i][q] = v[i][q];
        }
      }
    }
  }
}

template <typename T, int MODE, int V, int NV>
static int launch_postnorm_nv(PostnormParams p, int threads, cudaStream_t st) {
  int grid = p.n_rows;
  p.rows_per_cta = 1;
  if (MODE != STREAM_FINAL && p.n_mix) {
    static int per_sm[33] = {};
    int& occ = per_sm[threads / 32];
    if (occ == 0 && (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, postnorm_kernel<T, MODE, V, NV>, threads, 0) !=
                         cudaSuccess || occ < 1))
      occ = 1;
    const int slots = occ * sm_count();
    p.rows_per_cta = (p.n_rows + slots - 1) / slots;
    if (p.rows_per_cta > 32) p.rows_per_cta = 32;
    grid = (p.n_rows + p.rows_per_cta - 1) / p.rows_per_cta;
  }
  postnorm_kernel<T, MODE, V, NV><<<grid, threads, 0, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T, int MODE>
static int launch_postnorm(const PostnormParams& p, cudaStream_t st) {
  const bool vec = p.W % 4 == 0 && p.y_ld % 4 == 0 && p.state_ld % 4 == 0;
  const int nvec = vec ? p.W / 4 : p.W, cap = vec ? 512 : 1024;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > cap) threads = cap;
  const int nv = (nvec + threads - 1) / threads;
  if (vec) {
    if (nv <= 1) return launch_postnorm_nv<T, MODE, 4, 1>(p, threads, st);
    if (nv <= 2) return launch_postnorm_nv<T, MODE, 4, 2>(p, threads, st);
    if (nv <= 4) return launch_postnorm_nv<T, MODE, 4, 4>(p, threads, st);
    if (nv <= 8) return launch_postnorm_nv<T, MODE, 4, 8>(p, threads, st);
    return -11;
  }
  if (nv <= 1) return launch_postnorm_nv<T, MODE, 1, 1>(p, threads, st);
  if (nv <= 8) return launch_postnorm_nv<T, MODE, 1, 8>(p, threads, st);
  return -11;
}

struct PrenormParams {
  const long long* tok;        // embedding source: [T]
  const void* embed;           // [vocab][W]
  int vocab;
  const float* x_in;           // sublayer source: [T][W]
  const void* y;               // [T][y_ld] or nullptr
  long long y_ld;
  const float* y_gate;         // logit of y's factor, stride y_gate_ld per row (nullptr: 1)
  long long y_gate_ld;
  const void* e_gate;          // [T][e_gate_ld] logits of a factor of every element of y, activation type (nullptr: 1)
  long long e_gate_ld;
  const float* e_bias;         // [W], added to them
  const void* experts;         // expert outputs, W wide, or nullptr
  const int* dest;             // [T * k] row of every routed slot (nullptr: the slot itself)
  const float* route_w;        // [T * k]
  int k;
  const float* w;              // [W]
  float w_base;                // the norm multiplies by w_base + w
  float eps;
  float* x_out;                // [T][W] (not for FINAL)
  void* h;                     // [rows][W]
  const int* rows;             // FINAL: the rows to produce
  int W;
};

// grid: rows
template <typename T, int MODE, int V, int NV>
__global__ void __launch_bounds__(V == 4 ? 512 : 1024)
prenorm_kernel(PrenormParams p) {
  constexpr int AHEAD = NV == 1 ? 8 : (NV == 2 ? 4 : 2);      // expert rows in flight
  __shared__ float scratch[32];
  const int nvec = p.W / V, t = MODE == STREAM_FINAL ? p.rows[blockIdx.x] : blockIdx.x;
  const size_t base = static_cast<size_t>(t) * p.W;
  float v[NV][V];
  if (MODE == STREAM_EMBED) {
    long long tok = p.tok[t];
    if (tok < 0 || tok >= p.vocab) {
      if (threadIdx.x == 0) ts_report_error(ERR_BOUNDS, 8002, static_cast<unsigned int>(tok));
      tok = 0;
    }
    const T* e = reinterpret_cast<const T*>(p.embed) + static_cast<size_t>(tok) * p.W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) VecIO<T>::template load<V>(e + c * V, v[i]);
    }
  } else {
    const float f = p.y_gate ? sigmoid(p.y_gate[t * p.y_gate_ld]) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nvec) {
        VecIO<float>::load<V>(p.x_in + base + c * V, v[i]);
        if (p.y) {
          float a[V];
          VecIO<T>::template load<V>(reinterpret_cast<const T*>(p.y) + t * p.y_ld + c * V, a);
          if (p.e_gate) {
            float g[V], b[V];
            VecIO<T>::template load<V>(reinterpret_cast<const T*>(p.e_gate) + t * p.e_gate_ld + c * V, g);
            VecIO<float>::load<V>(p.e_bias + c * V, b);
#pragma unroll
            for (int q = 0; q < V; ++q) a[q] *= sigmoid(g[q] + b[q]);
          }
#pragma unroll
          for (int q = 0; q < V; ++q) v[i][q] += f * a[q];
        }
      }
    }
    if (p.experts) {
#pragma unroll AHEAD
      for (int j = 0; j < p.k; ++j) {
        const int slot = t * p.k + j;
        const float w = p.route_w[slot];
        const T* src = reinterpret_cast<const T*>(p.experts) + static_cast<size_t>(p.dest ? p.dest[slot] : slot) * p.W;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < nvec) {
            float a[V];
            VecIO<T>::template load<V>(src + c * V, a);
#pragma unroll
            for (int q = 0; q < V; ++q) v[i][q] += w * a[q];
          }
        }
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < nvec) {
      if (MODE != STREAM_FINAL) VecIO<float>::store<V>(p.x_out + base + c * V, v[i]);
#pragma unroll
      for (int q = 0; q < V; ++q) ss += v[i][q] * v[i][q];
    }
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.W) + p.eps);
  T* h = reinterpret_cast<T*>(p.h) + static_cast<size_t>(blockIdx.x) * p.W;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < nvec) {
      float g[V];
      VecIO<float>::load<V>(p.w + c * V, g);
#pragma unroll
      for (int q = 0; q < V; ++q) v[i][q] = v[i][q] * inv * (p.w_base + g[q]);
      VecIO<T>::template store<V>(h + c * V, v[i]);
    }
  }
}

template <typename T, int MODE>
static int launch_prenorm(const PrenormParams& p, int rows, cudaStream_t st) {
  const bool vec = p.W % 4 == 0 && p.y_ld % 4 == 0 && p.e_gate_ld % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.e_gate)) % (4 * sizeof(T)) == 0;
  const int nvec = vec ? p.W / 4 : p.W, cap = vec ? 512 : 1024;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > cap) threads = cap;
  const int nv = (nvec + threads - 1) / threads;
  if (vec) {
    if (nv <= 1) prenorm_kernel<T, MODE, 4, 1><<<rows, threads, 0, st>>>(p);
    else if (nv <= 2) prenorm_kernel<T, MODE, 4, 2><<<rows, threads, 0, st>>>(p);
    else if (nv <= 4) prenorm_kernel<T, MODE, 4, 4><<<rows, threads, 0, st>>>(p);
    else if (nv <= 8) prenorm_kernel<T, MODE, 4, 8><<<rows, threads, 0, st>>>(p);
    else return -11;
  } else {
    if (nv <= 1) prenorm_kernel<T, MODE, 1, 1><<<rows, threads, 0, st>>>(p);
    else if (nv <= 8) prenorm_kernel<T, MODE, 1, 8><<<rows, threads, 0, st>>>(p);
    else return -11;
  }
  return (int)cudaGetLastError();
}

}  // namespace ts

TS_DEFINE_ERROR_API(ts_stream)
using namespace ts;

// X_0 of every row -> hist[0]; h, hs of the first layer.  fp32_act: activations and tables are fp32 (else bf16).
extern "C" int ts_stream_embed(const long long* tok, const int* prev_tok, const void* embed, const void* bigram, int vocab,
                               int buckets, long long mul_prev, long long mul_cur, float* hist, const float* gain,
                               float eps, const float* shift, void* h, void* hs, const int* row_prev,
                               const int* row_next, float* state, int rows, int W, int fp32_act, void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || buckets <= 0) return -10;
  StreamParams p = {};
  p.tok = tok; p.prev_tok = prev_tok; p.embed = embed; p.bigram = bigram; p.vocab = vocab; p.buckets = buckets;
  p.mul_prev = mul_prev; p.mul_cur = mul_cur; p.hist = hist; p.gain = gain; p.eps = eps; p.shift = shift; p.h = h;
  p.hs = hs; p.row_prev = row_prev; p.row_next = row_next; p.state = state; p.n_rows = rows; p.W = W;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32_act ? launch_stream<float, STREAM_EMBED>(p, st) : launch_stream<__nv_bfloat16, STREAM_EMBED>(p, st);
}

// Layer boundary: X_n -> hist[n_hist], depth average -> x_out, norm and token shift of the NEXT layer -> h, hs.
// `rows_list` (with n_out entries): last boundary - only those rows are produced, h only, nothing else is written.
extern "C" int ts_stream_layer(const float* x_in, const void* mixer, int mixer_ld, const void* y, const int* dest,
                               const float* route_w, int k, float* hist, long long hist_stride, const float* dwa,
                               int n_hist, float* x_out, const float* gain, float eps, const float* shift, void* h,
                               void* hs, const int* row_prev, const int* row_next, float* state, int rows,
                               const int* rows_list, int n_out, int W, int fp32_act, void* stream) {
  if (rows_list ? n_out <= 0 : rows <= 0) return 0;
  if (W <= 0 || n_hist < 1 || (y && k <= 0)) return -10;
  StreamParams p = {};
  p.x_in = x_in; p.mixer = mixer; p.mixer_ld = mixer_ld; p.y = y; p.dest = dest; p.route_w = route_w; p.k = k;
  p.hist = hist; p.hist_stride = hist_stride; p.dwa = dwa; p.n_hist = n_hist; p.x_out = x_out; p.gain = gain;
  p.eps = eps; p.shift = shift; p.h = h; p.hs = hs; p.row_prev = row_prev; p.row_next = row_next; p.state = state;
  p.rows = rows_list; p.n_rows = rows_list ? n_out : rows; p.W = W;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (rows_list)
    return fp32_act ? launch_stream<float, STREAM_FINAL>(p, st) : launch_stream<__nv_bfloat16, STREAM_FINAL>(p, st);
  return fp32_act ? launch_stream<float, STREAM_LAYER>(p, st) : launch_stream<__nv_bfloat16, STREAM_LAYER>(p, st);
}

// Boundary of output-normed decoders.  `tok`: embedding source (then x_in, y, w are unused).  `mu` with n_mix rows: h
// receives the token-shift mixes [rows][n_mix][W] and the state row of `row_next` the row itself.
extern "C" int ts_stream_postnorm(const long long* tok, const void* embed, int vocab, float embed_scale, const float* x_in,
                                  const void* y, long long y_ld, const float* w, float eps, float* x_out, void* h,
                                  const float* mu, int n_mix, const int* row_prev, const int* row_next, float* state,
                                  long long state_ld, int rows, int W, int fp32_act, void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || n_mix < 0 || (n_mix && (!mu || !state || state_ld < W))) return -10;
  PostnormParams p = {};
  p.tok = tok; p.embed = embed; p.vocab = vocab; p.embed_scale = embed_scale; p.x_in = x_in; p.y = y; p.y_ld = y_ld;
  p.w = w; p.eps = eps; p.x_out = x_out; p.h = h; p.mu = mu; p.n_mix = n_mix; p.row_prev = row_prev;
  p.row_next = row_next; p.state = state; p.state_ld = state_ld; p.n_rows = rows; p.W = W;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (tok)
    return fp32_act ? launch_postnorm<float, STREAM_EMBED>(p, st) : launch_postnorm<__nv_bfloat16, STREAM_EMBED>(p, st);
  return fp32_act ? launch_postnorm<float, STREAM_LAYER>(p, st) : launch_postnorm<__nv_bfloat16, STREAM_LAYER>(p, st);
}

// Last boundary: the rows `rows_list`, residual sum and final norm -> h [n_out][W].
extern "C" int ts_stream_postnorm_final(const float* x_in, const void* y, long long y_ld, const float* w,
                                        const float* final_w, float eps, void* h, const int* rows_list, int n_out, int W,
                                        int fp32_act, void* stream) {
  if (n_out <= 0) return 0;
  if (W <= 0) return -10;
  PostnormParams p = {};
  p.x_in = x_in; p.y = y; p.y_ld = y_ld; p.w = w; p.final_w = final_w; p.eps = eps; p.h = h; p.rows = rows_list;
  p.n_rows = n_out; p.W = W;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32_act ? launch_postnorm<float, STREAM_FINAL>(p, st) : launch_postnorm<__nv_bfloat16, STREAM_FINAL>(p, st);
}

// Boundary of input-normed decoders.  `tok`: embedding source (then x_in, y and the experts are unused).  y_gate: logits of a
// factor of y, one per row; e_gate (with e_bias [W]): logits of one per element.  The norm multiplies by w_base + w.  experts with dest (nullptr: slot order) and route_w [rows * k]: weighted sum of a row's slots.
// `rows_list` (with n_out entries): last boundary - h of those rows only, nothing else is written.
extern "C" int ts_stream_prenorm(const long long* tok, const void* embed, int vocab, const float* x_in, const void* y,
                                 long long y_ld, const float* y_gate, long long y_gate_ld, const void* e_gate, long long e_gate_ld,
                                 const float* e_bias, const void* experts, const int* dest, const float* route_w, int k,
                                 const float* w, float w_base, float eps, float* x_out, void* h, int rows, const int* rows_list, int n_out, int W, int fp32_act, void* stream) {
  if (rows_list ? n_out <= 0 : rows <= 0) return 0;
  if (W <= 0 || (experts && (k <= 0 || !route_w)) || (tok && rows_list) || (e_gate && (!y || !e_bias))) return -10;
  PrenormParams p = {};
  p.tok = tok; p.embed = embed; p.vocab = vocab; p.x_in = x_in; p.y = y; p.y_ld = y_ld; p.y_gate = y_gate;
  p.y_gate_ld = y_gate_ld; p.e_gate = e_gate; p.e_gate_ld = e_gate_ld; p.e_bias = e_bias; p.w_base = w_base; p.experts = experts; p.dest = dest; p.route_w = route_w; p.k = k; p.w = w; p.eps = eps;
  p.x_out = x_out; p.h = h; p.rows = rows_list; p.W = W;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (tok) return fp32_act ? launch_prenorm<float, STREAM_EMBED>(p, rows, st) : launch_prenorm<__nv_bfloat16, STREAM_EMBED>(p, rows, st);
  if (rows_list)
    return fp32_act ? launch_prenorm<float, STREAM_FINAL>(p, n_out, st) : launch_prenorm<__nv_bfloat16, STREAM_FINAL>(p, n_out, st);
  return fp32_act ? launch_prenorm<float, STREAM_LAYER>(p, rows, st) : launch_prenorm<__nv_bfloat16, STREAM_LAYER>(p, rows, st);
}
