// filters.cu — the input side of pre-norm sublayers and short causal filters over time.
//
//   prenorm : x' = x + y (y: the result of the sublayer before, optional) ; n = x' / sqrt(mean(x'^2) + eps) * w ;
//             h = n, or with an input filter  h_t = n_t + sum_i c[i] n_{t - (taps - 1) + i}   per channel, zeros before
//             the start of the sequence: residual sum, norm and filter in one launch.  Without w: h = x' itself.
//   filter  : out = act(b + sum_i c[i] (in + in_bias)_{t - (taps - 1) + i})                   act: none or silu
//
// The residual, norms, filter sums and filter states are fp32; T is the activation type of y, in, h and out.  Per
// sequence slot a filter keeps its last taps - 1 inputs [slot, taps - 1, channels] (fp32).  A portion that starts at
// position 0 reads zeros whatever the slot holds.  Rows of a sequence are cut into chunks, one CTA each; a chunk works
// out the rows before it that its filter needs by itself.  Where every portion of the step is one chunk the CTA writes
// the new state; otherwise a second launch does, after all chunks have read the old one.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kPnThreads = 256;
constexpr int kMaxTaps = 16;

enum { SRC_NONE = 0, SRC_ROWS = 1, SRC_PARTIALS = 2 };

// v[0 .. 3] of a row; n valid channels (vec: all four, on a 4-element boundary)
template <typename T>
__device__ __forceinline__ void get4(const T* __restrict__ p, float (&v)[4], int n, bool vec) {
  if (vec) {
    load4<T>(p, v);
  } else {
#pragma unroll
    for (int k = 0; k < 4; ++k) v[k] = k < n ? Num<T>::to_f(p[k]) : 0.0f;
  }
}
template <typename T>
__device__ __forceinline__ void put4(T* __restrict__ p, const float (&v)[4], int n, bool vec) {
  if (vec) {
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      *reinterpret_cast<uint2*>(p) = make_uint2(Num<T>::pack(v[0], v[1]), Num<T>::pack(v[2], v[3]));
    }
  } else {
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k < n) p[k] = Num<T>::from_f(v[k]);
  }
}

struct PrenormArgs {
  float* x_out;            // nullable (no y, or nobody needs the sum)
  void* h_out;
  int64_t ldh;
  const float* x_in;
  const void* y;           // SRC_ROWS: rows of T with stride ldy (0: the same row for all)
  int64_t ldy;
  const float* partials;   // SRC_PARTIALS: fp32 [slots][rows][W]
  int64_t slot_stride;
  W4Plan plan;
  const float* w;          // nullable without a filter: no norm
  const float* filt;       // [taps][W], oldest tap first
  float* state;            // [slot][taps - 1][W]
  const int *q_cu, *positions, *state_slots;
  int W, taps, chunk;
  float eps;
  int carry;               // 1: no outputs, only the new filter state
  int write_state;
  int vec;
};

// x' of one row into dst [W] (shared memory); returns this thread's part of the sum of squares
template <typename T, int SRC>
__device__ __forceinline__ float residual_row(const PrenormArgs& a, float* dst, size_t row, bool store) {
  const float* x = a.x_in + row * a.W;
  float* xo = a.x_out + row * a.W;
  float ss = 0.0f;
  if constexpr (SRC == SRC_PARTIALS) {
    const float* prow = a.partials + row * a.W;
    for (int v = threadIdx.x; v < a.W / 8; v += kPnThreads) {
      float s[8];
      w4_sum_partials8(s, prow + v * 8, a.slot_stride, w4_contrib_col(a.plan, v * 8));
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float r = x[v * 8 + i] + rnd<T>(s[i]);     // what the product's own reduction pass would have stored
        dst[v * 8 + i] = r;
        if (store) xo[v * 8 + i] = r;
        ss += r * r;
      }
    }
  } else {
    const T* y = SRC == SRC_ROWS ? static_cast<const T*>(a.y) + row * a.ldy : nullptr;
    for (int i = threadIdx.x * 4; i < a.W; i += kPnThreads * 4) {
      float v[4];
      get4<float>(x + i, v, a.W - i, a.vec);
      if constexpr (SRC == SRC_ROWS) {
        float u[4];
        get4<T>(y + i, u, a.W - i, a.vec);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] += u[k];
        if (store) put4<float>(xo + i, v, a.W - i, a.vec);
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) ss += v[k] * v[k];
      put4<float>(dst + i, v, a.W - i, a.vec);           // (channels past W do not exist: n says so)
    }
  }
  return ss;
}

template <typename T, int SRC>
__global__ void __launch_bounds__(kPnThreads) prenorm_kernel(const PrenormArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  const float ss = block_sum<kPnThreads>(residual_row<T, SRC>(a, sm, row, a.x_out != nullptr), red);
  const float r = 1.0f / sqrtf(ss / (float)a.W + a.eps);
  T* h = static_cast<T*>(a.h_out) + row * a.ldh;
  for (int i = threadIdx.x * 4; i < a.W; i += kPnThreads * 4) {
    float v[4], w[4];
    get4<float>(sm + i, v, a.W - i, a.vec);
    if (a.w) {
      get4<float>(a.w + i, w, a.W - i, a.vec);
#pragma unroll
      for (int k = 0; k < 4; ++k) v[k] *= r * w[k];
    }
    put4<T>(h + i, v, a.W - i, a.vec);
  }
}

template <typename T, int SRC>
__global__ void __launch_bounds__(kPnThreads) prenorm_filter_kernel(const PrenormArgs a) {
  extern __shared__ __align__(16) float ring[];          // [taps][W]: in-step row r at slot r mod taps
  __shared__ float red[2][32];
  const int W = a.W, taps = a.taps, seq = blockIdx.y;
  const int q0 = a.q_cu[seq], n = a.q_cu[seq + 1] - q0;
  const int r0 = a.carry ? (n - (taps - 1) > 0 ? n - (taps - 1) : 0) : (int)blockIdx.x * a.chunk;
  if (r0 >= n) return;
  const int r1 = a.carry ? n : (r0 + a.chunk < n ? r0 + a.chunk : n);
  const int pos0 = a.positions[q0];
  float* st = a.state + (size_t)a.state_slots[seq] * (taps - 1) * W;
  // thread t owns channels [4 t, 4 t + 4) + 1024 k of every ring slot
  for (int r = r0 - (taps - 1); r < 0; ++r)
    for (int i = threadIdx.x * 4; i < W; i += kPnThreads * 4) {
      float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (pos0 + r >= 0) get4<float>(st + (size_t)(taps - 1 + r) * W + i, v, W - i, a.vec);
      put4<float>(ring + (size_t)((r + taps) % taps) * W + i, v, W - i, a.vec);
    }
  const int first = a.carry ? r0 : (r0 - (taps - 1) > 0 ? r0 - (taps - 1) : 0);
  for (int r = first; r < r1; ++r) {
    const bool own = r >= r0 && !a.carry;
    const size_t row = (size_t)q0 + r;
    float* cur = ring + (size_t)(r % taps) * W;
    if constexpr (SRC == SRC_PARTIALS) __syncthreads();  // other threads' channels of the slot are still being read
    const float ss = block_sum<kPnThreads>(residual_row<T, SRC>(a, cur, row, own && a.x_out), red[r & 1]);
    const float rr = 1.0f / sqrtf(ss / (float)W + a.eps);
    T* h = static_cast<T*>(a.h_out) + row * W;
    for (int i = threadIdx.x * 4; i < W; i += kPnThreads * 4) {
      float v[4], w[4];
      get4<float>(cur + i, v, W - i, a.vec);
      get4<float>(a.w + i, w, W - i, a.vec);
#pragma unroll
      for (int k = 0; k < 4; ++k) v[k] *= rr * w[k];
      put4<float>(cur + i, v, W - i, a.vec);
      if (own) {
        float acc[4], c[4];
        get4<float>(a.filt + (size_t)(taps - 1) * W + i, c, W - i, a.vec);
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[k] = c[k] * v[k];
        for (int lag = 1; lag < taps; ++lag) {
          float u[4];
          get4<float>(ring + (size_t)((r - lag + taps) % taps) * W + i, u, W - i, a.vec);
          get4<float>(a.filt + (size_t)(taps - 1 - lag) * W + i, c, W - i, a.vec);
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[k] += c[k] * u[k];
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] += acc[k];
        put4<T>(h + i, v, W - i, a.vec);
      }
    }
  }
  if (a.write_state)
    for (int e = 0; e < taps - 1; ++e) {
      const int r = n - (taps - 1) + e;
      for (int i = threadIdx.x * 4; i < W; i += kPnThreads * 4) {
        float v[4];
        get4<float>(ring + (size_t)((r + taps) % taps) * W + i, v, W - i, a.vec);
        put4<float>(st + (size_t)e * W + i, v, W - i, a.vec);
      }
    }
}

// The same for filters of at most TP taps on rows of whole 4-channel groups: the last TP - 1 normalised rows stay in
// registers (thread t owns groups t, t + threads, ...: NG of them), and R rows at a time are loaded and summed, so that
// their loads are in flight together and share a barrier.
template <typename T, int SRC, int TP, int NG, int R>
__global__ void __launch_bounds__(512) prenorm_walk_kernel(const PrenormArgs a) {
  __shared__ float red[2][R][16];
  const int W = a.W, taps = a.taps, seq = blockIdx.y, nt = blockDim.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = nt >> 5;
  const int q0 = a.q_cu[seq], n = a.q_cu[seq + 1] - q0;
  const int r0 = (int)blockIdx.x * a.chunk;
  if (r0 >= n) return;
  const int r1 = r0 + a.chunk < n ? r0 + a.chunk : n;
  const int pos0 = a.positions[q0];
  float* st = a.state + (size_t)a.state_slots[seq] * (taps - 1) * W;
  const int first = r0 - (taps - 1) > 0 ? r0 - (taps - 1) : 0;
  float win[TP - 1][NG][4];                              // rows r - (TP - 1) .. r - 1
#pragma unroll
  for (int j = 0; j < TP - 1; ++j) {
    const int r = first - (TP - 1) + j;                  // (rows of the step before `first` are not looked at)
    const int e = taps - 1 + r;                          // state entry of a row before the step
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      const int i = (threadIdx.x + g * nt) * 4;
      win[j][g][0] = win[j][g][1] = win[j][g][2] = win[j][g][3] = 0.0f;
      if (r < 0 && e >= 0 && pos0 + r >= 0 && i < W) load4<float>(st + (size_t)e * W + i, win[j][g]);
    }
  }
  int par = 0;
  for (int rb = first; rb < r1; rb += R, par ^= 1) {
    float v[R][NG][4], ss[R];
#pragma unroll
    for (int k = 0; k < R; ++k) {
      const size_t row = (size_t)q0 + rb + k;
#pragma unroll
      for (int g = 0; g < NG; ++g) {
        const int i = (threadIdx.x + g * nt) * 4;
        v[k][g][0] = v[k][g][1] = v[k][g][2] = v[k][g][3] = 0.0f;
        if (i < W && rb + k < r1) load4<float>(a.x_in + row * W + i, v[k][g]);
      }
    }
    if constexpr (SRC == SRC_ROWS) {
      float y[R][NG][4];
#pragma unroll
      for (int k = 0; k < R; ++k)
#pragma unroll
        for (int g = 0; g < NG; ++g) {
          const int i = (threadIdx.x + g * nt) * 4;
          y[k][g][0] = y[k][g][1] = y[k][g][2] = y[k][g][3] = 0.0f;
          if (i < W && rb + k < r1)
            load4<T>(static_cast<const T*>(a.y) + ((size_t)q0 + rb + k) * a.ldy + i, y[k][g]);
        }
#pragma unroll
      for (int k = 0; k < R; ++k)
#pragma unroll
        for (int g = 0; g < NG; ++g) {
          const int i = (threadIdx.x + g * nt) * 4;
#pragma unroll
          for (int c = 0; c < 4; ++c) v[k][g][c] += y[k][g][c];
          if (i < W && rb + k < r1 && rb + k >= r0) put4<float>(a.x_out + ((size_t)q0 + rb + k) * W + i, v[k][g], 4, true);
        }
    }
#pragma unroll
    for (int k = 0; k < R; ++k) {
      ss[k] = 0.0f;
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int c = 0; c < 4; ++c) ss[k] += v[k][g][c] * v[k][g][c];
      ss[k] = warp_sum(ss[k]);
      if (lane == 0) red[par][k][warp] = ss[k];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < R; ++k)
      ss[k] = 1.0f / sqrtf(warp_sum(lane < n_warps ? red[par][k][lane] : 0.0f) / (float)W + a.eps);
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      const int i = (threadIdx.x + g * nt) * 4;
      if (i >= W) continue;
      float w[4], co[TP][4];
      load4<float>(a.w + i, w);
#pragma unroll
      for (int j = 0; j < TP; ++j) {
        const int tap = j - (TP - taps);                 // negative: none
        co[j][0] = co[j][1] = co[j][2] = co[j][3] = 0.0f;
        if (tap >= 0) load4<float>(a.filt + (size_t)tap * W + i, co[j]);
      }
#pragma unroll
      for (int k = 0; k < R; ++k) {
        if (rb + k >= r1) break;
        float acc[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float nv = v[k][g][c] * (ss[k] * w[c]);
          acc[c] = nv + co[TP - 1][c] * nv;
#pragma unroll
          for (int j = 0; j < TP - 1; ++j) acc[c] += co[j][c] * win[j][g][c];
#pragma unroll
          for (int j = 0; j + 1 < TP - 1; ++j) win[j][g][c] = win[j + 1][g][c];
          win[TP - 2][g][c] = nv;
        }
        if (rb + k >= r0) put4<T>(static_cast<T*>(a.h_out) + ((size_t)q0 + rb + k) * W + i, acc, 4, true);
      }
    }
  }
  if (a.write_state) {
#pragma unroll
    for (int j = 0; j < TP - 1; ++j) {
      const int e = j - (TP - taps);
      if (e < 0) continue;
#pragma unroll
      for (int g = 0; g < NG; ++g) {
        const int i = (threadIdx.x + g * nt) * 4;
        if (i < W) put4<float>(st + (size_t)e * W + i, win[j][g], 4, true);
      }
    }
  }
}

template <typename T, int SRC>
int launch_prenorm(PrenormArgs& a, int64_t rows, int64_t n_seq, int64_t q_max, cudaStream_t st) {
  if (!a.filt) {
    const size_t smem = (size_t)(a.W + 4) * sizeof(float);
    auto kern = prenorm_kernel<T, SRC>;
    if (smem > 48 * 1024)
      B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<(unsigned)rows, kPnThreads, smem, st>>>(a);
    B200_LAUNCH_OK("prenorm_kernel");
    return B200_OK;
  }
  const size_t smem = (size_t)a.taps * a.W * sizeof(float);
  auto kern = prenorm_filter_kernel<T, SRC>;
  if (smem > 48 * 1024)
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  // long chunks redo fewer rows, short ones fill the SMs
  int chunk = rows >= 64 * sm_count() ? 29 : (rows >= 16 * sm_count() ? 13 : 5);
  if (q_max <= chunk) chunk = (int)q_max;
  const unsigned n_chunks = (unsigned)((q_max + chunk - 1) / chunk);
  a.chunk = chunk;
  a.carry = 0;
  a.write_state = a.taps > 1 && n_chunks == 1;
  bool walked = false;
  if constexpr (SRC != SRC_PARTIALS) {
    const int groups = a.W / 4;
    if (a.vec && a.taps <= 4 && groups <= 4 * 512) {
      const int ng = groups <= 256 ? 1 : (groups <= 1024 ? 2 : 4);
      const int threads = ((groups + ng - 1) / ng + 31) / 32 * 32;
      const dim3 grid(n_chunks, (unsigned)n_seq);
#define PN_WALK(TP)                                                                  \
  do {                                                                               \
    if (ng == 1) prenorm_walk_kernel<T, SRC, TP, 1, 4><<<grid, threads, 0, st>>>(a);     \
    else if (ng == 2) prenorm_walk_kernel<T, SRC, TP, 2, 2><<<grid, threads, 0, st>>>(a); \
    else prenorm_walk_kernel<T, SRC, TP, 4, 1><<<grid, threads, 0, st>>>(a);             \
  } while (0)
      if (a.taps <= 2) PN_WALK(2);
      else PN_WALK(4);
#undef PN_WALK
      walked = true;
    }
  }
  if (!walked) kern<<<dim3(n_chunks, (unsigned)n_seq), kPnThreads, smem, st>>>(a);
  B200_LAUNCH_OK("prenorm_filter_kernel");
  if (a.taps > 1 && n_chunks > 1) {
    // the last taps - 1 rows of every portion again, from the stored sums (the same numbers in the same order)
    if (a.x_out) a.x_in = a.x_out;
    a.carry = a.write_state = 1;
    auto kern2 = prenorm_filter_kernel<T, SRC_NONE>;
    if (smem > 48 * 1024)
      B200_CUDA_OK(cudaFuncSetAttribute(kern2, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern2<<<dim3(1, (unsigned)n_seq), kPnThreads, smem, st>>>(a);
    B200_LAUNCH_OK("prenorm_filter_kernel (state)");
  }
  return B200_OK;
}

template <typename T>
int dispatch_prenorm(PrenormArgs& a, int64_t rows, int64_t n_seq, int64_t q_max, cudaStream_t st) {
  if (a.partials) return launch_prenorm<T, SRC_PARTIALS>(a, rows, n_seq, q_max, st);
  if (a.y) return launch_prenorm<T, SRC_ROWS>(a, rows, n_seq, q_max, st);
  return launch_prenorm<T, SRC_NONE>(a, rows, n_seq, q_max, st);
}

// silu of an fp32 sum; where the result is rounded to 16 bits at once the fast exponential and division do
template <typename T>
__device__ __forceinline__ float silu_for(float x) {
  if constexpr (sizeof(T) == 4) return x / (1.0f + expf(-x));
  else return __fdividef(x, 1.0f + __expf(-x));
}

// ------------------------------------------------------------------------------------------------------------
// Plain short filter: one thread walks a chunk of rows for V neighbouring channels with the last TP - 1 inputs in
// registers (TP >= taps; the surplus taps are zero).
// ------------------------------------------------------------------------------------------------------------
constexpr int kFiThreads = 128;

template <typename T, int TP, int V>
__global__ void __launch_bounds__(kFiThreads)
causal_filter_kernel(T* __restrict__ out, int64_t ldo, const T* __restrict__ in, int64_t ld,
                     const float* __restrict__ filt, const float* __restrict__ in_bias, const float* __restrict__ bias,
                     float* __restrict__ state, const int* __restrict__ q_cu, const int* __restrict__ positions,
                     const int* __restrict__ state_slots, int C, int taps, int chunk, int silu, int write_state) {
  const int seq = blockIdx.z;
  const int q0 = q_cu[seq], n = q_cu[seq + 1] - q0;
  const int r0 = (int)blockIdx.x * chunk;
  if (r0 >= n) return;
  const int r1 = r0 + chunk < n ? r0 + chunk : n;
  const int c0 = ((int)blockIdx.y * kFiThreads + threadIdx.x) * V;
  if (c0 >= C) return;
  const int pos0 = positions[q0];
  float* st = state + (size_t)state_slots[seq] * (taps - 1) * C + c0;
  float win[TP][V], co[TP][V], b[V], ib[V];              // win[0]: the oldest
#pragma unroll
  for (int v = 0; v < V; ++v) ib[v] = in_bias ? in_bias[c0 + v] : 0.0f;
#pragma unroll
  for (int j = 0; j < TP; ++j) {
    const int tap = j - (TP - taps);                     // filter column; negative: none
#pragma unroll
    for (int v = 0; v < V; ++v) co[j][v] = tap >= 0 ? filt[(size_t)tap * C + c0 + v] : 0.0f;
    const int r = r0 - (TP - 1) + j;                     // the input that stands at place j when row r0 is made
#pragma unroll
    for (int v = 0; v < V; ++v) {
      win[j][v] = 0.0f;
      if (tap >= 0 && j < TP - 1 && pos0 + r >= 0)
        win[j][v] = r >= 0 ? Num<T>::to_f(in[(size_t)(q0 + r) * ld + c0 + v]) + ib[v] : st[(size_t)(taps - 1 + r) * C + v];
    }
  }
#pragma unroll
  for (int v = 0; v < V; ++v) b[v] = bias ? bias[c0 + v] : 0.0f;
#pragma unroll 4
  for (int r = r0; r < r1; ++r) {
    float o[V];
    if constexpr (V == 4) {
      float x[4];
      load4<T>(in + (size_t)(q0 + r) * ld + c0, x);
#pragma unroll
      for (int v = 0; v < 4; ++v) win[TP - 1][v] = x[v] + ib[v];
    } else {
      win[TP - 1][0] = Num<T>::to_f(in[(size_t)(q0 + r) * ld + c0]) + ib[0];
    }
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float acc = b[v];
#pragma unroll
      for (int j = 0; j < TP; ++j) acc += co[j][v] * win[j][v];
      o[v] = silu ? silu_for<T>(acc) : acc;
#pragma unroll
      for (int j = 0; j + 1 < TP; ++j) win[j][v] = win[j + 1][v];
    }
    T* dst = out + (size_t)(q0 + r) * ldo + c0;
    if constexpr (V == 4) {
      put4<T>(dst, o, 4, true);
    } else {
      dst[0] = Num<T>::from_f(o[0]);
    }
  }
  if (write_state) {
    // the window has moved past the last row: places TP - taps .. TP - 2 hold the last taps - 1 inputs
#pragma unroll
    for (int j = 0; j < TP - 1; ++j) {
      const int e = j - (TP - taps);
      if (e >= 0)
#pragma unroll
        for (int v = 0; v < V; ++v) st[(size_t)e * C + v] = win[j][v];
    }
  }
}

// state[slot, e] <- the input at in-step row n - (taps - 1) + e, or the old entry e + n where that is before the step
template <typename T>
__global__ void causal_filter_carry_kernel(float* __restrict__ state, const T* __restrict__ in, int64_t ld,
                                           const float* __restrict__ in_bias,
                                           const int* __restrict__ q_cu, const int* __restrict__ positions,
                                           const int* __restrict__ state_slots, int C, int taps) {
  const int seq = blockIdx.y;
  const int q0 = q_cu[seq], n = q_cu[seq + 1] - q0;
  if (n <= 0) return;
  const int pos0 = positions[q0];
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  float* st = state + (size_t)state_slots[seq] * (taps - 1) * C + c;
  for (int e = 0; e < taps - 1; ++e) {                   // ascending: entry e reads entry e + n > e of the old state
    const int r = n - (taps - 1) + e;
    float v = 0.0f;
    if (r >= 0) v = Num<T>::to_f(in[(size_t)(q0 + r) * ld + c]) + (in_bias ? in_bias[c] : 0.0f);
    else if (pos0 + r >= 0) v = st[(size_t)(e + n) * C];
    st[(size_t)e * C] = v;
  }
}

template <typename T, int TP, int V>
int launch_filter(void* out, int64_t ldo, const void* in, int64_t ld, const float* filt, const float* in_bias,
                  const float* bias, float* state, const int* q_cu, const int* positions, const int* slots, int64_t rows, int64_t n_seq,
                  int64_t q_max, int C, int taps, int silu, cudaStream_t st) {
  const unsigned cy = (unsigned)((C + kFiThreads * V - 1) / (kFiThreads * V));
  int chunk = rows * cy >= 64 * sm_count() * 4 ? 32 : 8;
  if (q_max <= chunk) chunk = (int)q_max;
  const unsigned n_chunks = (unsigned)((q_max + chunk - 1) / chunk);
  causal_filter_kernel<T, TP, V><<<dim3(n_chunks, cy, (unsigned)n_seq), kFiThreads, 0, st>>>(
      static_cast<T*>(out), ldo, static_cast<const T*>(in), ld, filt, in_bias, bias, state, q_cu, positions, slots, C, taps, chunk,
      silu, taps > 1 && n_chunks == 1);
  B200_LAUNCH_OK("causal_filter_kernel");
  if (taps > 1 && n_chunks > 1) {
    causal_filter_carry_kernel<T><<<dim3((unsigned)((C + 255) / 256), (unsigned)n_seq), 256, 0, st>>>(
        state, static_cast<const T*>(in), ld, in_bias, q_cu, positions, slots, C, taps);
    B200_LAUNCH_OK("causal_filter_carry_kernel");
  }
  return B200_OK;
}

}  // namespace
}  // namespace b200

using namespace b200;

#define FILTERS_DISPATCH(dtype, ...)                                             \
  switch (dtype) {                                                               \
    case B200_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }             \
    case B200_FP16: { using T = __half; __VA_ARGS__; break; }                    \
    case B200_FP32: { using T = float; __VA_ARGS__; break; }                     \
    default: return set_error(B200_ERR_INVALID_ARG, "bad dtype %d", dtype);      \
  }

extern "C" {

int b200_prenorm(float* x_out, void* h_out, int64_t ldh, const float* x_in, const void* y, int64_t ldy, const float* partials,
                 int64_t n_slots, const int32_t* plan6, const float* weight, const float* filter, int64_t taps,
                 float* filter_state, const int32_t* q_cu_lens, const int32_t* positions, const int32_t* state_slots,
                 int64_t n_seq, int64_t q_max, int64_t rows, int64_t W, float eps, int dtype, b200_stream_t stream) {
  if (rows == 0) return B200_OK;
  B200_CHECK_ARG(h_out && x_in && (weight || !filter), "prenorm: null pointer");
  B200_CHECK_ARG(rows > 0 && W > 0 && !(y && partials) && (!y || ldy >= W || (ldy == 0 && !filter)) &&
                     (filter ? ldh == W : ldh >= W) && (W + 4) * 4 <= 200 * 1024,
                 "prenorm: bad shape (at most ~50K channels), or rows and partials both given");
  B200_CHECK_ARG(!(y || partials) || (x_out && x_out != x_in), "prenorm: the sum goes to a buffer of its own");
  B200_CHECK_ARG(!partials || (plan6 && W % 8 == 0 && n_slots == plan6[4] && n_slots <= W4_MAX_SLOTS &&
                               is_aligned(partials, 16)),
                 "prenorm: the partials are not those of the given partition");
  B200_CHECK_ARG(!filter || (taps >= 1 && taps <= kMaxTaps && taps * W * 4 <= 200 * 1024 &&
                             (taps == 1 || filter_state) && q_cu_lens && positions && state_slots && n_seq > 0 &&
                             n_seq <= 65535 && q_max > 0),
                 "prenorm: bad filter (1 to 16 taps, taps * channels at most ~50K)");
  PrenormArgs a{};
  a.x_out = (y || partials) ? x_out : nullptr;
  a.h_out = h_out; a.ldh = ldh; a.x_in = x_in; a.y = y; a.ldy = ldy; a.partials = partials; a.slot_stride = rows * W;
  if (plan6 && partials) {
    a.plan.units = plan6[0]; a.plan.P = plan6[1]; a.plan.KT = plan6[2]; a.plan.NT = plan6[3]; a.plan.slots = plan6[4];
    a.plan.nsub_log2 = plan6[5];
  }
  a.w = weight; a.filt = filter; a.state = filter_state; a.q_cu = q_cu_lens; a.positions = positions;
  a.state_slots = state_slots; a.W = (int)W; a.taps = (int)taps; a.eps = eps;
  a.vec = W % 4 == 0 && is_aligned(x_in, 16) && (!a.x_out || is_aligned(x_out, 16)) && is_aligned(h_out, 16) &&
          ldh % 4 == 0 && (!y || (ldy % 4 == 0 && is_aligned(y, 16))) && (!weight || is_aligned(weight, 16)) &&
          (!filter || (is_aligned(filter, 16) && (taps == 1 || is_aligned(filter_state, 16))));
  auto st = static_cast<cudaStream_t>(stream);
  FILTERS_DISPATCH(dtype, return dispatch_prenorm<T>(a, rows, n_seq, q_max, st));
  return B200_OK;
}

int b200_causal_filter(void* out, int64_t ldo, const void* in, int64_t ld, const float* filter,
                       const float* in_bias, const float* bias, int64_t taps, float* filter_state, const int32_t* q_cu_lens, const int32_t* positions,
                       const int32_t* state_slots, int64_t n_seq, int64_t q_max, int64_t rows, int64_t channels, int silu,
                       int dtype, b200_stream_t stream) {
  if (rows == 0 || n_seq == 0) return B200_OK;
  B200_CHECK_ARG(out && in && filter && (taps == 1 || filter_state) && q_cu_lens && positions && state_slots,
                 "causal_filter: null pointer");
  B200_CHECK_ARG(rows > 0 && n_seq > 0 && n_seq <= 65535 && q_max > 0 && channels > 0 && channels < (1ll << 30) &&
                     taps >= 1 && taps <= kMaxTaps && ld >= channels && ldo >= channels && out != in,
                 "causal_filter: bad shape (1 to 16 taps)");
  auto st = static_cast<cudaStream_t>(stream);
  const size_t esz = dtype == B200_FP32 ? 4 : 2;
  const bool vec = channels % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && is_aligned(in, 4 * esz) && is_aligned(out, 4 * esz);
#define CF_CALL(TP, V)                                                                                          \
  return (launch_filter<T, TP, V>(out, ldo, in, ld, filter, in_bias, bias, filter_state, q_cu_lens, positions, state_slots, \
                                  rows, n_seq, q_max, (int)channels, (int)taps, silu, st))
  FILTERS_DISPATCH(dtype, {
    if (vec) {
      if (taps <= 2) CF_CALL(2, 4);
      if (taps <= 4) CF_CALL(4, 4);
      if (taps <= 8) CF_CALL(8, 4);
    }
    if (taps <= 2) CF_CALL(2, 1);
    if (taps <= 4) CF_CALL(4, 1);
    if (taps <= 8) CF_CALL(8, 1);
    CF_CALL(16, 1);
  });
#undef CF_CALL
  return B200_OK;
}

}  // extern "C"
