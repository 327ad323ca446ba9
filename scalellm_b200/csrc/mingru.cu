// mingru.cu — gated linear recurrences with one state value per channel whose decay and input depend on the current
// token only:  S_t = a_t S_{t-1} + b_t (fp32), out_t = S_t * g_t.
//
//   minimal gated unit : z = sigmoid(pz + bz) ; u = px + bx ; c = u + 1/2 (u >= 0) | sigmoid(u) (u < 0) ;
//                        a = 1 - z, b = z c ; g = silu(pg)           pz | px | pg: column blocks [width] of one matrix
//   real-gated unit    : r = sigmoid(pr + br), i = sigmoid(pi + bi) ; log a = rate r softplus(lam) ;
//                        b = sqrt(1 - a^2) i u ; g = gelu_tanh(py + by)
//                        pr, pi: fp32 [blocks][rows][2 n] as a block-diagonal product leaves them (n = width / blocks)
//
// The state of a sequence lives in its state slot [n_slots, width]; a portion whose first row has position 0 starts
// from 0.  One thread per (sequence, channel) walks the step's tokens of that sequence in order; the inputs of the
// following tokens are loaded ahead, since nothing of them depends on the recurrence.
// Long portions are cut into chunks of `chunk_len` tokens that run side by side: a first kernel reduces every chunk to
// (A, B) with S_end = A S_start + B, and a second one starts every chunk from the fold of the chunks before it.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kAhead = 4;

template <typename T>
struct MinGruCell {
  const T* proj;
  int64_t ld;
  const float *z_bias, *x_bias;
  int width;

  struct Channel { int c; float bz, bx; };
  struct In { float z, x; };
  __device__ __forceinline__ Channel channel(int c) const {
    return {c, z_bias ? z_bias[c] : 0.0f, x_bias ? x_bias[c] : 0.0f};
  }
  __device__ __forceinline__ In load(int t, const Channel& ch) const {
    const T* p = proj + (size_t)t * ld + ch.c;
    return {Num<T>::to_f(p[0]), Num<T>::to_f(p[width])};
  }
  __device__ __forceinline__ float load_gate(int t, const Channel& ch) const {
    return Num<T>::to_f(proj[(size_t)t * ld + ch.c + 2 * (size_t)width]);
  }
  __device__ __forceinline__ void coef(const In& in, const Channel& ch, float& a, float& b) const {
    const float z = 1.0f / (1.0f + expf(-(in.z + ch.bz)));
    const float u = in.x + ch.bx;
    const float cand = u >= 0.0f ? u + 0.5f : 1.0f / (1.0f + expf(-u));
    a = 1.0f - z;
    b = z * cand;
  }
  __device__ __forceinline__ float gate(float g, const Channel&) const { return g / (1.0f + expf(-g)); }
};

template <typename T>
struct RealGatedCell {
  const T *u, *y;
  int64_t ld_u, ld_y;
  const float* gates;      // [blocks][rows][2 n]: r then i
  int64_t rows;
  const float *r_bias, *i_bias, *lam, *y_bias;
  float rate;
  int n;                   // channels of a block

  struct Channel { int c; const float* g; float br, bi, k, by; };
  struct In { float u, r, i; };
  __device__ __forceinline__ Channel channel(int c) const {
    const float l = lam[c];
    return {c, gates + (size_t)(c / n) * rows * 2 * n + c % n, r_bias[c], i_bias[c],
            rate * (fmaxf(l, 0.0f) + log1pf(expf(-fabsf(l)))), y_bias ? y_bias[c] : 0.0f};
  }
  __device__ __forceinline__ In load(int t, const Channel& ch) const {
    const float* g = ch.g + (size_t)t * 2 * n;
    return {Num<T>::to_f(u[(size_t)t * ld_u + ch.c]), g[0], g[n]};
  }
  __device__ __forceinline__ float load_gate(int t, const Channel& ch) const {
    return Num<T>::to_f(y[(size_t)t * ld_y + ch.c]);
  }
  __device__ __forceinline__ void coef(const In& in, const Channel& ch, float& a, float& b) const {
    const float r = 1.0f / (1.0f + expf(-(in.r + ch.br))), i = 1.0f / (1.0f + expf(-(in.i + ch.bi)));
    const float log_a = ch.k * r;
    a = expf(log_a);
    b = sqrtf(-expm1f(2.0f * log_a)) * i * in.u;         // 1 - a^2 without cancellation
  }
  __device__ __forceinline__ float gate(float p, const Channel& ch) const {
    const float z = p + ch.by;
    return 0.5f * z * (1.0f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
  }
};

template <typename T, typename Cell>
__global__ void __launch_bounds__(128)
channel_scan_kernel(T* __restrict__ out, int64_t ldo, const Cell cell, float* __restrict__ state,
                    const int* __restrict__ q_cu, const int* __restrict__ positions,
                    const int* __restrict__ state_slots, int width) {
  const int seq = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int t0 = q_cu[seq], t1 = q_cu[seq + 1];
  if (c >= width || t0 >= t1) return;
  float* slot = state + (size_t)state_slots[seq] * width + c;
  float S = positions[t0] == 0 ? 0.0f : *slot;
  const typename Cell::Channel ch = cell.channel(c);
  typename Cell::In ahead[kAhead];
  float ahead_g[kAhead];
  auto load = [&](int t, int k) {
    ahead[k] = cell.load(t, ch);
    ahead_g[k] = cell.load_gate(t, ch);
  };
#pragma unroll
  for (int k = 0; k < kAhead; ++k)
    if (t0 + k < t1) load(t0 + k, k);
  for (int t = t0; t < t1; t += kAhead) {
    typename Cell::In now[kAhead];
    float now_g[kAhead];
#pragma unroll
    for (int k = 0; k < kAhead; ++k) { now[k] = ahead[k]; now_g[k] = ahead_g[k]; }
#pragma unroll
    for (int k = 0; k < kAhead; ++k)
      if (t + kAhead + k < t1) load(t + kAhead + k, k);
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      if (t + k < t1) {
        float a, b;
        cell.coef(now[k], ch, a, b);
        S = a * S + b;
        out[(size_t)(t + k) * ldo + c] = Num<T>::from_f(S * cell.gate(now_g[k], ch));
      }
    }
  }
  *slot = S;
}

// (A, B) of every chunk, and the state every sequence starts from (its slot, or 0 at position 0)
template <typename Cell>
__global__ void __launch_bounds__(128)
channel_chunk_summary_kernel(float* __restrict__ A_ws, float* __restrict__ B_ws, float* __restrict__ S0_ws,
                             const Cell cell, const float* __restrict__ state, const int* __restrict__ q_cu,
                             const int* __restrict__ positions, const int* __restrict__ state_slots, int width,
                             int chunk_len, int n_chunks) {
  const int seq = blockIdx.x, chunk = blockIdx.y;
  const int c = blockIdx.z * blockDim.x + threadIdx.x;
  const int q0 = q_cu[seq], q1 = q_cu[seq + 1];
  const int t0 = q0 + chunk * chunk_len;
  if (c >= width || t0 >= q1) return;
  const int t1 = t0 + chunk_len < q1 ? t0 + chunk_len : q1;
  if (chunk == 0)
    S0_ws[(size_t)seq * width + c] = positions[q0] == 0 ? 0.0f : state[(size_t)state_slots[seq] * width + c];
  if (t1 == q1) return;                       // nothing follows the portion's last chunk
  const typename Cell::Channel ch = cell.channel(c);
  float A = 1.0f, B = 0.0f;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float a, b;
    cell.coef(cell.load(t, ch), ch, a, b);
    A *= a;
    B = a * B + b;
  }
  const size_t o = ((size_t)seq * n_chunks + chunk) * width + c;
  A_ws[o] = A;
  B_ws[o] = B;
}

template <typename T, typename Cell>
__global__ void __launch_bounds__(128)
channel_chunk_apply_kernel(T* __restrict__ out, int64_t ldo, const Cell cell, float* __restrict__ state,
                           const float* __restrict__ A_ws, const float* __restrict__ B_ws,
                           const float* __restrict__ S0_ws, const int* __restrict__ q_cu,
                           const int* __restrict__ state_slots, int width, int chunk_len, int n_chunks) {
  const int seq = blockIdx.x, chunk = blockIdx.y;
  const int c = blockIdx.z * blockDim.x + threadIdx.x;
  const int q0 = q_cu[seq], q1 = q_cu[seq + 1];
  const int t0 = q0 + chunk * chunk_len;
  if (c >= width || t0 >= q1) return;
  const int t1 = t0 + chunk_len < q1 ? t0 + chunk_len : q1;
  float S = S0_ws[(size_t)seq * width + c];
  for (int k = 0; k < chunk; ++k) {
    const size_t o = ((size_t)seq * n_chunks + k) * width + c;
    S = A_ws[o] * S + B_ws[o];
  }
  const typename Cell::Channel ch = cell.channel(c);
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float a, b;
    cell.coef(cell.load(t, ch), ch, a, b);
    const float g = cell.load_gate(t, ch);
    S = a * S + b;
    out[(size_t)t * ldo + c] = Num<T>::from_f(S * cell.gate(g, ch));
  }
  if (t1 == q1) state[(size_t)state_slots[seq] * width + c] = S;
}

template <typename T, typename Cell>
int launch_scan(T* out, int64_t ldo, const Cell& cell, float* state, const int* q_cu, const int* positions,
                const int* slots, int64_t n_seq, int64_t width, cudaStream_t st) {
  dim3 grid((unsigned)n_seq, (unsigned)((width + 127) / 128));
  channel_scan_kernel<T, Cell><<<grid, 128, 0, st>>>(out, ldo, cell, state, q_cu, positions, slots, (int)width);
  B200_LAUNCH_OK("channel_scan_kernel");
  return B200_OK;
}

template <typename T, typename Cell>
int launch_chunked(T* out, int64_t ldo, const Cell& cell, float* state, const int* q_cu, const int* positions,
                   const int* slots, int64_t n_seq, int64_t width, int64_t q_max, int64_t chunk_len, float* ws,
                   int64_t ws_floats, cudaStream_t st) {
  B200_CHECK_ARG(q_max > 0 && chunk_len > 0 && ws, "channel scan: chunks without a length or a workspace");
  const int64_t n_chunks = (q_max + chunk_len - 1) / chunk_len;
  B200_CHECK_ARG(n_chunks <= 65535 && (width + 127) / 128 <= 65535 &&
                     ws_floats >= b200_mingru_chunked_workspace_floats(n_seq, width, q_max, chunk_len),
                 "channel scan: too many chunks or a workspace too small");
  float* A_ws = ws;
  float* B_ws = A_ws + n_seq * n_chunks * width;
  float* S0_ws = B_ws + n_seq * n_chunks * width;
  dim3 grid((unsigned)n_seq, (unsigned)n_chunks, (unsigned)((width + 127) / 128));
  channel_chunk_summary_kernel<Cell><<<grid, 128, 0, st>>>(A_ws, B_ws, S0_ws, cell, state, q_cu, positions, slots,
                                                           (int)width, (int)chunk_len, (int)n_chunks);
  B200_LAUNCH_OK("channel_chunk_summary_kernel");
  channel_chunk_apply_kernel<T, Cell><<<grid, 128, 0, st>>>(out, ldo, cell, state, A_ws, B_ws, S0_ws, q_cu, slots,
                                                            (int)width, (int)chunk_len, (int)n_chunks);
  B200_LAUNCH_OK("channel_chunk_apply_kernel");
  return B200_OK;
}

}  // namespace
}  // namespace b200

using namespace b200;

#define CHANNEL_DISPATCH(dtype, ...)                                             \
  switch (dtype) {                                                               \
    case B200_BF16: { using T = __nv_bfloat16; __VA_ARGS__; }                    \
    case B200_FP16: { using T = __half; __VA_ARGS__; }                           \
    case B200_FP32: { using T = float; __VA_ARGS__; }                            \
    default: return set_error(B200_ERR_INVALID_ARG, "bad dtype %d", dtype);      \
  }

extern "C" {

int b200_mingru_scan(void* out, int64_t ldo, const void* proj, int64_t ld, const float* z_bias,
                     const float* x_bias, float* state, const int32_t* q_cu_lens, const int32_t* positions,
                     const int32_t* state_slots, int64_t n_seq, int64_t width, int dtype, b200_stream_t stream) {
  if (n_seq == 0) return B200_OK;
  B200_CHECK_ARG(out && proj && state && q_cu_lens && positions && state_slots, "mingru_scan: null pointer");
  B200_CHECK_ARG(n_seq > 0 && width > 0 && width < (1ll << 23) && ldo >= width && ld >= 3 * width,
                 "mingru_scan: bad shape");
  auto st = static_cast<cudaStream_t>(stream);
  CHANNEL_DISPATCH(dtype, return (launch_scan<T>(
      static_cast<T*>(out), ldo, MinGruCell<T>{static_cast<const T*>(proj), ld, z_bias, x_bias, (int)width}, state,
      q_cu_lens, positions, state_slots, n_seq, width, st)));
}

int64_t b200_mingru_chunked_workspace_floats(int64_t n_seq, int64_t width, int64_t q_max, int64_t chunk_len) {
  if (n_seq <= 0 || width <= 0 || q_max <= 0 || chunk_len <= 0) return 0;
  const int64_t n_chunks = (q_max + chunk_len - 1) / chunk_len;
  return n_seq * (2 * n_chunks + 1) * width;
}

int b200_mingru_scan_chunked(void* out, int64_t ldo, const void* proj, int64_t ld, const float* z_bias,
                             const float* x_bias, float* state, const int32_t* q_cu_lens, const int32_t* positions,
                             const int32_t* state_slots, int64_t n_seq, int64_t width, int64_t q_max,
                             int64_t chunk_len, float* workspace, int64_t workspace_floats, int dtype,
                             b200_stream_t stream) {
  if (n_seq == 0 || q_max == 0) return B200_OK;
  B200_CHECK_ARG(out && proj && state && q_cu_lens && positions && state_slots && workspace,
                 "mingru_scan_chunked: null pointer");
  B200_CHECK_ARG(n_seq > 0 && width > 0 && width < (1ll << 23) && ldo >= width && ld >= 3 * width,
                 "mingru_scan_chunked: bad shape");
  auto st = static_cast<cudaStream_t>(stream);
  CHANNEL_DISPATCH(dtype, return (launch_chunked<T>(
      static_cast<T*>(out), ldo, MinGruCell<T>{static_cast<const T*>(proj), ld, z_bias, x_bias, (int)width}, state,
      q_cu_lens, positions, state_slots, n_seq, width, q_max, chunk_len, workspace, workspace_floats, st)));
}

int b200_real_gated_scan(void* out, int64_t ldo, const void* u, int64_t ld_u, const void* y, int64_t ld_y,
                         const float* gates, int64_t rows, int64_t blocks, const float* r_bias, const float* i_bias,
                         const float* lam, const float* y_bias, float rate, float* state, const int32_t* q_cu_lens,
                         const int32_t* positions, const int32_t* state_slots, int64_t n_seq, int64_t width,
                         int64_t q_max, int64_t chunk_len, float* workspace, int64_t workspace_floats, int dtype,
                         b200_stream_t stream) {
  if (n_seq == 0 || rows == 0) return B200_OK;
  B200_CHECK_ARG(out && u && y && gates && r_bias && i_bias && lam && state && q_cu_lens && positions && state_slots,
                 "real_gated_scan: null pointer");
  B200_CHECK_ARG(n_seq > 0 && rows > 0 && width > 0 && width < (1ll << 23) && blocks > 0 && width % blocks == 0 &&
                     ldo >= width && ld_u >= width && ld_y >= width && chunk_len >= 0,
                 "real_gated_scan: bad shape (the width in equal blocks)");
  auto st = static_cast<cudaStream_t>(stream);
  CHANNEL_DISPATCH(dtype, {
    const RealGatedCell<T> cell{static_cast<const T*>(u), static_cast<const T*>(y), ld_u, ld_y, gates, rows, r_bias,
                                i_bias, lam, y_bias, rate, (int)(width / blocks)};
    if (chunk_len > 0)
      return (launch_chunked<T>(static_cast<T*>(out), ldo, cell, state, q_cu_lens, positions, state_slots, n_seq, width,
                                q_max, chunk_len, workspace, workspace_floats, st));
    return (launch_scan<T>(static_cast<T*>(out), ldo, cell, state, q_cu_lens, positions, state_slots, n_seq, width, st));
  });
}

}  // extern "C"
