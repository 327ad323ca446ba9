// linear_scan.cu — linear recurrences with a matrix state per head whose decay does not look at the state.
//
//     S_t = diag(a_t) S_{t-1} + k_t v_t^T ,   o_t = S_t^T q_t           S [N (key) x V (value)], fp32, per head
//
//   forget : a = f, k = 1 - f, f = low + (1 - low) sigmoid(fl + b) per head and key channel, q = silu(ql);
//            out = mul * o / sqrt(mean_head(o^2) + eps) * w                              (what is forgotten is written)
//   ssd    : a = exp(-exp(A_h) d) for the whole head, k = d B, q = C (one B, C per group of heads),
//            d = softplus(dl + bias_h);  y = o + D_h v                                   (state-space duality form)
//   memory : f = log sigmoid(cap tanh((fl + bf_h) / cap)), i = cap tanh((il + bi_h) / cap), m' = max(f + m, i) from m = 0 ;
//            a = exp(f + m - m'), k = exp(i - m') kl, q = c ql ; a sum of keys n <- a n + k goes along ;
//            y = o / (max(|n . q|, exp(-m')) + 1e-6)                                     (matrix memory with exponential gates)
//
// The elements of S do not meet except in o's sum over the key channels, so a thread keeps a tile of RL key rows x 4
// value columns in registers (packed pairs of key rows: two multiply-adds an instruction) and LP neighbouring lanes
// share a column group; a warp walks 128 / LP columns.  One CTA per (sequence, head[, column part]); up to 16 tokens
// at a time are turned into fp32 decay / key / query rows in shared memory by all threads (so no transcendental sits
// in the walk), then the walk runs with no barrier, its read-outs collected in shared memory for the norm.
// A portion that starts at position 0 starts from S = 0 instead of reading the slot.
//
//   part_norm : out = u / sqrt(mean_part(u^2) + eps) * w, u = y silu(z), the row in equal parts    (after the ssd walk)
//               or u = y and sigmoid(z) on the way out                                             (after the memory walk)
#include <type_traits>

#include "common.cuh"

namespace b200 {
namespace {

constexpr int kScanTokens = 16;
constexpr int kScanWarps = 8;

constexpr float kMemoryDenEps = 1e-6f;

enum { MODE_FORGET = 0, MODE_SSD = 1, MODE_MEMORY = 2 };

// Column parts a head is walked in (the walk on CUDA cores).
__host__ __device__ constexpr int scan_col_parts(int N, int V) {
  const int lp = N <= 128 ? 4 : (N <= 256 ? 8 : 16);
  const int warps = (V + 128 / lp - 1) / (128 / lp);
  return (warps + kScanWarps - 1) / kScanWarps;
}
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.0f) - log1pf(expf(-fabsf(x))); }

template <typename T>
struct ScanArgs {
  T* out;                  // forget: rows of stride ldo (when the CTA holds the whole head)
  int64_t ldo;
  float* raw;              // fp32 [rows, H * V]: read-outs before the norm (forget in column parts), or y (ssd)
  const T *q, *k, *v;      // forget: query, forget and value logits; ssd: C, B, x
  int64_t ld;
  const float *f_bias, *f_low, *norm_w;
  const T* dt;
  int64_t ld_dt;
  const float *dt_bias, *a_log, *skip;
  const float *gi, *gf;    // memory: gate logits, fp32 rows of stride ld_g; one bias per head each
  int64_t ld_g;
  const float *gi_bias, *gf_bias;
  float cap, q_scale;
  float* key_sum;          // memory: [slot][H][column part][N + 1]: n, then m (one copy per column part of the walk)
  float* state;            // [slot][H][N][V]
  const int *q_cu, *positions, *state_slots;
  int H, G, N, V, CB, chunk;
  float eps, mul;
  int vec_in, vec_state;
};

template <typename T>
__device__ __forceinline__ void get4c(const T* __restrict__ p, float (&v)[4], int n, bool vec) {
  if (vec) {
    load4<T>(p, v);
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = i < n ? Num<T>::to_f(p[i]) : 0.0f;
  }
}

template <typename T, int MODE, int RL, int LP>
__global__ void __launch_bounds__(kScanWarps * 32)
linear_scan_kernel(const ScanArgs<T> a) {
  constexpr int NP = RL * LP;                             // key rows, padded
  extern __shared__ __align__(16) float sm[];
  const int CH = a.chunk, CBP = (int)(blockDim.x >> 5) * (128 / LP);
  float* k_s = sm;                                        // [CH][NP]
  float* q_s = k_s + CH * NP;                             // [CH][NP]
  float* a_s = q_s + CH * NP;                             // forget: [CH][NP]; ssd: [CH]; memory: log gates f, i [2][CH4]
  const int CH4 = (CH + 3) / 4 * 4;
  float* v_s = a_s + (MODE == MODE_FORGET ? CH * NP : (MODE == MODE_MEMORY ? 2 * CH4 : CH4));   // [CH][CBP]
  float* o_s = v_s + CH * CBP;                            // [CH][CBP]
  const int seq = blockIdx.x, h = blockIdx.y, cb0 = (int)blockIdx.z * a.CB;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int t0 = a.q_cu[seq], t1 = a.q_cu[seq + 1];
  if (t0 >= t1) return;
  const int N = a.N, V = a.V;
  const int ncol = V - cb0 < a.CB ? V - cb0 : a.CB;
  const int p = lane % LP, cq = warp * (32 / LP) + lane / LP;
  const int c0 = cq * 4;                                  // this thread's columns c0 .. c0 + 3 of the part
  float* Sg = a.state + (((size_t)a.state_slots[seq] * a.H + h) * N) * V + cb0;
  const bool fresh = a.positions[t0] == 0;
  // the state is asked for first and made into pairs of key rows only after the first tokens are staged, so that its
  // latency and theirs overlap (a decoded token's step is little else)
  float raw[RL][4];
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int n = p * 4 + (i / 4) * 4 * LP + (i & 3);
    raw[i][0] = raw[i][1] = raw[i][2] = raw[i][3] = 0.0f;
    if (!fresh && c0 < ncol && n < N) get4c<float>(Sg + (size_t)n * V + c0, raw[i], ncol - c0, a.vec_state);
  }
  float* key_sum = nullptr;
  float m = 0.0f;
  float raw_n[MODE == MODE_MEMORY ? RL : 1];
  if constexpr (MODE == MODE_MEMORY) {
    key_sum = a.key_sum + (((size_t)a.state_slots[seq] * a.H + h) * gridDim.z + blockIdx.z) * (N + 1);
    if (!fresh) m = key_sum[N];
#pragma unroll
    for (int i = 0; i < RL; ++i) {
      const int n = p * 4 + (i / 4) * 4 * LP + (i & 3);
      raw_n[i] = !fresh && n < N ? key_sum[n] : 0.0f;
    }
  }
  const int g = MODE == MODE_SSD ? h / (a.H / a.G) : h;
  float neg_a = 0.0f, dbias = 0.0f, skip = 0.0f;
  if constexpr (MODE == MODE_SSD) {
    neg_a = -expf(a.a_log[h]);
    dbias = a.dt_bias[h];
    skip = a.skip[h];
  }
  auto stage = [&](int tc, int nt) {
    for (int tok = warp; tok < nt; tok += n_warps) {
      const size_t row = (size_t)(tc + tok);
      const T* qr = a.q + row * a.ld + (size_t)g * N;
      const T* kr = a.k + row * a.ld + (size_t)g * N;
      float dt = 0.0f;
      if constexpr (MODE == MODE_SSD) {
        dt = softplus_f(Num<T>::to_f(a.dt[row * a.ld_dt + h]) + dbias);
        if (lane == 0) a_s[tok] = expf(neg_a * dt);
      }
      if constexpr (MODE == MODE_MEMORY) {
        if (lane < 2) {
          const float z = lane == 0 ? a.gf[row * a.ld_g + h] + a.gf_bias[h] : a.gi[row * a.ld_g + h] + a.gi_bias[h];
          const float t = a.cap * tanhf(z / a.cap);
          a_s[lane * CH4 + tok] = lane == 0 ? log_sigmoid_f(t) : t;
        }
      }
      for (int c = lane * 4; c < NP; c += 128) {
        float qv[4] = {0.0f, 0.0f, 0.0f, 0.0f}, kv[4] = {0.0f, 0.0f, 0.0f, 0.0f}, av[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        if (c < N) {
          get4c<T>(qr + c, qv, N - c, a.vec_in);
          get4c<T>(kr + c, kv, N - c, a.vec_in);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if constexpr (MODE == MODE_FORGET) {
              if (c + i < N) {
                const float l = a.f_low[h * N + c + i];
                const float z = kv[i] + a.f_bias[h * N + c + i];
                const float e = expf(-fabsf(z));          // sigmoid(z) and sigmoid(-z) without cancellation
                const float big = 1.0f / (1.0f + e), small = e * big;
                av[i] = l + (1.0f - l) * (z >= 0.0f ? big : small);
                kv[i] = (1.0f - l) * (z >= 0.0f ? small : big);
                qv[i] = qv[i] * sigmoid_f(qv[i]);
              }
            } else if constexpr (MODE == MODE_SSD) {
              kv[i] *= dt;
            }
          }
        }
        *reinterpret_cast<float4*>(k_s + tok * NP + c) = make_float4(kv[0], kv[1], kv[2], kv[3]);
        *reinterpret_cast<float4*>(q_s + tok * NP + c) = make_float4(qv[0], qv[1], qv[2], qv[3]);
        if constexpr (MODE == MODE_FORGET)
          *reinterpret_cast<float4*>(a_s + tok * NP + c) = make_float4(av[0], av[1], av[2], av[3]);
      }
      const T* vr = a.v + row * a.ld + (size_t)h * V + cb0;
      for (int c = lane * 4; c < CBP; c += 128) {
        float vv[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        if (c < ncol) get4c<T>(vr + c, vv, ncol - c, a.vec_in);
        *reinterpret_cast<float4*>(v_s + tok * CBP + c) = make_float4(vv[0], vv[1], vv[2], vv[3]);
      }
    }
  };
  stage(t0, t1 - t0 < CH ? t1 - t0 : CH);
  f32x2 S[RL / 2][4];
#pragma unroll
  for (int i = 0; i < RL / 2; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) S[i][c] = pack2(raw[2 * i][c], raw[2 * i + 1][c]);
  f32x2 n2[MODE == MODE_MEMORY ? RL / 2 : 1];             // every column group keeps the sum of keys of its rows
  if constexpr (MODE == MODE_MEMORY) {
#pragma unroll
    for (int i = 0; i < RL / 2; ++i) n2[i] = pack2(raw_n[2 * i], raw_n[2 * i + 1]);
  }
  for (int tc = t0; tc < t1; tc += CH) {
    const int nt = t1 - tc < CH ? t1 - tc : CH;
    if (tc != t0) {
      __syncthreads();                                    // the read-outs and rows of the chunk before are done with
      stage(tc, nt);
    }
    __syncthreads();
    for (int tok = 0; tok < nt; ++tok) {
      float4 vv = *reinterpret_cast<const float4*>(v_s + tok * CBP + c0);
      f32x2 da = 0ull, w2 = 0ull, nq2 = 0ull;
      if constexpr (MODE == MODE_SSD) da = pack2(a_s[tok], a_s[tok]);
      if constexpr (MODE == MODE_MEMORY) {
        const float fm = a_s[tok] + m, li = a_s[CH4 + tok];
        m = fmaxf(fm, li);
        const float keep = expf(fm - m), write = expf(li - m);
        da = pack2(keep, keep);
        w2 = pack2(write, write);
        vv.x *= write; vv.y *= write; vv.z *= write; vv.w *= write;
      }
      const f32x2 v2[4] = {pack2(vv.x, vv.x), pack2(vv.y, vv.y), pack2(vv.z, vv.z), pack2(vv.w, vv.w)};
      f32x2 o2[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) o2[c] = 0ull;
#pragma unroll
      for (int i = 0; i < RL / 4; ++i) {
        const int n0 = tok * NP + p * 4 + i * 4 * LP;
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(k_s + n0);
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(q_s + n0);
        ulonglong2 f2;
        if constexpr (MODE == MODE_FORGET) f2 = *reinterpret_cast<const ulonglong2*>(a_s + n0);
        else f2.x = f2.y = da;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[i * 2][c] = fma2(f2.x, S[i * 2][c], mul2(k2.x, v2[c]));
          o2[c] = fma2(S[i * 2][c], q2.x, o2[c]);
          S[i * 2 + 1][c] = fma2(f2.y, S[i * 2 + 1][c], mul2(k2.y, v2[c]));
          o2[c] = fma2(S[i * 2 + 1][c], q2.y, o2[c]);
        }
        if constexpr (MODE == MODE_MEMORY) {
          n2[i * 2] = fma2(da, n2[i * 2], mul2(k2.x, w2));
          nq2 = fma2(n2[i * 2], q2.x, nq2);
          n2[i * 2 + 1] = fma2(da, n2[i * 2 + 1], mul2(k2.y, w2));
          nq2 = fma2(n2[i * 2 + 1], q2.y, nq2);
        }
      }
      float o[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float2 t = unpack2(o2[c]);
        o[c] = t.x + t.y;
      }
      // sum over the LP lanes of the column group; two exchanges leave one column with each of four lanes
      const bool b0 = p & 1, b1 = p & 2;
      float s0 = b0 ? o[0] : o[2], s1 = b0 ? o[1] : o[3], r0 = b0 ? o[2] : o[0], r1 = b0 ? o[3] : o[1];
      r0 += __shfl_xor_sync(0xffffffffu, s0, 1);
      r1 += __shfl_xor_sync(0xffffffffu, s1, 1);
      const float s = b1 ? r0 : r1;
      float r = b1 ? r1 : r0;
      r += __shfl_xor_sync(0xffffffffu, s, 2);
#pragma unroll
      for (int d = 4; d < LP; d <<= 1) r += __shfl_xor_sync(0xffffffffu, r, d);
      if constexpr (MODE == MODE_MEMORY) {
        const float2 t = unpack2(nq2);
        float nq = t.x + t.y;
#pragma unroll
        for (int d = 1; d < LP; d <<= 1) nq += __shfl_xor_sync(0xffffffffu, nq, d);
        r = r * a.q_scale / (fmaxf(fabsf(nq * a.q_scale), expf(-m)) + kMemoryDenEps);
      }
      if (p < 4) o_s[tok * CBP + c0 + (b0 ? 2 : 0) + (b1 ? 1 : 0)] = r;
    }
    __syncthreads();
    for (int tok = warp; tok < nt; tok += n_warps) {
      const size_t row = (size_t)(tc + tok);
      const float* ot = o_s + tok * CBP;
      if constexpr (MODE == MODE_SSD) {
        float* dst = a.raw + row * (size_t)a.H * V + (size_t)h * V + cb0;
        for (int c = lane; c < ncol; c += 32) dst[c] = ot[c] + skip * v_s[tok * CBP + c];
      } else if (MODE == MODE_MEMORY || a.raw) {
        float* dst = a.raw + row * (size_t)a.H * V + (size_t)h * V + cb0;
        for (int c = lane; c < ncol; c += 32) dst[c] = ot[c];
      } else {
        float ss = 0.0f;
        for (int c = lane; c < V; c += 32) ss += ot[c] * ot[c];
        ss = warp_sum(ss);
        const float inv = a.mul / sqrtf(ss / (float)V + a.eps);
        T* dst = a.out + row * a.ldo + (size_t)h * V;
        for (int c = lane; c < V; c += 32) dst[c] = Num<T>::from_f(ot[c] * inv * a.norm_w[c]);
      }
    }
  }
  if constexpr (MODE == MODE_MEMORY) {
    if (cq == 0) {                                        // LP threads, each with the rows of its p
      if (p == 0) key_sum[N] = m;
#pragma unroll
      for (int i = 0; i < RL / 2; ++i) {
        const int n = p * 4 + (i / 2) * 4 * LP + (i & 1) * 2;
        const float2 t = unpack2(n2[i]);
        if (n < N) key_sum[n] = t.x;
        if (n + 1 < N) key_sum[n + 1] = t.y;
      }
    }
  }
  if (c0 < ncol) {
#pragma unroll
    for (int i = 0; i < RL / 2; ++i) {
      const int n = p * 4 + (i / 2) * 4 * LP + (i & 1) * 2;
      float2 t[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) t[c] = unpack2(S[i][c]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (n + e >= N) continue;
        float* dst = Sg + (size_t)(n + e) * V + c0;
        if (a.vec_state) {
          *reinterpret_cast<float4*>(dst) = e == 0 ? make_float4(t[0].x, t[1].x, t[2].x, t[3].x)
                                                   : make_float4(t[0].y, t[1].y, t[2].y, t[3].y);
        } else {
#pragma unroll
          for (int c = 0; c < 4; ++c)
            if (c0 + c < ncol) dst[c] = e == 0 ? t[c].x : t[c].y;
        }
      }
    }
  }
}

// out[row, h] = mul * raw / sqrt(mean(raw^2) + eps) * w: a warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256)
head_norm_kernel(T* __restrict__ out, int64_t ldo, const float* __restrict__ raw, const float* __restrict__ w,
                 int64_t n_units, int H, int V, float eps, float mul) {
  const int64_t u = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (u >= n_units) return;
  const int64_t row = u / H;
  const int h = (int)(u - row * H);
  const float* r = raw + (size_t)u * V;
  float ss = 0.0f;
  for (int i = lane; i < V; i += 32) ss += r[i] * r[i];
  ss = warp_sum(ss);
  const float inv = mul / sqrtf(ss / (float)V + eps);
  for (int i = lane; i < V; i += 32) out[(size_t)row * ldo + (size_t)h * V + i] = Num<T>::from_f(r[i] * inv * w[i]);
}

// out = u / sqrt(mean_part(u^2) + eps) * w, u = y silu(z), or (GATE_AFTER) out = y / sqrt(mean_part(y^2) + eps) * w *
// sigmoid(z); one CTA per row, the row in `parts` equal parts.  With fewer parts than warps several warps share a part.
constexpr int kPartThreads = 256;
template <typename T, bool GATE_AFTER>
__global__ void __launch_bounds__(kPartThreads)
gated_part_norm_kernel(T* __restrict__ out, int64_t ldo, const float* __restrict__ y, const T* __restrict__ z,
                       int64_t ldz, const float* __restrict__ w, int n, int parts, float eps, int vec) {
  extern __shared__ __align__(16) float sm[];
  float* u_s = sm;                                        // [n]
  float* r_s = sm + (n + 3) / 4 * 4;                      // [units] partial sums of squares
  constexpr int NW = kPartThreads / 32;
  const size_t row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x * 4; i < n; i += kPartThreads * 4) {
    float yv[4], zv[4];
    get4c<float>(y + row * n + i, yv, n - i, vec);
    if constexpr (!GATE_AFTER) get4c<T>(z + row * ldz + i, zv, n - i, vec);
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (i + k < n) {
        if constexpr (GATE_AFTER) u_s[i + k] = yv[k];
        else if constexpr (sizeof(T) == 4) u_s[i + k] = yv[k] * zv[k] * sigmoid_f(zv[k]);
        else u_s[i + k] = yv[k] * __fdividef(zv[k], 1.0f + __expf(-zv[k]));
      }
  }
  __syncthreads();
  const int ps = n / parts;
  const int per = parts >= NW ? 1 : NW / parts;           // warps of a part
  for (int un = warp; un < parts * per; un += NW) {
    const int part = un / per, sub = un - part * per;
    float ss = 0.0f;
    for (int i = sub * 32 + lane; i < ps; i += per * 32) {
      const float v = u_s[part * ps + i];
      ss += v * v;
    }
    ss = warp_sum(ss);
    if (lane == 0) r_s[un] = ss;
  }
  __syncthreads();
  for (int part = threadIdx.x; part < parts; part += kPartThreads) {
    float ss = 0.0f;
    for (int k = 0; k < per; ++k) ss += r_s[part * per + k];
    r_s[part * per] = 1.0f / sqrtf(ss / (float)ps + eps);
  }
  __syncthreads();
  for (int i = threadIdx.x * 4; i < n; i += kPartThreads * 4) {
    float wv[4], o[4];
    get4c<float>(w + i, wv, n - i, vec);
    if (ps % 4 == 0) {                                    // four channels of one part
      const float r = r_s[i / ps * per];
      const float4 u = *reinterpret_cast<const float4*>(u_s + i);
      o[0] = u.x * r * wv[0]; o[1] = u.y * r * wv[1]; o[2] = u.z * r * wv[2]; o[3] = u.w * r * wv[3];
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] = i + k < n ? u_s[i + k] * r_s[(i + k) / ps * per] * wv[k] : 0.0f;
    }
    if constexpr (GATE_AFTER) {
      float zv[4];
      get4c<T>(z + row * ldz + i, zv, n - i, vec);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if constexpr (sizeof(T) == 4) o[k] *= sigmoid_f(zv[k]);
        else o[k] = __fdividef(o[k], 1.0f + __expf(-zv[k]));
      }
    }
    T* dst = out + row * ldo + i;
    if (vec) {
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = make_float4(o[0], o[1], o[2], o[3]);
      else *reinterpret_cast<uint2*>(dst) = make_uint2(Num<T>::pack(o[0], o[1]), Num<T>::pack(o[2], o[3]));
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (i + k < n) dst[k] = Num<T>::from_f(o[k]);
    }
  }
}

template <typename T, int MODE, int RL, int LP>
int launch_scan_n(ScanArgs<T>& a, int64_t n_seq, int64_t q_max, cudaStream_t st) {
  constexpr int CW = 128 / LP;                            // columns of a warp
  int warps = (a.V + CW - 1) / CW;
  const int parts = scan_col_parts(a.N, a.V);
  warps = (warps + parts - 1) / parts;
  a.CB = warps * CW;
  a.chunk = q_max < kScanTokens ? (int)q_max : kScanTokens;
  constexpr int NP = RL * LP;
  const size_t smem = ((size_t)a.chunk * (NP * (MODE == MODE_FORGET ? 3 : 2) + 2 * a.CB) +
                       (MODE == MODE_FORGET ? 0 : (a.chunk + 3) / 4 * 4 * (MODE == MODE_MEMORY ? 2 : 1))) *
                      sizeof(float);
  auto kern = linear_scan_kernel<T, MODE, RL, LP>;
  if (smem > 48 * 1024)
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<dim3((unsigned)n_seq, (unsigned)a.H, (unsigned)((a.V + a.CB - 1) / a.CB)), warps * 32, smem, st>>>(a);
  B200_LAUNCH_OK("linear_scan_kernel");
  return B200_OK;
}

template <typename T, int MODE>
int launch_scan(ScanArgs<T>& a, int64_t n_seq, int64_t q_max, cudaStream_t st) {
  if (a.N <= 16) return launch_scan_n<T, MODE, 4, 4>(a, n_seq, q_max, st);
  if (a.N <= 32) return launch_scan_n<T, MODE, 8, 4>(a, n_seq, q_max, st);
  if (a.N <= 64) return launch_scan_n<T, MODE, 16, 4>(a, n_seq, q_max, st);
  if (a.N <= 128) return launch_scan_n<T, MODE, 32, 4>(a, n_seq, q_max, st);
  if (a.N <= 256) return launch_scan_n<T, MODE, 32, 8>(a, n_seq, q_max, st);
  return launch_scan_n<T, MODE, 32, 16>(a, n_seq, q_max, st);
}


// ------------------------------------------------------------------------------------------------------------
// Portions in bf16 on the tensor cores (mma.sync m16n8k16, fp32 accumulation): 16 tokens of a sequence at a time.
// S^T [V x N] stays in fp32 accumulators over the whole portion, a warp holding 16 MT value rows: the accumulator
// layout of S^T is the operand layout of S in  o_i = q_i . S,  so the state never passes through memory between tiles.
// fp32 factors enter a product as two bf16 terms (hi + lo, 16 mantissa bits); inputs that are bf16 already enter as
// they are.
//   ssd    : with c_i = sum_{t <= i} log a_t inside the tile,  o_i = exp(c_i) (C_i . S) + sum_{j <= i} (C_i . B_j)
//            exp(c_i - c_j) d_j x_j ;  S <- exp(c_last) S + sum_j exp(c_last - c_j) d_j B_j x_j^T    (exponents <= 0)
//   memory : with F_t = sum of the tile's log forget gates up to t, u_t = i_t - F_t and M_t = max(m, u_1 .. u_t) the running
//            maximum is m_t = F_t + M_t, the decay since the tile's start exp(m - M_t) and the weight of token j in row t
//            exp(u_j - M_t) (exponents <= 0): the ssd form with other exponents.  n rides along in shared memory: n . q
//            of the state before the tile is 16 dot products shared out over the CTA, the tile's own part the sum of a
//            row of weighted scores
//   forget : everything relative to the middle of the tile, per key channel: with r_t the product of the gates between
//            token t and the middle, q and k become q / r, k r before it and q r, k / r after it; S is decayed to the
//            middle, o = q . S + (masked q k^T) v, S <- S + k v^T, and S is decayed to the end.  Where a product of a
//            half tile falls below kMinSpan the tile is cut to 4 tokens, and to one (which needs no division) if need be.
// ------------------------------------------------------------------------------------------------------------
constexpr int kTile = 16;
constexpr float kMinSpan = 1e-16f;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = Num<__nv_bfloat16>::pack(x, y);
  const float2 h = Num<__nv_bfloat16>::unpack(hi);
  lo = Num<__nv_bfloat16>::pack(x - h.x, y - h.y);
}

// Shared-memory rows of a forget tile (bf16, 8 elements of padding per row): q hi, q lo, k hi, k lo.
template <int KN>
struct TileRows {
  static constexpr int NS = 16 * KN + 8;
  static constexpr int kRows = 4 * kTile * NS;            // the four key-channel arrays
};

__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gsrc, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem_dst)), "l"(gsrc), "r"(valid ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// One token of two neighbouring key channels of a forget tile: gates a, written shares k and silu(q) from the raw pairs.
__device__ __forceinline__ void forget_token(uint32_t qraw, uint32_t fraw, float2 bias, float2 low, float2& q, float2& a,
                                             float2& k) {
  const float2 qv = Num<__nv_bfloat16>::unpack(qraw), fv = Num<__nv_bfloat16>::unpack(fraw);
  auto gate = [](float z, float l, float& ga, float& gk) {
    const float e = __expf(-fabsf(z));
    const float big = __fdividef(1.0f, 1.0f + e), small = e * big;
    ga = l + (1.0f - l) * (z >= 0.0f ? big : small);
    gk = (1.0f - l) * (z >= 0.0f ? small : big);
  };
  gate(fv.x + bias.x, low.x, a.x, k.x);
  gate(fv.y + bias.y, low.y, a.y, k.y);
  q = make_float2(__fdividef(qv.x, 1.0f + __expf(-qv.x)), __fdividef(qv.y, 1.0f + __expf(-qv.y)));
}

// Channels c, c + 1 of one half of a forget tile of L tokens from row o on, whose middle is after token o + HA - 1.
// BEFORE: rows o + HA - 1 .. 0, else rows o + HA .. 15 (zeros outside the tile).  FULL: o = 0, HA = 8, L = 16.  raw: the
// window's query and forget logits [2][16][16 KN].  Returns the product of the half's gates.
template <int KN, bool BEFORE, bool FULL>
__device__ __forceinline__ float2 stage_forget_half(__nv_bfloat16* rows, const __nv_bfloat16* raw, int c, float2 bias,
                                                    float2 low, int o_rt, int HA_rt, int L_rt) {
  constexpr int NS = TileRows<KN>::NS, NP = 16 * KN;
  const int o = FULL ? 0 : o_rt, HA = FULL ? 8 : HA_rt, L = FULL ? kTile : L_rt;
  float2 r = make_float2(1.0f, 1.0f);
  auto put = [&](int t) {
    uint32_t qh = 0u, ql = 0u, kh = 0u, kl = 0u;
    if (FULL || (t >= o && t < o + L)) {
      const __nv_bfloat16* src = raw + t * NP + c;
      float2 qs, a, k;
      forget_token(*reinterpret_cast<const uint32_t*>(src), *reinterpret_cast<const uint32_t*>(src + kTile * NP), bias,
                   low, qs, a, k);
      if constexpr (BEFORE) {
        split_bf16(__fdividef(qs.x, r.x), __fdividef(qs.y, r.y), qh, ql);
        split_bf16(k.x * r.x, k.y * r.y, kh, kl);
        r.x *= a.x;
        r.y *= a.y;
      } else {
        r.x *= a.x;
        r.y *= a.y;
        split_bf16(qs.x * r.x, qs.y * r.y, qh, ql);
        split_bf16(__fdividef(k.x, r.x), __fdividef(k.y, r.y), kh, kl);
      }
    }
    __nv_bfloat16* dst = rows + t * NS + c;
    *reinterpret_cast<uint32_t*>(dst) = qh;
    *reinterpret_cast<uint32_t*>(dst + kTile * NS) = ql;
    *reinterpret_cast<uint32_t*>(dst + 2 * kTile * NS) = kh;
    *reinterpret_cast<uint32_t*>(dst + 3 * kTile * NS) = kl;
  };
  if constexpr (FULL) {
#pragma unroll
    for (int s = 0; s < 8; ++s) put(BEFORE ? 7 - s : 8 + s);
  } else if constexpr (BEFORE) {
    for (int t = o + HA - 1; t >= 0; --t) put(t);
  } else {
    for (int t = o + HA; t < kTile; ++t) put(t);
  }
  return r;
}

// The walk goes by windows of 16 tokens, whose raw rows are copied one window ahead (two buffers); a window is one tile
// unless its gates are too small.  The decay to the end of a tile is applied together with the next tile's decay to the
// middle.
template <int KN, int MT>
__global__ void __launch_bounds__(MT == 1 ? 128 : kScanWarps * 32, MT == 1 ? 2 : 1)
forget_scan_tc_kernel(const ScanArgs<__nv_bfloat16> a) {
  using bf16 = __nv_bfloat16;
  constexpr int NP = 16 * KN, NS = TileRows<KN>::NS, PIECES = NP / 8;
  extern __shared__ __align__(16) unsigned char smraw[];
  const int N = a.N, V = a.V, VS = V + 8, OS = V + 4;
  bf16* rows = reinterpret_cast<bf16*>(smraw);            // [q hi, q lo, k hi, k lo][16][NS]
  bf16* raw_s = rows + TileRows<KN>::kRows;               // [2 buffers][q, f][16][NP]
  bf16* v_s = raw_s + 4 * kTile * NP;                     // [2 buffers][16][VS]
  float* e_s = reinterpret_cast<float*>(v_s + 2 * kTile * VS);   // [NP] to the middle, [2][NP] to the end (two tiles')
  float* c_s = e_s + 3 * NP;                              // [2][NP] bias, lower bound
  float* o_s = c_s + 2 * NP;                              // [16][OS]
  const int seq = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int t0 = a.q_cu[seq], t1 = a.q_cu[seq + 1];
  if (t0 >= t1) return;
  const int gr = lane >> 2, qc = (lane & 3) * 2;
  const int v0 = warp * 16 * MT;                          // this warp's value rows v0 .. v0 + 16 MT - 1
  const int n_windows = (t1 - t0 + kTile - 1) / kTile;
  const bf16* qg = a.q + (size_t)h * N;
  const bf16* fg = a.k + (size_t)h * N;
  const bf16* vg = a.v + (size_t)h * V;
  const int vp = V / 8;
  auto copy_window = [&](int it) {
    const int buf = it & 1, tc = t0 + it * kTile;
    bf16* dst = raw_s + buf * 2 * kTile * NP;
    for (int x = threadIdx.x; x < 2 * kTile * PIECES; x += blockDim.x) {
      const int t = x / (2 * PIECES), p = x % (2 * PIECES);
      const bool is_f = p >= PIECES;
      const int ch = (is_f ? p - PIECES : p) * 8;
      const bool ok = tc + t < t1 && ch < N;              // (channels past N: zeros make q = k = 0, the gate 1)
      const bf16* src = is_f ? fg : qg;
      cp_async16(dst + ((is_f ? kTile : 0) + t) * NP + ch, ok ? src + (size_t)(tc + t) * a.ld + ch : src, ok);
    }
    bf16* vd = v_s + buf * kTile * VS;
    for (int t = warp; t < kTile; t += n_warps)
      for (int p = lane; p < vp; p += 32) {
        const bool ok = tc + t < t1;
        cp_async16(vd + t * VS + p * 8, ok ? vg + (size_t)(tc + t) * a.ld + p * 8 : vg, ok);
      }
    cp_async_commit();
  };
  copy_window(0);
  float* Sg = a.state + (((size_t)a.state_slots[seq] * a.H + h) * N) * V;
  const bool fresh = a.positions[t0] == 0;
  float S[MT][2 * KN][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2 * KN; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + qc + (e & 1), v = v0 + mt * 16 + gr + (e >> 1) * 8;
        S[mt][nt][e] = (!fresh && n < N && v < V) ? Sg[(size_t)n * V + v] : 0.0f;
      }
  for (int i = threadIdx.x; i < NP; i += blockDim.x) {
    c_s[i] = i < N ? a.f_bias[h * N + i] : 0.0f;
    c_s[NP + i] = i < N ? a.f_low[h * N + i] : 1.0f;
    e_s[NP + i] = 1.0f;                                    // the first tile's decay from a tile before it
  }
  const int a_off = (lane & 15) * NS + (lane >> 4) * 8;
  const int b_off = ((lane & 7) + (lane >> 4) * 8) * NS + ((lane >> 3) & 1) * 8;
  const int t_off = (lane & 7) + ((lane >> 3) & 1) * 8;
  const bf16* q_hi = rows;
  const bf16* q_lo = rows + kTile * NS;
  const bf16* k_hi = rows + 2 * kTile * NS;
  const bf16* k_lo = rows + 3 * kTile * NS;
  int par = 0;                                             // which of the two end decays is the tile before's
  for (int it = 0; it < n_windows; ++it) {
    const int tc = t0 + it * kTile, nt_w = t1 - tc < kTile ? t1 - tc : kTile;
    const bf16* raw = raw_s + (it & 1) * 2 * kTile * NP;
    const bf16* v_t = v_s + (it & 1) * kTile * VS;
    cp_async_wait_all();
    __syncthreads();                                       // the window's raw rows stand
    if (it + 1 < n_windows) copy_window(it + 1);
    int L = 0;
    for (int o = 0; o < nt_w; o += L) {
      // ---- stage the tile: rows o .. o + L - 1 of the window
      L = nt_w - o;
      while (true) {
        const int HA = (L + 1) / 2;
        bool bad = false;
        for (int u = threadIdx.x; u < NP; u += blockDim.x) {
          const bool before = u < NP / 2;
          const int c = (before ? u : u - NP / 2) * 2;
          const float2 bias = *reinterpret_cast<const float2*>(c_s + c), low = *reinterpret_cast<const float2*>(c_s + NP + c);
          float2 r;
          if (L == kTile) {
            r = before ? stage_forget_half<KN, true, true>(rows, raw, c, bias, low, o, HA, L)
                       : stage_forget_half<KN, false, true>(rows, raw, c, bias, low, o, HA, L);
          } else {
            r = before ? stage_forget_half<KN, true, false>(rows, raw, c, bias, low, o, HA, L)
                       : stage_forget_half<KN, false, false>(rows, raw, c, bias, low, o, HA, L);
          }
          *reinterpret_cast<float2*>(e_s + (before ? 0 : NP + (par ^ 1) * NP) + c) = r;
          bad |= !(fminf(r.x, r.y) >= kMinSpan);
        }
        const int any_bad = __syncthreads_or(bad);         // (also: the tile stands)
        if (L == 1 || !any_bad) break;
        L = L > 4 ? 4 : 1;
      }
      // ---- products
#pragma unroll
      for (int nt = 0; nt < 2 * KN; ++nt) {                // from the tile before to the middle of this one
        float2 e = *reinterpret_cast<const float2*>(e_s + nt * 8 + qc);
        const float2 ep = *reinterpret_cast<const float2*>(e_s + NP + par * NP + nt * 8 + qc);
        e.x *= ep.x;
        e.y *= ep.y;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          S[mt][nt][0] *= e.x; S[mt][nt][1] *= e.y; S[mt][nt][2] *= e.x; S[mt][nt][3] *= e.y;
        }
      }
      par ^= 1;
      float sc[2][4], y[MT * 2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.0f;
#pragma unroll
      for (int i = 0; i < MT * 2; ++i) y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.0f;
#pragma unroll
      for (int ks = 0; ks < KN; ++ks) {
        uint32_t ah[4], b[4];
        ldsm_x4(ah, q_hi + a_off + ks * 16);
        uint32_t al[4], bl[4];
        ldsm_x4(al, q_lo + a_off + ks * 16);
        ldsm_x4(b, k_hi + b_off + ks * 16);
        ldsm_x4(bl, k_lo + b_off + ks * 16);
        mma_bf16(sc[0], ah, b[0], b[1]);  mma_bf16(sc[1], ah, b[2], b[3]);
        mma_bf16(sc[0], ah, bl[0], bl[1]); mma_bf16(sc[1], ah, bl[2], bl[3]);
        mma_bf16(sc[0], al, b[0], b[1]);  mma_bf16(sc[1], al, b[2], b[3]);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            uint32_t h0, l0, h1, l1;
            split_bf16(S[mt][2 * ks][2 * hf], S[mt][2 * ks][2 * hf + 1], h0, l0);
            split_bf16(S[mt][2 * ks + 1][2 * hf], S[mt][2 * ks + 1][2 * hf + 1], h1, l1);
            mma_bf16(y[mt * 2 + hf], ah, h0, h1);
            mma_bf16(y[mt * 2 + hf], ah, l0, l1);
            mma_bf16(y[mt * 2 + hf], al, h0, h1);
          }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (n * 8 + qc + (e & 1) > gr + (e >> 1) * 8) sc[n][e] = 0.0f;
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        split_bf16(sc[n][0], sc[n][1], ph[n * 2], pl[n * 2]);
        split_bf16(sc[n][2], sc[n][3], ph[n * 2 + 1], pl[n * 2 + 1]);
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const int vc = v0 + mt * 16;
        if (vc < V) {                                        // (the same for the whole warp)
          uint32_t b[4];
          ldsm_x4_t(b, v_t + t_off * VS + vc + (lane >> 4) * 8);
          mma_bf16(y[mt * 2], ph, b[0], b[1]); mma_bf16(y[mt * 2 + 1], ph, b[2], b[3]);
          mma_bf16(y[mt * 2], pl, b[0], b[1]); mma_bf16(y[mt * 2 + 1], pl, b[2], b[3]);
        }
      }
      // ---- the new state
      uint32_t va[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const int vc = v0 + mt * 16;
        va[mt][0] = va[mt][1] = va[mt][2] = va[mt][3] = 0u;
        if (vc < V) ldsm_x4_t(va[mt], v_t + ((lane & 7) + (lane >> 4) * 8) * VS + vc + ((lane >> 3) & 1) * 8);
      }
#pragma unroll
      for (int ks = 0; ks < KN; ++ks) {
        uint32_t b[4], bl[4];
        ldsm_x4_t(b, k_hi + t_off * NS + ks * 16 + (lane >> 4) * 8);
        ldsm_x4_t(bl, k_lo + t_off * NS + ks * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(S[mt][2 * ks], va[mt], b[0], b[1]);
          mma_bf16(S[mt][2 * ks + 1], va[mt], b[2], b[3]);
          mma_bf16(S[mt][2 * ks], va[mt], bl[0], bl[1]);
          mma_bf16(S[mt][2 * ks + 1], va[mt], bl[2], bl[3]);
        }
      }
      // ---- out: eight lanes a token
#pragma unroll
      for (int i = 0; i < MT * 2; ++i) {
        const int v = v0 + i * 8 + qc;
        if (v < V) {
          *reinterpret_cast<float2*>(o_s + gr * OS + v) = make_float2(y[i][0], y[i][1]);
          *reinterpret_cast<float2*>(o_s + (gr + 8) * OS + v) = make_float2(y[i][2], y[i][3]);
        }
      }
      __syncthreads();                                     // the read-outs stand; the tile's rows are done with
      for (int tb = o + warp * 4; tb < o + L; tb += n_warps * 4) {
        const int t = tb + (lane >> 3), sub = lane & 7;
        const bool ok = t < o + L;
        const float* ot = o_s + (ok ? t : o) * OS;
        float ss = 0.0f;
        for (int c = sub * 2; c < V; c += 16) {
          const float2 w = *reinterpret_cast<const float2*>(ot + c);
          ss += w.x * w.x + w.y * w.y;
        }
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        if (!ok) continue;
        const float inv = a.mul / sqrtf(ss / (float)V + a.eps);
        bf16* dst = a.out + (size_t)(tc + t) * a.ldo + (size_t)h * V;
        for (int c = sub * 2; c < V; c += 16) {
          const float2 w = *reinterpret_cast<const float2*>(ot + c), nw = *reinterpret_cast<const float2*>(a.norm_w + c);
          *reinterpret_cast<uint32_t*>(dst + c) = Num<bf16>::pack(w.x * inv * nw.x, w.y * inv * nw.y);
        }
      }
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2 * KN; ++nt) {
      const float2 ep = *reinterpret_cast<const float2*>(e_s + NP + par * NP + nt * 8 + qc);   // the last tile's end
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + qc + (e & 1), v = v0 + mt * 16 + gr + (e >> 1) * 8;
        if (n < N && v < V) Sg[(size_t)n * V + v] = S[mt][nt][e] * (e & 1 ? ep.y : ep.x);
      }
    }
}

// The ssd walk, and (MEM) the matrix memory's with C = q, B = k, x = v.  A tile's C, B and x rows are copied one tile ahead (two buffers); its decay exponents are worked out one tile ahead by
// one warp, which takes turns.
template <int KN, int MT, bool MEM>
__global__ void __launch_bounds__(MT == 1 ? 128 : kScanWarps * 32, MT == 1 ? (MEM ? 2 : 3) : 1)
ssd_scan_tc_kernel(const ScanArgs<__nv_bfloat16> a) {
  using bf16 = __nv_bfloat16;
  constexpr int NP = 16 * KN, NS = TileRows<KN>::NS, PIECES = NP / 8;
  extern __shared__ __align__(16) unsigned char smraw[];
  const int N = a.N, V = a.V, VS = V + 8;
  bf16* cb_s = reinterpret_cast<bf16*>(smraw);            // [2 buffers][C, B][16][NS]
  bf16* k_s = cb_s + 4 * kTile * NS;                      // [hi, lo][16][NS]: B with its step size and decay to the end
  bf16* v_s = k_s + 2 * kTile * NS;                       // [2 buffers][16][VS]
  float* e_s = reinterpret_cast<float*>(v_s + 2 * kTile * VS);   // ssd: [2 buffers][c_i | d_i | d_i exp(c_last - c_i)][16]
  constexpr int ES = MEM ? 5 : 3;                         // memory: [2][M_i | u_i | exp(u_i - M_last) | exp(-m_i) | m, m'][16]
  float* n_s = e_s + 2 * ES * kTile;                      // memory: [NP] the sum of keys before the tile
  float* nq_s = n_s + NP;                                 // memory: [16] its products with the tile's queries
  const int seq = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int t0 = a.q_cu[seq], t1 = a.q_cu[seq + 1];
  if (t0 >= t1) return;
  const int gr = lane >> 2, qc = (lane & 3) * 2;
  const int v0 = warp * 16 * MT;                          // this warp's value rows v0 .. v0 + 16 MT - 1
  float neg_a = 0.0f, dbias = 0.0f, skip = 0.0f, ibias = 0.0f;
  if constexpr (MEM) {
    dbias = a.gf_bias[h];
    ibias = a.gi_bias[h];
  } else {
    neg_a = -expf(a.a_log[h]);
    dbias = a.dt_bias[h];
    skip = a.skip[h];
  }
  const int n_tiles = (t1 - t0 + kTile - 1) / kTile;
  const bf16* cg = a.q + (size_t)g * N;
  const bf16* bg = a.k + (size_t)g * N;
  const bf16* vg = a.v + (size_t)h * V;
  const int vp = V / 8;
  auto copy_tile = [&](int it) {
    const int buf = it & 1, tc = t0 + it * kTile;
    bf16* dst = cb_s + buf * 2 * kTile * NS;
    for (int x = threadIdx.x; x < 2 * kTile * PIECES; x += blockDim.x) {
      const int t = x / (2 * PIECES), p = x % (2 * PIECES);
      const bool is_b = p >= PIECES;
      const int ch = (is_b ? p - PIECES : p) * 8;
      const bool ok = tc + t < t1 && ch < N;
      const bf16* src = is_b ? bg : cg;
      cp_async16(dst + ((is_b ? kTile : 0) + t) * NS + ch, ok ? src + (size_t)(tc + t) * a.ld + ch : src, ok);
    }
    bf16* vd = v_s + buf * kTile * VS;
    for (int t = warp; t < kTile; t += n_warps)
      for (int p = lane; p < vp; p += 32) {
        const bool ok = tc + t < t1;
        cp_async16(vd + t * VS + p * 8, ok ? vg + (size_t)(tc + t) * a.ld + p * 8 : vg, ok);
      }
    cp_async_commit();
  };
  auto load_dt = [&](int it) {                            // lane t holds token t of the tile (-inf: no step)
    const int t = t0 + it * kTile + lane;
    const bool ok = lane < kTile && t < t1;
    if constexpr (MEM)
      return make_float2(ok ? a.gf[(size_t)t * a.ld_g + h] + dbias : -INFINITY,
                         ok ? a.gi[(size_t)t * a.ld_g + h] + ibias : 0.0f);
    else
      return ok ? Num<bf16>::to_f(a.dt[(size_t)t * a.ld_dt + h]) + dbias : -INFINITY;
  };
  using Gate = typename std::conditional<MEM, float2, float>::type;
  auto exponents_mem = [&](int it, float2 z, float m) {   // m: the running maximum before the tile
    const bool ok = z.x != -INFINITY;
    const float ft = a.cap * tanhf((ok ? z.x : 0.0f) / a.cap), iv = a.cap * tanhf(z.y / a.cap);
    float F = ok ? log_sigmoid_f(ft) : 0.0f;
#pragma unroll
    for (int s = 1; s < kTile; s <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, F, s);
      if (lane >= s) F += up;
    }
    const float u = ok ? iv - F : -INFINITY;
    float M = fmaxf(m, u);
#pragma unroll
    for (int s = 1; s < kTile; s <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, M, s);
      if (lane >= s) M = fmaxf(M, up);
    }
    const float M_last = __shfl_sync(0xffffffffu, M, kTile - 1);
    if (lane < kTile) {
      float* e = e_s + (it & 1) * ES * kTile;
      e[lane] = M;
      e[kTile + lane] = u;
      e[2 * kTile + lane] = expf(u - M_last);
      e[3 * kTile + lane] = expf(-(F + M));
      if (lane == kTile - 1) {
        e[4 * kTile] = m;
        e[4 * kTile + 1] = F + M;
      }
    }
  };
  auto exponents_ssd = [&](int it, float z) {
    const float d = z == -INFINITY ? 0.0f : softplus_f(z);
    float c = neg_a * d;
#pragma unroll
    for (int s = 1; s < kTile; s <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, c, s);
      if (lane >= s) c += up;
    }
    const float c_last = __shfl_sync(0xffffffffu, c, kTile - 1);
    if (lane < kTile) {
      float* e = e_s + (it & 1) * ES * kTile;
      e[lane] = c;
      e[kTile + lane] = d;
      e[2 * kTile + lane] = d * expf(c_last - c);
    }
  };
  copy_tile(0);
  const bool fresh = a.positions[t0] == 0;
  float* key_sum = nullptr;
  if constexpr (MEM) {
    key_sum = a.key_sum + ((size_t)a.state_slots[seq] * a.H + h) * scan_col_parts(N, V) * (N + 1);
    if (warp == 0) exponents_mem(0, load_dt(0), fresh ? 0.0f : key_sum[N]);
    for (int i = threadIdx.x; i < NP; i += blockDim.x) n_s[i] = !fresh && i < N ? key_sum[i] : 0.0f;
  } else {
    if (warp == 0) exponents_ssd(0, load_dt(0));
  }
  float* Sg = a.state + (((size_t)a.state_slots[seq] * a.H + h) * N) * V;
  float S[MT][2 * KN][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2 * KN; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + qc + (e & 1), v = v0 + mt * 16 + gr + (e >> 1) * 8;
        S[mt][nt][e] = (!fresh && n < N && v < V) ? Sg[(size_t)n * V + v] : 0.0f;
      }
  const int a_off = (lane & 15) * NS + (lane >> 4) * 8;
  const int b_off = ((lane & 7) + (lane >> 4) * 8) * NS + ((lane >> 3) & 1) * 8;
  const int t_off = (lane & 7) + ((lane >> 3) & 1) * 8;
  for (int it = 0; it < n_tiles; ++it) {
    const int buf = it & 1;
    cp_async_wait_all();
    __syncthreads();                                       // tile `it` stands; everyone is done with the tile before
    const bool ahead = it + 1 < n_tiles, mine = ahead && it % n_warps == warp;
    Gate z{};
    if (ahead) copy_tile(it + 1);
    if (mine) z = load_dt(it + 1);
    const bf16* c_t = cb_s + buf * 2 * kTile * NS;
    const bf16* b_t = c_t + kTile * NS;
    const bf16* v_t = v_s + buf * kTile * VS;
    const float* e = e_s + buf * ES * kTile;
    for (int x = threadIdx.x; x < kTile * PIECES; x += blockDim.x) {
      const int t = x / PIECES, ch = (x % PIECES) * 8;
      const uint4 raw = *reinterpret_cast<const uint4*>(b_t + t * NS + ch);
      const float wt = e[2 * kTile + t];
      const uint32_t in[4] = {raw.x, raw.y, raw.z, raw.w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 bv = Num<bf16>::unpack(in[i]);
        split_bf16(bv.x * wt, bv.y * wt, hi[i], lo[i]);
      }
      *reinterpret_cast<uint4*>(k_s + t * NS + ch) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(k_s + (kTile + t) * NS + ch) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    if constexpr (MEM) {
      // n . q: eight lanes a token
      for (int t = threadIdx.x >> 3; t < kTile; t += blockDim.x >> 3) {
        float s = 0.0f;
        for (int c = (threadIdx.x & 7) * 2; c < NP; c += 16) {
          const float2 qv = Num<bf16>::unpack(*reinterpret_cast<const uint32_t*>(c_t + t * NS + c));
          const float2 nv = *reinterpret_cast<const float2*>(n_s + c);
          s += qv.x * nv.x + qv.y * nv.y;
        }
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
        if ((threadIdx.x & 7) == 0) nq_s[t] = s;
      }
    }
    // ---- read-outs: C . S and the scores C . B
    float sc[2][4], y[MT * 2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.0f;
#pragma unroll
    for (int i = 0; i < MT * 2; ++i) y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < KN; ++ks) {
      uint32_t ca[4], b[4];
      ldsm_x4(ca, c_t + a_off + ks * 16);
      ldsm_x4(b, b_t + b_off + ks * 16);
      mma_bf16(sc[0], ca, b[0], b[1]);
      mma_bf16(sc[1], ca, b[2], b[3]);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          uint32_t h0, l0, h1, l1;
          split_bf16(S[mt][2 * ks][2 * hf], S[mt][2 * ks][2 * hf + 1], h0, l0);
          split_bf16(S[mt][2 * ks + 1][2 * hf], S[mt][2 * ks + 1][2 * hf + 1], h1, l1);
          mma_bf16(y[mt * 2 + hf], ca, h0, h1);
          mma_bf16(y[mt * 2 + hf], ca, l0, l1);
        }
    }
    const float ci[2] = {e[gr], e[gr + 8]};
    float gi[2], c_end, rs[2] = {0.0f, 0.0f};               // rs: row sums of the weighted scores
    if constexpr (MEM) {
      const float m = e[4 * kTile];
      gi[0] = expf(m - ci[0]);
      gi[1] = expf(m - ci[1]);
      c_end = expf(m - e[kTile - 1]);
    } else {
      gi[0] = __expf(ci[0]);
      gi[1] = __expf(ci[1]);
      c_end = __expf(e[kTile - 1]);
    }
#pragma unroll
    for (int i = 0; i < MT * 2; ++i) { y[i][0] *= gi[0]; y[i][1] *= gi[0]; y[i][2] *= gi[1]; y[i][3] *= gi[1]; }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float2 cj = *reinterpret_cast<const float2*>(e + n * 8 + qc);
      const float2 dj = *reinterpret_cast<const float2*>(e + kTile + n * 8 + qc);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int i = gr + (r >> 1) * 8, j = n * 8 + qc + (r & 1);
        if constexpr (MEM) {
          sc[n][r] = j <= i ? sc[n][r] * expf((r & 1 ? dj.y : dj.x) - ci[r >> 1]) : 0.0f;
          rs[r >> 1] += sc[n][r];
        } else {
          const float w = __expf(ci[r >> 1] - (r & 1 ? cj.y : cj.x)) * (r & 1 ? dj.y : dj.x);
          sc[n][r] = j <= i ? sc[n][r] * w : 0.0f;
        }
      }
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      split_bf16(sc[n][0], sc[n][1], ph[n * 2], pl[n * 2]);
      split_bf16(sc[n][2], sc[n][3], ph[n * 2 + 1], pl[n * 2 + 1]);
    }
    uint32_t va[MT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const int vc = v0 + mt * 16;
      va[mt][0] = va[mt][1] = va[mt][2] = va[mt][3] = 0u;
      if (vc < V) {                                        // (the same for the whole warp)
        uint32_t b[4];
        ldsm_x4_t(b, v_t + t_off * VS + vc + (lane >> 4) * 8);
        ldsm_x4_t(va[mt], v_t + ((lane & 7) + (lane >> 4) * 8) * VS + vc + ((lane >> 3) & 1) * 8);
        mma_bf16(y[mt * 2], ph, b[0], b[1]); mma_bf16(y[mt * 2 + 1], ph, b[2], b[3]);
        mma_bf16(y[mt * 2], pl, b[0], b[1]); mma_bf16(y[mt * 2 + 1], pl, b[2], b[3]);
      }
    }
    const int tc = t0 + it * kTile;
    auto write_out = [&]() {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = gr + r * 8;
        float f = 1.0f;
        if constexpr (MEM) {
          rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 1);
          rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 2);
          f = a.q_scale / (fmaxf(fabsf((gi[r] * nq_s[t] + rs[r]) * a.q_scale), e[3 * kTile + t]) + kMemoryDenEps);
        }
        if (tc + t < t1) {
          float* dst = a.raw + ((size_t)(tc + t) * a.H + h) * V + v0 + qc;
          const bf16* xr = v_t + t * VS + v0 + qc;
#pragma unroll
          for (int i = 0; i < MT * 2; ++i)
            if (v0 + i * 8 < V) {
              if constexpr (MEM) {
                *reinterpret_cast<float2*>(dst + i * 8) = make_float2(y[i][2 * r] * f, y[i][2 * r + 1] * f);
              } else {
                const float2 x = Num<bf16>::unpack(*reinterpret_cast<const uint32_t*>(xr + i * 8));
                *reinterpret_cast<float2*>(dst + i * 8) = make_float2(y[i][2 * r] + skip * x.x, y[i][2 * r + 1] + skip * x.y);
              }
            }
        }
      }
    };
    if constexpr (!MEM) write_out();
    // ---- the new state
    __syncthreads();                                       // k_s stands (memory: and n . q)
    if constexpr (MEM) {
      write_out();
      for (int c = threadIdx.x; c < NP; c += blockDim.x) {
        float n = n_s[c] * c_end;
#pragma unroll 4
        for (int t = 0; t < kTile; ++t) n += Num<bf16>::to_f(b_t[t * NS + c]) * e[2 * kTile + t];
        n_s[c] = n;
      }
    }
#pragma unroll
    for (int ks = 0; ks < KN; ++ks) {
      uint32_t b[4], bl[4];
      ldsm_x4_t(b, k_s + t_off * NS + ks * 16 + (lane >> 4) * 8);
      ldsm_x4_t(bl, k_s + (kTile + t_off) * NS + ks * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          S[mt][2 * ks][r] *= c_end;
          S[mt][2 * ks + 1][r] *= c_end;
        }
        mma_bf16(S[mt][2 * ks], va[mt], b[0], b[1]);
        mma_bf16(S[mt][2 * ks + 1], va[mt], b[2], b[3]);
        mma_bf16(S[mt][2 * ks], va[mt], bl[0], bl[1]);
        mma_bf16(S[mt][2 * ks + 1], va[mt], bl[2], bl[3]);
      }
    }
    if (mine) {
      if constexpr (MEM) exponents_mem(it + 1, z, e[4 * kTile + 1]);
      else exponents_ssd(it + 1, z);
    }
  }
  if constexpr (MEM) {
    __syncthreads();                                       // n stands
    const float* e = e_s + ((n_tiles - 1) & 1) * ES * kTile;
    const int parts = scan_col_parts(N, V);                // every copy: a walk of another form may follow
    for (int i = threadIdx.x; i < parts * (N + 1); i += blockDim.x) {
      const int c = i % (N + 1);
      key_sum[i] = c < N ? n_s[c] : e[4 * kTile + 1];
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < 2 * KN; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + qc + (e & 1), v = v0 + mt * 16 + gr + (e >> 1) * 8;
        if (n < N && v < V) Sg[(size_t)n * V + v] = S[mt][nt][e];
      }
}

template <int KN, int MT>
int launch_tc_n(int mode, const ScanArgs<__nv_bfloat16>& a, int64_t n_seq, cudaStream_t st) {
  const int warps = (a.V + 16 * MT - 1) / (16 * MT);
  constexpr int NS = TileRows<KN>::NS;
  size_t smem;
  if (mode == MODE_FORGET)
    smem = (size_t)(4 * kTile * (NS + 16 * KN) + 2 * kTile * (a.V + 8)) * sizeof(__nv_bfloat16) +
           (size_t)(5 * 16 * KN + kTile * (a.V + 4)) * sizeof(float);
  else
    smem = (size_t)(6 * kTile * NS + 2 * kTile * (a.V + 8)) * sizeof(__nv_bfloat16) +
           (mode == MODE_SSD ? 6 * kTile : 11 * kTile + 16 * KN) * sizeof(float);
  auto kern = mode == MODE_FORGET ? forget_scan_tc_kernel<KN, MT>
                                  : (mode == MODE_SSD ? ssd_scan_tc_kernel<KN, MT, false> : ssd_scan_tc_kernel<KN, MT, true>);
  if (smem > 48 * 1024)
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<dim3((unsigned)n_seq, (unsigned)a.H), warps * 32, smem, st>>>(a);
  B200_LAUNCH_OK("scan_tc_kernel");
  return B200_OK;
}

int launch_scan_tc(int mode, const ScanArgs<__nv_bfloat16>& a, int64_t n_seq, cudaStream_t st) {
  const bool two = a.V > 64;                              // 16 value rows a warp, or 32
  if (a.N <= 32) return two ? launch_tc_n<2, 2>(mode, a, n_seq, st) : launch_tc_n<2, 1>(mode, a, n_seq, st);
  if (a.N <= 64) return two ? launch_tc_n<4, 2>(mode, a, n_seq, st) : launch_tc_n<4, 1>(mode, a, n_seq, st);
  return two ? launch_tc_n<8, 2>(mode, a, n_seq, st) : launch_tc_n<8, 1>(mode, a, n_seq, st);
}
int launch_scan_tc(int, const ScanArgs<float>&, int64_t, cudaStream_t) {
  return set_error(B200_ERR_UNSUPPORTED, "linear_scan: the tensor-core form takes bf16");
}

bool scan_tc_fits(int64_t N, int64_t V, int dtype) {
  return dtype == B200_BF16 && N > 0 && N % 8 == 0 && N <= 128 && V > 0 && V % 16 == 0 && V <= 32 * kScanWarps;
}

}  // namespace
}  // namespace b200

using namespace b200;

#define SCAN_DISPATCH(dtype, ...)                                                            \
  switch (dtype) {                                                                           \
    case B200_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }                         \
    case B200_FP32: { using T = float; __VA_ARGS__; break; }                                 \
    default: return set_error(B200_ERR_INVALID_ARG, "linear_scan: bf16 or fp32, got %d", dtype); \
  }

extern "C" {

int b200_linear_scan_parts(int64_t N, int64_t V) { return scan_col_parts((int)N, (int)V); }

int b200_linear_scan_tc_supported(int64_t N, int64_t V, int dtype) { return scan_tc_fits(N, V, dtype); }

int b200_forget_scan(void* out, int64_t ldo, const void* q, const void* f, const void* v, int64_t ld,
                     const float* f_bias, const float* f_low, const float* norm_weight, float* state,
                     const int32_t* q_cu_lens, const int32_t* positions, const int32_t* state_slots, int64_t n_seq,
                     int64_t q_max, int64_t rows, int64_t H, int64_t N, int64_t V, float eps, float mul, float* raw,
                     int tensor_cores, int dtype, b200_stream_t stream) {
  if (rows == 0 || n_seq == 0) return B200_OK;
  B200_CHECK_ARG(out && q && f && v && f_bias && f_low && norm_weight && state && q_cu_lens && positions && state_slots,
                 "forget_scan: null pointer");
  B200_CHECK_ARG(rows > 0 && n_seq > 0 && q_max > 0 && H > 0 && H <= 65535 && N > 0 && N <= 512 && V > 0 && V <= 4096 &&
                     ldo >= H * V && ld >= H * (N > V ? N : V),
                 "forget_scan: bad shape (key size <= 512)");
  B200_CHECK_ARG(!tensor_cores || (scan_tc_fits(N, V, dtype) && ld % 8 == 0 && ldo % 2 == 0 && is_aligned(q, 16) &&
                                   is_aligned(f, 16) && is_aligned(v, 16) && is_aligned(out, 4) &&
                                   is_aligned(norm_weight, 8)),
                 "forget_scan: sizes or alignment do not fit the tensor-core tiles");
  B200_CHECK_ARG(tensor_cores || raw || scan_col_parts((int)N, (int)V) == 1, "forget_scan: heads in several column parts need a workspace");
  auto st = static_cast<cudaStream_t>(stream);
  SCAN_DISPATCH(dtype, {
    ScanArgs<T> a{};
    a.out = static_cast<T*>(out); a.ldo = ldo; a.raw = raw;
    a.q = static_cast<const T*>(q); a.k = static_cast<const T*>(f); a.v = static_cast<const T*>(v); a.ld = ld;
    a.f_bias = f_bias; a.f_low = f_low; a.norm_w = norm_weight; a.state = state;
    a.q_cu = q_cu_lens; a.positions = positions; a.state_slots = state_slots;
    a.H = (int)H; a.G = (int)H; a.N = (int)N; a.V = (int)V; a.eps = eps; a.mul = mul;
    a.vec_in = N % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && is_aligned(q, 4 * sizeof(T)) && is_aligned(f, 4 * sizeof(T)) &&
               is_aligned(v, 4 * sizeof(T));
    a.vec_state = V % 4 == 0 && is_aligned(state, 16);
    if (tensor_cores) return launch_scan_tc(MODE_FORGET, a, n_seq, st);
    const int rc = launch_scan<T, MODE_FORGET>(a, n_seq, q_max, st);
    if (rc != B200_OK) return rc;
    if (raw) {
      const int64_t n_units = rows * H;
      head_norm_kernel<T><<<(unsigned)((n_units + 7) / 8), 256, 0, st>>>(static_cast<T*>(out), ldo, raw, norm_weight,
                                                                         n_units, (int)H, (int)V, eps, mul);
      B200_LAUNCH_OK("head_norm_kernel");
    }
  });
  return B200_OK;
}

int b200_ssd_scan(float* y, const void* x, const void* B, const void* Cm, int64_t ld, const void* dt, int64_t ld_dt,
                  const float* dt_bias, const float* a_log, const float* skip, float* state, const int32_t* q_cu_lens,
                  const int32_t* positions, const int32_t* state_slots, int64_t n_seq, int64_t q_max, int64_t rows,
                  int64_t H, int64_t G, int64_t N, int64_t V, int tensor_cores, int dtype, b200_stream_t stream) {
  if (rows == 0 || n_seq == 0) return B200_OK;
  B200_CHECK_ARG(y && x && B && Cm && dt && dt_bias && a_log && skip && state && q_cu_lens && positions && state_slots,
                 "ssd_scan: null pointer");
  B200_CHECK_ARG(rows > 0 && n_seq > 0 && q_max > 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && N > 0 && N <= 512 &&
                     V > 0 && V <= 4096 && ld >= H * V && ld >= G * N && ld_dt >= H,
                 "ssd_scan: bad shape (state size <= 512, heads a multiple of groups)");
  B200_CHECK_ARG(!tensor_cores || (scan_tc_fits(N, V, dtype) && ld % 8 == 0 && is_aligned(x, 16) && is_aligned(B, 16) &&
                                   is_aligned(Cm, 16) && is_aligned(y, 8)),
                 "ssd_scan: sizes or alignment do not fit the tensor-core tiles");
  auto st = static_cast<cudaStream_t>(stream);
  SCAN_DISPATCH(dtype, {
    ScanArgs<T> a{};
    a.raw = y;
    a.q = static_cast<const T*>(Cm); a.k = static_cast<const T*>(B); a.v = static_cast<const T*>(x); a.ld = ld;
    a.dt = static_cast<const T*>(dt); a.ld_dt = ld_dt; a.dt_bias = dt_bias; a.a_log = a_log; a.skip = skip;
    a.state = state; a.q_cu = q_cu_lens; a.positions = positions; a.state_slots = state_slots;
    a.H = (int)H; a.G = (int)G; a.N = (int)N; a.V = (int)V; a.mul = 1.0f;
    a.vec_in = N % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && is_aligned(x, 4 * sizeof(T)) && is_aligned(B, 4 * sizeof(T)) &&
               is_aligned(Cm, 4 * sizeof(T));
    a.vec_state = V % 4 == 0 && is_aligned(state, 16);
    if (tensor_cores) return launch_scan_tc(MODE_SSD, a, n_seq, st);
    return (launch_scan<T, MODE_SSD>(a, n_seq, q_max, st));
  });
  return B200_OK;
}

int b200_memory_scan(float* y, const void* q, const void* k, const void* v, int64_t ld, const float* i_logits,
                     const float* f_logits, int64_t ld_g, const float* i_bias, const float* f_bias, float cap,
                     float q_scale, float* state, float* key_sum, const int32_t* q_cu_lens, const int32_t* positions,
                     const int32_t* state_slots, int64_t n_seq, int64_t q_max, int64_t rows, int64_t H, int64_t N,
                     int64_t V, int tensor_cores, int dtype, b200_stream_t stream) {
  if (rows == 0 || n_seq == 0) return B200_OK;
  B200_CHECK_ARG(y && q && k && v && i_logits && f_logits && i_bias && f_bias && state && key_sum && q_cu_lens &&
                     positions && state_slots,
                 "memory_scan: null pointer");
  B200_CHECK_ARG(rows > 0 && n_seq > 0 && q_max > 0 && H > 0 && H <= 65535 && N > 0 && N <= 512 && V > 0 && V <= 4096 &&
                     ld >= H * (N > V ? N : V) && ld_g >= H && cap > 0.0f,
                 "memory_scan: bad shape (key size <= 512)");
  B200_CHECK_ARG(!tensor_cores || (scan_tc_fits(N, V, dtype) && ld % 8 == 0 && is_aligned(q, 16) && is_aligned(k, 16) &&
                                   is_aligned(v, 16) && is_aligned(y, 8)),
                 "memory_scan: sizes or alignment do not fit the tensor-core tiles");
  auto st = static_cast<cudaStream_t>(stream);
  SCAN_DISPATCH(dtype, {
    ScanArgs<T> a{};
    a.raw = y;
    a.q = static_cast<const T*>(q); a.k = static_cast<const T*>(k); a.v = static_cast<const T*>(v); a.ld = ld;
    a.gi = i_logits; a.gf = f_logits; a.ld_g = ld_g; a.gi_bias = i_bias; a.gf_bias = f_bias; a.cap = cap;
    a.q_scale = q_scale; a.key_sum = key_sum;
    a.state = state; a.q_cu = q_cu_lens; a.positions = positions; a.state_slots = state_slots;
    a.H = (int)H; a.G = (int)H; a.N = (int)N; a.V = (int)V; a.mul = 1.0f;
    a.vec_in = N % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && is_aligned(q, 4 * sizeof(T)) && is_aligned(k, 4 * sizeof(T)) &&
               is_aligned(v, 4 * sizeof(T));
    a.vec_state = V % 4 == 0 && is_aligned(state, 16);
    if (tensor_cores) return launch_scan_tc(MODE_MEMORY, a, n_seq, st);
    return (launch_scan<T, MODE_MEMORY>(a, n_seq, q_max, st));
  });
  return B200_OK;
}

int b200_gated_part_norm(void* out, int64_t ldo, const float* y, const void* z, int64_t ldz, const float* weight,
                         int64_t rows, int64_t n, int64_t parts, float eps, int gate_after, int dtype, b200_stream_t stream) {
  if (rows == 0) return B200_OK;
  B200_CHECK_ARG(out && y && z && weight, "gated_part_norm: null pointer");
  B200_CHECK_ARG(rows > 0 && n > 0 && parts > 0 && n % parts == 0 && ldo >= n && ldz >= n && (n + parts + 16) * 4 <= 200 * 1024,
                 "gated_part_norm: bad shape (the row in equal parts, at most ~50K channels)");
  auto st = static_cast<cudaStream_t>(stream);
  const size_t smem = (size_t)((n + 3) / 4 * 4 + (parts < 8 ? 8 : parts)) * sizeof(float);
  SCAN_DISPATCH(dtype, {
    const int vec = n % 4 == 0 && ldo % 4 == 0 && ldz % 4 == 0 && is_aligned(out, 4 * sizeof(T)) &&
                    is_aligned(z, 4 * sizeof(T)) && is_aligned(y, 16) && is_aligned(weight, 16);
    auto kern = gate_after ? gated_part_norm_kernel<T, true> : gated_part_norm_kernel<T, false>;
    if (smem > 48 * 1024)
      B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<(unsigned)rows, kPartThreads, smem, st>>>(static_cast<T*>(out), ldo, y, static_cast<const T*>(z), ldz, weight,
                                                     (int)n, (int)parts, eps, vec);
  });
  B200_LAUNCH_OK("gated_part_norm_kernel");
  return B200_OK;
}

}  // extern "C"
