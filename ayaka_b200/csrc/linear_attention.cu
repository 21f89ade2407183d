// Linear attention with a matrix state per head: a gated delta rule (decay per head or per key
// channel) and retention (a fixed decay per head), over a step's rows. Per head, with S [N x P],
//   S <- g S;   u = beta (v - S^T k)  (delta) or  u = v;   S <- S + k u^T;   o = S^T q,
// where g scales the rows of S (one factor per key channel, or the same for all of a head).
// Everything here is fp32.
//
// A request's state in its slot: S as [head][N][P] from the slot's start, then (layers with a
// short causal convolution) a ring of the last `taps` inputs, [taps][channels]: the input of
// position p lies at p % taps. A decode step only writes the ring at its own position and only
// reads the others, so every CTA of a step may read while one writes.
//
// Steps of single rows: decode_kernel, one launch from the projection's row to the normed and
// gated row that the output product reads (convolution, unit keys, decay, the state's update,
// the head's norm, the gate).
//
// Portions: rows are taken in chunks of C = 16, and a chunk is turned into small matrices by
// prepare_kernel (a CTA per chunk and head, all in parallel) so that the sequential part,
// scan_kernel, touches the state once per chunk. With S_0 the state ahead of the chunk, row i's
// cumulative decay G_i = g_0 ... g_i (per channel) and D_ij = g_(j+1) ... g_i:
//   u_i = beta_i (v_i - (G_i k_i) S_0 - sum_(j<i) A_ij u_j),   A_ij = k_i . (D_ij k_j)
//   o_i = (G_i q_i) S_0 + sum_(j<=i) B_ij u_j,                 B_ij = q_i . (D_ij k_j)
//   S_C = G_(C-1) S_0 + sum_j (D_(C-1)j k_j) u_j^T.
// The first line is a lower triangular system, U = T W with W = V - (G k) S_0 and
// T = (I + diag(beta) A)^-1 diag(beta); T is folded into what multiplies U, so that
//   W = V - Kt S_0,   O = Qt S_0 + R W,   S_C = G S_0 + Kh^T W
// with Kt = G k, Qt = G q, R = B T, Kh = T^T (D_(C-1) k) is all the scan computes. Decays only
// ever appear as products of factors in [0, 1] (never as quotients), so nothing overflows and a
// channel that forgets at once is exact. A chunk's missing rows have k = q = 0, beta = 0, g = 1.
#include "common.cuh"
#include "rope.cuh"

namespace ayk {

constexpr int LA_C = 16;           // rows of a chunk
constexpr int LA_COLS = 16;        // columns of the state per CTA of the scan
constexpr int LA_MAX_N = 512;      // key channels of a head
constexpr int LA_MAX_TAPS = 16;
constexpr int LA_CONV_ROWS = 8;    // rows per CTA of the portions' convolution
constexpr int LA_THREADS = 256;

enum DecayMode : int { DECAY_FIXED = 0, DECAY_HEAD = 1, DECAY_CHANNEL = 2 };
enum HeadGate : int { HEAD_GATE_NONE = 0, HEAD_GATE_SIGMOID = 1, HEAD_GATE_SILU = 2 };

// What both paths need to know of a layer and a step (packed once per call by the host).
struct LinearArgs {
  // rows: q, k, v (and for decode the raw gate, decay and beta) at columns of `in`
  const float* in;         // portions: after the convolution; decode: the projection itself
  const float* raw;        // portions: where decay and beta columns are (the projection)
  const float* decay_raw;  // portions, DECAY_CHANNEL: rows of heads * N raw decays
  const float* a_log;      // [heads] (not DECAY_FIXED)
  const float* dt_bias;    // [heads] or [heads * N]
  const float* fixed;      // [heads] (DECAY_FIXED)
  const double* freq;      // rotation frequencies or null
  const int* positions;
  const int* row_start;
  const int* state_slot;
  float* state;
  float* scratch;          // portions: chunk matrices
  float* out;              // portions: heads * P answers a row
  // decode only
  const float* conv_weight;  // [channels][taps] or null
  const void* decay_up;      // [heads * N][decay_rank] (compute type)
  const void* gate_up;       // [heads * P][gate_rank] (compute type) or null
  const float* norm_weight;  // [P] or null
  void* gated;               // rows of heads * P, compute type
  long long state_stride;
  int ld_in, ld_raw, ld_decay, ld_out, ld_gated;
  int q_at, k_at, v_at, decay_at, beta_at, gate_at;
  int heads, kv_heads, N, P, taps, channels, ring_at;
  int decay_mode, delta, unit, gate_mode, decay_rank, gate_rank;
  int rot_dims, rot_layout;
  int requests, chunks;
  float q_scale, k_scale, eps, unit_eps;
};

__device__ __forceinline__ float la_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float la_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float la_softplus(float z) {  // log(1 + e^z), for any z
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}
// a decay; rate = -exp(A_log)
__device__ __forceinline__ float la_decay(float rate, float raw) {
  return expf(rate * la_softplus(raw));
}
__device__ __forceinline__ void la_sincos(int position, double f, float& s, float& c) {
  // the angle and its reduction to [-pi, pi] in double precision (see rope.cuh)
  const double two_pi = 6.283185307179586476925287, inv_two_pi = 0.159154943091895335768884;
  const double angle = (double)position * f;
  sincosf((float)(angle - two_pi * rint(angle * inv_two_pi)), &s, &c);
}

// ---------------------------------------------------------------------------------------------
// The portions' convolution: out[r][c] = silu(sum_l w[c][taps - 1 - l] in[row of t - l][c]), from
// this step's rows or, ahead of a request's first row, from its ring. A request's first
// taps - 1 rows and its ring belong to the CTA that holds its first row (the only reader and the
// only writer of the ring); every other row is the CTA's that holds it.
template <int TAPS>
__global__ void __launch_bounds__(128)
la_conv_kernel(const float* __restrict__ in, int ld_in, const float* __restrict__ w,
               float* __restrict__ ring, long long state_stride,
               const int* __restrict__ request_of_row, const int* __restrict__ row_start,
               const int* __restrict__ state_slot, const int* __restrict__ positions,
               float* __restrict__ out, int ld_out, int rows, int channels, int taps) {
  pdl_launch_dependents();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  float wv[TAPS];
#pragma unroll
  for (int l = 0; l < TAPS; ++l) wv[l] = l < taps ? w[(size_t)c * taps + taps - 1 - l] : 0.f;
  pdl_wait_for(in, ring);
  const int first = blockIdx.x * LA_CONV_ROWS, last = min(rows, first + LA_CONV_ROWS);
  if (TAPS <= 4 && last - first == LA_CONV_ROWS) {
    // the usual case, all rows well inside one request: every input is fetched once
    const int b = request_of_row[first];
    if (b >= 0 && b == request_of_row[last - 1] && state_slot[b] >= 0 &&
        first - row_start[b] >= taps - 1) {
      float u[LA_CONV_ROWS + TAPS - 1];
#pragma unroll
      for (int i = 0; i < LA_CONV_ROWS + TAPS - 1; ++i) {
        const int r = first + i - (TAPS - 1);
        u[i] = r >= first - (taps - 1) ? in[(size_t)r * ld_in + c] : 0.f;
      }
#pragma unroll
      for (int i = 0; i < LA_CONV_ROWS; ++i) {
        float acc = 0.f;
#pragma unroll
        for (int l = 0; l < TAPS; ++l) acc = fmaf(wv[l], u[i + TAPS - 1 - l], acc);
        out[(size_t)(first + i) * ld_out + c] = la_silu(acc);
      }
      return;
    }
  }
  for (int r = first; r < last; ++r) {
    const int b = request_of_row[r];
    if (b < 0 || state_slot[b] < 0) continue;
    const int r0 = row_start[b], j = r - r0;
    if (j == 0) {
      float* mine = ring + (size_t)state_slot[b] * state_stride;
      const int p = positions[r], count = row_start[b + 1] - r0;
      float kept[TAPS];  // kept[l]: the input l + 1 rows ahead of the request's first row
#pragma unroll
      for (int l = 0; l < TAPS; ++l) {
        kept[l] = (l + 1 < taps && p - l - 1 >= 0)
                      ? mine[(size_t)((p - l - 1) % taps) * channels + c] : 0.f;
      }
#pragma unroll
      for (int t = 0; t < TAPS; ++t) {
        if (t < taps - 1 && t < count) {
          float acc = 0.f;
#pragma unroll
          for (int l = 0; l < TAPS; ++l) {
            if (l < taps) {
              const float u = l <= t ? in[(size_t)(r + t - l) * ld_in + c]
                                     : kept[l - t - 1 >= 0 ? l - t - 1 : 0];
              acc = fmaf(wv[l], u, acc);
            }
          }
          out[(size_t)(r + t) * ld_out + c] = la_silu(acc);
        }
      }
      for (int t = max(0, count - taps); t < count; ++t) {
        mine[(size_t)((p + t) % taps) * channels + c] = in[(size_t)(r + t) * ld_in + c];
      }
    }
    if (j >= taps - 1) {
      float acc = 0.f;
#pragma unroll
      for (int l = 0; l < TAPS; ++l) {
        if (l < taps) acc = fmaf(wv[l], in[(size_t)(r - l) * ld_in + c], acc);
      }
      out[(size_t)r * ld_out + c] = la_silu(acc);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// A chunk's matrices in the scratch, per (chunk, head): M [N][2 C] (Kt of the C rows, then Qt),
// Kh [N][C], G [N] (padded to a multiple of 4), R [C][C].
__host__ __device__ __forceinline__ int la_pad4(int n) { return (n + 3) & ~3; }
__host__ __device__ __forceinline__ int la_chunk_floats(int N) {
  return 3 * LA_C * N + la_pad4(N) + LA_C * LA_C;
}

// The request that owns chunk `index` of the step and the chunk's first row in it.
__device__ __forceinline__ bool la_find_chunk(const int* row_start, int requests, int index, int& b,
                                              int& t0, int& count) {
  for (b = 0; b < requests; ++b) {
    const int rows = row_start[b + 1] - row_start[b];
    const int chunks = (rows + LA_C - 1) / LA_C;
    if (index < chunks) {
      t0 = index * LA_C;
      count = min(LA_C, rows - t0);
      return true;
    }
    index -= chunks;
  }
  return false;
}

// grid (chunks, heads). Shared memory: k, q, g and D_(C-1) k as [C][NS], NS = N padded to a
// multiple of 4 (the padding holds k = q = 0, g = 1). This kernel lets the scan start only when it
// has ended: CTAs of the scan that took their places beside it would crowd on the SMs that empty
// first, two or three on one (measured: 190 instead of 90 microseconds for 128 CTAs).
template <int NREG, bool CHANNEL>  // ceil(N / 32); a decay per channel, or one per row
__global__ void __launch_bounds__(LA_THREADS)
la_prepare_kernel(const LinearArgs a) {
  extern __shared__ __align__(16) float la_smem[];
  __shared__ __align__(16) float A[LA_C][LA_C], B[LA_C][LA_C], T[LA_C][LA_C];
  __shared__ float beta_s[LA_C];
  const int N = a.N, NS = la_pad4(N), h = blockIdx.y, kv = h / (a.heads / a.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* k_s = la_smem;
  float* q_s = k_s + LA_C * NS;
  float* g_s = q_s + LA_C * NS;
  float* w_s = g_s + LA_C * NS;
  int b, t0, count;
  const bool found = la_find_chunk(a.row_start, a.requests, blockIdx.x, b, t0, count);
  const float* in = a.in;
  const float* raw = a.raw;
  const float* decay_raw = a.decay_raw;
  float* scratch = a.scratch;
  pdl_wait_for(in, raw, decay_raw, scratch);
  if (!found) return;
  const int r0 = a.row_start[b] + t0;
  const float rate = a.decay_mode == DECAY_FIXED ? 0.f : -expf(a.a_log[h]);
  if (tid < LA_C * LA_C) {
    A[tid / LA_C][tid % LA_C] = 0.f;
    B[tid / LA_C][tid % LA_C] = 0.f;
  }
  // a warp per row: q and k (rotated, of unit length, scaled), the decays, beta
  for (int i = warp; i < LA_C; i += LA_THREADS / 32) {
    const bool row = i < count;
    const float* src = in + (size_t)(r0 + i) * a.ld_in;
    float k[NREG], q[NREG], g[NREG];
    float shared_g = 1.f;
    if (!CHANNEL && row) {
      shared_g = a.decay_mode == DECAY_FIXED
                     ? a.fixed[h]
                     : la_decay(rate, raw[(size_t)(r0 + i) * a.ld_raw + a.decay_at + h] +
                                          a.dt_bias[h]);
    }
#pragma unroll
    for (int m = 0; m < NREG; ++m) {
      const int n = lane + 32 * m;
      const bool live = row && n < N;
      k[m] = live ? src[a.k_at + kv * N + n] : 0.f;
      q[m] = live ? src[a.q_at + kv * N + n] : 0.f;
      g[m] = shared_g;
      if (CHANNEL) {
        g[m] = live ? la_decay(rate, decay_raw[(size_t)(r0 + i) * a.ld_decay + h * N + n] +
                                         a.dt_bias[h * N + n])
                    : 1.f;
      }
    }
    if (lane == 0) {
      beta_s[i] = (a.delta && row)
                      ? la_sigmoid(raw[(size_t)(r0 + i) * a.ld_raw + a.beta_at + h]) : 0.f;
    }
    float* kr = k_s + i * NS;
    float* qr = q_s + i * NS;
    if (a.rot_dims > 0) {
#pragma unroll
      for (int m = 0; m < NREG; ++m) {
        const int n = lane + 32 * m;
        if (n < N) {
          kr[n] = k[m];
          qr[n] = q[m];
        }
      }
      __syncwarp();
      if (row) {
        for (int pair = lane; pair < a.rot_dims / 2; pair += 32) {
          int x, y;
          rope_members(pair, a.rot_dims, a.rot_layout, x, y);
          float s, c;
          la_sincos(a.positions[r0 + i], a.freq[pair], s, c);
          const float ku = kr[x], kw = kr[y], qu = qr[x], qw = qr[y];
          kr[x] = ku * c - kw * s;
          kr[y] = kw * c + ku * s;
          qr[x] = qu * c - qw * s;
          qr[y] = qw * c + qu * s;
        }
      }
      __syncwarp();
#pragma unroll
      for (int m = 0; m < NREG; ++m) {
        const int n = lane + 32 * m;
        k[m] = n < N ? kr[n] : 0.f;
        q[m] = n < N ? qr[n] : 0.f;
      }
    }
    float kf = a.k_scale, qf = a.q_scale;
    if (a.unit) {
      float kk = 0.f, qq = 0.f;
#pragma unroll
      for (int m = 0; m < NREG; ++m) {
        kk = fmaf(k[m], k[m], kk);
        qq = fmaf(q[m], q[m], qq);
      }
      kf /= sqrtf(warp_sum(kk) + a.unit_eps);
      qf /= sqrtf(warp_sum(qq) + a.unit_eps);
    }
#pragma unroll
    for (int m = 0; m < NREG; ++m) {
      const int n = lane + 32 * m;
      if (n < NS) {
        kr[n] = k[m] * kf;
        qr[n] = q[m] * qf;
        g_s[i * NS + n] = g[m];
      }
    }
  }
  __syncthreads();
  float* chunk = scratch + ((size_t)blockIdx.x * a.heads + h) * la_chunk_floats(N);
  float* m_out = chunk;
  float* kh_out = m_out + 2 * LA_C * N;
  float* g_out = kh_out + LA_C * N;
  float* r_out = g_out + la_pad4(N);
  {
    // A, B and D_(C-1) k: warp w takes columns w and C - 1 - w, half a warp each, four
    // neighbouring channels a lane at a time
    constexpr int M = (NREG + 1) / 2;  // pieces of 16 lanes x 4 channels
    const int half = lane >> 4, l = lane & 15, j = half ? LA_C - 1 - warp : warp;
    float4 d[M];  // D_ij k_j (CHANNEL), else k_j, whose decays are one factor `dd`
    float dd = 1.f;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int n = 4 * (l + 16 * m);
      d[m] = n < NS ? *reinterpret_cast<const float4*>(k_s + j * NS + n)
                    : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int i = warp; i < LA_C; ++i) {  // (warp: the smaller of the two columns)
      float sa = 0.f, sb = 0.f;
      if (!CHANNEL && i > j) dd *= g_s[i * NS];
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int n = 4 * (l + 16 * m);
        if (n < NS) {
          const float4 k = *reinterpret_cast<const float4*>(k_s + i * NS + n);
          const float4 q = *reinterpret_cast<const float4*>(q_s + i * NS + n);
          if (CHANNEL && i > j) {
            const float4 g = *reinterpret_cast<const float4*>(g_s + i * NS + n);
            d[m].x *= g.x;
            d[m].y *= g.y;
            d[m].z *= g.z;
            d[m].w *= g.w;
          }
          sa = fmaf(k.x, d[m].x, fmaf(k.y, d[m].y, fmaf(k.z, d[m].z, fmaf(k.w, d[m].w, sa))));
          sb = fmaf(q.x, d[m].x, fmaf(q.y, d[m].y, fmaf(q.z, d[m].z, fmaf(q.w, d[m].w, sb))));
        }
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) {
        sa += __shfl_xor_sync(0xffffffffu, sa, o);
        sb += __shfl_xor_sync(0xffffffffu, sb, o);
      }
      if (l == 0 && i >= j) {
        A[i][j] = sa * dd;
        B[i][j] = sb * dd;
      }
    }
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int n = 4 * (l + 16 * m);
      if (n < NS) {
        *reinterpret_cast<float4*>(w_s + j * NS + n) =
            make_float4(d[m].x * dd, d[m].y * dd, d[m].z * dd, d[m].w * dd);
      }
    }
  }
  __syncthreads();
  if (warp == 0) {
    if (lane < LA_C) {  // column `lane` of T, from the top (x[m] is 0 above the diagonal)
      float x[LA_C];
#pragma unroll
      for (int i = 0; i < LA_C; ++i) {
        float s = i == lane ? 1.f : 0.f;
        if (a.delta) {
#pragma unroll
          for (int m = 0; m < i; ++m) s = fmaf(-A[i][m], x[m], s);
          s *= beta_s[i];
        }
        x[i] = s;
        T[i][lane] = s;
      }
    }
  } else {  // meanwhile Kt and Qt (four rows of a channel a thread) and G
    for (int idx = tid - 32; idx < N * 8; idx += LA_THREADS - 32) {
      const int n = idx >> 3, part = idx & 7, first = (part & 3) * 4;
      const float* x = part < 4 ? k_s : q_s;
      float g = 1.f;
      for (int i = 0; i < first; ++i) g *= g_s[i * NS + n];
      float v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        g *= g_s[(first + i) * NS + n];
        v[i] = g * x[(first + i) * NS + n];
      }
      *reinterpret_cast<float4*>(m_out + (size_t)n * 2 * LA_C + part * 4) =
          make_float4(v[0], v[1], v[2], v[3]);
      if (part == 3) g_out[n] = g;
    }
  }
  __syncthreads();
  if (tid < LA_C * LA_C) {  // (B and T are zero above the diagonal)
    const int i = tid / LA_C, j = tid % LA_C;
    float s = 0.f;
#pragma unroll
    for (int m = 0; m < LA_C; ++m) s = fmaf(B[i][m], T[m][j], s);
    r_out[tid] = s;
  }
  for (int idx = tid; idx < N * (LA_C / 4); idx += LA_THREADS) {
    const int n = idx / (LA_C / 4), j = idx % (LA_C / 4) * 4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < LA_C; ++i) {
      const float d = w_s[i * NS + n];
      const float4 t = *reinterpret_cast<const float4*>(&T[i][j]);
      s.x = fmaf(t.x, d, s.x);
      s.y = fmaf(t.y, d, s.y);
      s.z = fmaf(t.z, d, s.z);
      s.w = fmaf(t.w, d, s.w);
    }
    *reinterpret_cast<float4*>(kh_out + (size_t)n * LA_C + j) = s;
  }
}

// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ void la_copy16(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void la_copy4(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void la_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// floats of one stage (a chunk's matrices and its values) and of the rest of shared memory
__host__ __device__ __forceinline__ int la_stage_floats(int N) {
  return la_chunk_floats(N) + LA_C * LA_COLS;
}
__host__ __device__ __forceinline__ int la_fixed_floats(int N) {
  return N * LA_COLS + 8 * 2 * LA_C * LA_COLS + LA_C * LA_COLS;
}

// grid (heads, requests, tiles of LA_COLS columns). Per chunk: [Kt; Qt] S_0 with the channels
// shared out over the eight warps (a warp's lanes hold 4 x 4 pieces of the 32 x 16 result), the
// warps' shares added up, W; then O and the new state from W.
template <int STAGES>
__global__ void __launch_bounds__(LA_THREADS)
la_scan_kernel(const LinearArgs a, int vec) {
  extern __shared__ __align__(16) float la_smem[];
  pdl_launch_dependents();
  const int N = a.N, P = a.P, h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * LA_COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int stage_floats = la_stage_floats(N), chunk_floats = la_chunk_floats(N);
  float* s_s = la_smem + (size_t)STAGES * stage_floats;  // [N][LA_COLS]
  float* red = s_s + N * LA_COLS;                        // [8 warps][4][32 lanes][4]
  float* w_s = red + 8 * 2 * LA_C * LA_COLS;             // [C][LA_COLS]
  const int r0 = a.row_start[b], rows = a.row_start[b + 1] - r0;
  if (a.state_slot[b] < 0 || rows <= 0) return;
  int before = 0;  // chunks of the requests ahead
  for (int i = 0; i < b; ++i) {
    before += (a.row_start[i + 1] - a.row_start[i] + LA_C - 1) / LA_C;
  }
  float* mine = a.state + (size_t)a.state_slot[b] * a.state_stride + (size_t)h * N * P;
  const float* in = a.in;
  const float* scratch = a.scratch;
  pdl_wait_for(in, scratch, mine);
  const int chunks = (rows + LA_C - 1) / LA_C;
  auto stage = [&](int c) {
    float* at = la_smem + (size_t)(STAGES == 1 ? 0 : c % STAGES) * stage_floats;
    const float* from = scratch + ((size_t)(before + c) * a.heads + h) * chunk_floats;
    for (int i = tid * 4; i < chunk_floats; i += LA_THREADS * 4) la_copy16(at + i, from + i);
    float* v_s = at + chunk_floats;
    const int t0 = c * LA_C, count = min(LA_C, rows - t0);
    const float* v = in + (size_t)(r0 + t0) * a.ld_in + a.v_at + h * P + p0;
    if (vec) {
      if (tid < LA_C * LA_COLS / 4) {
        const int i = tid / (LA_COLS / 4), j = tid % (LA_COLS / 4) * 4;
        if (i < count && p0 + j < P) {
          la_copy16(v_s + i * LA_COLS + j, v + (size_t)i * a.ld_in + j);
        } else {
          *reinterpret_cast<float4*>(v_s + i * LA_COLS + j) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
    } else {
      const int i = tid / LA_COLS, j = tid % LA_COLS;
      if (i < count && p0 + j < P) {
        la_copy4(v_s + tid, v + (size_t)i * a.ld_in + j);
      } else {
        v_s[tid] = 0.f;
      }
    }
  };
  if (STAGES > 1) {
#pragma unroll
    for (int c = 0; c < STAGES - 1; ++c) {
      if (c < chunks) stage(c);
      la_commit();
    }
  }
  for (int idx = tid; idx < N * LA_COLS; idx += LA_THREADS) {
    const int n = idx / LA_COLS, c = idx % LA_COLS;
    s_s[idx] = p0 + c < P ? mine[(size_t)n * P + p0 + c] : 0.f;
  }
  const int rg = lane >> 2, cg = lane & 3;
  // the result's element this thread finishes: its two rows of a warp lie in different quads of
  // rows at the same place, so that a warp reads 32 neighbouring floats of a share
  const int pr = tid >> 4, col = tid & 15;
  const int row = (pr & 1) * 4 + ((pr >> 1) & 3) + (pr >> 3) * 8;
  const int red_at = ((row & 3) * 32 + (row >> 2) * 4) * 4 + col;
  for (int c = 0; c < chunks; ++c) {
    if (STAGES == 1) {
      __syncthreads();
      stage(c);
      la_commit();
      la_wait<0>();
      __syncthreads();
    } else {
      la_wait<(STAGES > 1 ? STAGES - 2 : 0)>();
      __syncthreads();  // chunk c has landed, and everyone is done with chunk c - 1
      if (c + STAGES - 1 < chunks) stage(c + STAGES - 1);
      la_commit();
    }
    const float* m_s = la_smem + (size_t)(STAGES == 1 ? 0 : c % STAGES) * stage_floats;
    const float* kh_s = m_s + 2 * LA_C * N;
    const float* g_s = kh_s + LA_C * N;
    const float* r_s = g_s + la_pad4(N);
    const float* v_s = m_s + chunk_floats;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 4
    for (int n = warp; n < N; n += 8) {
      const float4 m = *reinterpret_cast<const float4*>(m_s + (size_t)n * 2 * LA_C + rg * 4);
      const float4 s = *reinterpret_cast<const float4*>(s_s + n * LA_COLS + cg * 4);
      const float mv[4] = {m.x, m.y, m.z, m.w}, sv[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(mv[i], sv[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      *reinterpret_cast<float4*>(red + ((warp * 4 + i) * 32 + lane) * 4) =
          make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    }
    __syncthreads();
    float seen = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      seen += red[w * 512 + red_at];
      o += red[w * 512 + red_at + 64];  // the same place of the rows of Qt (16 rows on)
    }
    const float v = v_s[row * LA_COLS + col];
    w_s[row * LA_COLS + col] = a.delta ? v - seen : v;
    __syncthreads();
    float wc[LA_C];
#pragma unroll
    for (int j = 0; j < LA_C; ++j) wc[j] = w_s[j * LA_COLS + col];
#pragma unroll
    for (int j = 0; j < LA_C; j += 4) {
      const float4 r = *reinterpret_cast<const float4*>(r_s + row * LA_C + j);
      o = fmaf(r.x, wc[j], o);
      o = fmaf(r.y, wc[j + 1], o);
      o = fmaf(r.z, wc[j + 2], o);
      o = fmaf(r.w, wc[j + 3], o);
    }
    const int t = c * LA_C + row;
    if (t < rows && p0 + col < P) a.out[(size_t)(r0 + t) * a.ld_out + h * P + p0 + col] = o;
    for (int item = tid; item < N * 4; item += LA_THREADS) {
      const int n = item >> 2, cq = (item & 3) * 4;
      float4 s = *reinterpret_cast<float4*>(s_s + n * LA_COLS + cq);
      const float g = g_s[n];
      s.x *= g;
      s.y *= g;
      s.z *= g;
      s.w *= g;
#pragma unroll
      for (int j = 0; j < LA_C; j += 4) {
        const float4 k = *reinterpret_cast<const float4*>(kh_s + n * LA_C + j);
        const float kv[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 w = *reinterpret_cast<const float4*>(w_s + (j + e) * LA_COLS + cq);
          s.x = fmaf(kv[e], w.x, s.x);
          s.y = fmaf(kv[e], w.y, s.y);
          s.z = fmaf(kv[e], w.z, s.z);
          s.w = fmaf(kv[e], w.w, s.w);
        }
      }
      *reinterpret_cast<float4*>(s_s + n * LA_COLS + cq) = s;
    }
  }
  __syncthreads();
  for (int idx = tid; idx < N * LA_COLS; idx += LA_THREADS) {
    const int n = idx / LA_COLS, c = idx % LA_COLS;
    if (p0 + c < P) mine[(size_t)n * P + p0 + c] = s_s[idx];
  }
}

// ---------------------------------------------------------------------------------------------
// Single rows. grid (heads, rows). A tile of PT columns of S at a time: thread (group, column)
// holds the entries group, group + G, ... of its column (G = threads / PT groups), which meet in
// shared memory. `first_of_kv` heads write the ring's query and key inputs for their group.
template <typename T> struct LaPiece;
template <> struct LaPiece<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ float dot(const float* w, const float* x) {
    const float4 v = *reinterpret_cast<const float4*>(w);
    return fmaf(v.x, x[0], fmaf(v.y, x[1], fmaf(v.z, x[2], v.w * x[3])));
  }
};
template <> struct LaPiece<__nv_bfloat16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ float dot(const __nv_bfloat16* w, const float* x) {
    const uint4 raw = *reinterpret_cast<const uint4*>(w);
    const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 v = __bfloat1622float2(pair[i]);
      s = fmaf(v.x, x[2 * i], s);
      s = fmaf(v.y, x[2 * i + 1], s);
    }
    return s;
  }
};

// out[o] = sum_r W[o][r] x[r] for o < count, four lanes an output
template <typename T, typename F>
__device__ __forceinline__ void la_matvec(const T* W, const float* x, int rank, int count, F store) {
  const int part = threadIdx.x & 3;
  const bool pieces = rank % LaPiece<T>::N == 0 && ((uintptr_t)W % 16) == 0;
  for (int o0 = 0; o0 < count; o0 += blockDim.x / 4) {  // (uniform: every lane shuffles)
    const int o = o0 + threadIdx.x / 4;
    float s = 0.f;
    if (o < count) {
      const T* w = W + (size_t)o * rank;
      if (pieces) {
        for (int r = part * LaPiece<T>::N; r < rank; r += 4 * LaPiece<T>::N) {
          s += LaPiece<T>::dot(w + r, x + r);
        }
      } else {
        for (int r = part; r < rank; r += 4) s = fmaf(ldf(w + r), x[r], s);
      }
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    if (o < count && part == 0) store(o, s);
  }
}

// `bytes` from p on towards L2, shared out over the CTA. (A prefetch reads nothing, so what the
// kernel ahead may still be writing may be named ahead of the dependency wait.)
__device__ __forceinline__ void la_prefetch(const void* p, size_t bytes) {
  const char* at = reinterpret_cast<const char*>(p);
  for (size_t o = (size_t)threadIdx.x * 128; o < bytes; o += (size_t)blockDim.x * 128) {
    asm volatile("prefetch.global.L2 [%0];" ::"l"(at + o));
  }
}

template <typename T, int RN>
__global__ void __launch_bounds__(512)
la_decode_kernel(const LinearArgs a, int PT) {
  extern __shared__ __align__(16) float la_smem[];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  const int N = a.N, P = a.P, h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
  const int threads = blockDim.x, lane = tid & 31, warp = tid >> 5;
  const int per = a.heads / a.kv_heads, kv = h / per;
  float* q_s = la_smem;
  float* k_s = q_s + N;
  float* g_s = k_s + N;
  float* v_s = g_s + N;
  float* z_s = v_s + P;        // the output gate's factor
  float* o_s = z_s + P;        // the head's answers
  float* low_s = o_s + P;      // the low-rank inputs of the decay and of the gate
  float* red = low_s + a.decay_rank + a.gate_rank;  // [2][threads]
  const int slot = a.state_slot[r], position = a.positions[r];
  T* dst = reinterpret_cast<T*>(a.gated) + (size_t)r * a.ld_gated + (size_t)h * P;
  const float* in = a.in;
  float* state = a.state;
  if (slot >= 0) {
    const float* own = state + (size_t)slot * a.state_stride;
    la_prefetch(own + (size_t)h * N * P, (size_t)N * P * sizeof(float));
    if (a.decay_rank > 0) {
      la_prefetch((const T*)a.decay_up + (size_t)h * N * a.decay_rank,
                  (size_t)N * a.decay_rank * sizeof(T));
    }
    if (a.gate_rank > 0) {
      la_prefetch((const T*)a.gate_up + (size_t)h * P * a.gate_rank,
                  (size_t)P * a.gate_rank * sizeof(T));
    }
  }
  pdl_wait_for(in, state);
  if (slot < 0) {  // a row of padding (a graph's bucket): no request, no state
    for (int p = tid; p < P; p += threads) stf(dst + p, 0.f);
    return;
  }
  const float* row = in + (size_t)r * a.ld_in;
  float* mine = state + (size_t)slot * a.state_stride + (size_t)h * N * P;
  const int G = threads / PT, group = tid / PT, column = tid % PT;
  float s[RN];  // the first tile's entries are on their way while the row's factors are formed
  auto fetch = [&](int p0) {
#pragma unroll
    for (int m = 0; m < RN; ++m) {
      const int n = group + G * m;
      s[m] = (n < N && p0 + column < P) ? mine[(size_t)n * P + p0 + column] : 0.f;
    }
  };
  fetch(0);
  for (int i = tid; i < a.decay_rank; i += threads) low_s[i] = row[a.decay_at + i];
  for (int i = tid; i < a.gate_rank; i += threads) low_s[a.decay_rank + i] = row[a.gate_at + i];
  if (a.conv_weight != nullptr) {
    float* ring = state + (size_t)slot * a.state_stride + a.ring_at;
    const int taps = a.taps, now = position % taps;
    for (int idx = tid; idx < 2 * N + P; idx += threads) {
      const int part = idx < N ? 0 : (idx < 2 * N ? 1 : 2);
      const int e = idx - part * N;
      const int c = part == 0 ? a.q_at + kv * N + e
                              : (part == 1 ? a.k_at + kv * N + e : a.v_at + h * P + e);
      const int channel = c - a.q_at;  // (q, k and v lie side by side from q_at on)
      const float* w = a.conv_weight + (size_t)channel * taps;
      const float x = row[c];
      float acc = w[taps - 1] * x;
      for (int l0 = 1; l0 < taps; l0 += 3) {  // three earlier inputs on their way at once
        float u[3], f[3];
#pragma unroll
        for (int e = 0; e < 3; ++e) {
          const int l = l0 + e;
          int at = now - l;
          if (at < 0) at += taps;
          const bool live = l < taps && l <= position;
          u[e] = live ? ring[(size_t)at * a.channels + channel] : 0.f;
          f[e] = live ? w[taps - 1 - l] : 0.f;
        }
#pragma unroll
        for (int e = 0; e < 3; ++e) acc = fmaf(f[e], u[e], acc);
      }
      (part == 0 ? q_s : (part == 1 ? k_s : v_s))[e] = la_silu(acc);
      if (part == 2 || h % per == 0) ring[(size_t)now * a.channels + channel] = x;
    }
  } else {
    for (int i = tid; i < N; i += threads) {
      q_s[i] = row[a.q_at + kv * N + i];
      k_s[i] = row[a.k_at + kv * N + i];
    }
    for (int i = tid; i < P; i += threads) v_s[i] = row[a.v_at + h * P + i];
  }
  if (a.gate_mode != HEAD_GATE_NONE && a.gate_rank == 0) {
    for (int p = tid; p < P; p += threads) {
      const float z = row[a.gate_at + h * P + p];
      z_s[p] = a.gate_mode == HEAD_GATE_SILU ? la_silu(z) : la_sigmoid(z);
    }
  }
  if (a.decay_mode == DECAY_HEAD) {
    const float g = la_decay(-expf(a.a_log[h]), row[a.decay_at + h] + a.dt_bias[h]);
    for (int n = tid; n < N; n += threads) g_s[n] = g;
  } else if (a.decay_mode == DECAY_FIXED) {
    for (int n = tid; n < N; n += threads) g_s[n] = a.fixed[h];
  }
  const float beta = a.delta ? la_sigmoid(row[a.beta_at + h]) : 1.f;
  __syncthreads();
  if (a.decay_mode == DECAY_CHANNEL) {
    const float rate = -expf(a.a_log[h]);
    la_matvec((const T*)a.decay_up + (size_t)h * N * a.decay_rank, low_s, a.decay_rank, N,
              [&](int n, float z) { g_s[n] = la_decay(rate, z + a.dt_bias[h * N + n]); });
  }
  if (a.gate_rank > 0) {
    la_matvec((const T*)a.gate_up + (size_t)h * P * a.gate_rank, low_s + a.decay_rank,
              a.gate_rank, P, [&](int p, float z) {
                z_s[p] = a.gate_mode == HEAD_GATE_SILU ? la_silu(z) : la_sigmoid(z);
              });
  }
  if (a.rot_dims > 0) {
    for (int i = tid; i < a.rot_dims / 2; i += threads) {
      int x, y;
      rope_members(i, a.rot_dims, a.rot_layout, x, y);
      float sn, cs;
      la_sincos(position, a.freq[i], sn, cs);
      const float ku = k_s[x], kw = k_s[y], qu = q_s[x], qw = q_s[y];
      k_s[x] = ku * cs - kw * sn;
      k_s[y] = kw * cs + ku * sn;
      q_s[x] = qu * cs - qw * sn;
      q_s[y] = qw * cs + qu * sn;
    }
    __syncthreads();
  }
  if (warp < 2) {  // one warp per vector: its length and scale
    float* x = warp == 0 ? q_s : k_s;
    float f = warp == 0 ? a.q_scale : a.k_scale;
    if (a.unit) {
      float ss = 0.f;
      for (int n = lane; n < N; n += 32) ss = fmaf(x[n], x[n], ss);
      f /= sqrtf(warp_sum(ss) + a.unit_eps);
    }
    for (int n = lane; n < N; n += 32) x[n] *= f;
  }
  __syncthreads();
  for (int p0 = 0; p0 < P; p0 += PT) {
    if (p0 > 0) fetch(p0);
    const int p = p0 + column;
    float seen = 0.f;
#pragma unroll
    for (int m = 0; m < RN; ++m) {
      const int n = group + G * m;
      if (n < N) {
        s[m] *= g_s[n];
        seen = fmaf(s[m], k_s[n], seen);
      }
    }
    float u = p < P ? v_s[p] : 0.f;
    if (a.delta) {
      red[tid] = seen;
      __syncthreads();
      float total = 0.f;
      for (int g = 0; g < G; ++g) total += red[g * PT + column];
      u = beta * (u - total);
    }
    float o = 0.f;
#pragma unroll
    for (int m = 0; m < RN; ++m) {
      const int n = group + G * m;
      if (n < N) {
        s[m] = fmaf(k_s[n], u, s[m]);
        o = fmaf(s[m], q_s[n], o);
        if (p < P) mine[(size_t)n * P + p] = s[m];
      }
    }
    red[threads + tid] = o;
    __syncthreads();
    if (group == 0 && p < P) {
      float total = 0.f;
      for (int g = 0; g < G; ++g) total += red[threads + g * PT + column];
      o_s[p] = total;
    }
    if (p0 + PT < P) __syncthreads();  // (the next tile writes `red` again)
  }
  float ss = 0.f;
  __syncthreads();
  for (int p = tid; p < P; p += threads) ss = fmaf(o_s[p], o_s[p], ss);
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)P + a.eps);
  for (int p = tid; p < P; p += threads) {
    float v = o_s[p] * inv;
    if (a.norm_weight != nullptr) v *= a.norm_weight[p];
    if (a.gate_mode != HEAD_GATE_NONE) v *= z_s[p];
    stf(dst + p, v);
  }
}

template <typename T>
int la_decode(const LinearArgs& a, int rows, cudaStream_t s) {
  const int threads = a.N > 256 || a.N * a.P > 4096 ? 512 : 256;
  int PT = 256;
  while (PT > 32 && (PT / 2 >= a.P || a.N > 32 * (threads / PT))) PT /= 2;
  const int entries = (a.N + threads / PT - 1) / (threads / PT);
  const size_t smem = (size_t)(3 * a.N + 3 * a.P + a.decay_rank + a.gate_rank + 2 * threads) *
                      sizeof(float);
#define AYK_LA_DECODE(RN)                                                                       \
  {                                                                                             \
    static const bool allowed =                                                                 \
        (cudaFuncSetAttribute(la_decode_kernel<T, RN>,                                          \
                              cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024), true);   \
    (void)allowed;                                                                              \
    return launch_kernel(la_decode_kernel<T, RN>, dim3(a.heads, rows), dim3(threads), smem, s,  \
                         1, a, PT);                                                             \
  }
  if (entries <= 8) AYK_LA_DECODE(8)
  if (entries <= 16) AYK_LA_DECODE(16)
  AYK_LA_DECODE(32)
#undef AYK_LA_DECODE
}

static bool la_common_ok(const LinearArgs& a) {
  return a.heads >= 1 && a.kv_heads >= 1 && a.heads % a.kv_heads == 0 && a.N >= 1 && a.P >= 1 &&
         a.in != nullptr && a.state != nullptr && a.state_slot != nullptr &&
         a.positions != nullptr && a.rot_dims >= 0 && a.rot_dims % 2 == 0 && a.rot_dims <= a.N &&
         (a.rot_dims == 0 || a.freq != nullptr) && a.eps > 0.f &&
         (a.decay_mode == DECAY_FIXED ? a.fixed != nullptr
                                      : a.a_log != nullptr && a.dt_bias != nullptr) &&
         a.decay_mode >= DECAY_FIXED && a.decay_mode <= DECAY_CHANNEL && a.q_at >= 0 &&
         a.k_at >= 0 && a.v_at >= 0 && a.ld_in >= a.v_at + a.heads * a.P &&
         a.ld_in >= a.k_at + a.kv_heads * a.N && a.ld_in >= a.q_at + a.kv_heads * a.N &&
         a.state_stride >= (long long)a.heads * a.N * a.P;
}

}  // namespace ayk

AYK_API void ayk_set_pdl(int on) { ayk::pdl_enabled() = on; }

AYK_API int ayk_linear_chunk_rows() { return ayk::LA_C; }
AYK_API int ayk_linear_args_bytes() { return (int)sizeof(ayk::LinearArgs); }
// floats of the scratch per (chunk, head)
AYK_API int ayk_linear_chunk_floats(int n) { return ayk::la_chunk_floats(n); }

// `ring`: the first float of slot 0's ring; slots are state_stride floats apart.
AYK_API int ayk_conv_ring(const float* in, int ld_in, const float* w, float* ring,
                          long long state_stride, const int* request_of_row,
                          const int* row_start, const int* state_slot, const int* positions,
                          float* out, int ld_out, int rows, int channels, int taps,
                          void* stream) {
  using namespace ayk;
  if (rows == 0 || channels == 0) return AYK_OK;
  if (rows < 0 || channels < 0 || taps < 1 || in == nullptr || w == nullptr || ring == nullptr ||
      request_of_row == nullptr || row_start == nullptr || state_slot == nullptr ||
      positions == nullptr || out == nullptr || ld_in < channels || ld_out < channels) {
    return AYK_BAD_ARGUMENT;
  }
  const int tiles = (channels + 127) / 128;
  if (taps > LA_MAX_TAPS || tiles > 65535) return AYK_TOO_LARGE;
  const dim3 grid((rows + LA_CONV_ROWS - 1) / LA_CONV_ROWS, tiles);
  if (taps <= 4) {
    return launch_kernel(la_conv_kernel<4>, grid, dim3(128), 0, (cudaStream_t)stream, 1, in, ld_in,
                         w, ring, state_stride, request_of_row, row_start, state_slot, positions,
                         out, ld_out, rows, channels, taps);
  }
  return launch_kernel(la_conv_kernel<LA_MAX_TAPS>, grid, dim3(128), 0, (cudaStream_t)stream, 1,
                       in, ld_in, w, ring, state_stride, request_of_row, row_start, state_slot,
                       positions, out, ld_out, rows, channels, taps);
}

// A step's rows in chunks: two launches. `args->chunks` is the step's count of chunks (the sum
// over requests of their rows over LA_C, rounded up); the scratch holds chunks * heads *
// ayk_linear_chunk_floats(N) floats and starts on 16 bytes.
AYK_API int ayk_linear_chunks(const ayk::LinearArgs* args, void* stream) {
  using namespace ayk;
  if (args == nullptr) return AYK_BAD_ARGUMENT;
  const LinearArgs& a = *args;
  if (a.chunks == 0 || a.requests == 0) return AYK_OK;
  if (!la_common_ok(a) || a.chunks < 0 || a.requests < 0 || a.row_start == nullptr ||
      a.scratch == nullptr || a.out == nullptr || a.ld_out < a.heads * a.P ||
      (a.decay_mode == DECAY_CHANNEL &&
       (a.decay_raw == nullptr || a.ld_decay < a.heads * a.N)) ||
      ((a.delta || a.decay_mode == DECAY_HEAD) && a.raw == nullptr) ||
      (a.delta && a.ld_raw < a.beta_at + a.heads) ||
      (a.decay_mode == DECAY_HEAD && a.ld_raw < a.decay_at + a.heads)) {
    return AYK_BAD_ARGUMENT;
  }
  if (((uintptr_t)a.scratch % 16) != 0) return AYK_BAD_ALIGNMENT;
  const int tiles = (a.P + LA_COLS - 1) / LA_COLS;
  if (a.N > LA_MAX_N || a.heads > 65535 || a.requests > 65535 || tiles > 65535) {
    return AYK_TOO_LARGE;
  }
  cudaStream_t s = (cudaStream_t)stream;
  const size_t smem = (size_t)4 * LA_C * la_pad4(a.N) * sizeof(float);
  int status;
#define AYK_LA_PREPARE_AS(NREG, CHANNEL)                                                         \
  {                                                                                              \
    static const bool allowed =                                                                  \
        (cudaFuncSetAttribute(la_prepare_kernel<NREG, CHANNEL>,                                  \
                              cudaFuncAttributeMaxDynamicSharedMemorySize,                       \
                              4 * LA_C * 32 * NREG * (int)sizeof(float)), true);                 \
    (void)allowed;                                                                               \
    status = launch_kernel(la_prepare_kernel<NREG, CHANNEL>, dim3(a.chunks, a.heads),            \
                           dim3(LA_THREADS), smem, s, 1, a);                                     \
  }
#define AYK_LA_PREPARE(NREG)                                                                     \
  {                                                                                              \
    if (a.decay_mode == DECAY_CHANNEL) AYK_LA_PREPARE_AS(NREG, true)                             \
    else AYK_LA_PREPARE_AS(NREG, false)                                                          \
  }
  if (a.N <= 32) AYK_LA_PREPARE(1)
  else if (a.N <= 64) AYK_LA_PREPARE(2)
  else if (a.N <= 128) AYK_LA_PREPARE(4)
  else if (a.N <= 256) AYK_LA_PREPARE(8)
  else AYK_LA_PREPARE(16)
#undef AYK_LA_PREPARE
#undef AYK_LA_PREPARE_AS
  if (status != AYK_OK) return status;
  const int vec = ((uintptr_t)a.in % 16) == 0 && a.ld_in % 4 == 0 && a.v_at % 4 == 0 &&
                  a.P % 4 == 0;
  const dim3 grid(a.heads, a.requests, tiles);
#define AYK_LA_SCAN(STAGES)                                                                      \
  {                                                                                              \
    static const bool allowed =                                                                  \
        (cudaFuncSetAttribute(la_scan_kernel<STAGES>,                                            \
                              cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024), true);   \
    (void)allowed;                                                                               \
    return launch_kernel(la_scan_kernel<STAGES>, grid, dim3(LA_THREADS),                         \
                         ((size_t)STAGES * la_stage_floats(a.N) + la_fixed_floats(a.N)) *        \
                             sizeof(float),                                                      \
                         s, 1, a, vec);                                                          \
  }
  if (a.N <= 128) AYK_LA_SCAN(3)
  if (a.N <= 320) AYK_LA_SCAN(2)
  AYK_LA_SCAN(1)
#undef AYK_LA_SCAN
}

// A step of single rows, row r of request r: one launch. type: 0 = float32, 1 = bfloat16, of
// `gated`, `decay_up` and `gate_up`.
AYK_API int ayk_linear_decode(const ayk::LinearArgs* args, int rows, int type, void* stream) {
  using namespace ayk;
  if (rows == 0) return AYK_OK;
  if (args == nullptr) return AYK_BAD_ARGUMENT;
  const LinearArgs& a = *args;
  if (!la_common_ok(a) || rows < 0 || a.gated == nullptr || a.ld_gated < a.heads * a.P ||
      a.decay_rank < 0 || a.gate_rank < 0 || a.gate_mode < HEAD_GATE_NONE ||
      a.gate_mode > HEAD_GATE_SILU || (type != 0 && type != 1) ||
      ((a.decay_mode == DECAY_CHANNEL) != (a.decay_rank > 0)) ||
      (a.decay_rank > 0 && (a.decay_up == nullptr || a.ld_in < a.decay_at + a.decay_rank)) ||
      (a.gate_rank > 0 && (a.gate_up == nullptr || a.ld_in < a.gate_at + a.gate_rank)) ||
      (a.gate_rank == 0 && a.gate_mode != HEAD_GATE_NONE &&
       a.ld_in < a.gate_at + a.heads * a.P) ||
      (a.delta && a.ld_in < a.beta_at + a.heads) ||
      (a.decay_mode == DECAY_HEAD && a.ld_in < a.decay_at + a.heads) ||
      (a.conv_weight != nullptr &&
       (a.taps < 1 || a.k_at != a.q_at + a.kv_heads * a.N || a.v_at != a.k_at + a.kv_heads * a.N ||
        a.channels != 2 * a.kv_heads * a.N + a.heads * a.P || a.ring_at < a.heads * a.N * a.P ||
        a.state_stride < (long long)a.ring_at + (long long)a.taps * a.channels))) {
    return AYK_BAD_ARGUMENT;
  }
  if (a.N > LA_MAX_N || a.P > 2048 || a.decay_rank > 2048 || a.gate_rank > 2048 ||
      rows > 65535) {
    return AYK_TOO_LARGE;
  }
  if (type == 0) return la_decode<float>(a, rows, (cudaStream_t)stream);
  return la_decode<__nv_bfloat16>(a, rows, (cudaStream_t)stream);
}
