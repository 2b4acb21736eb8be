// Recurrences with a matrix state per head and one decay per head: the gated delta rule and the linear attention with a
// fixed decay (retention). All arithmetic is float32; the states live in the cache's per-sequence regions [slots, H, N, P]
// (N key channels, P value channels) and are indexed by the step's slots.
//
//   rotate_rows_kernel     the first channels of every unit of a float32 row turn in pairs, in place
//   delta_prep_kernel      q and k units divided by their length, in place (q also scaled); beta = sigmoid(b);
//                          log decay = -exp(A_log) softplus(a + dt_bias)
//   state_walk_kernel      either recurrence token by token: S <- g S, u = beta (v - S^T k) or v, S <- S + k u^T, o = S^T q
//   chunk_solve_kernel, chunk_state_kernel, chunk_out_kernel   the same for long portions, in chunks of 64 tokens (below)
//   state_token_kernel     a whole single-token step of either recurrence behind the projections: what the two kernels above
//                          (or the rotation) do, the recurrence, the head's norm and the silu gate, in one launch
#include <math.h>

#include "common.cuh"

namespace slb {

__device__ __forceinline__ float sigmoid_of(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_of(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_of(float v) { return v > 20.0f ? v : log1pf(expf(v)); }

// One thread per (token, unit, pair). rows: [tokens, stride], the first units * dim values of a row are the units.
__global__ void __launch_bounds__(256) rotate_rows_kernel(float* __restrict__ rows, long long stride, const float* __restrict__ cos,
                                                          const float* __restrict__ sin, const int* __restrict__ tok_pos,
                                                          long long total, int units, int dim, int half, int neighbours) {
  pdl_enter();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int pair = (int)(i % half);
  const long long r = i / half;
  const int u = (int)(r % units);
  const long long t = r / units;
  float* x = rows + (size_t)t * stride + (size_t)u * dim + (neighbours ? 2 * pair : pair);
  float* y = x + (neighbours ? 1 : half);
  const size_t at = (size_t)tok_pos[t] * half + pair;
  const float c = cos[at], s = sin[at], a = *x, b = *y;
  *x = a * c - b * s;
  *y = b * c + a * s;
}

// One warp per (token, q or k unit) and one per token for the scalars of its H heads.
__global__ void __launch_bounds__(256) delta_prep_kernel(float* __restrict__ rows, long long stride, int units, int q_units, int dim,
                                                         float q_scale, float unit_eps, const float* __restrict__ raw_beta,
                                                         const float* __restrict__ raw_step, long long raw_stride,
                                                         const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                                                         float* __restrict__ beta, float* __restrict__ log_decay, int tokens, int H) {
  pdl_enter();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)tokens * (units + 1)) return;
  const int t = (int)(item / (units + 1)), u = (int)(item - (long long)t * (units + 1));
  if (u == units) {
    for (int h = lane; h < H; h += 32) {
      const size_t i = (size_t)t * raw_stride + h;
      beta[(size_t)t * H + h] = sigmoid_of(raw_beta[i]);
      log_decay[(size_t)t * H + h] = -expf(a_log[h]) * softplus_of(raw_step[i] + dt_bias[h]);
    }
    return;
  }
  float* x = rows + (size_t)t * stride + (size_t)u * dim;
  float v[8];                          // dim is at most 256
  float ss = 0.0f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = lane + 32 * j;
    v[j] = c < dim ? x[c] : 0.0f;
    ss = fmaf(v[j], v[j], ss);
  }
  const float r = (1.0f / sqrtf(warp_sum(ss) + unit_eps)) * (u < q_units ? q_scale : 1.0f);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = lane + 32 * j;
    if (c < dim) x[c] = v[j] * r;
  }
}

struct ScanArgs {
  const float *q, *k, *v;              // float32 rows of G * N, G * N and H * P values
  long long q_stride, k_stride, v_stride;
  const float* log_decay;              // [tokens, H], or (decay_stride 0, the only form without beta) [H]
  long long decay_stride;
  const float* beta;                   // [tokens, H]; null: no correction, u = v
  float* state;                        // [slots, H, N, P]
  const int* slots;
  const int* seq_start;
  float* out;                          // [tokens, H * P]
  int n_seqs, H, G, N, P;
  float q_scale;
  // the chunked form
  int chunks;                          // chunks of the longest portion
  float* w;                            // [n_seqs, chunks, H, N, 64]
  float* ends;                         // [n_seqs, chunks, H, 68]: decays from a token to its chunk's end, then the whole chunk's
  float* starts;                       // [n_seqs, chunks, H, N, P]
  int vec;                             // q, k and v rows may be read 16 bytes at a time
};

// Four neighbouring lanes share a column p of a head's state (rows n, n + 4, ...) and walk the sequence's tokens of the
// step; the two inner products are joined by shuffles inside the four lanes.
template <int NB>
__global__ void __launch_bounds__(128) state_walk_kernel(ScanArgs a) {
  pdl_enter();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const long long col = i >> 2;
  if (col >= (long long)a.n_seqs * a.H * a.P) return;        // the four lanes of a column leave together
  const int l = (int)(i & 3);
  const unsigned mask = 0xfu << (threadIdx.x & 28);
  const int p = (int)(col % a.P), h = (int)((col / a.P) % a.H), seq = (int)(col / ((long long)a.P * a.H));
  const int g = h / (a.H / a.G);
  float* st = a.state + (((size_t)a.slots[seq] * a.H + h) * a.N) * a.P + p;
  float S[NB];
#pragma unroll
  for (int j = 0; j < NB; ++j) S[j] = 4 * j + l < a.N ? st[(size_t)(4 * j + l) * a.P] : 0.0f;
  const int t1 = a.seq_start[seq + 1];
  for (int t = a.seq_start[seq]; t < t1; ++t) {
    const float* kr = a.k + (size_t)t * a.k_stride + (size_t)g * a.N;
    const float* qr = a.q + (size_t)t * a.q_stride + (size_t)g * a.N;
    const float decay = expf(a.log_decay[(size_t)t * a.decay_stride + h]);
    const float v = a.v[(size_t)t * a.v_stride + (size_t)h * a.P + p];
    float kk[NB], d = 0.0f, o = 0.0f, u = v;
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      kk[j] = 4 * j + l < a.N ? kr[4 * j + l] : 0.0f;
      S[j] *= decay;
      d = fmaf(S[j], kk[j], d);
    }
    if (a.beta != nullptr) {
      d += __shfl_xor_sync(mask, d, 1);
      d += __shfl_xor_sync(mask, d, 2);
      u = a.beta[(size_t)t * a.H + h] * (v - d);
    }
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      S[j] = fmaf(kk[j], u, S[j]);
      o = fmaf(S[j], 4 * j + l < a.N ? qr[4 * j + l] : 0.0f, o);
    }
    o += __shfl_xor_sync(mask, o, 1);
    o += __shfl_xor_sync(mask, o, 2);
    if (l == 0) a.out[(size_t)t * ((size_t)a.H * a.P) + (size_t)h * a.P + p] = o * a.q_scale;
  }
#pragma unroll
  for (int j = 0; j < NB; ++j)
    if (4 * j + l < a.N) st[(size_t)(4 * j + l) * a.P] = S[j];
}

// ---- long portions in chunks of 64 tokens --------------------------------------------------------------------------
// Within a chunk let L_i be the sum of the log decays of its tokens up to i, and S the state in front of it. Then
//   u = U - W S with (I + A) [U | W] = [beta v | beta e^L k], A_ij = beta_i e^(L_i - L_j) (k_i . k_j) for j < i   (delta rule)
//   u = v                                                                                                   (no correction)
//   o_i = e^(L_i) S^T q_i + sum_(j <= i) e^(L_i - L_j) (q_i . k_j) u_j
//   S after the chunk = e^(L_last) S + sum_j e^(L_last - L_j) k_j u_j^T
// so everything but the two small products with S is independent of the chunks in front (Yang, Wang, Shen, Panda, Kim:
// "Parallelizing Linear Transformers with the Delta Rule over Sequence Length", with decays). Three kernels: the triangular
// systems of all chunks, the states chunk after chunk, the outputs of all chunks. All float32; e^x of differences that are
// never positive, formed from sums in double.
constexpr int kChunk = 64;
constexpr int kPad = kChunk + 4;       // row length of a transposed tile: 16-byte pieces of neighbouring rows fall into other banks
constexpr int kOutCols = 64;           // value columns of a block of the output kernel

// Sums of the chunk's log decays, each as a pair of floats whose sum is the sum to double precision (constant beyond the
// chunk's tokens); called by one whole warp.
__device__ __forceinline__ void chunk_log_sums(const ScanArgs& a, int t0, int cnt, int h, float2* L) {
  const int lane = threadIdx.x & 31;
  double lo = 2 * lane < cnt ? (double)a.log_decay[(size_t)(t0 + 2 * lane) * a.decay_stride + h] : 0.0;
  double hi = 2 * lane + 1 < cnt ? (double)a.log_decay[(size_t)(t0 + 2 * lane + 1) * a.decay_stride + h] : 0.0;
  lo = fmax(lo, -1e30);                // a decay of zero
  hi = fmax(hi, -1e30);
  double run = lo + hi;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += v;
  }
  const double first = run - hi;
  const float f0 = (float)first, f1 = (float)run;
  L[2 * lane] = make_float2(f0, (float)(first - (double)f0));
  L[2 * lane + 1] = make_float2(f1, (float)(run - (double)f1));
}

__device__ __forceinline__ float decay_between(const float2& to, const float2& from) { return expf((to.x - from.x) + (to.y - from.y)); }
__device__ __forceinline__ float decay_since_start(const float2& to) { return expf(to.x + to.y); }

// A [64, N] tile of rows transposed into shared memory, dst[n][i]; rows from cnt on are zero.
template <int THREADS>
__device__ __forceinline__ void load_transposed(float* dst, const float* src, long long stride, int cnt, int N) {
  auto quad = [&](int n, int i) {
    const float* p = src + (size_t)i * stride + n;
    float4 v;
    v.x = i < cnt ? p[0] : 0.0f;
    v.y = i + 1 < cnt ? p[stride] : 0.0f;
    v.z = i + 2 < cnt ? p[2 * stride] : 0.0f;
    v.w = i + 3 < cnt ? p[3 * stride] : 0.0f;
    *reinterpret_cast<float4*>(dst + n * kPad + i) = v;
  };
  if (N == 64 || N == 128) {           // the usual widths: shifts instead of divisions
    const int sh = N == 64 ? 6 : 7, n = threadIdx.x & (N - 1);
#pragma unroll 4
    for (int i = (threadIdx.x >> sh) * 4; i < kChunk; i += (THREADS >> sh) * 4) quad(n, i);
  } else {
    for (int idx = threadIdx.x; idx < N * (kChunk / 4); idx += THREADS) quad(idx % N, idx / N * 4);
  }
}

__device__ __forceinline__ void fma4(float4& acc, float s, const float4& v) {
  acc.x = fmaf(s, v.x, acc.x);
  acc.y = fmaf(s, v.y, acc.y);
  acc.z = fmaf(s, v.z, acc.z);
  acc.w = fmaf(s, v.w, acc.w);
}

__device__ __forceinline__ void copy_async(float* dst, const float* src, bool valid, bool bytes16) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  if (bytes16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(valid ? 16 : 0) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(valid ? 4 : 0) : "memory");
}

// ROWS rows of COLS floats into shared memory; rows from `valid` on and columns from `live` on become zero. vec: `live` and the
// source's addresses are multiples of 4 floats.
template <int THREADS, int ROWS, int COLS>
__device__ __forceinline__ void copy_tile(float* dst, const float* src, long long stride, int valid, int live, bool vec) {
  if (vec) {
    constexpr int per = COLS / 4;
    const int c = (threadIdx.x % per) * 4;
    const float* p = src + c + (long long)(threadIdx.x / per) * stride;
#pragma unroll
    for (int m = 0; m < ROWS * per / THREADS; ++m) {
      const int r = threadIdx.x / per + m * (THREADS / per);
      const bool in = r < valid && c < live;
      copy_async(dst + r * COLS + c, in ? p + (long long)m * (THREADS / per) * stride : src, in, true);
    }
  } else {
    const int c = threadIdx.x % COLS;
    for (int r = threadIdx.x / COLS; r < ROWS; r += THREADS / COLS) {
      const bool in = r < valid && c < live;
      copy_async(dst + r * COLS + c, in ? src + (long long)r * stride + c : src, in, false);
    }
  }
}

// grid (chunks, H, sequences), 128 threads: U into `out`, W transposed into `w`, the decays from every token to the chunk's end
// (and behind them the whole chunk's) into `ends`.
__global__ void __launch_bounds__(128) chunk_solve_kernel(ScanArgs a) {
  pdl_enter();
  extern __shared__ __align__(16) float sm[];
  __shared__ float2 L[kChunk];
  __shared__ float sbeta[kChunk], sgrow[kChunk];
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int t0 = a.seq_start[seq] + chunk * kChunk, cnt = min(kChunk, a.seq_start[seq + 1] - t0);
  if (cnt <= 0) return;
  const int N = a.N, P = a.P, g = h / (a.H / a.G);
  float* KT = sm;                      // [N][kPad], then W in the same layout
  float* AT = KT + N * kPad;           // [64][kPad]: AT[j][i] = A_ij
  const float* krow = a.k + (size_t)t0 * a.k_stride + (size_t)g * N;
  load_transposed<128>(KT, krow, a.k_stride, cnt, N);
  if (tid < 32) chunk_log_sums(a, t0, cnt, h, L);
  if (tid >= 64) sbeta[tid - 64] = tid - 64 < cnt ? a.beta[(size_t)(t0 + tid - 64) * a.H + h] : 0.0f;
  __syncthreads();
  float* ends = a.ends + (((size_t)seq * a.chunks + chunk) * a.H + h) * (kChunk + 4);
  if (tid < kChunk) {
    const float grow = decay_since_start(L[tid]);
    sgrow[tid] = grow;
    ends[tid] = tid < cnt ? decay_between(L[cnt - 1], L[tid]) : 0.0f;
    if (tid == cnt - 1) ends[kChunk] = grow;
  }
  {
    // a warp takes 32 rows x 32 keys or so: lanes 8 (rows, 4 each) x 4 (keys, 8 each)
    const int warp = tid >> 5, lane = tid & 31;
    const int i0 = (warp & 1) * 32 + (lane & 7) * 4, j0 = (warp >> 1) * 32 + (lane >> 3) * 8;
    if ((warp >> 1) <= (warp & 1)) {
      float4 acc[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int n = 0; n < N; ++n) {
        const float4 ki = *reinterpret_cast<const float4*>(KT + n * kPad + i0);
        const float4 ka = *reinterpret_cast<const float4*>(KT + n * kPad + j0), kb = *reinterpret_cast<const float4*>(KT + n * kPad + j0 + 4);
        fma4(acc[0], ka.x, ki); fma4(acc[1], ka.y, ki); fma4(acc[2], ka.z, ki); fma4(acc[3], ka.w, ki);
        fma4(acc[4], kb.x, ki); fma4(acc[5], kb.y, ki); fma4(acc[6], kb.z, ki); fma4(acc[7], kb.w, ki);
      }
      float2 li[4];
      float bi[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { li[i] = L[i0 + i]; bi[i] = sbeta[i0 + i]; }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int jj = j0 + j;
        const float2 lj = L[jj];
        float4 r;
        r.x = i0 > jj ? bi[0] * decay_between(li[0], lj) * acc[j].x : 0.0f;
        r.y = i0 + 1 > jj ? bi[1] * decay_between(li[1], lj) * acc[j].y : 0.0f;
        r.z = i0 + 2 > jj ? bi[2] * decay_between(li[2], lj) * acc[j].z : 0.0f;
        r.w = i0 + 3 > jj ? bi[3] * decay_between(li[3], lj) * acc[j].w : 0.0f;
        *reinterpret_cast<float4*>(AT + jj * kPad + i0) = r;
      }
    }
  }
  __syncthreads();
  // forward substitution, a column of [beta v | beta e^L k] a thread, in registers; nothing is shared but A
  const float* vrow = a.v + (size_t)t0 * a.v_stride + (size_t)h * P;
  for (int c0 = 0; c0 < P + N; c0 += 128) {
    const int c = c0 + tid;
    const bool is_v = c < P;
    if (c < P + N) {
      float x[kChunk];
      if (is_v) {
        const float* p = vrow + c;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) x[i] = i < cnt ? p[(size_t)i * a.v_stride] : 0.0f;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) x[i] *= sbeta[i];
      } else {
        const float* p = KT + (c - P) * kPad;
#pragma unroll
        for (int i = 0; i < kChunk; i += 4) {
          const float4 v = *reinterpret_cast<const float4*>(p + i);
          x[i] = v.x * (sbeta[i] * sgrow[i]);
          x[i + 1] = v.y * (sbeta[i + 1] * sgrow[i + 1]);
          x[i + 2] = v.z * (sbeta[i + 2] * sgrow[i + 2]);
          x[i + 3] = v.w * (sbeta[i + 3] * sgrow[i + 3]);
        }
      }
#pragma unroll
      for (int j = 0; j < kChunk - 1; ++j) {
        const float f = -x[j];
        const float* ar = AT + j * kPad;
#pragma unroll
        for (int i = (j + 1) & ~3; i < kChunk; i += 4) {
          const float4 m = *reinterpret_cast<const float4*>(ar + i);
          if (i > j) x[i] = fmaf(m.x, f, x[i]);
          if (i + 1 > j) x[i + 1] = fmaf(m.y, f, x[i + 1]);
          if (i + 2 > j) x[i + 2] = fmaf(m.z, f, x[i + 2]);
          if (i + 3 > j) x[i + 3] = fmaf(m.w, f, x[i + 3]);
        }
      }
      if (is_v) {
        float* p = a.out + (size_t)t0 * ((size_t)a.H * P) + (size_t)h * P + c;
#pragma unroll
        for (int i = 0; i < kChunk; ++i)
          if (i < cnt) p[(size_t)i * ((size_t)a.H * P)] = x[i];
      } else {                         // this thread's own column of KT: nobody else reads it any more
        float* p = KT + (c - P) * kPad;
#pragma unroll
        for (int i = 0; i < kChunk; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
      }
    }
  }
  __syncthreads();
  float* wt = a.w + ((((size_t)seq * a.chunks + chunk) * a.H + h) * N) * kChunk;
  for (int i = tid; i < N * (kChunk / 4); i += 128)
    reinterpret_cast<float4*>(wt)[i] = *reinterpret_cast<const float4*>(KT + (i >> 4) * kPad + (i & 15) * 4);
}

// grid (slices of PS value columns, H, sequences), TH threads: walks the sequence's chunks with its slice of the state; leaves
// every chunk's start state in `starts`, u in `out` (delta rule) and the last state in the slot. Both products run as 4 x 2 (RN x 2)
// outputs a thread with the inner dimension cut into KS pieces whose partial sums meet in shared memory; behind them a thread owns
// elements tid, tid + TH, ... of the chunk's u and of the state. The next chunk's W, k and values are on their way meanwhile.
template <int RN, int PS, int TH, bool DELTA>
__global__ void __launch_bounds__(TH) chunk_state_kernel(ScanArgs a) {
  pdl_enter();
  extern __shared__ __align__(16) float sm[];
  constexpr int NP = 16 * RN;          // rows of the state, padded
  constexpr int CG = PS / 2;           // pairs of columns
  constexpr int KS = TH / (16 * CG);   // pieces of the inner dimension
  constexpr int OS = (NP * PS + TH - 1) / TH, OU = (kChunk * PS + TH - 1) / TH;      // elements of the state and of u that a thread owns
  constexpr int PARTS = KS * (NP > kChunk ? NP : kChunk) * PS;
  float* sS = sm;                      // [NP][PS]
  float* sV = sS + NP * PS;            // [64][PS]: u times the decay to the chunk's end
  float* sP = sV + kChunk * PS;        // partial sums
  float* sE = sP + PARTS;              // [2][68]: decays to the chunk's end, then the whole chunk's
  float* sK = sE + 2 * (kChunk + 4);   // [2][64][NP]
  float* sW = sK + 2 * kChunk * NP;    // [2][NP][64] (delta rule)
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int N = a.N, P = a.P, g = h / (a.H / a.G);
  const int first = a.seq_start[seq], total = a.seq_start[seq + 1] - first;
  const int live = (total + kChunk - 1) / kChunk;
  if (live <= 0) return;
  const int tp = tid % CG, tr = (tid / CG) & 15, piece = tid / (16 * CG);
  const int c0 = blockIdx.x * PS, cols = min(PS, P - c0);
  const size_t out_stride = (size_t)a.H * P;
  const float log_fixed = DELTA ? 0.0f : fmaxf(a.log_decay[h], -1e30f);
  if (DELTA && NP > N)                 // W's rows beyond N stay zero in every chunk
    for (int i = tid; i < 2 * NP * kChunk; i += TH) sW[i] = 0.0f;
  // element e = tid + TH r of the state: (row part e / (16 PS), row group (e / PS) % 16, column e % PS) -> row group * RN + part
  auto state_row = [&](int e) { return ((e / PS) & 15) * RN + e / (16 * PS); };
  float* st = a.state + (((size_t)a.slots[seq] * a.H + h) * N) * P + c0;
  float S[OS];
#pragma unroll
  for (int r = 0; r < OS; ++r) {
    const int e = tid + TH * r, n = state_row(e), p = e % PS;
    S[r] = n < N && p < cols ? st[(size_t)n * P + p] : 0.0f;
    if (e < NP * PS) sS[n * PS + p] = S[r];
  }
  __syncthreads();
  auto fetch = [&](int c) {            // one commit group a chunk
    if (c < live) {
      const int cnt = min(kChunk, total - c * kChunk), b = c & 1;
      copy_tile<TH, kChunk, NP>(sK + b * kChunk * NP, a.k + (size_t)(first + c * kChunk) * a.k_stride + (size_t)g * N, a.k_stride, cnt, N, a.vec);
      if (DELTA) {
        const size_t at = ((size_t)seq * a.chunks + c) * a.H + h;
        float* wd = sW + b * NP * kChunk;
        const float* ws = a.w + at * N * kChunk;
#pragma unroll
        for (int m = 0; m < (NP * kChunk / 4 + TH - 1) / TH; ++m) {
          const int i = (tid + m * TH) * 4;
          if (i < N * kChunk) copy_async(wd + i, ws + i, true, true);
        }
        if (tid < kChunk / 4 + 1) copy_async(sE + b * (kChunk + 4) + tid * 4, a.ends + at * (kChunk + 4) + tid * 4, true, true);
      } else if (tid <= kChunk) {      // a fixed decay: its powers
        const float left = tid == kChunk ? (float)cnt : (float)(cnt - 1 - tid);
        sE[b * (kChunk + 4) + tid] = left < 0.0f ? 0.0f : (left == 0.0f ? 1.0f : expf(left * log_fixed));
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float uv[OU];                        // this thread's elements of U (or v) of the chunk, element e as for the state with 4 parts
  auto u_row = [&](int e) { return ((e / PS) & 15) * 4 + e / (16 * PS); };
  auto values = [&](int c) {
    const int t0 = first + c * kChunk, cnt = c < live ? min(kChunk, total - c * kChunk) : 0;
#pragma unroll
    for (int r = 0; r < OU; ++r) {
      const int e = tid + TH * r, i = u_row(e), p = e % PS;
      uv[r] = i < cnt && p < cols ? (DELTA ? a.out[(size_t)(t0 + i) * out_stride + (size_t)h * P + c0 + p] : a.v[(size_t)(t0 + i) * a.v_stride + (size_t)h * P + c0 + p]) : 0.0f;
    }
  };
  fetch(0);
  values(0);
  for (int c = 0; c < live; ++c) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                   // chunk c is here; the other buffers are free; sS holds the state
    fetch(c + 1);
    const int t0 = first + c * kChunk, cnt = min(kChunk, total - c * kChunk), b = c & 1;
    const float* ends = sE + b * (kChunk + 4);
    float* start = a.starts + ((((size_t)seq * a.chunks + c) * a.H + h) * N) * P + c0;
#pragma unroll
    for (int r = 0; r < OS; ++r) {
      const int e = tid + TH * r, n = state_row(e), p = e % PS;
      if (n < N && p < cols) start[(size_t)n * P + p] = S[r];
    }
    if (DELTA) {
      const float* w = sW + b * NP * kChunk + tr * 4;
      float acc[4][2];
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0.0f;
      const int lo = piece * (NP / KS);
#pragma unroll 8
      for (int n = lo; n < lo + NP / KS; ++n) {
        const float4 w4 = *reinterpret_cast<const float4*>(w + n * kChunk);
        const float2 s2 = *reinterpret_cast<const float2*>(sS + n * PS + 2 * tp);
        acc[0][0] = fmaf(w4.x, s2.x, acc[0][0]); acc[0][1] = fmaf(w4.x, s2.y, acc[0][1]);
        acc[1][0] = fmaf(w4.y, s2.x, acc[1][0]); acc[1][1] = fmaf(w4.y, s2.y, acc[1][1]);
        acc[2][0] = fmaf(w4.z, s2.x, acc[2][0]); acc[2][1] = fmaf(w4.z, s2.y, acc[2][1]);
        acc[3][0] = fmaf(w4.w, s2.x, acc[3][0]); acc[3][1] = fmaf(w4.w, s2.y, acc[3][1]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float2*>(sP + piece * kChunk * PS + (i * 16 + tr) * PS + 2 * tp) = make_float2(acc[i][0], acc[i][1]);
      __syncthreads();
#pragma unroll
      for (int r = 0; r < OU; ++r) {
        const int e = tid + TH * r, i = u_row(e), p = e % PS;
        float sum = 0.0f;
#pragma unroll
        for (int k = 0; k < KS; ++k) sum += sP[k * kChunk * PS + e];
        uv[r] -= sum;
        if (i < cnt && p < cols) a.out[(size_t)(t0 + i) * out_stride + (size_t)h * P + c0 + p] = uv[r];
      }
    }
#pragma unroll
    for (int r = 0; r < OU; ++r) {
      const int e = tid + TH * r, i = u_row(e), p = e % PS;
      if (e < kChunk * PS) sV[i * PS + p] = uv[r] * ends[i];
    }
    __syncthreads();
    values(c + 1);
    {
      const float* kk = sK + b * kChunk * NP + tr * RN;
      float acc[RN][2];
#pragma unroll
      for (int r = 0; r < RN; ++r) acc[r][0] = acc[r][1] = 0.0f;
      const int lo = piece * (kChunk / KS);
#pragma unroll 8
      for (int i = lo; i < lo + kChunk / KS; ++i) {
        const float2 u2 = *reinterpret_cast<const float2*>(sV + i * PS + 2 * tp);
        if constexpr (RN >= 4) {
#pragma unroll
          for (int r = 0; r < RN; r += 4) {
            const float4 k4 = *reinterpret_cast<const float4*>(kk + i * NP + r);
            acc[r][0] = fmaf(k4.x, u2.x, acc[r][0]); acc[r][1] = fmaf(k4.x, u2.y, acc[r][1]);
            acc[r + 1][0] = fmaf(k4.y, u2.x, acc[r + 1][0]); acc[r + 1][1] = fmaf(k4.y, u2.y, acc[r + 1][1]);
            acc[r + 2][0] = fmaf(k4.z, u2.x, acc[r + 2][0]); acc[r + 2][1] = fmaf(k4.z, u2.y, acc[r + 2][1]);
            acc[r + 3][0] = fmaf(k4.w, u2.x, acc[r + 3][0]); acc[r + 3][1] = fmaf(k4.w, u2.y, acc[r + 3][1]);
          }
        } else {
          const float2 k2 = *reinterpret_cast<const float2*>(kk + i * NP);
          acc[0][0] = fmaf(k2.x, u2.x, acc[0][0]); acc[0][1] = fmaf(k2.x, u2.y, acc[0][1]);
          acc[1][0] = fmaf(k2.y, u2.x, acc[1][0]); acc[1][1] = fmaf(k2.y, u2.y, acc[1][1]);
        }
      }
#pragma unroll
      for (int r = 0; r < RN; ++r)
        *reinterpret_cast<float2*>(sP + piece * NP * PS + (r * 16 + tr) * PS + 2 * tp) = make_float2(acc[r][0], acc[r][1]);
    }
    __syncthreads();
    const float keep = ends[kChunk];
#pragma unroll
    for (int r = 0; r < OS; ++r) {
      const int e = tid + TH * r;
      if (e >= NP * PS) break;
      float sum = 0.0f;
#pragma unroll
      for (int k = 0; k < KS; ++k) sum += sP[k * NP * PS + e];
      S[r] = fmaf(keep, S[r], sum);
      sS[state_row(e) * PS + e % PS] = S[r];
    }
  }
#pragma unroll
  for (int r = 0; r < OS; ++r) {
    const int e = tid + TH * r, n = state_row(e), p = e % PS;
    if (n < N && p < cols) st[(size_t)n * P + p] = S[r];
  }
}

// Row length of the output kernel's tiles of queries and keys: a multiple of 4 floats, and 4 more than a multiple of 32, so that
// 16-byte pieces of eight neighbouring rows lie in different banks.
__host__ __device__ constexpr int out_row(int N) { return (N + 31) / 32 * 32 + 4; }
__host__ __device__ constexpr int out_keys_floats(int N) {      // the keys' tile, later the start state [N rounded up to 16][64]
  return kChunk * out_row(N) > (N + 15) / 16 * 16 * kOutCols ? kChunk * out_row(N) : (N + 15) / 16 * 16 * kOutCols;
}

// A [64, N] tile of rows into shared memory (row length `ld`), zeros behind N up to a multiple of 4 and in rows from cnt on.
__device__ __forceinline__ void copy_rows(float* dst, int ld, const float* src, long long stride, int cnt, int N, bool vec) {
  const int step = vec ? 4 : 1, per = ((N + 3) & ~3) / step;
  const int r0 = threadIdx.x / 32;                         // a warp a row, eight rows at a time
  for (int r = r0; r < kChunk; r += 8)
    for (int c = threadIdx.x & 31; c < per; c += 32) {
      const bool in = r < cnt && c * step < N;
      copy_async(dst + r * ld + c * step, in ? src + (size_t)r * stride + c * step : src, in, vec);
    }
}

// grid (chunks, H * slices of 64 value columns, sequences), 256 threads: the chunk's outputs. A warp takes 16 rows x 32 columns,
// lanes 4 x 8; a lane's four rows lie 4 apart, its four keys 8 apart (scores) and its four value columns side by side. Inner
// dimensions go four values at a time: 8 loads of 16 bytes for 64 multiply-adds.
__global__ void __launch_bounds__(256) chunk_out_kernel(ScanArgs a) {
  pdl_enter();
  extern __shared__ __align__(16) float sm[];
  __shared__ float2 L[kChunk];
  const int slices = (a.P + kOutCols - 1) / kOutCols;
  const int chunk = blockIdx.x, h = blockIdx.y / slices, c0 = (blockIdx.y % slices) * kOutCols, seq = blockIdx.z, tid = threadIdx.x;
  const int t0 = a.seq_start[seq] + chunk * kChunk, cnt = min(kChunk, a.seq_start[seq + 1] - t0);
  if (cnt <= 0) return;
  const int N = a.N, N4 = (N + 3) & ~3, P = a.P, g = h / (a.H / a.G), cols = min(kOutCols, P - c0), ld = out_row(N);
  float* Q = sm;                       // [64][ld]
  float* K = Q + kChunk * ld;          // [64][ld], then the start state [N4][64]
  float* A = K + out_keys_floats(N);   // [64][kPad]: A[i][j] = e^(L_i - L_j) (q_i . k_j)
  float* V = A + kChunk * kPad;        // [64][64]: u
  copy_rows(Q, ld, a.q + (size_t)t0 * a.q_stride + (size_t)g * N, a.q_stride, cnt, N, a.vec);
  copy_rows(K, ld, a.k + (size_t)t0 * a.k_stride + (size_t)g * N, a.k_stride, cnt, N, a.vec);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const bool from_out = a.beta != nullptr;
  const float* u = from_out ? a.out + (size_t)t0 * ((size_t)a.H * P) + (size_t)h * P + c0 : a.v + (size_t)t0 * a.v_stride + (size_t)h * P + c0;
  copy_tile<256, kChunk, kOutCols>(V, u, from_out ? (long long)a.H * P : a.v_stride, cnt, cols, a.vec);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (tid < 32) chunk_log_sums(a, t0, cnt, h, L);
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31;
  const int i0 = (warp >> 1) * 16 + (lane >> 3), j0 = (warp & 1) * 32 + (lane & 7), p0 = (warp & 1) * 32 + (lane & 7) * 4;
  const int rows_end = (warp >> 1) * 16 + 16;               // keys from here on are behind all rows of the warp
  {
    float acc[4][4];                   // [row][key]
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    if ((warp & 1) * 32 < rows_end) {
#pragma unroll 2
      for (int n = 0; n < N4; n += 4) {
        float4 q4[4], k4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) q4[i] = *reinterpret_cast<const float4*>(Q + (i0 + 4 * i) * ld + n);
#pragma unroll
        for (int j = 0; j < 4; ++j) k4[j] = *reinterpret_cast<const float4*>(K + (j0 + 8 * j) * ld + n);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j)
            acc[i][j] = fmaf(q4[i].w, k4[j].w, fmaf(q4[i].z, k4[j].z, fmaf(q4[i].y, k4[j].y, fmaf(q4[i].x, k4[j].x, acc[i][j]))));
      }
    }
    float2 lj[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) lj[j] = L[j0 + 8 * j];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 li = L[i0 + 4 * i];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        A[(i0 + 4 * i) * kPad + j0 + 8 * j] = i0 + 4 * i >= j0 + 8 * j ? acc[i][j] * decay_between(li, lj[j]) : 0.0f;
    }
  }
  __syncthreads();                     // the keys have been read: their place takes the start state
  const float* start = a.starts + ((((size_t)seq * a.chunks + chunk) * a.H + h) * N) * P + c0;
  for (int n = 0; n < N; n += 16) copy_tile<256, 16, kOutCols>(K + n * kOutCols, start + (size_t)n * P, P, N - n, cols, a.vec);
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  float4 o[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  auto accumulate = [&](const float* rows, int row_len, const float* col) {      // four inner values
    float4 r4[4], v4[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) r4[i] = *reinterpret_cast<const float4*>(rows + 4 * i * row_len);
#pragma unroll
    for (int k = 0; k < 4; ++k) v4[k] = *reinterpret_cast<const float4*>(col + k * kOutCols);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      fma4(o[i], r4[i].x, v4[0]);
      fma4(o[i], r4[i].y, v4[1]);
      fma4(o[i], r4[i].z, v4[2]);
      fma4(o[i], r4[i].w, v4[3]);
    }
  };
#pragma unroll 2
  for (int n = 0; n < N4; n += 4) accumulate(Q + i0 * ld + n, ld, K + n * kOutCols + p0);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float f = decay_since_start(L[i0 + 4 * i]);
    o[i] = make_float4(o[i].x * f, o[i].y * f, o[i].z * f, o[i].w * f);
  }
#pragma unroll 2
  for (int j = 0; j < rows_end; j += 4) accumulate(A + i0 * kPad + j, kPad, V + j * kOutCols + p0);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = i0 + 4 * i;
    if (row >= cnt) continue;
    float* dst = a.out + (size_t)(t0 + row) * ((size_t)a.H * P) + (size_t)h * P + c0 + p0;
    const float r[4] = {o[i].x * a.q_scale, o[i].y * a.q_scale, o[i].z * a.q_scale, o[i].w * a.q_scale};
    if (a.vec && p0 + 3 < cols) {
      *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (p0 + e < cols) dst[e] = r[e];
    }
  }
}

struct StateTokenArgs {
  const float *q, *k, *v;              // rows of G * N, G * N and H * P values, one row a sequence
  long long q_stride, k_stride, v_stride;
  const float* gate;                   // rows of H * P pre-activations
  long long gate_stride;
  const float* decay;                  // fixed decay: [H]; null for the delta rule, which reads the next four
  const float *raw_beta, *raw_step;    // rows of H values
  long long raw_stride;
  const float *dt_bias, *a_log;        // [H]
  const float *cos, *sin;              // [positions, half] or null: rotation of the first 2 * half channels of q and k
  const int* tok_pos;
  int half, neighbours;
  float* state;
  const int* slots;
  const float* gain;                   // [P] or null (ones)
  void* out;                           // [n, H * P] in the run dtype
  int H, G, N, P, PB;                  // PB: columns of a block, rounded up to whole warps
  int team;                            // blocks of a cluster that share a head, 64 columns each
  float q_scale, unit_eps, eps;
};

constexpr int kStateThreads = 512, kTeamCols = 64, kTeamMost = 8;

// grid (H * team, sequences), clusters of `team` blocks. Thread (r, c), c = tid % PB, holds rows r, r + R, ... of column c of its
// block's part of the head's state; the blocks of a head meet once, for the head's sum of squares.
template <typename T, int NB>
__global__ void __launch_bounds__(kStateThreads, NB <= 16 ? 2 : 1) state_token_kernel(StateTokenArgs a) {
  pdl_enter();
  __shared__ float sq[256], sk[256], part_k[kStateThreads], part_q[kStateThreads], scratch[33];
  __shared__ float team_ss[kTeamMost];
  if (a.team > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // this block runs
  const int h = blockIdx.x / a.team, rank = blockIdx.x % a.team, seq = blockIdx.y, tid = threadIdx.x;
  const int N = a.N, P = a.P, R = blockDim.x / a.PB;
  const int cb = tid % a.PB, r = tid / a.PB;               // column within the block
  const int c = rank * kTeamCols + cb;
  const bool mine = c < P && r < R;
  const int g = h / (a.H / a.G);
  float* st = a.state + ((size_t)a.slots[seq] * a.H + h) * N * P + c;
  float S[NB];
#pragma unroll
  for (int j = 0; j < NB; ++j) S[j] = mine && r + j * R < N ? st[(r + j * R) * P] : 0.0f;
  const float v = mine ? a.v[(size_t)seq * a.v_stride + (size_t)h * P + c] : 0.0f;
  const float gate = mine && r == 0 ? a.gate[(size_t)seq * a.gate_stride + (size_t)h * P + c] : 0.0f;
  const float gain = mine && r == 0 && a.gain ? a.gain[c] : 1.0f;
  float qv = tid < N ? a.q[(size_t)seq * a.q_stride + (size_t)g * N + tid] : 0.0f;
  float kv = tid < N ? a.k[(size_t)seq * a.k_stride + (size_t)g * N + tid] : 0.0f;
  float decay, beta = 1.0f;
  if (a.decay != nullptr) {
    decay = a.decay[h];
    if (a.half > 0) {
      if (tid < N) { sq[tid] = qv; sk[tid] = kv; }
      __syncthreads();
      if (tid < 2 * a.half) {
        const int pair = a.neighbours ? tid >> 1 : (tid < a.half ? tid : tid - a.half);
        const bool second = a.neighbours ? (tid & 1) : tid >= a.half;
        const int other = a.neighbours ? tid ^ 1 : (second ? tid - a.half : tid + a.half);
        const size_t at = (size_t)a.tok_pos[seq] * a.half + pair;
        const float co = a.cos[at], si = second ? a.sin[at] : -a.sin[at];
        qv = qv * co + sq[other] * si;
        kv = kv * co + sk[other] * si;
      }
      __syncthreads();
    }
  } else {
    const float x = a.raw_step[(size_t)seq * a.raw_stride + h] + a.dt_bias[h];
    decay = expf(-expf(a.a_log[h]) * softplus_of(x));
    beta = sigmoid_of(a.raw_beta[(size_t)seq * a.raw_stride + h]);
    qv *= 1.0f / sqrtf(block_sum(qv * qv, scratch) + a.unit_eps);
    kv *= 1.0f / sqrtf(block_sum(kv * kv, scratch) + a.unit_eps);
  }
  qv *= a.q_scale;
  if (tid < N) { sq[tid] = qv; sk[tid] = kv; }
  const float kq = block_sum(qv * kv, scratch);              // (its barriers also publish sq and sk)
  float dk = 0.0f, dq = 0.0f;
#pragma unroll
  for (int j = 0; j < NB; ++j) {
    const int n = r + j * R;
    if (n < N) {
      S[j] *= decay;
      dk = fmaf(S[j], sk[n], dk);
      dq = fmaf(S[j], sq[n], dq);
    }
    if ((j & 3) == 3) asm volatile("" ::: "memory");       // four rows' keys and queries at a time in registers, not all
  }
  part_k[tid] = dk;
  part_q[tid] = dq;
  __syncthreads();
  dk = dq = 0.0f;
  for (int i = 0; i < R; ++i) {
    dk += part_k[i * a.PB + cb];
    dq += part_q[i * a.PB + cb];
  }
  const float u = a.decay != nullptr ? v : beta * (v - dk);
  float* back = st;
  asm volatile("" : "+l"(back));       // the addresses are worked out again instead of being kept since the loads
#pragma unroll
  for (int j = 0; j < NB; ++j) {
    const int n = r + j * R;
    if (mine && n < N) back[n * P] = fmaf(sk[n], u, S[j]);
    if ((j & 3) == 3) asm volatile("" ::: "memory");
  }
  const float o = mine && r == 0 ? fmaf(u, kq, dq) : 0.0f;   // S_new^T q = (decayed S)^T q + u (k . q)
  float ss = block_sum(o * o, scratch);
  if (a.team > 1) {
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");                              // every block of the head runs
    if (tid < a.team) {
      uint32_t at;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"((uint32_t)__cvta_generic_to_shared(&team_ss[rank])), "r"(tid));
      asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(at), "f"(ss) : "memory");
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    ss = 0.0f;
    for (int i = 0; i < a.team; ++i) ss += team_ss[i];
  }
  const float inv = 1.0f / sqrtf(ss / (float)P + a.eps);
  if (mine && r == 0) ((T*)a.out)[((size_t)seq * a.H + h) * P + c] = from_f32<T>(o * inv * gain * silu_of(gate));
}

template <typename T, int NB>
static void launch_state_token_nb(const StateTokenArgs& a, int n, cudaStream_t s) {
  const dim3 grid(a.H * a.team, n), block(kStateThreads);
  if (a.team > 1) launch_clusters(pdl_mode() == 1, a.team, state_token_kernel<T, NB>, grid, block, 0, s, a);
  else launch(state_token_kernel<T, NB>, grid, block, 0, s, a);
}

template <typename T>
static void launch_state_token(const StateTokenArgs& a, int n, int rows, cudaStream_t s) {
  if (rows <= 4) launch_state_token_nb<T, 4>(a, n, s);
  else if (rows <= 8) launch_state_token_nb<T, 8>(a, n, s);
  else if (rows <= 16) launch_state_token_nb<T, 16>(a, n, s);
  else launch_state_token_nb<T, 32>(a, n, s);
}

}  // namespace slb

using namespace slb;

extern "C" int slb_rotate_rows(float* rows, long long stride, const float* cos, const float* sin, const int* tok_pos, int tokens,
                               int units, int dim, int rot, int neighbours, void* stream) {
  SLB_REQUIRE(tokens >= 0 && units > 0 && dim > 0 && rot >= 0 && rot % 2 == 0 && rot <= dim && stride >= (long long)units * dim,
              "rotate_rows: units=%d dim=%d rotated=%d", units, dim, rot);
  SLB_REQUIRE(rot == 0 || (cos != nullptr && sin != nullptr), "rotate_rows: a rotation needs its tables");
  if (tokens == 0 || rot == 0) return 0;
  const long long total = (long long)tokens * units * (rot / 2);
  launch(rotate_rows_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, rows, stride, cos, sin, tok_pos,
         total, units, dim, rot / 2, neighbours);
  return check_launch("rotate_rows");
}

extern "C" int slb_delta_prep(float* rows, long long stride, int groups, int dim, float q_scale, float unit_eps, const float* raw_beta,
                              const float* raw_step, long long raw_stride, const float* dt_bias, const float* a_log, float* beta,
                              float* log_decay, int tokens, int H, void* stream) {
  SLB_REQUIRE(tokens >= 0 && groups > 0 && dim > 0 && dim <= 256 && H > 0 && stride >= 2ll * groups * dim && raw_stride >= H,
              "delta_prep: groups=%d dim=%d (at most 256) heads=%d", groups, dim, H);
  if (tokens == 0) return 0;
  const long long warps = (long long)tokens * (2 * groups + 1);
  launch(delta_prep_kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, (cudaStream_t)stream, rows, stride, 2 * groups, groups, dim,
         q_scale, unit_eps, raw_beta, raw_step, raw_stride, dt_bias, a_log, beta, log_decay, tokens, H);
  return check_launch("delta_prep");
}

// Portions of more than kWalkTokens tokens run in chunks (states of up to 128 key channels).
constexpr int kWalkTokens = 24;
static bool runs_in_chunks(int max_count, int N) { return max_count > kWalkTokens && N <= 128; }

// Floats of scratch memory that a step whose longest portion has max_count tokens needs (0: token by token).
extern "C" long long slb_state_scan_scratch_floats(int n_seqs, int max_count, int H, int N, int P, int delta) {
  if (!runs_in_chunks(max_count, N)) return 0;
  const long long chunks = (max_count + kChunk - 1) / kChunk;
  const long long starts = (((long long)n_seqs * chunks * H * N * P) + 3) & ~3ll;
  return starts + (delta ? (long long)n_seqs * chunks * H * ((long long)N * kChunk + kChunk + 4) : 0);
}

template <int RN, int PS, int TH>
static int launch_chunk_state(const ScanArgs& a, cudaStream_t s) {
  const dim3 grid((a.P + PS - 1) / PS, a.H, a.n_seqs), block(TH);
  const bool delta = a.beta != nullptr;
  constexpr int NP = 16 * RN, KS = TH / (8 * PS);
  const int smem = (NP * PS + kChunk * PS + KS * (NP > kChunk ? NP : kChunk) * PS + 2 * (kChunk + 4) + (delta ? 4 : 2) * kChunk * NP) * 4;
  static bool configured[2] = {false, false};
  if (!configured[delta]) {
    const cudaError_t e = delta ? cudaFuncSetAttribute(chunk_state_kernel<RN, PS, TH, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem)
                                : cudaFuncSetAttribute(chunk_state_kernel<RN, PS, TH, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(2, "state_scan: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(e));
    configured[delta] = true;
  }
  if (delta) launch(chunk_state_kernel<RN, PS, TH, true>, grid, block, (size_t)smem, s, a);
  else launch(chunk_state_kernel<RN, PS, TH, false>, grid, block, (size_t)smem, s, a);
  return check_launch("state_scan (states)");
}

extern "C" int slb_state_scan(const float* q, long long q_stride, const float* k, long long k_stride, const float* v, long long v_stride,
                              const float* log_decay, long long decay_stride, const float* beta, float* state, const int* slots,
                              const int* seq_start, float* out, int n_seqs, int H, int G, int N, int P, float q_scale, int max_count,
                              float* scratch, long long scratch_floats, void* stream) {
  SLB_REQUIRE(n_seqs >= 0 && n_seqs < 65536 && H > 0 && G > 0 && H % G == 0 && N > 0 && N <= 256 && P > 0,
              "state_scan: heads=%d groups=%d N=%d (at most 256) P=%d", H, G, N, P);
  SLB_REQUIRE(decay_stride == 0 || (beta != nullptr && decay_stride >= H), "state_scan: decay rows of %lld values for %d heads", decay_stride, H);
  if (n_seqs == 0 || max_count <= 0) return 0;
  ScanArgs a{q, k, v, q_stride, k_stride, v_stride, log_decay, decay_stride, beta, state, slots, seq_start, out, n_seqs, H, G, N, P, q_scale,
             0, nullptr, nullptr, nullptr, 0};
  cudaStream_t s = (cudaStream_t)stream;
  const bool delta = beta != nullptr;
  const long long need = slb_state_scan_scratch_floats(n_seqs, max_count, H, N, P, delta);
  if (need == 0) {
    const long long total = (long long)n_seqs * H * P * 4;
    const dim3 grid((unsigned)((total + 127) / 128)), block(128);
    if (N <= 32) launch(state_walk_kernel<8>, grid, block, 0, s, a);
    else if (N <= 64) launch(state_walk_kernel<16>, grid, block, 0, s, a);
    else if (N <= 128) launch(state_walk_kernel<32>, grid, block, 0, s, a);
    else launch(state_walk_kernel<64>, grid, block, 0, s, a);
    return check_launch("state_scan");
  }
  SLB_REQUIRE(scratch != nullptr && scratch_floats >= need, "state_scan: %lld floats of scratch memory are needed, %lld were given", need, scratch_floats);
  a.chunks = (max_count + kChunk - 1) / kChunk;
  const size_t per = (size_t)n_seqs * a.chunks * H;
  a.w = scratch;
  a.ends = a.w + (delta ? per * N * kChunk : 0);
  a.starts = a.ends + (delta ? per * (kChunk + 4) : 0);
  a.vec = N % 4 == 0 && P % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 &&
          ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)out | (uintptr_t)scratch) % 16 == 0;
  SLB_REQUIRE((uintptr_t)scratch % 16 == 0, "state_scan: the scratch memory must be 16-byte aligned");
  SLB_REQUIRE(H < 65536 && (long long)H * ((P + kOutCols - 1) / kOutCols) < 65536, "state_scan: too many heads (%d)", H);
  if (delta) {
    const int smem = (N * kPad + kChunk * kPad) * 4;
    static int most = 0;
    if (smem > most) {
      const cudaError_t e = cudaFuncSetAttribute(chunk_solve_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return fail(2, "state_scan: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(e));
      most = smem;
    }
    launch(chunk_solve_kernel, dim3(a.chunks, H, n_seqs), dim3(128), (size_t)smem, s, a);
    const int rc = check_launch("state_scan (triangular systems)");
    if (rc) return rc;
  }
  {
    // slices of 8 columns while all their blocks can be resident at once, else of 16 (with 128 rows one block fits an SM)
    const bool narrow = (long long)((P + 7) / 8) * H * n_seqs <= (long long)sm_count() * (N <= 64 ? 2 : 1);
    int rc;
    if (N <= 32) rc = narrow ? launch_chunk_state<2, 8, 256>(a, s) : launch_chunk_state<2, 16, 256>(a, s);
    else if (N <= 64) rc = narrow ? launch_chunk_state<4, 8, 512>(a, s) : launch_chunk_state<4, 16, 512>(a, s);
    else rc = narrow ? launch_chunk_state<8, 8, 512>(a, s) : launch_chunk_state<8, 16, 512>(a, s);
    if (rc) return rc;
  }
  const int smem = (kChunk * out_row(N) + out_keys_floats(N) + kChunk * kPad + kChunk * kOutCols) * 4;
  static int most_out = 0;
  if (smem > most_out) {
    const cudaError_t e = cudaFuncSetAttribute(chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return fail(2, "state_scan: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(e));
    most_out = smem;
  }
  launch(chunk_out_kernel, dim3(a.chunks, H * ((P + kOutCols - 1) / kOutCols), n_seqs), dim3(256), (size_t)smem, s, a);
  return check_launch("state_scan (outputs)");
}

// 1 when slb_state_token takes heads of N key and P value channels.
extern "C" int slb_state_token_supported(int N, int P) {
  return N >= 1 && N <= 256 && P >= 1 && P <= kTeamCols * kTeamMost;
}

extern "C" int slb_state_token(const float* q, long long q_stride, const float* k, long long k_stride, const float* v, long long v_stride,
                               const float* gate, long long gate_stride, const float* decay, const float* raw_beta,
                               const float* raw_step, long long raw_stride, const float* dt_bias, const float* a_log, const float* cos,
                               const float* sin, const int* tok_pos, int rot, int neighbours, float* state, const int* slots,
                               const float* gain, void* out, int n, int H, int G, int N, int P, float q_scale, float unit_eps, float eps,
                               int dtype, void* stream) {
  SLB_REQUIRE(n >= 0 && n < 65536 && H > 0 && G > 0 && H % G == 0 && slb_state_token_supported(N, P), "state_token: heads=%d groups=%d N=%d P=%d", H, G, N, P);
  SLB_REQUIRE(decay != nullptr || (raw_beta != nullptr && raw_step != nullptr && dt_bias != nullptr && a_log != nullptr && raw_stride >= H),
              "state_token: a fixed decay, or the delta rule's step sizes and strengths");
  SLB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= N && (rot == 0 || (decay != nullptr && cos != nullptr && sin != nullptr)), "state_token: %d rotated channels of %d", rot, N);
  if (n == 0) return 0;
  const int team = P <= kTeamCols ? 1 : (P + kTeamCols - 1) / kTeamCols;
  const int PB = team > 1 ? kTeamCols : (P + 31) / 32 * 32, R = kStateThreads / PB;
  SLB_REQUIRE((long long)H * team < 65536, "state_token: too many heads (%d)", H);
  const StateTokenArgs a{q, k, v, q_stride, k_stride, v_stride, gate, gate_stride, decay, raw_beta, raw_step, raw_stride, dt_bias, a_log,
                         cos, sin, tok_pos, rot / 2, neighbours, state, slots, gain, out, H, G, N, P, PB, team, q_scale, unit_eps, eps};
  if (dtype == kF32) launch_state_token<float>(a, n, (N + R - 1) / R, (cudaStream_t)stream);
  else if (dtype == kBF16) launch_state_token<__nv_bfloat16>(a, n, (N + R - 1) / R, (cudaStream_t)stream);
  else return fail(1, "state_token: unknown dtype %d", dtype);
  return check_launch("state_token");
}
