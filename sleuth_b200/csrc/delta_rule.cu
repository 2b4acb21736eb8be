// Recurrences with a matrix state per head and one decay per head: the gated delta rule and the linear attention with a
// fixed decay (retention). All arithmetic is float32; the states live in the cache's per-sequence regions [slots, H, N, P]
// (N key channels, P value channels) and are indexed by the step's slots.
//
//   rotate_rows_kernel     the first channels of every unit of a float32 row turn in pairs, in place
//   delta_prep_kernel      q and k units divided by their length, in place (q also scaled); beta = sigmoid(b);
//                          log decay = -exp(A_log) softplus(a + dt_bias)
//   delta_scan_kernel      the gated delta rule token by token: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q
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

struct DeltaArgs {
  const float *q, *k, *v;              // float32 rows of G * N, G * N and H * P values (unit vectors; q scaled)
  long long q_stride, k_stride, v_stride;
  const float* log_decay;              // [tokens, H]
  const float* beta;                   // [tokens, H]
  float* state;                        // [slots, H, N, P]
  const int* slots;
  const int* seq_start;
  float* out;                          // [tokens, H * P]
  int n_seqs, H, G, N, P;
};

// Four neighbouring lanes share a column p of a head's state (rows n, n + 4, ...) and walk the sequence's tokens of the
// step; the two inner products are joined by shuffles inside the four lanes.
template <int NB>
__global__ void __launch_bounds__(128) delta_scan_kernel(DeltaArgs a) {
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
    const float decay = expf(a.log_decay[(size_t)t * a.H + h]), beta = a.beta[(size_t)t * a.H + h];
    const float v = a.v[(size_t)t * a.v_stride + (size_t)h * a.P + p];
    float kk[NB], d = 0.0f, o = 0.0f;
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      kk[j] = 4 * j + l < a.N ? kr[4 * j + l] : 0.0f;
      S[j] *= decay;
      d = fmaf(S[j], kk[j], d);
    }
    d += __shfl_xor_sync(mask, d, 1);
    d += __shfl_xor_sync(mask, d, 2);
    const float u = beta * (v - d);
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      S[j] = fmaf(kk[j], u, S[j]);
      o = fmaf(S[j], 4 * j + l < a.N ? qr[4 * j + l] : 0.0f, o);
    }
    o += __shfl_xor_sync(mask, o, 1);
    o += __shfl_xor_sync(mask, o, 2);
    if (l == 0) a.out[(size_t)t * ((size_t)a.H * a.P) + (size_t)h * a.P + p] = o;
  }
#pragma unroll
  for (int j = 0; j < NB; ++j)
    if (4 * j + l < a.N) st[(size_t)(4 * j + l) * a.P] = S[j];
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
  int H, G, N, P, PB;                  // PB: P rounded up to whole warps
  float q_scale, unit_eps, eps;
};

constexpr int kStateThreads = 512;

// grid (H, sequences). Thread (r, c), c = tid % PB, holds rows r, r + R, ... of column c of the head's state.
template <typename T, int NB>
__global__ void __launch_bounds__(kStateThreads) state_token_kernel(StateTokenArgs a) {
  pdl_enter();
  __shared__ float sq[256], sk[256], part_k[kStateThreads], part_q[kStateThreads], scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int N = a.N, P = a.P, R = blockDim.x / a.PB;
  const int c = tid % a.PB, r = tid / a.PB;
  const bool mine = c < P && r < R;
  const int g = h / (a.H / a.G);
  float* st = a.state + ((size_t)a.slots[seq] * a.H + h) * N * P + c;
  float S[NB];
#pragma unroll
  for (int j = 0; j < NB; ++j) S[j] = mine && r + j * R < N ? st[(size_t)(r + j * R) * P] : 0.0f;
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
  }
  part_k[tid] = dk;
  part_q[tid] = dq;
  __syncthreads();
  dk = dq = 0.0f;
  for (int i = 0; i < R; ++i) {
    dk += part_k[i * a.PB + c];
    dq += part_q[i * a.PB + c];
  }
  const float u = a.decay != nullptr ? v : beta * (v - dk);
#pragma unroll
  for (int j = 0; j < NB; ++j) {
    const int n = r + j * R;
    if (mine && n < N) st[(size_t)n * P] = fmaf(sk[n], u, S[j]);
  }
  const float o = mine && r == 0 ? fmaf(u, kq, dq) : 0.0f;   // S_new^T q = (decayed S)^T q + u (k . q)
  const float inv = 1.0f / sqrtf(block_sum(o * o, scratch) / (float)P + a.eps);
  if (mine && r == 0) ((T*)a.out)[((size_t)seq * a.H + h) * P + c] = from_f32<T>(o * inv * gain * silu_of(gate));
}

template <typename T>
static void launch_state_token(const StateTokenArgs& a, int n, int rows, cudaStream_t s) {
  const dim3 grid(a.H, n), block(kStateThreads);
  if (rows <= 8) launch(state_token_kernel<T, 8>, grid, block, 0, s, a);
  else if (rows <= 16) launch(state_token_kernel<T, 16>, grid, block, 0, s, a);
  else if (rows <= 32) launch(state_token_kernel<T, 32>, grid, block, 0, s, a);
  else launch(state_token_kernel<T, 64>, grid, block, 0, s, a);
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

extern "C" int slb_delta_scan(const float* q, long long q_stride, const float* k, long long k_stride, const float* v, long long v_stride,
                              const float* log_decay, const float* beta, float* state, const int* slots, const int* seq_start, float* out,
                              int n_seqs, int H, int G, int N, int P, void* stream) {
  SLB_REQUIRE(n_seqs >= 0 && H > 0 && G > 0 && H % G == 0 && N > 0 && N <= 256 && P > 0, "delta_scan: heads=%d groups=%d N=%d (at most 256) P=%d", H, G, N, P);
  if (n_seqs == 0) return 0;
  const DeltaArgs a{q, k, v, q_stride, k_stride, v_stride, log_decay, beta, state, slots, seq_start, out, n_seqs, H, G, N, P};
  const long long total = (long long)n_seqs * H * P * 4;
  const dim3 grid((unsigned)((total + 127) / 128)), block(128);
  cudaStream_t s = (cudaStream_t)stream;
  if (N <= 32) launch(delta_scan_kernel<8>, grid, block, 0, s, a);
  else if (N <= 64) launch(delta_scan_kernel<16>, grid, block, 0, s, a);
  else if (N <= 128) launch(delta_scan_kernel<32>, grid, block, 0, s, a);
  else launch(delta_scan_kernel<64>, grid, block, 0, s, a);
  return check_launch("delta_scan");
}

// 1 when slb_state_token takes heads of N key and P value channels.
extern "C" int slb_state_token_supported(int N, int P) {
  if (N < 1 || N > 256 || P < 1 || P > kStateThreads) return 0;
  const int PB = (P + 31) / 32 * 32, R = kStateThreads / PB;
  return (N + R - 1) / R <= 64;
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
  const int PB = (P + 31) / 32 * 32, R = kStateThreads / PB;
  const StateTokenArgs a{q, k, v, q_stride, k_stride, v_stride, gate, gate_stride, decay, raw_beta, raw_step, raw_stride, dt_bias, a_log,
                         cos, sin, tok_pos, rot / 2, neighbours, state, slots, gain, out, H, G, N, P, PB, q_scale, unit_eps, eps};
  if (dtype == kF32) launch_state_token<float>(a, n, (N + R - 1) / R, (cudaStream_t)stream);
  else if (dtype == kBF16) launch_state_token<__nv_bfloat16>(a, n, (N + R - 1) / R, (cudaStream_t)stream);
  else return fail(1, "state_token: unknown dtype %d", dtype);
  return check_launch("state_token");
}
