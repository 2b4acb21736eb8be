// Single-token steps of attention through low-rank latents (bfloat16): one token a sequence, few sequences. The arithmetic
// is that of latent_attention.cu; what differs is the shape of the work, a handful of rows against whole weight matrices
// and long caches, so each kernel here spreads one step over all SMs and does in one launch what would be several.
//
//   latent_decode_attn_kernel   scores, online softmax and weighted sum of latents for all heads of a sequence over a slice
//                               of its cache rows. Sixteen warps share a chunk of 64 rows: for the scores a warp takes eight
//                               of the keys and half of the columns, for the weighted sum a share of the latent's columns,
//                               so that all of them work although a sequence brings no more rows than it has heads
//   latent_query_kernel         norm of the query latent, query up-projection, the step into the latent space, norm of the
//                               key/value latent, rotation of the key part and the cache write; a cluster of blocks a head
//   latent_value_kernel         joining of the slices with the head's sink, value up-projection, output gate; a cluster of
//                               blocks a head
#include "mma_sync.cuh"
#include "tcgen05.cuh"

namespace slb {

constexpr size_t kLdMaxSmem = 227 * 1024;      // dynamic shared memory a block may ask for
constexpr float kLdLn2 = 0.6931471805599453f;

struct LatentDecodeArgs {
  const __nv_bfloat16* q_lat;      // [H, n, R]
  const __nv_bfloat16* q_raw;      // [n, H, dn + P]; the rotated part starts at dn
  const __nv_bfloat16* pool;       // [pages, 64, R + P]
  __nv_bfloat16* out;              // [H, n, R]; splits == 1
  float* parts;                    // splits > 1: [splits, n * H, R + 2] (sum, then running maximum and mass)
  const float* cos_t;
  const float* sin_t;
  const int* past;                 // [n]: the token's position, its sequence's earlier tokens
  const int* table;                // [n, stride]
  const float* sinks;              // [H] or null
  int stride, n, H, R, P, dn, rot, window, splits, buffers;
  float scale;
};

constexpr int kLdWarps = 16, kLdThreads = kLdWarps * 32;

// Shared memory of a block: queries [16 MT][ks], `buffers` chunks of 64 cache rows [64][ks], the scores of each half of the
// columns float [2][16 MT][68], weights bfloat16 [16 MT][72], the rows' factors float [16 MT].
__host__ __device__ inline size_t latent_decode_smem(int mt, int W, int buffers) {
  const size_t rows = 16 * mt;
  return (rows + (size_t)64 * buffers) * (W + 8) * 2 + 2 * rows * 68 * 4 + rows * 72 * 2 + rows * 4;
}

// Grid: (slice, sequence, tile of 16 MT heads). NP: pairs of 8-column tiles of the latent that a warp owns (R <= 256 NP).
// KQ > 0 (one row tile, R + P = 32 KQ): a warp keeps the queries of its half of the columns, KQ steps of 16, in registers; read
// from shared memory by sixteen warps at every chunk they would be two fifths of all that is read there.
template <int MT, int NP, int KQ>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_attn_kernel(const LatentDecodeArgs a) {
  pdl_enter();
  extern __shared__ __align__(16) unsigned char ld_raw[];
  constexpr int ROWS = 16 * MT, TPR = kLdThreads / ROWS, KPT = 64 / TPR;      // threads a row, keys a thread in the softmax
  const int W = a.R + a.P, ks = W + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(ld_raw);
  __nv_bfloat16* Ks = Qs + ROWS * ks;
  float* Ss = reinterpret_cast<float*>(Ks + (size_t)a.buffers * 64 * ks);
  __nv_bfloat16* Ps = reinterpret_cast<__nv_bfloat16*>(Ss + 2 * ROWS * 68);
  float* As = reinterpret_cast<float*>(Ps + ROWS * 72);
  const int slice = blockIdx.x, seq = blockIdx.y, h0 = blockIdx.z * ROWS, nh = min(ROWS, a.H - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int pos = a.past[seq];
  const int key_lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int first = key_lo / 64 * 64;
  const int n_chunks = (pos - first) / 64 + 1;
  const int per = (n_chunks + a.splits - 1) / a.splits;
  const int c_lo = slice * per, c_hi = min(n_chunks, c_lo + per);
  const int* trow = a.table + (size_t)seq * a.stride;
  const int pieces = W / 8;

  // a chunk of 64 cache rows (a page, whose number was looked up a chunk earlier) into buffer `buf`; rows past the token
  // become zeros, never stale values
  auto page_of = [&](int c) { return c < c_hi ? trow[first / 64 + c] : 0; };
  auto load_chunk = [&](int c, int page, int buf) {
    const int k0 = first + c * 64, nk = min(64, pos - k0 + 1);
    const __nv_bfloat16* src = a.pool + (size_t)page * 64 * W;
    __nv_bfloat16* base = Ks + (size_t)buf * 64 * ks;
    for (int j = warp; j < 64; j += kLdWarps)
      for (int p = lane; p < pieces; p += 32) {
        __nv_bfloat16* dst = base + (size_t)j * ks + p * 8;
        if (j < nk) cp_async16(smem_u32(dst), src + (size_t)j * W + p * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
  };
  // one group of copies per chunk, empty past the end, so that "all but the newest groups" always means the same chunks
  const int ahead = a.buffers - 1;
  for (int i = 0; i < ahead; ++i) {
    if (c_lo + i < c_hi) load_chunk(c_lo + i, page_of(c_lo + i), i);
    cp_async_commit();
  }
  int next_page = page_of(c_lo + ahead);
  // queries: the latent part as it is, the rotated part turned by the token's angle
  const int half = a.rot / 2;
  for (int r = warp; r < ROWS; r += kLdWarps) {
    __nv_bfloat16* qs = Qs + (size_t)r * ks;
    if (r >= nh) {
      for (int i = lane * 8; i < W; i += 256) *reinterpret_cast<uint4*>(qs + i) = make_uint4(0, 0, 0, 0);
      continue;
    }
    const int h = h0 + r;
    const __nv_bfloat16* ql = a.q_lat + ((size_t)h * a.n + seq) * a.R;
    for (int i = lane * 8; i < a.R; i += 256) *reinterpret_cast<uint4*>(qs + i) = *reinterpret_cast<const uint4*>(ql + i);
    const __nv_bfloat16* qr = a.q_raw + ((size_t)seq * a.H + h) * (a.dn + a.P) + a.dn;
    for (int i = lane; i < a.P; i += 32) {
      float v = __bfloat162float(qr[i]);
      if (i < a.rot) {
        const int f = i < half ? i : i - half;
        const float c = a.cos_t[(size_t)pos * half + f], sn = a.sin_t[(size_t)pos * half + f];
        v = i < half ? v * c - __bfloat162float(qr[i + half]) * sn : v * c + __bfloat162float(qr[i - half]) * sn;
      }
      qs[a.R + i] = __float2bfloat16_rn(v);
    }
  }

  float o[MT][2 * NP][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  // the softmax state of row tid / TPR: the maximum is the row's, the mass this thread's share
  const int my_row = tid / TPR, my_key = tid % TPR;
  float m = -INFINITY, l = 0.f;
  const float scale_log2 = a.scale * 1.4426950408889634f;
  const uint32_t q_base = smem_u32(Qs), p_base = smem_u32(Ps);
  const int k16 = W / 16, k_mid = (k16 + 1) / 2;            // the columns' halves, in steps of 16
  const int kt = warp & 7, kb_lo = warp < 8 ? 0 : k_mid, kb_hi = warp < 8 ? min(k_mid, k16) : k16;
  uint32_t qr[KQ > 0 ? KQ : 1][4];
  if constexpr (KQ > 0) {
    __syncthreads();           // the queries are in shared memory
#pragma unroll
    for (int i = 0; i < KQ; ++i) ldmatrix_x4(qr[i], q_base + 2 * ((lane & 15) * ks + (kb_lo + i) * 16 + ((lane >> 4) << 3)));
  }
  int buf = 0, fill = ahead;      // the buffer of this chunk, and the one that the next load fills
  for (int c = c_lo; c < c_hi; ++c) {
    if (a.buffers == 4) cp_async_wait<2>();
    else if (a.buffers == 3) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();           // this chunk has arrived, and the one before is no longer read
    if (c + ahead < c_hi) load_chunk(c + ahead, next_page, fill);
    cp_async_commit();
    next_page = page_of(c + ahead + 1);
    const uint32_t k_base = smem_u32(Ks + (size_t)buf * 64 * ks);
    // scores of this warp's eight keys over its half of the columns, two sums a row tile so that products do not wait for one another
    float s[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[mt][0][e] = s[mt][1][e] = 0.f;
    const uint32_t k_at = k_base + 2 * ((kt * 8 + (lane & 7)) * ks + (lane >> 3) * 8);
    const uint32_t q_at = q_base + 2 * ((lane & 15) * ks + ((lane >> 4) << 3));
    if constexpr (KQ > 0) {
#pragma unroll
      for (int i = 0; i < KQ; i += 2) {
        uint32_t kf[4];
        ldmatrix_x4(kf, k_at + 2 * (kb_lo + i) * 16);
        mma_bf16(s[0][0], qr[i], kf[0], kf[1]);
        if (i + 1 < KQ) mma_bf16(s[0][1], qr[i + 1 < KQ ? i + 1 : i], kf[2], kf[3]);
      }
    } else {
#pragma unroll 4
      for (int kb = kb_lo; kb < kb_hi; kb += 2) {
        uint32_t kf[4];          // two steps of 16 columns; behind an odd last step lies padding or the next row, not used
        ldmatrix_x4(kf, k_at + 2 * kb * 16);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          uint32_t qf[4];
          ldmatrix_x4(qf, q_at + 2 * (mt * 16 * ks + kb * 16));
          mma_bf16(s[mt][0], qf, kf[0], kf[1]);
          if (kb + 1 < kb_hi) {
            ldmatrix_x4(qf, q_at + 2 * (mt * 16 * ks + kb * 16 + 16));
            mma_bf16(s[mt][1], qf, kf[2], kf[3]);
          }
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float* at = Ss + ((warp >> 3) * ROWS + mt * 16 + g) * 68 + kt * 8 + 2 * t4;
      *reinterpret_cast<float2*>(at) = make_float2(s[mt][0][0] + s[mt][1][0], s[mt][0][1] + s[mt][1][1]);
      *reinterpret_cast<float2*>(at + 8 * 68) = make_float2(s[mt][0][2] + s[mt][1][2], s[mt][0][3] + s[mt][1][3]);
    }
    __syncthreads();
    {
      const int k0 = first + c * 64;
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int key = k0 + my_key + TPR * i;
        v[i] = (Ss[my_row * 68 + my_key + TPR * i] + Ss[(ROWS + my_row) * 68 + my_key + TPR * i]) * scale_log2;
        if (key > pos || key < key_lo) v[i] = -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int w = TPR / 2; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float m_new = fmaxf(m, mx);         // finite: every chunk of a slice holds a key that the token sees
      const float alpha = exp2f(m - m_new);
      m = m_new;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const float p = exp2f(v[i] - m_new);
        sum += p;
        Ps[my_row * 72 + my_key + TPR * i] = __float2bfloat16_rn(p);
      }
      l = l * alpha + sum;
      if (my_key == 0) As[my_row] = alpha;
    }
    __syncthreads();
    // this warp's columns of the weighted sum
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float a0 = As[mt * 16 + g], a1 = As[mt * 16 + g + 8];
#pragma unroll
      for (int i = 0; i < 2 * NP; ++i) {
        o[mt][i][0] *= a0; o[mt][i][1] *= a0;
        o[mt][i][2] *= a1; o[mt][i][3] *= a1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(pf[mt], p_base + 2 * ((mt * 16 + (lane & 15)) * 72 + kk * 16 + ((lane >> 4) << 3)));
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int col = (warp + kLdWarps * i) * 16;
        if (col < a.R) {
          uint32_t vf[4];
          ldmatrix_x4_trans(vf, k_base + 2 * ((kk * 16 + (lane & 15)) * ks + col + ((lane >> 4) << 3)));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16(o[mt][2 * i], pf[mt], vf[0], vf[1]);
            mma_bf16(o[mt][2 * i + 1], pf[mt], vf[2], vf[3]);
          }
        }
      }
    }
    buf = buf + 1 == a.buffers ? 0 : buf + 1;
    fill = fill + 1 == a.buffers ? 0 : fill + 1;
  }
  cp_async_wait<0>();
  __syncthreads();             // the last chunk's factors have been read
#pragma unroll
  for (int w = TPR / 2; w > 0; w >>= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
  if (my_key == 0 && my_row < nh) {
    const int h = h0 + my_row;
    const float m_e = m == -INFINITY ? -INFINITY : m * kLdLn2;
    if (a.splits == 1) {
      float f = 1.0f, mass = l;
      if (a.sinks != nullptr) {
        const float top = fmaxf(m_e, a.sinks[h]);
        f = expf(m_e - top);
        mass = l * f + expf(a.sinks[h] - top);
      }
      As[my_row] = f / mass;
    } else {
      float* dst = a.parts + ((size_t)slice * a.n * a.H + (size_t)seq * a.H + h) * (a.R + 2);
      dst[a.R] = m_e;
      dst[a.R + 1] = l;
    }
  }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = mt * 16 + g + 8 * e;
      if (r >= nh) continue;
      const int h = h0 + r;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int col = (warp + kLdWarps * i) * 16 + 2 * t4;
        if ((warp + kLdWarps * i) * 16 >= a.R) continue;
        if (a.splits == 1) {
          const float f = As[r];
          __nv_bfloat16* dst = a.out + ((size_t)h * a.n + seq) * a.R + col;
          *reinterpret_cast<uint32_t*>(dst) = pack_bf16(o[mt][2 * i][2 * e] * f, o[mt][2 * i][2 * e + 1] * f);
          *reinterpret_cast<uint32_t*>(dst + 8) = pack_bf16(o[mt][2 * i + 1][2 * e] * f, o[mt][2 * i + 1][2 * e + 1] * f);
        } else {
          float* dst = a.parts + ((size_t)slice * a.n * a.H + (size_t)seq * a.H + h) * (a.R + 2) + col;
          *reinterpret_cast<float2*>(dst) = make_float2(o[mt][2 * i][2 * e], o[mt][2 * i][2 * e + 1]);
          *reinterpret_cast<float2*>(dst + 8) = make_float2(o[mt][2 * i + 1][2 * e], o[mt][2 * i + 1][2 * e + 1]);
        }
      }
    }
}

// ---- products of a few token rows with the matrices of one head, shared by a cluster of blocks ----
constexpr int kTeam = 8;          // blocks of a cluster: one head's rows are dealt to them
constexpr int kGroup = 8;         // tokens a cluster serves (the columns of an m16n8k16 product)
constexpr int kTeamWarps = 8;
constexpr int kAheadK = 4;        // blocks of 32 inner values whose weights a warp has in flight at once
constexpr int kRowPad = 32;       // elements behind a token row in shared memory (64 bytes, against bank conflicts)

__device__ __forceinline__ uint4 ldg_weights(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];\n" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ void st_cluster_bf16(uint32_t addr, __nv_bfloat16 v) {
  asm volatile("st.shared::cluster.b16 [%0], %1;" ::"r"(addr), "h"(*reinterpret_cast<unsigned short*>(&v)) : "memory");
}

// Sixteen weight rows times eight token rows. Lane (g, t) of a warp holds eight consecutive inner values 8t .. 8t + 7 of a
// block of 32 for weight rows g and g + 8 and for token g: two products' worth of operands (the sum over k does not care
// about the order of k as long as both sides agree). The eight warps take every eighth block of 32.
struct TeamTile {
  const __nv_bfloat16* row0;      // this lane's rows, at its first inner value, or null beyond the matrix
  const __nv_bfloat16* row1;
  uint4 wa[kAheadK], wb[kAheadK];
  // rows first .. of `limit` rows (absolute row numbers of w [.., K])
  __device__ __forceinline__ void aim(const __nv_bfloat16* w, int first, int limit, int K) {
    const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    row0 = first + g < limit ? w + (size_t)(first + g) * K + 8 * t : nullptr;
    row1 = first + g + 8 < limit ? w + (size_t)(first + g + 8) * K + 8 * t : nullptr;
  }
  __device__ __forceinline__ void fetch(int kb, int k_blocks) {
    const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int u = 0; u < kAheadK; ++u) {
      const int k = kb + u * kTeamWarps;
      wa[u] = (k < k_blocks && row0) ? ldg_weights(row0 + k * 32) : zero;
      wb[u] = (k < k_blocks && row1) ? ldg_weights(row1 + k * 32) : zero;
    }
  }
  // Products with the token rows xs [8][stride]; the first batch of weights has been fetched. acc: rows g (0, 1) and g + 8
  // (2, 3), tokens 2t and 2t + 1.
  __device__ __forceinline__ void multiply(const __nv_bfloat16* xs, int stride, int k_blocks, float (&acc)[4]) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const __nv_bfloat16* x = xs + (size_t)g * stride + 8 * t;
    acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
    for (int kb = warp; kb < k_blocks; kb += kAheadK * kTeamWarps) {
      if (kb != warp) fetch(kb, k_blocks);
#pragma unroll
      for (int u = 0; u < kAheadK; ++u) {
        const int k = kb + u * kTeamWarps;
        if (k >= k_blocks) break;
        const uint4 xv = *reinterpret_cast<const uint4*>(x + k * 32);
        const uint32_t lo[4] = {wa[u].x, wb[u].x, wa[u].y, wb[u].y}, hi[4] = {wa[u].z, wb[u].z, wa[u].w, wb[u].w};
        mma_bf16(acc, lo, xv.x, xv.y);
        mma_bf16(acc, hi, xv.z, xv.w);
      }
    }
  }
};

// The warps' partial products joined in warp order: thread (row, token) = (i / 8, i % 8) of the first 128 threads gets its sum.
__device__ __forceinline__ float team_reduce(float (*red)[16][kGroup + 1], const float (&acc)[4]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  red[warp][g][2 * t] = acc[0];
  red[warp][g][2 * t + 1] = acc[1];
  red[warp][g + 8][2 * t] = acc[2];
  red[warp][g + 8][2 * t + 1] = acc[3];
  __syncthreads();
  float v = 0.f;
  if (threadIdx.x < 16 * kGroup) {
#pragma unroll
    for (int w = 0; w < kTeamWarps; ++w) v += red[w][threadIdx.x / kGroup][threadIdx.x % kGroup];
  }
  __syncthreads();
  return v;
}

struct LatentQueryArgs {
  const float* lat;                // [n, lat_stride]: q_rank values, then R + P (and whatever follows)
  const float* q_gain;             // [q_rank]
  const float* c_gain;             // [R]
  const __nv_bfloat16* h;          // [n, K]: the queries' input when q_rank is 0
  const __nv_bfloat16* w_uq;       // [H * (dn + P), K]
  const __nv_bfloat16* w_ukt;      // [H, R, dn]: the key up-projection, transposed head by head
  const float* cos_t;
  const float* sin_t;
  __nv_bfloat16* q_lat;            // [H, n, R]
  __nv_bfloat16* q_raw;            // [n, H, dn + P]: only the rotated parts are written
  __nv_bfloat16* pool;             // [pages, 64, R + P], or null: nothing is stored
  const int* pos;                  // [n]
  const int* table;                // [n, stride]
  long long lat_stride;
  int stride, n, H, K, q_rank, R, P, dn, rot;
  float eps;
};

// Grid: x = 8 H blocks in clusters of 8 (one head each), y = groups of eight tokens. Dynamic shared memory: the token rows
// [8][K + pad], then the head's queries [8][dn + pad], every block of the cluster holding all of both.
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentQueryArgs a) {
  extern __shared__ __align__(16) unsigned char lq_raw[];
  __shared__ float red[kTeamWarps][16][kGroup + 1];
  __shared__ float scratch[33];
  const int xstride = a.K + kRowPad, qstride = a.dn + kRowPad;
  __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(lq_raw);
  __nv_bfloat16* qs = xs + kGroup * xstride;
  const int head = blockIdx.x / kTeam, rank = (int)cluster_ctarank();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = blockIdx.y * kGroup, nt = min(kGroup, a.n - t0);
  const int rows = a.dn + a.P, share = (rows + kTeam - 1) / kTeam;           // this block's rows of the up-projection
  const int r_lo = rank * share, r_hi = min(rows, r_lo + share);
  const int kb1 = a.K / 32;
  TeamTile tile;
  pdl_launch_dependents();
  tile.aim(a.w_uq + (size_t)head * rows * a.K, r_lo, r_hi, a.K);             // weights: written by no kernel
  tile.fetch(warp, kb1);
  const int cshare = (a.R + kTeam - 1) / kTeam, c_lo = rank * cshare, c_hi = min(a.R, c_lo + cshare);
  if (tid == 0 && c_lo < c_hi) {
    const NextRead second{reinterpret_cast<const char*>(a.w_ukt + ((size_t)head * a.R + c_lo) * a.dn), (long long)(c_hi - c_lo) * a.dn * 2};
    prefetch_share(second, 0, 1);
  }
  cluster_sync_all();            // every block of the cluster runs: its shared memory may be written
  pdl_wait();
  // the token rows: a warp takes one
  {
    __nv_bfloat16* x = xs + warp * xstride;
    if (warp >= nt) {
      for (int i = lane * 8; i < a.K; i += 256) *reinterpret_cast<uint4*>(x + i) = make_uint4(0, 0, 0, 0);
    } else if (a.q_rank > 0) {
      const float* row = a.lat + (size_t)(t0 + warp) * a.lat_stride;
      float ss = 0.f;
      for (int i = lane; i < a.K; i += 32) ss = fmaf(row[i], row[i], ss);
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.K + a.eps);
      for (int i = lane; i < a.K; i += 32) x[i] = __float2bfloat16_rn((row[i] * inv) * a.q_gain[i]);
    } else {
      const __nv_bfloat16* row = a.h + (size_t)(t0 + warp) * a.K;
      for (int i = lane * 8; i < a.K; i += 256) *reinterpret_cast<uint4*>(x + i) = *reinterpret_cast<const uint4*>(row + i);
    }
  }
  __syncthreads();
  // up-projection: this block's rows, given to every block of the cluster
  for (int r0 = r_lo; r0 < r_lo + share; r0 += 16) {
    if (r0 != r_lo) {
      tile.aim(a.w_uq + (size_t)head * rows * a.K, r0, r_hi, a.K);
      tile.fetch(warp, kb1);
    }
    float acc[4];
    tile.multiply(xs, xstride, kb1, acc);
    const float v = team_reduce(red, acc);
    const int r = r0 + tid / kGroup, t = tid % kGroup;
    if (tid < 16 * kGroup && r < r_hi) {
      const __nv_bfloat16 q = __float2bfloat16_rn(v);
      if (r < a.dn) {
        const uint32_t at = smem_addr(qs + t * qstride + r);
#pragma unroll
        for (int b = 0; b < kTeam; ++b) st_cluster_bf16(cluster_map(at, b), q);
      } else if (t < nt) {
        a.q_raw[((size_t)(t0 + t) * a.H + head) * rows + r] = q;
      }
    }
  }
  const int kb2 = a.dn / 32;
  tile.aim(a.w_ukt + (size_t)head * a.R * a.dn, c_lo, c_hi, a.dn);
  tile.fetch(warp, kb2);
  cluster_sync_all();            // the head's queries are complete here
  for (int r0 = c_lo; r0 < c_hi; r0 += 16) {
    if (r0 != c_lo) {
      tile.aim(a.w_ukt + (size_t)head * a.R * a.dn, r0, c_hi, a.dn);
      tile.fetch(warp, kb2);
    }
    float acc[4];
    tile.multiply(qs, qstride, kb2, acc);
    const float v = team_reduce(red, acc);
    const int r = r0 + tid / kGroup, t = tid % kGroup;
    if (tid < 16 * kGroup && r < c_hi && t < nt) a.q_lat[((size_t)head * a.n + t0 + t) * a.R + r] = __float2bfloat16_rn(v);
  }
  // the cache rows of the group's tokens, one block each
  const int mine = (int)blockIdx.x / a.H;
  if (a.pool == nullptr || (int)blockIdx.x % a.H != 0 || mine >= nt) return;
  const int t = t0 + mine, pos = a.pos[t];
  const float* row = a.lat + (size_t)t * a.lat_stride + a.q_rank;
  __nv_bfloat16* dst = a.pool + ((size_t)a.table[(size_t)t * a.stride + pos / 64] * 64 + pos % 64) * (a.R + a.P);
  float ss = 0.f;
  for (int i = tid; i < a.R; i += 256) ss = fmaf(row[i], row[i], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)a.R + a.eps);
  for (int i = tid; i < a.R; i += 256) dst[i] = __float2bfloat16_rn((row[i] * inv) * a.c_gain[i]);
  const float* kr = row + a.R;
  const int half = a.rot / 2;
  for (int i = tid; i < a.P; i += 256) {
    float v = kr[i];
    if (i < a.rot) {
      const int f = i < half ? i : i - half;
      const float c = a.cos_t[(size_t)pos * half + f], s = a.sin_t[(size_t)pos * half + f];
      v = i < half ? v * c - kr[i + half] * s : v * c + kr[i - half] * s;
    }
    dst[a.R + i] = __float2bfloat16_rn(v);
  }
}

struct LatentValueArgs {
  const float* parts;              // splits > 1: [splits, n * H, R + 2]
  const __nv_bfloat16* o_lat;      // splits == 1: [H, n, R]
  const float* sinks;              // [H] or null (with slices; without, the sink has joined already)
  const __nv_bfloat16* w_uv;       // [H * dv, R]
  const float* gate;               // [n, gate_stride] pre-activations, or null: no gate
  __nv_bfloat16* y;                // [n, H * dv]
  long long gate_stride;
  int n, H, R, dv, splits, gate_per_head;
};

// Grid as above. Dynamic shared memory: the head's weighted sums [8][R + pad], every block of the cluster holding all.
__global__ void __launch_bounds__(256) latent_value_kernel(const LatentValueArgs a) {
  extern __shared__ __align__(16) unsigned char lv_raw[];
  __shared__ float red[kTeamWarps][16][kGroup + 1];
  __shared__ float factor[kGroup][64];
  const int ostride = a.R + kRowPad;
  __nv_bfloat16* os = reinterpret_cast<__nv_bfloat16*>(lv_raw);
  const int head = blockIdx.x / kTeam, rank = (int)cluster_ctarank();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = blockIdx.y * kGroup, nt = min(kGroup, a.n - t0);
  const int share = (a.dv + kTeam - 1) / kTeam, r_lo = rank * share, r_hi = min(a.dv, r_lo + share);
  const int kb = a.R / 32;
  const __nv_bfloat16* w = a.w_uv + (size_t)head * a.dv * a.R;
  TeamTile tile;
  pdl_launch_dependents();
  tile.aim(w, r_lo, r_hi, a.R);
  tile.fetch(warp, kb);
  cluster_sync_all();            // every block of the cluster runs: its shared memory may be written
  pdl_wait();
  if (a.splits == 1) {           // every block reads the finished rows
    for (int i = tid * 8; i < kGroup * a.R; i += 2048) {
      const int t = i / a.R, c = i - t * a.R;
      *reinterpret_cast<uint4*>(os + t * ostride + c) =
          t < nt ? *reinterpret_cast<const uint4*>(a.o_lat + ((size_t)head * a.n + t0 + t) * a.R + c) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
  } else {
    // a warp forms the slices' factors of one token: exp(m_s - m) / mass, the mass summed in slice order
    const size_t rows = (size_t)a.n * a.H;
    if (warp < nt) {
      const size_t row = (size_t)(t0 + warp) * a.H + head;
      auto stat = [&](int s, int k) { return a.parts[((size_t)s * rows + row) * (a.R + 2) + a.R + k]; };
      const float m0 = lane < a.splits ? stat(lane, 0) : -INFINITY, m1 = lane + 32 < a.splits ? stat(lane + 32, 0) : -INFINITY;
      const float l0 = lane < a.splits ? stat(lane, 1) : 0.f, l1 = lane + 32 < a.splits ? stat(lane + 32, 1) : 0.f;
      float mx = warp_max(fmaxf(m0, m1));
      if (a.sinks != nullptr) mx = fmaxf(mx, a.sinks[head]);
      const float f0 = m0 == -INFINITY ? 0.f : expf(m0 - mx), f1 = m1 == -INFINITY ? 0.f : expf(m1 - mx);
      factor[warp][lane] = f0 * l0;
      factor[warp][lane + 32] = f1 * l1;
      __syncwarp();
      float mass = 0.f;
      if (lane == 0) {
        for (int s = 0; s < a.splits; ++s) mass += factor[warp][s];
        if (a.sinks != nullptr) mass += expf(a.sinks[head] - mx);
      }
      mass = __shfl_sync(0xffffffffu, mass, 0);
      const float inv = mass > 0.f ? 1.0f / mass : 0.f;
      __syncwarp();
      factor[warp][lane] = f0 * inv;
      factor[warp][lane + 32] = f1 * inv;
    }
    __syncthreads();
    // this block's share of the columns of every token's sum, given to every block of the cluster
    const int pairs = a.R / 2, pshare = (pairs + kTeam - 1) / kTeam, p_lo = rank * pshare, p_n = min(pairs, p_lo + pshare) - p_lo;
    for (int i = tid; i < kGroup * p_n; i += 256) {
      const int t = i / p_n, p = p_lo + i - t * p_n;
      float vx = 0.f, vy = 0.f;
      if (t < nt) {
        const float* src = a.parts + ((size_t)(t0 + t) * a.H + head) * (a.R + 2) + 2 * p;
        const size_t step = rows * (a.R + 2);
        constexpr int kBatch = 12;                // loads in flight; a slice without keys left zeros
        for (int s0 = 0; s0 < a.splits; s0 += kBatch) {
          float2 v[kBatch];
#pragma unroll
          for (int u = 0; u < kBatch; ++u)
            v[u] = s0 + u < a.splits ? *reinterpret_cast<const float2*>(src + (size_t)(s0 + u) * step) : make_float2(0.f, 0.f);
#pragma unroll
          for (int u = 0; u < kBatch; ++u) {
            const float f = factor[t][min(s0 + u, 63)];
            vx = fmaf(v[u].x, f, vx);
            vy = fmaf(v[u].y, f, vy);
          }
        }
      }
      const uint32_t at = smem_addr(os + t * ostride + 2 * p), two = pack_bf16(vx, vy);
#pragma unroll
      for (int b = 0; b < kTeam; ++b)
        asm volatile("st.shared::cluster.b32 [%0], %1;" ::"r"(cluster_map(at, b)), "r"(two) : "memory");
    }
    cluster_sync_all();          // the head's sums are complete here
  }
  for (int r0 = r_lo; r0 < r_hi; r0 += 16) {
    if (r0 != r_lo) {
      tile.aim(w, r0, r_hi, a.R);
      tile.fetch(warp, kb);
    }
    float acc[4];
    tile.multiply(os, ostride, kb, acc);
    float v = team_reduce(red, acc);
    const int j = r0 + tid / kGroup, t = tid % kGroup;
    if (tid < 16 * kGroup && j < r_hi && t < nt) {
      const int col = head * a.dv + j;
      if (a.gate != nullptr) v = v / (1.0f + expf(-a.gate[(size_t)(t0 + t) * a.gate_stride + (a.gate_per_head ? head : col)]));
      a.y[(size_t)(t0 + t) * a.H * a.dv + col] = __float2bfloat16_rn(v);
    }
  }
}

}  // namespace slb

using namespace slb;

// How the attention kernel is launched for these sizes: row tiles of 16 heads a block, chunks in shared memory (as many of
// four as fit). false: not taken.
struct DecodeShape {
  int mt, buffers;
};
static bool decode_shape(int H, int R, int P, DecodeShape& s) {
  const int W = R + P;
  if (H <= 0 || R <= 0 || P < 0 || R % 16 != 0 || W % 16 != 0 || R > 512) return false;
  for (int mt = H <= 16 ? 1 : (H <= 32 ? 2 : 4); mt >= 1; mt /= 2) {
    for (int buffers = 4; buffers >= 2; --buffers)
      if (latent_decode_smem(mt, W, buffers) <= kLdMaxSmem) { s = {mt, buffers}; return true; }
  }
  return false;
}

extern "C" int slb_latent_decode_supported(int H, int R, int P) {
  DecodeShape s;
  return decode_shape(H, R, P, s) ? 1 : 0;
}

// Into how many slices the keys of a single-token step of n sequences are cut (at most max_len keys a sequence): as many as
// keep every SM busy once, a slice being at least a page.
extern "C" int slb_latent_decode_splits(int n, int H, int R, int P, int max_len) {
  DecodeShape s;
  if (n <= 0 || !decode_shape(H, R, P, s)) return 1;
  const int blocks = n * ((H + 16 * s.mt - 1) / (16 * s.mt)), pages = (max_len + 63) / 64;
  int splits = sm_count() / blocks;
  if (splits > pages) splits = pages;
  if (splits > 64) splits = 64;
  return splits < 1 ? 1 : splits;
}

// One token a sequence. parts: scratch [splits, n * H, R + 2] float32 when splits > 1 (slb_latent_value joins them), else the
// result goes to out [H, n, R].
extern "C" int slb_latent_decode_attention(const void* q_lat, const void* q_raw, const void* pool, void* out, float* parts,
                                           const float* cos_t, const float* sin_t, const int* past, const int* table, int stride,
                                           int n, int H, int R, int P, int dn, int rot, int window, float scale, int splits,
                                           const float* sinks, void* stream) {
  DecodeShape shape;
  SLB_REQUIRE(decode_shape(H, R, P, shape), "latent_decode_attention: %d heads, latent %d, rotated part %d are not taken", H, R, P);
  SLB_REQUIRE(n >= 0 && stride > 0 && rot >= 0 && rot <= P && rot % 2 == 0 && window >= 0 && splits >= 1 && splits <= 64 &&
                  (splits == 1 ? out != nullptr : parts != nullptr),
              "latent_decode_attention: n=%d rot=%d window=%d splits=%d", n, rot, window, splits);
  SLB_REQUIRE(((uintptr_t)q_lat | (uintptr_t)pool | (uintptr_t)out | (uintptr_t)parts) % 16 == 0, "latent_decode_attention: 16-byte alignment");
  if (n == 0) return 0;
  LatentDecodeArgs a;
  a.q_lat = (const __nv_bfloat16*)q_lat; a.q_raw = (const __nv_bfloat16*)q_raw; a.pool = (const __nv_bfloat16*)pool;
  a.out = (__nv_bfloat16*)out; a.parts = parts; a.cos_t = cos_t; a.sin_t = sin_t; a.past = past; a.table = table; a.sinks = sinks;
  a.stride = stride; a.n = n; a.H = H; a.R = R; a.P = P; a.dn = dn; a.rot = rot; a.window = window; a.splits = splits;
  a.buffers = shape.buffers; a.scale = scale;
  const size_t smem = latent_decode_smem(shape.mt, R + P, shape.buffers);
  const dim3 grid(splits, n, (H + 16 * shape.mt - 1) / (16 * shape.mt)), block(kLdThreads);
  cudaStream_t s = (cudaStream_t)stream;
  const bool one = R <= 256;
#define SLB_LD(MT, NP, KQ)                                                                                                   \
  do {                                                                                                                       \
    static bool raised = false;                                                                                              \
    if (!raised) {                                                                                                           \
      cudaFuncSetAttribute(latent_decode_attn_kernel<MT, NP, KQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLdMaxSmem); \
      raised = true;                                                                                                         \
    }                                                                                                                        \
    launch(latent_decode_attn_kernel<MT, NP, KQ>, grid, block, smem, s, a);                                                      \
  } while (0)
#define SLB_LD_NP(MT) \
  do { if (one) SLB_LD(MT, 1, 0); else SLB_LD(MT, 2, 0); } while (0)
  if (shape.mt == 1) {
    const int width = R + P;
    if (one && width == 64) SLB_LD(1, 1, 2); else if (one && width == 128) SLB_LD(1, 1, 4);
    else if (one && width == 256) SLB_LD(1, 1, 8); else if (one && width == 288) SLB_LD(1, 1, 9);
    else if (!one && width == 512) SLB_LD(1, 2, 16); else if (!one && width == 576) SLB_LD(1, 2, 18);
    else SLB_LD_NP(1);
  } else if (shape.mt == 2) SLB_LD_NP(2); else SLB_LD_NP(4);
#undef SLB_LD_NP
#undef SLB_LD
  return check_launch("latent_decode_attention");
}

static size_t query_smem(int K, int dn) { return (size_t)kGroup * (K + dn + 2 * kRowPad) * 2; }
static size_t value_smem(int R) { return (size_t)kGroup * (R + kRowPad) * 2; }

// Whether the two cluster kernels take these sizes (K: inner width of the query up-projection).
extern "C" int slb_latent_team_supported(int K, int dn, int R) {
  return K >= 32 && K % 32 == 0 && dn >= 32 && dn % 32 == 0 && R >= 32 && R % 32 == 0 && query_smem(K, dn) <= kLdMaxSmem - 8 * 1024 &&
                 value_smem(R) <= kLdMaxSmem - 8 * 1024 ? 1 : 0;
}

extern "C" int slb_latent_query(const float* lat, long long lat_stride, const float* q_gain, const float* c_gain, const void* h,
                                const void* w_uq, const void* w_ukt, const float* cos_t, const float* sin_t, void* q_lat, void* q_raw,
                                void* pool, const int* pos, const int* table, int stride, int n, int H, int K, int q_rank, int R,
                                int P, int dn, int rot, float eps, void* stream) {
  SLB_REQUIRE(slb_latent_team_supported(K, dn, R), "latent_query: inner widths %d, %d, %d are not taken", K, dn, R);
  SLB_REQUIRE(n >= 0 && H > 0 && (q_rank == 0 ? h != nullptr : q_rank == K && q_gain != nullptr) && P >= 0 && rot >= 0 && rot <= P && rot % 2 == 0 &&
                  lat_stride >= q_rank + R + P && eps > 0.f && (pool == nullptr || stride > 0) && (P == 0 || q_raw != nullptr),
              "latent_query: n=%d heads=%d q_rank=%d rot_dim=%d", n, H, q_rank, P);
  SLB_REQUIRE(((uintptr_t)h | (uintptr_t)w_uq | (uintptr_t)w_ukt) % 16 == 0, "latent_query: 16-byte alignment");
  if (n == 0) return 0;
  LatentQueryArgs a;
  a.lat = lat; a.lat_stride = lat_stride; a.q_gain = q_gain; a.c_gain = c_gain; a.h = (const __nv_bfloat16*)h;
  a.w_uq = (const __nv_bfloat16*)w_uq; a.w_ukt = (const __nv_bfloat16*)w_ukt; a.cos_t = cos_t; a.sin_t = sin_t;
  a.q_lat = (__nv_bfloat16*)q_lat; a.q_raw = (__nv_bfloat16*)q_raw; a.pool = (__nv_bfloat16*)pool; a.pos = pos; a.table = table;
  a.stride = stride; a.n = n; a.H = H; a.K = K; a.q_rank = q_rank; a.R = R; a.P = P; a.dn = dn; a.rot = rot; a.eps = eps;
  static bool raised = false;
  if (!raised) {
    cudaFuncSetAttribute(latent_query_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLdMaxSmem - 8 * 1024);
    raised = true;
  }
  launch_clusters(pdl_mode() != 0, kTeam, latent_query_kernel, dim3(kTeam * H, (n + kGroup - 1) / kGroup), dim3(256), query_smem(K, dn),
                  (cudaStream_t)stream, a);
  return check_launch("latent_query");
}

extern "C" int slb_latent_value(const float* parts, const void* o_lat, const float* sinks, const void* w_uv, const float* gate,
                                long long gate_stride, int gate_per_head, void* y, int n, int H, int R, int dv, int splits, void* stream) {
  SLB_REQUIRE(R >= 32 && R % 32 == 0 && value_smem(R) <= kLdMaxSmem - 8 * 1024, "latent_value: a latent of %d values is not taken", R);
  SLB_REQUIRE(n >= 0 && H > 0 && dv > 0 && splits >= 1 && splits <= 64 && (splits == 1 ? o_lat != nullptr : parts != nullptr) &&
                  (gate == nullptr || gate_stride >= (gate_per_head ? H : (long long)H * dv)),
              "latent_value: n=%d heads=%d width=%d slices=%d", n, H, dv, splits);
  SLB_REQUIRE(((uintptr_t)parts | (uintptr_t)o_lat | (uintptr_t)w_uv) % 16 == 0, "latent_value: 16-byte alignment");
  if (n == 0) return 0;
  LatentValueArgs a;
  a.parts = parts; a.o_lat = (const __nv_bfloat16*)o_lat; a.sinks = sinks; a.w_uv = (const __nv_bfloat16*)w_uv; a.gate = gate;
  a.y = (__nv_bfloat16*)y; a.gate_stride = gate_stride; a.n = n; a.H = H; a.R = R; a.dv = dv; a.splits = splits; a.gate_per_head = gate_per_head;
  static bool raised = false;
  if (!raised) {
    cudaFuncSetAttribute(latent_value_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLdMaxSmem - 8 * 1024);
    raised = true;
  }
  launch_clusters(pdl_mode() != 0, kTeam, latent_value_kernel, dim3(kTeam * H, (n + kGroup - 1) / kGroup), dim3(256), value_smem(R),
                  (cudaStream_t)stream, a);
  return check_launch("latent_value");
}
