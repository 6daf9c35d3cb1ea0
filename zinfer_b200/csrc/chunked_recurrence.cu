// Long portions of the recurrences with one decay per head and token (linear_attention.cu has the form that walks the
// tokens one by one), in chunks of 64 tokens whose work is matrix products:
//
//     S <- g_t S ;  u_t = beta_t (v_t - S^T k_t) (delta rule)  or  u_t = beta_t v_t ;  S <- S + k_t u_t^T ;  o_t = S^T q_t
//
// With c_t = log g_1 + .. + log g_t inside a chunk that begins from S0, the chunk's updates U solve a triangular system,
// (I + L) U = diag(beta) (V - diag(e^c) K S0) with L_ts = beta_t e^(c_t - c_s) (k_t . k_s) for s < t, so that U = U0 - W S0
// with (I + L) [W | U0] = diag(beta) [diag(e^c) K | V]; then
//
//     O = diag(e^c) Q S0 + P U,  P_ts = e^(c_t - c_s) (q_t . k_s) for s <= t ;   S1 = e^(c_64) S0 + K^T diag(e^(c_64 - c)) U
//
// (the chunked form of "Parallelizing Linear Transformers with the Delta Rule over Sequence Length", Yang et al., 2024, and
// of "Gated Delta Networks", Yang et al., 2024; without the delta rule W = 0 and U = diag(beta) V, the state-space duality of
// Dao and Gu, 2024).  The kernels:
//   1. chunk_scores   per chunk and key head: q . k and k . k (32-bit multiply-adds), Q and K as pairs of bfloat16
//                     values (high part and remainder: 16 bits of mantissa together), the sums c of every head
//   2. chunk_weights  per chunk and head: P as pairs of bfloat16 values
//      chunk_solve    (delta rule) per chunk and head: the triangular system by forward substitution in 32-bit, a
//                     thread per column of [W | U0]; W as pairs of bfloat16 values
//   3. chunk_walk     per request, head and 32 value channels: the chunks in order; the products with the state on the
//                     tensor cores (mma.sync, each operand as two bfloat16 parts, three products, 32-bit sums); the state
//                     stays in 32-bit accumulators
// The first ones do all chunks side by side; only the last walks.  A request's chunks begin with its portion; the places of
// its chunks in the workspace follow from cu_q alone: chunk i of request s lies at cu_q[s] / 64 + s + i.
#include "api.h"
#include "common.cuh"

namespace {
constexpr int CK = 64;               // tokens per chunk
constexpr int CK_VP = 32;            // value channels per block of the walk
constexpr int CK_PAD = 8;            // bfloat16 elements behind every row in shared memory: rows start 16 bytes further on
using bf = __nv_bfloat16;

struct Chunked {
  const float* q;      // [T][G * D] rows, ready (unit vectors, scale)
  const float* k;
  const float* v;      // [T][H * V]
  int ldq, ldk, ldv;
  const float* logg;   // [T][H] logarithms of the decays
  const float* beta;   // [T][H]
  float* state;
  long long slot_stride;
  int H, G, D, V;
  const int* cu_q;
  const int* state_slots;
  int n_seqs, slots;
  float* out;          // [T][H * V]
  int ldo;
  // workspace
  bf* qs;              // [slots][G][2][CK][D]
  bf* ks;
  float* qk;           // [slots][G][CK][CK]
  float* kk;           // delta rule only
  float* c;            // [slots][H][CK] sums of the logarithms, to base 2
  bf* p;               // [slots][H][2][CK][CK] P
  bf* w;               // [slots][H][2][CK][D]
  float* u0;           // [slots][H][CK][V]
};

__device__ __forceinline__ bool chunk_of(const Chunked& j, int slot, int& seq, int& first, int& n) {
  int lo = 0, hi = j.n_seqs - 1;      // the last request whose first place is at or before this one
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (j.cu_q[mid] / CK + mid <= slot) lo = mid; else hi = mid - 1;
  }
  seq = lo;
  const int tok0 = j.cu_q[lo], qlen = j.cu_q[lo + 1] - tok0, i = slot - (tok0 / CK + lo);
  first = tok0 + i * CK;
  n = min(CK, qlen - i * CK);
  return qlen > 1 && i >= 0 && n > 0;                 // single tokens are not done here
}

__device__ __forceinline__ void split2(float x, bf& hi, bf& lo) {
  hi = __float2bfloat16_rn(x);
  lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
__device__ __forceinline__ uint32_t pack2(bf a, bf b) {
  const __nv_bfloat162 p = __halves2bfloat162(a, b);
  return *reinterpret_cast<const uint32_t*>(&p);
}

// ------------------------------------------------------------------------------------------- 1. scores
constexpr float LOG2E = 1.4426950408889634f;
constexpr int CS_THREADS = 256, CS_PITCH = CK + 4;

template <bool DELTA>
__global__ void __launch_bounds__(CS_THREADS)
chunk_scores_kernel(const Chunked j) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float cs[];
  float* qt = cs;                                     // [D][CS_PITCH]: transposed, so that four tokens are one read
  float* kt = qt + j.D * CS_PITCH;
  const int slot = blockIdx.x, g = blockIdx.y, tid = threadIdx.x, D = j.D;
  int seq, first, n;
  if (!chunk_of(j, slot, seq, first, n)) {            // uniform in the block
    pdl_wait();
    return;
  }
  pdl_wait();
  bf* qo = j.qs + ((size_t)slot * j.G + g) * 2 * CK * D;
  bf* ko = j.ks + ((size_t)slot * j.G + g) * 2 * CK * D;
  // a warp takes 4 tokens x 32 channels at a time: whole lines of memory, few lanes on one bank
  for (int e = tid; e < CK * 8 * ((D + 31) / 32); e += CS_THREADS) {
    const int unit = e >> 5, l = e & 31;
    const int t = (unit & 15) * 4 + (l >> 3), i = (unit >> 4) * 32 + (l & 7) * 4;
    if (i >= D) continue;
    float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
    if (t < n) {
      const float* pq = j.q + (size_t)(first + t) * j.ldq + (size_t)g * D + i;
      const float* pk = j.k + (size_t)(first + t) * j.ldk + (size_t)g * D + i;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        a[u] = pq[u];
        b[u] = pk[u];
      }
    }
    bf ah[4], al[4], bh[4], bl[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      qt[(i + u) * CS_PITCH + t] = a[u];
      kt[(i + u) * CS_PITCH + t] = b[u];
      split2(a[u], ah[u], al[u]);
      split2(b[u], bh[u], bl[u]);
    }
    const size_t at = (size_t)t * D + i;
    *reinterpret_cast<uint2*>(qo + at) = make_uint2(pack2(ah[0], ah[1]), pack2(ah[2], ah[3]));
    *reinterpret_cast<uint2*>(qo + CK * D + at) = make_uint2(pack2(al[0], al[1]), pack2(al[2], al[3]));
    *reinterpret_cast<uint2*>(ko + at) = make_uint2(pack2(bh[0], bh[1]), pack2(bh[2], bh[3]));
    *reinterpret_cast<uint2*>(ko + CK * D + at) = make_uint2(pack2(bl[0], bl[1]), pack2(bl[2], bl[3]));
  }
  // the sums of the logarithms, two tokens per lane, a warp per head of this key head's group
  const int warp = tid >> 5, lane = tid & 31, rep = j.H / j.G;
  for (int r = warp; r < rep; r += CS_THREADS / 32) {
    const int h = g * rep + r;
    float a = 2 * lane < n ? j.logg[(size_t)(first + 2 * lane) * j.H + h] * LOG2E : 0.f;
    float b = 2 * lane + 1 < n ? j.logg[(size_t)(first + 2 * lane + 1) * j.H + h] * LOG2E : 0.f;
    b += a;
    float run = b;                                    // both tokens; then of all lanes up to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += x;
    }
    float before = __shfl_up_sync(0xffffffffu, run, 1);
    if (lane == 0) before = 0.f;
    float* co = j.c + ((size_t)slot * j.H + h) * CK;
    co[2 * lane] = before + a;
    co[2 * lane + 1] = before + b;
  }
  __syncthreads();
  const int ty = tid >> 4, tx = tid & 15;             // four tokens t x four tokens s per thread
  if (tx > ty) return;                                // s > t throughout: never read
  float qk[4][4], kk[4][4];
#pragma unroll
  for (int a = 0; a < 4; ++a)
#pragma unroll
    for (int b = 0; b < 4; ++b) qk[a][b] = kk[a][b] = 0.f;
  for (int i = 0; i < D; ++i) {
    const float4 q4 = *reinterpret_cast<const float4*>(qt + i * CS_PITCH + 4 * ty);
    const float4 s4 = *reinterpret_cast<const float4*>(kt + i * CS_PITCH + 4 * tx);
    const float qa[4] = {q4.x, q4.y, q4.z, q4.w}, sa[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b) qk[a][b] = fmaf(qa[a], sa[b], qk[a][b]);
    if constexpr (DELTA) {
      const float4 k4 = *reinterpret_cast<const float4*>(kt + i * CS_PITCH + 4 * ty);
      const float ka[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
      for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) kk[a][b] = fmaf(ka[a], sa[b], kk[a][b]);
    }
  }
  const size_t base = ((size_t)slot * j.G + g) * CK * CK;
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    *reinterpret_cast<float4*>(j.qk + base + (4 * ty + a) * CK + 4 * tx) = make_float4(qk[a][0], qk[a][1], qk[a][2], qk[a][3]);
    if constexpr (DELTA)
      *reinterpret_cast<float4*>(j.kk + base + (4 * ty + a) * CK + 4 * tx) = make_float4(kk[a][0], kk[a][1], kk[a][2], kk[a][3]);
  }
}

// -------------------------------------------------------------------------------- 2. weights, the triangular system
// Per chunk and head: P as pairs of bfloat16 values.
constexpr int CP_THREADS = 256;

__global__ void __launch_bounds__(CP_THREADS)
chunk_weights_kernel(const Chunked j) {
  pdl_launch_dependents();
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  int seq, first, n;
  const bool on = chunk_of(j, slot, seq, first, n);
  pdl_wait();
  if (!on) return;
  const int g = h / (j.H / j.G);
  const float* c = j.c + ((size_t)slot * j.H + h) * CK;
  const float* qk = j.qk + ((size_t)slot * j.G + g) * CK * CK;
  bf* po = j.p + ((size_t)slot * j.H + h) * 2 * CK * CK;
  for (int e = tid; e < CK * CK / 4; e += CP_THREADS) {
    const int t = e / (CK / 4), s = (e - t * (CK / 4)) * 4;
    if (s >= (t & ~15) + 16) continue;                // 16 x 16 parts above the diagonal are never read
    const float4 q4 = s <= t ? *reinterpret_cast<const float4*>(qk + t * CK + s) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 c4 = *reinterpret_cast<const float4*>(c + s);
    const float ct = c[t];
    const float w[4] = {q4.x * exp2f(ct - c4.x), s + 1 <= t ? q4.y * exp2f(ct - c4.y) : 0.f, s + 2 <= t ? q4.z * exp2f(ct - c4.z) : 0.f,
                        s + 3 <= t ? q4.w * exp2f(ct - c4.w) : 0.f};
    bf hi[4], lo[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) split2(s + u <= t ? w[u] : 0.f, hi[u], lo[u]);
    *reinterpret_cast<uint2*>(po + t * CK + s) = make_uint2(pack2(hi[0], hi[1]), pack2(hi[2], hi[3]));
    *reinterpret_cast<uint2*>(po + CK * CK + t * CK + s) = make_uint2(pack2(lo[0], lo[1]), pack2(lo[2], lo[3]));
  }
}

// (delta rule) Per chunk and head: [W | U0] by forward substitution, a column per thread.
constexpr int SV_B = 16;             // rows per block of the substitution
constexpr int NT = 128;              // columns per block

__global__ void __launch_bounds__(NT)
chunk_solve_kernel(const Chunked j) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sv[];
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, D = j.D, V = j.V;
  float* lt = sv;                                     // [s][t]: L transposed, CS_PITCH apart
  float* bs = lt + CK * CS_PITCH;                     // beta, then beta e^c
  float* be = bs + CK;
  float* xs = be + CK;                                // [CK][NT]: solved rows of this block's columns
  int seq, first, n;
  const bool on_chunk = chunk_of(j, slot, seq, first, n);
  pdl_wait();
  if (!on_chunk) return;
  const int g = h / (j.H / j.G);
  const float* c = j.c + ((size_t)slot * j.H + h) * CK;
  const float* kk = j.kk + ((size_t)slot * j.G + g) * CK * CK;
  for (int t = tid; t < CK; t += NT) {
    const float b = t < n ? j.beta[(size_t)(first + t) * j.H + h] : 0.f;
    bs[t] = b;
    be[t] = b * exp2f(c[t]);
  }
  __syncthreads();
  for (int e = tid; e < CK * CK; e += NT) {
    const int s = e / CK, t = e - s * CK;
    lt[s * CS_PITCH + t] = s < t ? bs[t] * exp2f(c[t] - c[s]) * kk[t * CK + s] : 0.f;
  }
  __syncthreads();
  bf* wo = j.w + ((size_t)slot * j.H + h) * 2 * CK * D;
  float* uo = j.u0 + ((size_t)slot * j.H + h) * CK * V;
  const int col = blockIdx.z * NT + tid;
  const bool on = col < D + V, is_k = col < D;
  const float* src = is_k ? j.k + (size_t)first * j.ldk + (size_t)g * D + col : j.v + (size_t)first * j.ldv + (size_t)h * V + col - D;
  const int ld = is_k ? j.ldk : j.ldv;
  const float* mul = is_k ? be : bs;
  float next[SV_B];
#pragma unroll
  for (int r = 0; r < SV_B; ++r) next[r] = on && r < n ? src[(size_t)r * ld] : 0.f;
#pragma unroll 1
  for (int bi = 0; bi < CK; bi += SV_B) {
    float acc[SV_B];
#pragma unroll
    for (int r = 0; r < SV_B; ++r) acc[r] = mul[bi + r] * next[r];
    if (bi + SV_B < CK) {
#pragma unroll
      for (int r = 0; r < SV_B; ++r) next[r] = on && bi + SV_B + r < n ? src[(size_t)(bi + SV_B + r) * ld] : 0.f;
    }
#pragma unroll 4
    for (int s = 0; s < bi; ++s) {
      const float x = xs[s * NT + tid];
#pragma unroll
      for (int r = 0; r < SV_B; r += 4) {
        const float4 l = *reinterpret_cast<const float4*>(lt + s * CS_PITCH + bi + r);
        acc[r] = fmaf(-l.x, x, acc[r]);
        acc[r + 1] = fmaf(-l.y, x, acc[r + 1]);
        acc[r + 2] = fmaf(-l.z, x, acc[r + 2]);
        acc[r + 3] = fmaf(-l.w, x, acc[r + 3]);
      }
    }
#pragma unroll
    for (int s = 0; s < SV_B; ++s) {                  // only rows below the diagonal change
#pragma unroll
      for (int r = s & ~3; r < SV_B; r += 4) {
        const float4 l = *reinterpret_cast<const float4*>(lt + (bi + s) * CS_PITCH + bi + r);
        if (r > s) acc[r] = fmaf(-l.x, acc[s], acc[r]);
        if (r + 1 > s) acc[r + 1] = fmaf(-l.y, acc[s], acc[r + 1]);
        if (r + 2 > s) acc[r + 2] = fmaf(-l.z, acc[s], acc[r + 2]);
        if (r + 3 > s) acc[r + 3] = fmaf(-l.w, acc[s], acc[r + 3]);
      }
    }
#pragma unroll
    for (int r = 0; r < SV_B; ++r) {
      xs[(bi + r) * NT + tid] = acc[r];               // read by this thread only
      if (on) {
        if (is_k) {
          bf hi, lo;
          split2(acc[r], hi, lo);
          wo[(size_t)(bi + r) * D + col] = hi;
          wo[(size_t)CK * D + (size_t)(bi + r) * D + col] = lo;
        } else {
          uo[(size_t)(bi + r) * V + col - D] = acc[r];
        }
      }
    }
  }
}

// -------------------------------------------------------------------------------------------- 3. the walk
// Two groups of 8 warps share a chunk: the first moves the state on (W S, U, K^T U), the second reads out (Q S, P U).  In
// both, warp (row group wr of 16 tokens or key channels, column half wc of 16 value channels).
constexpr int CW_THREADS = 512;

__device__ __forceinline__ void ck_ldsm(uint32_t* r, const bf* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ck_ldsm_t(uint32_t* r, const bf* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ck_mma(float* d, const uint32_t* a, const uint32_t* b) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// Two neighbouring 16 x 8 tiles, both operands in two parts; the product of the remainders is below the sums' own
// rounding.  The tiles take turns, so that a product does not wait for the one right before it.
__device__ __forceinline__ void ck_mma3(float (&d)[2][4], const uint32_t* ah, const uint32_t* al, const uint32_t* bh, const uint32_t* bl) {
  ck_mma(d[0], al, bh);
  ck_mma(d[1], al, bh + 2);
  ck_mma(d[0], ah, bl);
  ck_mma(d[1], ah, bl + 2);
  ck_mma(d[0], ah, bh);
  ck_mma(d[1], ah, bh + 2);
}
__device__ __forceinline__ void ck_cp16(void* dst, const void* src) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}

constexpr int CW_PP = CK + CK_PAD;   // pitch of P

size_t ck_walk_smem(int D, bool delta) {
  const size_t tile = (size_t)2 * CK * (D + CK_PAD) * sizeof(bf);                   // Q, K or W in two parts
  return tile * (delta ? 4 : 3) + 2 * (size_t)2 * CK * CW_PP * sizeof(bf) + 2 * CK * sizeof(float)
         + (size_t)2 * D * (CK_VP + CK_PAD) * sizeof(bf) + (size_t)4 * CK * (CK_VP + CK_PAD) * sizeof(bf);
}

template <bool DELTA>
__global__ void __launch_bounds__(CW_THREADS)
chunk_walk_kernel(const Chunked j) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) char walk_smem[];
  const int D = j.D, DP = D + CK_PAD, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wr = warp & 3, wc = (warp >> 2) & 1;
  const bool moves = warp < 8;                        // of the first group
  constexpr int VP = CK_VP + CK_PAD;
  const int tile = 2 * CK * DP, ptile = 2 * CK * CW_PP;       // elements of a tile in two parts
  bf* Q = reinterpret_cast<bf*>(walk_smem);
  bf* K = Q + tile;                                   // twice
  bf* W = K + 2 * tile;                               // delta rule only
  bf* P = W + (DELTA ? tile : 0);                     // twice
  float* Cs = reinterpret_cast<float*>(P + 2 * ptile);        // sums of the logarithms, twice
  bf* Ss = reinterpret_cast<bf*>(Cs + 2 * CK);        // the state, two parts of [D][VP]
  bf* Us = Ss + 2 * D * VP;                           // U, two parts of [CK][VP]; then U e^(c_64 - c), two parts
  const int seq = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * CK_VP;
  const int tok0 = j.cu_q[seq], qlen = j.cu_q[seq + 1] - tok0;
  pdl_wait();
  if (qlen <= 1) return;                              // single tokens are not done here
  const int g = h / (j.H / j.G), chunks = (qlen + CK - 1) / CK, slot0 = tok0 / CK + seq;
  float* S = j.state + (size_t)j.state_slots[seq] * j.slot_stride + (size_t)h * D * j.V;
  const bool pairs = j.V % 2 == 0 && j.ldv % 2 == 0 && j.ldo % 2 == 0 && ((uintptr_t)j.v & 7) == 0 && ((uintptr_t)j.out & 7) == 0;
  const int fr = lane >> 2, fc = (lane & 3) * 2;      // an accumulator's first row and column
  const int lr = lane & 15, lc = (lane >> 4) * 8;     // ldmatrix: this lane's row and column offset within 16 x 16

  // the rolling loads of a chunk: Q and W once, K, P and the sums in two buffers
  auto load = [&](int i) {
    const int slot = slot0 + i, buf = i & 1;
    const size_t at = ((size_t)slot * j.G + g) * 2 * CK * D, wat = ((size_t)slot * j.H + h) * 2 * CK * D;
    const int x = (tid & 15) * 8;                     // 16 threads a row (D <= 128), rows of both parts
#pragma unroll
    for (int r = tid >> 4; r < 2 * CK; r += CW_THREADS / 16) {
      if (x >= D) break;
      ck_cp16(Q + r * DP + x, j.qs + at + (size_t)r * D + x);
      ck_cp16(K + buf * tile + r * DP + x, j.ks + at + (size_t)r * D + x);
      if (DELTA) ck_cp16(W + r * DP + x, j.w + wat + (size_t)r * D + x);
    }
    const bf* p = j.p + ((size_t)slot * j.H + h) * 2 * CK * CK;
#pragma unroll
    for (int r = tid >> 3; r < 2 * CK; r += CW_THREADS / 8) {
      const int s = (tid & 7) * 8;
      if (s < ((r & (CK - 1)) & ~15) + 16) ck_cp16(P + buf * ptile + r * CW_PP + s, p + r * CK + s);
    }
    if (tid < CK / 4) ck_cp16(Cs + buf * CK + tid * 4, j.c + ((size_t)slot * j.H + h) * CK + tid * 4);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0);

  // the state in the first group's accumulators: key channels 16 (wr + 4 m) .., value channels 16 wc + 8 n ..
  float acc[2][2][4] = {};
  auto each_state = [&](auto f) {
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      if (!moves || (wr + 4 * m) * 16 >= D) continue;
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int row = (wr + 4 * m) * 16 + fr + (e >> 1) * 8, col = wc * 16 + nn * 8 + fc + (e & 1);
          f(acc[m][nn][e], row, col);
        }
    }
  };
  each_state([&](float& x, int row, int col) { x = v0 + col < j.V ? S[(size_t)row * j.V + v0 + col] : 0.f; });
  auto share_state = [&] {                            // into shared memory, in two parts
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      if (!moves || (wr + 4 * m) * 16 >= D) continue;
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int row = (wr + 4 * m) * 16 + fr + (e >> 1) * 8, col = wc * 16 + nn * 8 + fc;
          bf ah, al, bh, bl;
          split2(acc[m][nn][e], ah, al);
          split2(acc[m][nn][e + 1], bh, bl);
          *reinterpret_cast<uint32_t*>(Ss + row * VP + col) = pack2(ah, bh);
          *reinterpret_cast<uint32_t*>(Ss + D * VP + row * VP + col) = pack2(al, bl);
        }
    }
  };
  share_state();

  for (int i = 0; i < chunks; ++i) {
    const int n = min(CK, qlen - i * CK), first = tok0 + i * CK, buf = i & 1;
    const float* cs = Cs + buf * CK;
    // what becomes U: asked for now, needed after the product with the state
    float u[2][4], step[2] = {1.f, 1.f};
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = wr * 16 + fr + r * 8;
      if (!DELTA) step[r] = moves && t < n ? j.beta[(size_t)(first + t) * j.H + h] : 0.f;
      const float* pu = DELTA ? j.u0 + (((size_t)(slot0 + i) * j.H + h) * CK + t) * j.V : j.v + (size_t)(first + t) * j.ldv + (size_t)h * j.V;
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
        const int col = v0 + wc * 16 + nn * 8 + fc;
        float2 x = make_float2(0.f, 0.f);
        if (moves && t < n && pairs && col < j.V) {
          x = *reinterpret_cast<const float2*>(pu + col);
        } else if (moves && t < n) {
          if (col < j.V) x.x = pu[col];
          if (col + 1 < j.V) x.y = pu[col + 1];
        }
        u[nn][2 * r] = x.x;
        u[nn][2 * r + 1] = x.y;
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                  // this chunk's tiles and the state are there; the chunk before is done with
    const float ct[2] = {cs[wr * 16 + fr], cs[wr * 16 + fr + 8]}, cend = cs[CK - 1];
    float so[2][4] = {};                              // W S, or Q S
    if (DELTA || !moves) {
      const bf* A = moves ? W : Q;
#pragma unroll 4
      for (int kk = 0; kk < D; kk += 16) {
        uint32_t bh[4], bl[4], ah[4], al[4];
        ck_ldsm_t(bh, Ss + (kk + lr) * VP + wc * 16 + lc);
        ck_ldsm_t(bl, Ss + D * VP + (kk + lr) * VP + wc * 16 + lc);
        ck_ldsm(ah, A + (wr * 16 + lr) * DP + kk + lc);
        ck_ldsm(al, A + CK * DP + (wr * 16 + lr) * DP + kk + lc);
        ck_mma3(so, ah, al, bh, bl);
      }
    }
    if (moves) {
      const float f[2] = {exp2f(cend - ct[0]), exp2f(cend - ct[1])};
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int row = wr * 16 + fr + (e >> 1) * 8, col = wc * 16 + nn * 8 + fc;
          const float x = DELTA ? u[nn][e] - so[nn][e] : step[e >> 1] * u[nn][e];
          const float y = DELTA ? u[nn][e + 1] - so[nn][e + 1] : step[e >> 1] * u[nn][e + 1];
          bf xh, xl, yh, yl;
          split2(x, xh, xl);
          split2(y, yh, yl);
          *reinterpret_cast<uint32_t*>(Us + row * VP + col) = pack2(xh, yh);
          *reinterpret_cast<uint32_t*>(Us + CK * VP + row * VP + col) = pack2(xl, yl);
          split2(x * f[e >> 1], xh, xl);
          split2(y * f[e >> 1], yh, yl);
          *reinterpret_cast<uint32_t*>(Us + 2 * CK * VP + row * VP + col) = pack2(xh, yh);
          *reinterpret_cast<uint32_t*>(Us + 3 * CK * VP + row * VP + col) = pack2(xl, yl);
        }
    }
    __syncthreads();                                  // U is there; nobody reads Q, W and the state any more
    if (i + 1 < chunks) load(i + 1);
    if (!moves) {                                     // O = e^c Q S + P U
      const float f[2] = {exp2f(ct[0]), exp2f(ct[1])};
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int e = 0; e < 4; ++e) so[nn][e] *= f[e >> 1];
      const bf* Pb = P + buf * ptile;
#pragma unroll
      for (int kb = 0; kb < CK / 16; ++kb) {
        if (kb > wr) break;
        uint32_t ah[4], al[4], bh[4], bl[4];
        ck_ldsm(ah, Pb + (wr * 16 + lr) * CW_PP + kb * 16 + lc);
        ck_ldsm(al, Pb + CK * CW_PP + (wr * 16 + lr) * CW_PP + kb * 16 + lc);
        ck_ldsm_t(bh, Us + (kb * 16 + lr) * VP + wc * 16 + lc);
        ck_ldsm_t(bl, Us + CK * VP + (kb * 16 + lr) * VP + wc * 16 + lc);
        ck_mma3(so, ah, al, bh, bl);
      }
#pragma unroll
      for (int nn = 0; nn < 2; ++nn)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int t = wr * 16 + fr + (e >> 1) * 8, col = v0 + wc * 16 + nn * 8 + fc;
          float* po = j.out + (size_t)(first + t) * j.ldo + (size_t)h * j.V + col;
          if (t < n && pairs && col < j.V) {
            *reinterpret_cast<float2*>(po) = make_float2(so[nn][e], so[nn][e + 1]);
          } else if (t < n) {
            if (col < j.V) po[0] = so[nn][e];
            if (col + 1 < j.V) po[1] = so[nn][e + 1];
          }
        }
    } else {                                          // S = e^(c_64) S + K^T U e^(c_64 - c)
      const float fend = exp2f(cend);
      const bf* Kb = K + buf * tile;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int nn = 0; nn < 2; ++nn)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[m][nn][e] *= fend;
#pragma unroll
      for (int kb = 0; kb < CK / 16; ++kb) {
        uint32_t bh[4], bl[4];
        ck_ldsm_t(bh, Us + 2 * CK * VP + (kb * 16 + lr) * VP + wc * 16 + lc);
        ck_ldsm_t(bl, Us + 3 * CK * VP + (kb * 16 + lr) * VP + wc * 16 + lc);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          const int c0 = (wr + 4 * m) * 16;
          if (c0 >= D) continue;
          // K lies by tokens: its transpose's 16 x 16 part, the halves of the tokens behind those of the channels
          uint32_t ah[4], al[4];
          const bf* kp = Kb + (kb * 16 + (lane & 7) + (lane >> 4) * 8) * DP + c0 + ((lane >> 3) & 1) * 8;
          ck_ldsm_t(ah, kp);
          ck_ldsm_t(al, kp + CK * DP);
          ck_mma3(acc[m], ah, al, bh, bl);
        }
      }
      if (i + 1 < chunks) share_state();
    }
  }
  each_state([&](float& x, int row, int col) { if (v0 + col < j.V) S[(size_t)row * j.V + v0 + col] = x; });
}

struct ChunkPlan {
  long long qs, qk, c, p, w, u0, total;     // floats
};
ChunkPlan chunk_plan(int slots, int H, int G, int D, int V, int delta) {
  ChunkPlan p = {};
  p.qs = (long long)slots * G * CK * D;                // Q, and as many for K: two bfloat16 parts are one float
  p.qk = (long long)slots * G * CK * CK;
  p.c = (long long)slots * H * CK;
  p.p = (long long)slots * H * CK * CK;
  p.w = delta ? (long long)slots * H * CK * D : 0;
  p.u0 = delta ? (long long)slots * H * CK * V : 0;
  p.total = 2 * p.qs + (delta ? 2 : 1) * p.qk + p.c + p.p + p.w + p.u0;
  return p;
}
}  // namespace

extern "C" int zi_chunked_recurrence_supported(int D, int V, int H, int G) {
  return D >= 16 && D <= 128 && D % 16 == 0 && V > 0 && H > 0 && G > 0 && H % G == 0 && H <= 65535 && (V + CK_VP - 1) / CK_VP <= 65535;
}
extern "C" long long zi_chunked_recurrence_workspace_floats(int T, int n_seqs, int H, int G, int D, int V, int delta) {
  return chunk_plan(T / CK + n_seqs + 1, H, G, D, V, delta).total;
}

// The portions of two tokens and more of a step; requests that bring one token are left alone.  logg: logarithms of the
// decays, beta: step sizes, float32 [T][H]; workspace: zi_chunked_recurrence_workspace_floats, 16-byte aligned.
extern "C" int zi_chunked_recurrence(float* out, int ldo, const float* q, int ldq, const float* k, int ldk, const float* v, int ldv,
                                     const float* logg, const float* beta, float* state, long long slot_stride, int T, int H, int G,
                                     int D, int V, int delta, const int* cu_q, const int* state_slots, int n_seqs, float* workspace,
                                     cudaStream_t stream) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (!zi_chunked_recurrence_supported(D, V, H, G)) return zi_refuse("chunked_recurrence: %d heads (%d of keys) of %d x %d", H, G, D, V);
  if (!workspace || ((uintptr_t)workspace & 15) || !logg || !beta) return zi_refuse("chunked_recurrence: needs decays, steps and an aligned workspace");
  const int slots = T / CK + n_seqs + 1;
  const ChunkPlan p = chunk_plan(slots, H, G, D, V, delta);
  Chunked j = {};
  j.q = q; j.k = k; j.v = v; j.ldq = ldq; j.ldk = ldk; j.ldv = ldv; j.logg = logg; j.beta = beta;
  j.state = state; j.slot_stride = slot_stride; j.H = H; j.G = G; j.D = D; j.V = V;
  j.cu_q = cu_q; j.state_slots = state_slots; j.n_seqs = n_seqs; j.slots = slots; j.out = out; j.ldo = ldo;
  float* at = workspace;
  j.qs = reinterpret_cast<bf*>(at); at += p.qs;
  j.ks = reinterpret_cast<bf*>(at); at += p.qs;
  j.qk = at; at += p.qk;
  if (delta) { j.kk = at; at += p.qk; }
  j.c = at; at += p.c;
  j.p = reinterpret_cast<bf*>(at); at += p.p;
  if (delta) {
    j.w = reinterpret_cast<bf*>(at); at += p.w;
    j.u0 = at;
  }
  auto launch = [&](auto kern, dim3 grid, int threads, size_t smem, const char* what) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return zi_refuse("%s: cannot get %zu bytes of shared memory", what, smem);
    zi_launch(kern, grid, dim3(threads), smem, stream, j);
    return zi_check_launch(what);
  };
  const size_t score_smem = (size_t)2 * D * CS_PITCH * sizeof(float);
  int rc = launch(delta ? chunk_scores_kernel<true> : chunk_scores_kernel<false>, dim3(slots, G), CS_THREADS, score_smem, "chunk_scores");
  if (rc) return rc;
  rc = launch(chunk_weights_kernel, dim3(slots, H), CP_THREADS, 0, "chunk_weights");
  if (rc) return rc;
  if (delta) {
    const size_t solve_smem = ((size_t)CK * CS_PITCH + 2 * CK + (size_t)CK * NT) * sizeof(float);
    rc = launch(chunk_solve_kernel, dim3(slots, H, (D + V + NT - 1) / NT), NT, solve_smem, "chunk_solve");
    if (rc) return rc;
  }
  const dim3 grid(n_seqs, H, (V + CK_VP - 1) / CK_VP);
  return delta ? launch(chunk_walk_kernel<true>, grid, CW_THREADS, ck_walk_smem(D, true), "chunk_walk")
               : launch(chunk_walk_kernel<false>, grid, CW_THREADS, ck_walk_smem(D, false), "chunk_walk");
}

ZI_TRACE_SETTER(chunked_recurrence)
