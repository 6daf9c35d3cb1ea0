// What follows a token's fused projection row when the changes span the whole row rather than one head:
//   zi_qkv_rows_prepare   [q heads | k heads | v heads | gate] -> biases, an RMS norm over ALL of q (and all of k)
//                         with a weight per element, rotation of the first rot_dims dimensions of every q and k head
//                         (pairs (i, i + rot_dims/2)), q into a tensor of its own, k and v into the token's page slot,
//                         the gate columns into a tensor of their own
//   zi_qkv_heads_prepare  [q heads | k heads | v heads] -> biases, an RMS norm per q and k head, rotation of the first
//                         rot_dims dimensions, values mixed with another layer's, q into a tensor of its own, k and v into
//                         the token's page slot; the row may come as split-K partial sums
//   zi_pool_blocks        one key and value per block of tokens: the means of the block's keys and values in the pages
//   zi_rmsnorm_rows       RMS norm of rows of activations (a latent between two projections)
// 32-bit arithmetic; the source may be 32-bit while the results have the activations' type, so that a bias or a norm
// meets the product's unrounded sums.  One block per token; every sum runs in an order that depends on the row only.
#include "api.h"
#include "common.cuh"

namespace {
// few tokens in bfloat16 (a decode step): more threads a token, since the walk is latency; the 32-bit path keeps one
// block size, so that its sums' order depends on nothing but the row
constexpr int ROW_THREADS = 256, ROW_THREADS_FEW = 1024;

template <typename TS>
__device__ __forceinline__ float row_at(const TS* x, const float* bias, int e) {
  return to_f32(x[e]) + (bias ? bias[e] : 0.f);
}

// One part (q or k) of the row: n_heads heads of d values starting at `x`, written to dst(head, i).
template <typename TS, typename T, class Dst>
__device__ __forceinline__ void finish_part(const TS* x, const float* bias, int n_heads, int d, const float* w, float eps,
                                            int rot_dims, const float* cs, const float* sn, float* scratch, Dst dst) {
  const int n = n_heads * d, half = rot_dims >> 1;
  float inv = 1.f;
  if (w) {
    float ss = 0.f;
    for (int e = threadIdx.x; e < n; e += blockDim.x) {
      const float v = row_at(x, bias, e);
      ss = fmaf(v, v, ss);
    }
    inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  }
  for (int e = threadIdx.x; e < n; e += blockDim.x) {
    const int hd = e / d, i = e - hd * d;
    float v = row_at(x, bias, e);
    if (w) v = norm_scale(v, w[e], inv);
    if (i < rot_dims) {
      const int p = i < half ? e + half : e - half;       // the other element of the pair
      float o = row_at(x, bias, p);
      if (w) o = norm_scale(o, w[p], inv);
      if (i < half) {
        rotate_pair(v, o, cs[i], sn[i]);
      } else {
        rotate_pair(o, v, cs[i - half], sn[i - half]);
      }
    }
    dst(hd, i, from_f32<T>(v));
  }
}

template <typename TS, typename T>
__global__ void __launch_bounds__(ROW_THREADS_FEW)
qkv_rows_kernel(const TS* __restrict__ src, int src_stride, const float* __restrict__ bias, T* __restrict__ q_out,
                int q_stride, T* __restrict__ gate_out, int gate_stride, int n_gate, int nq, int nkv, int d, int dv,
                const float* __restrict__ qw, const float* __restrict__ kw, float eps, int rot_dims,
                const float* __restrict__ cos_t, const float* __restrict__ sin_t, int n_table_pos,
                const int* __restrict__ positions, T* __restrict__ kcache, T* __restrict__ vcache,
                const int* __restrict__ slots, int page_size) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[33];
  const int t = blockIdx.x;
  const TS* row = src + (size_t)t * src_stride;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= n_table_pos && n_table_pos > 0 ? n_table_pos - 1 : pos);   // the host refuses such positions
  const int half = rot_dims >> 1;
  const float* cs = cos_t ? cos_t + (size_t)pos * half : nullptr;
  const float* sn = sin_t ? sin_t + (size_t)pos * half : nullptr;
  const int rd = cos_t ? rot_dims : 0;
  const int qn = nq * d, kn = nkv * d, vn = nkv * dv;
  T* qo = q_out + (size_t)t * q_stride;
  finish_part<TS, T>(row, bias, nq, d, qw, eps, rd, cs, sn, scratch,
                     [&](int hd, int i, T v) { qo[hd * d + i] = v; });
  for (int e = threadIdx.x; e < n_gate; e += blockDim.x)
    gate_out[(size_t)t * gate_stride + e] = from_f32<T>(row_at(row + qn + kn + vn, bias ? bias + qn + kn + vn : nullptr, e));
  const int slot = slots[t];
  if (slot < 0) return;        // a row that pads a captured batch
  const size_t page = (size_t)(slot / page_size), off = (size_t)(slot % page_size);
  finish_part<TS, T>(row + qn, bias ? bias + qn : nullptr, nkv, d, kw, eps, rd, cs, sn, scratch,
                     [&](int hd, int i, T v) { kcache[((page * nkv + hd) * page_size + off) * d + i] = v; });
  for (int e = threadIdx.x; e < vn; e += blockDim.x) {
    const int hd = e / dv, i = e - hd * dv;
    vcache[((page * nkv + hd) * page_size + off) * dv + i] = from_f32<T>(row_at(row + qn + kn, bias ? bias + qn + kn : nullptr, e));
  }
}

// One warp per (token, head).  The head's values (partial sums added in order, bias added) wait in the warp's shared
// memory between the sum of squares and the rotation, so the row is read once.  W = 4: 16-byte reads, W = 1: any sizes.
// With v_in, a value becomes v_keep * v + v_lambda * v_in[t] (v_in float32 [T, nkv * dv]: the same token's values of an
// earlier layer); with v_out the values go there as well, unrounded.  Tokens without a slot write no keys and values
// to pages.
constexpr int HEAD_WARPS = 4;

template <typename TS, typename T, int W>
__global__ void __launch_bounds__(HEAD_WARPS * 32)
qkv_heads_kernel(const TS* __restrict__ src, int src_stride, const float* __restrict__ part, int splits, size_t zstride,
                 const float* __restrict__ bias, T* __restrict__ q_out, int q_stride, int T_, int nq, int nkv, int d, int dv,
                 const float* __restrict__ qw, const float* __restrict__ kw, float eps, int rot_dims,
                 const float* __restrict__ cos_t, const float* __restrict__ sin_t, int n_table_pos,
                 const int* __restrict__ positions, T* __restrict__ kcache, T* __restrict__ vcache,
                 const int* __restrict__ slots, int page_size, const float* __restrict__ v_in, float v_keep, float v_lambda,
                 float* __restrict__ v_out) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float head_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_heads = nq + 2 * nkv;
  const long long wi = (long long)blockIdx.x * HEAD_WARPS + warp;
  if (wi >= (long long)T_ * n_heads) return;
  const int t = (int)(wi / n_heads), head = (int)(wi % n_heads);
  const bool is_v = head >= nq + nkv, is_q = head < nq;
  const int kvh = is_q ? 0 : (head - nq) % nkv;
  const int n = is_v ? dv : d;
  const int at = is_v ? (nq + nkv) * d + kvh * dv : head * d;
  float* x = head_smem + warp * (((d > dv ? d : dv) + 3) & ~3);
  float ss = 0.f;
  for (int i = lane * W; i < n; i += 32 * W) {
    float v[W];
    if (part) {
      const float* p = part + (size_t)t * src_stride + at + i;
#pragma unroll
      for (int u = 0; u < W; ++u) v[u] = 0.f;
      for (int z = 0; z < splits; ++z) {
        if constexpr (W == 4) {
          const float4 f = *reinterpret_cast<const float4*>(p + (size_t)z * zstride);
          v[0] += f.x; v[1] += f.y; v[2] += f.z; v[3] += f.w;
        } else {
          v[0] += p[(size_t)z * zstride];
        }
      }
    } else {
      const TS* p = src + (size_t)t * src_stride + at + i;
      if constexpr (W == 4 && sizeof(TS) == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
      } else {
#pragma unroll
        for (int u = 0; u < W; ++u) v[u] = to_f32(p[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < W; ++u) {
      if (bias) v[u] += bias[at + i + u];
      x[i + u] = v[u];
      ss = fmaf(v[u], v[u], ss);
    }
  }
  const int slot = is_q ? 0 : slots[t];
  const size_t page_at = slot < 0 ? 0 : ((size_t)(slot / page_size) * nkv + kvh) * page_size + (slot % page_size);
  if (is_v) {
    __syncwarp();
    const size_t vr = ((size_t)t * nkv + kvh) * dv;
    for (int i = lane * W; i < n; i += 32 * W) {
#pragma unroll
      for (int u = 0; u < W; ++u) {
        float v = x[i + u];
        if (v_in) v = fmaf(v_lambda, v_in[vr + i + u], v_keep * v);
        if (v_out) v_out[vr + i + u] = v;
        if (slot >= 0) vcache[page_at * dv + i + u] = from_f32<T>(v);
      }
    }
    return;
  }
  const float* w = is_q ? qw : kw;
  float inv = 1.f;
  if (w) inv = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);
  __syncwarp();
  if (!is_q && slot < 0) return;      // a row that pads a captured batch
  T* dst = is_q ? q_out + (size_t)t * q_stride + (size_t)head * d : kcache + page_at * d;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= n_table_pos && n_table_pos > 0 ? n_table_pos - 1 : pos);   // the host refuses such positions
  const int half = rot_dims >> 1;
  const float* cs = cos_t ? cos_t + (size_t)pos * half : nullptr;
  const float* sn = sin_t ? sin_t + (size_t)pos * half : nullptr;
  for (int i = lane * W; i < d; i += 32 * W) {
    T out[W];
#pragma unroll
    for (int u = 0; u < W; ++u) {
      const int e = i + u;
      float a = x[e];
      if (w) a = norm_scale(a, w[e], inv);
      if (cs && e < rot_dims) {
        const int p = e < half ? e + half : e - half;       // the other element of the pair
        float b = x[p];
        if (w) b = norm_scale(b, w[p], inv);
        if (e < half) rotate_pair(a, b, cs[e], sn[e]);
        else rotate_pair(b, a, cs[p], sn[p]);
      }
      out[u] = from_f32<T>(a);
    }
    if constexpr (W == 4 && sizeof(T) == 2) {
      *reinterpret_cast<uint2*>(dst + i) = *reinterpret_cast<const uint2*>(out);
    } else {
#pragma unroll
      for (int u = 0; u < W; ++u) dst[i + u] = out[u];
    }
  }
}

// The pooled entry of every block of `per` tokens that this step's tokens complete.  entry_slots[t] >= 0 for the token
// that completes its request's next block: the block's last position is positions[t], its keys and values lie in the
// tokens' own pages (block_tables), and their means go to entry entry_slots[t] of the pooled pages, in 32-bit sums in
// the order of the positions.  A block of threads looks through POOL_TOKENS neighbouring tokens (most complete nothing) and
// does the entries they complete for one kv head.
// C: elements per access (16 bytes, or one).
constexpr int POOL_TOKENS = 32, POOL_THREADS = 128, POOL_COLS = 16, POOL_TILE_BYTES = 32 * 1024;

template <typename T, int C>
__global__ void __launch_bounds__(POOL_THREADS)
pool_blocks_kernel(const T* __restrict__ kcache, const T* __restrict__ vcache, const int* __restrict__ block_tables, int bt_stride,
                   T* __restrict__ kpool, T* __restrict__ vpool, const int* __restrict__ entry_slots,
                   const int* __restrict__ positions, const int* __restrict__ cu_q, int n_seqs, int T_, int nkv, int d, int dv,
                   int per, int page_size, int tile) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float rows[];      // [tile][W]
  const int W = d + dv;
  const int t0 = blockIdx.x * POOL_TOKENS, kvh = blockIdx.y, lane = threadIdx.x & 31;
  // the step's own arrays: here before any kernel of the step
  const int mine = t0 + lane < T_ ? entry_slots[t0 + lane] : -1;
  unsigned todo = __ballot_sync(0xffffffffu, mine >= 0);
  pdl_wait();
  const float inv = 1.0f / (float)per;
  for (; todo; todo &= todo - 1) {
    const int k = __ffs(todo) - 1, t = t0 + k;
    const int entry = __shfl_sync(0xffffffffu, mine, k);
    int lo = 0, hi = n_seqs - 1;                      // the request that token t belongs to
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
    }
    const int* bt = block_tables + (size_t)lo * bt_stride;
    const int p0 = positions[t] - per + 1;
    const size_t out_at = ((size_t)(entry / page_size) * nkv + kvh) * page_size + (entry % page_size);
    // TILE rows [key | value] at a time into shared memory, all their loads in flight together; then a thread per column
    // adds them in the order of the positions
    float sum[POOL_COLS];
#pragma unroll
    for (int u = 0; u < POOL_COLS; ++u) sum[u] = 0.f;
    for (int j0 = 0; j0 < per; j0 += tile) {
      const int nj = min(tile, per - j0);
      __syncthreads();                                // the tile before is added up
      for (int e = threadIdx.x; e < nj * (W / C); e += POOL_THREADS) {
        const int r = e / (W / C), c = (e - r * (W / C)) * C, p = p0 + j0 + r;
        const int page = p < 0 ? -1 : bt[p / page_size];
        const size_t at = page < 0 ? 0 : ((size_t)page * nkv + kvh) * page_size + (p % page_size);
        const T* src = c < d ? kcache + at * d + c : vcache + at * dv + c - d;
        __align__(16) T v[C];
        if constexpr (C > 1) *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(src);
        else v[0] = *src;
#pragma unroll
        for (int u = 0; u < C; ++u) rows[r * W + c + u] = page < 0 ? 0.f : to_f32(v[u]);
      }
      __syncthreads();
#pragma unroll
      for (int u = 0; u < POOL_COLS; ++u) {
        const int c = threadIdx.x + u * POOL_THREADS;
        if (c < W)
          for (int r = 0; r < nj; ++r) sum[u] += rows[r * W + c];
      }
    }
#pragma unroll
    for (int u = 0; u < POOL_COLS; ++u) {
      const int c = threadIdx.x + u * POOL_THREADS;
      if (c < d) kpool[out_at * d + c] = from_f32<T>(sum[u] * inv);
      else if (c < W) vpool[out_at * dv + c - d] = from_f32<T>(sum[u] * inv);
    }
  }
}

template <typename TS, typename T>
__global__ void __launch_bounds__(ROW_THREADS)
rmsnorm_rows_kernel(T* __restrict__ out, int ldo, const TS* __restrict__ x, int ldx, const float* __restrict__ w, float eps,
                    int n) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[33];
  const TS* xr = x + (size_t)blockIdx.x * ldx;
  float ss = 0.f;
  for (int e = threadIdx.x; e < n; e += blockDim.x) {
    const float v = to_f32(xr[e]);
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  for (int e = threadIdx.x; e < n; e += blockDim.x)
    out[(size_t)blockIdx.x * ldo + e] = from_f32<T>(norm_scale(to_f32(xr[e]), w[e], inv));
}
}  // namespace

#define ZI_DISPATCH_SRC_OUT(sd, od, TS, TT, ...)                                                   \
  do {                                                                                             \
    if ((sd) == ZI_F32 && (od) == ZI_F32) { using TS = float; using TT = float; __VA_ARGS__; }      \
    else if ((sd) == ZI_F32 && (od) == ZI_BF16) { using TS = float; using TT = __nv_bfloat16; __VA_ARGS__; } \
    else if ((sd) == ZI_BF16 && (od) == ZI_BF16) { using TS = __nv_bfloat16; using TT = __nv_bfloat16; __VA_ARGS__; } \
    else return zi_refuse("a source of type %d cannot become results of type %d", (int)(sd), (int)(od)); \
  } while (0)

extern "C" int zi_qkv_rows_prepare(const void* src, int src_dtype, int src_stride, const float* bias, void* q_out,
                                   int q_stride, void* gate_out, int gate_stride, int n_gate, int out_dtype, int T, int nq,
                                   int nkv, int d, int dv, const float* qw, const float* kw, float eps, int rot_dims,
                                   const float* cos_t, const float* sin_t, int n_table_pos, const int* positions,
                                   void* kcache, void* vcache, const int* slots, int page_size, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0) return zi_refuse("qkv_rows_prepare: %d and %d heads of %d and %d", nq, nkv, d, dv);
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > d) return zi_refuse("qkv_rows_prepare: %d rotated dimensions of a head of %d", rot_dims, d);
  if ((cos_t == nullptr) != (sin_t == nullptr)) return zi_refuse("qkv_rows_prepare: cos and sin tables go together");
  if ((qw == nullptr) != (kw == nullptr)) return zi_refuse("qkv_rows_prepare: q and k are normed together or not at all");
  if (!kcache || !vcache || !slots || page_size <= 0) return zi_refuse("qkv_rows_prepare: keys and values need pages and slots");
  if (n_gate < 0 || (n_gate > 0 && !gate_out)) return zi_refuse("qkv_rows_prepare: %d gate columns without a place", n_gate);
  ZI_DISPATCH_SRC_OUT(src_dtype, out_dtype, TS, TT,
                      zi_launch(qkv_rows_kernel<TS, TT>, dim3(T), dim3(T <= 64 && out_dtype == ZI_BF16 ? ROW_THREADS_FEW : ROW_THREADS), 0, stream,
                                (const TS*)src, src_stride, bias,
                                (TT*)q_out, q_stride, (TT*)gate_out, gate_stride, n_gate, nq, nkv, d, dv, qw, kw, eps, rot_dims,
                                cos_t, sin_t, n_table_pos, positions, (TT*)kcache, (TT*)vcache, slots, page_size));
  return zi_check_launch("qkv_rows_prepare");
}

extern "C" int zi_qkv_heads_prepare(const void* src, int src_dtype, int src_stride, const float* part, int splits,
                                    long long zstride, const float* bias, void* q_out, int q_stride, int out_dtype, int T, int nq,
                                    int nkv, int d, int dv, const float* qw, const float* kw, float eps, int rot_dims,
                                    const float* cos_t, const float* sin_t, int n_table_pos, const int* positions, void* kcache,
                                    void* vcache, const int* slots, int page_size, const float* v_in, float v_lambda,
                                    float* v_out, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0) return zi_refuse("qkv_heads_prepare: %d and %d heads of %d and %d", nq, nkv, d, dv);
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > d) return zi_refuse("qkv_heads_prepare: %d rotated dimensions of a head of %d", rot_dims, d);
  if ((cos_t == nullptr) != (sin_t == nullptr)) return zi_refuse("qkv_heads_prepare: cos and sin tables go together");
  if ((src == nullptr) == (part == nullptr)) return zi_refuse("qkv_heads_prepare: give the rows either whole or as partial sums");
  if (!kcache || !vcache || !slots || page_size <= 0) return zi_refuse("qkv_heads_prepare: keys and values need pages and slots");
  auto al16 = [](const void* p) { return p == nullptr || ((uintptr_t)p & 15) == 0; };
  const bool vec = d % 4 == 0 && dv % 4 == 0 && src_stride % 4 == 0 && zstride % 4 == 0 && q_stride % 4 == 0 && al16(src) && al16(part) &&
                   al16(q_out) && al16(kcache) && al16(vcache);
  const size_t smem = (size_t)HEAD_WARPS * (((d > dv ? d : dv) + 3) & ~3) * sizeof(float);
  if (smem > 48 * 1024) return zi_refuse("qkv_heads_prepare: heads of %d and %d are more than this kernel holds", d, dv);
  const long long n = (long long)T * (nq + 2 * nkv);
  const unsigned blocks = (unsigned)((n + HEAD_WARPS - 1) / HEAD_WARPS);
#define ZI_QH(TS, TT, W)                                                                                                  \
  zi_launch(qkv_heads_kernel<TS, TT, W>, dim3(blocks), dim3(HEAD_WARPS * 32), smem, stream, (const TS*)src, src_stride, part, splits, \
            (size_t)zstride, bias, (TT*)q_out, q_stride, T, nq, nkv, d, dv, qw, kw, eps, cos_t ? rot_dims : 0, cos_t, sin_t,  \
            n_table_pos, positions, (TT*)kcache, (TT*)vcache, slots, page_size, v_in, 1.0f - v_lambda, v_lambda, v_out)
  ZI_DISPATCH_SRC_OUT(part ? ZI_F32 : src_dtype, out_dtype, TS, TT, { if (vec) ZI_QH(TS, TT, 4); else ZI_QH(TS, TT, 1); });
#undef ZI_QH
  return zi_check_launch("qkv_heads_prepare");
}

extern "C" int zi_pool_blocks(const void* kcache, const void* vcache, int dtype, const int* block_tables, int bt_stride, void* kpool,
                              void* vpool, const int* entry_slots, const int* positions, const int* cu_q, int n_seqs, int T,
                              int nkv, int d, int dv, int per, int page_size, cudaStream_t stream) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (nkv <= 0 || d <= 0 || dv <= 0 || per <= 0 || page_size <= 0) return zi_refuse("pool_blocks: blocks of %d tokens, heads of %d and %d", per, d, dv);
  if (nkv > 65535) return zi_refuse("pool_blocks: %d kv heads", nkv);
  if (d + dv > POOL_COLS * POOL_THREADS) return zi_refuse("pool_blocks: heads of %d and %d are more than this kernel holds", d, dv);
  const int per16 = dtype == ZI_BF16 ? 8 : 4;
  auto al16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = d % per16 == 0 && dv % per16 == 0 && al16(kcache) && al16(vcache);
  int tile = POOL_TILE_BYTES / (int)((d + dv) * sizeof(float));
  tile = tile < 1 ? 1 : (tile > per ? per : tile);
  const size_t smem = (size_t)tile * (d + dv) * sizeof(float);
  dim3 grid((T + POOL_TOKENS - 1) / POOL_TOKENS, nkv);
  ZI_DISPATCH_DTYPE(dtype, TT, {
    constexpr int C = 16 / (int)sizeof(TT);
    auto kern = vec ? pool_blocks_kernel<TT, C> : pool_blocks_kernel<TT, 1>;
    zi_launch(kern, grid, dim3(POOL_THREADS), smem, stream, (const TT*)kcache, (const TT*)vcache, block_tables, bt_stride, (TT*)kpool,
              (TT*)vpool, entry_slots, positions, cu_q, n_seqs, T, nkv, d, dv, per, page_size, tile);
  });
  return zi_check_launch("pool_blocks");
}

extern "C" int zi_rmsnorm_rows(void* out, int ldo, int out_dtype, const void* x, int ldx, int x_dtype, const float* w,
                               float eps, int T, int n, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  ZI_DISPATCH_SRC_OUT(x_dtype, out_dtype, TS, TT,
                      zi_launch(rmsnorm_rows_kernel<TS, TT>, dim3(T), dim3(ROW_THREADS), 0, stream, (TT*)out, ldo, (const TS*)x,
                                ldx, w, eps, n));
  return zi_check_launch("rmsnorm_rows");
}

ZI_TRACE_SETTER(projection_rows)
