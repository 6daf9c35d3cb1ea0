// From a projection's rows to what a mixer with short convolutions works on, in one kernel: the projection's bias, the
// causal convolution per channel, its bias and activation, what finishes a head (nothing, a unit vector, a rotation), the
// place the head goes to (a row of a tensor of its own, or the token's page slot), and the convolution's carried inputs.
//
//   u_t = projected row (whole, or split-K partial sums added in order) + in_bias
//   y_t = act(sum_i kern[i] * u_(t - taps + 1 + i) + out_bias)           per channel; kern is [taps][C]
//
// The inputs before a request's first token of this step come from tail[slot][taps-1][C] (oldest first; zero at a
// request's start); the blocks that walk a request's first tokens of the step are the only ones that touch its tail, and
// leave the last taps-1 inputs of the step there after they have read the old ones.
//
// The channels are cut into segments of equal heads.  A warp takes one head of one tile of up to CH_TILE tokens: a lane
// keeps the running inputs of its channels in registers while it walks the tile, so every input is read once (plus taps-1
// before the tile).  A lane's channels come in the pairs that a rotation turns: neighbours (2i, 2i+1), or (i, i + rot/2).
// 32-bit arithmetic throughout.
#include "api.h"
#include "common.cuh"

namespace {
constexpr int CH_WARPS = 4, CH_TILE = 16, CH_SEGMENTS = 3;

struct ConvSegment {
  int c0;            // first channel
  int n;             // channels
  int d;             // channels per head (the last head of a segment without a finish may be shorter)
  int first_head;    // heads before this segment
  int finish;        // 0 none, 1 unit vector times `scale`, 2 rotation
  int dest;          // 0 float32 rows, 1 rows in the activations' type, 2 pages
  int ldo;           // row pitch of dest 0 and 1
  float scale;
  void* out;         // row 0's first channel of this segment, or the pages
};
struct ConvJob {
  ConvSegment seg[CH_SEGMENTS];
  int n_seg, heads;
  const float* src;  // row 0, channel 0
  int ld, splits;
  long long zstride;
  const float* in_bias;
  const float* kern;
  const float* out_bias;
  int act;           // 1: silu
  float* tail;
  long long slot_stride;
  int C, taps;
  float unit_eps;
  const float* cos_t;
  const float* sin_t;
  int n_table_pos, rot_dims, neighbours;
  const int* positions;
  const int* slots;
  int page_size;
  const int* tile_seq;
  const int* tile_q0;
  const int* cu_q;
  const int* state_slots;
  int smem_head;     // floats per token of a warp's shared memory (unit vectors only)
  // what every token has once per head beside the channels: a step and a decay's logarithm (scalars 0: nothing to do)
  int scalars;       // 1: step = sigmoid(b), log decay = -exp(a_log) softplus(a + dt_bias); 2: step = softplus(a + dt_bias), log decay = -exp(a_log) step
  int n_scalar;      // heads
  const float* a;    // row 0, head 0 (rows as above: same pitch and splits)
  const float* b;
  const float* a_log;
  const float* dt_bias;
  float* decay;      // [T][n_scalar] logarithms
  float* step;
};

__device__ __forceinline__ float conv_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float conv_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float summed_at(const float* p, int splits, long long zstride) {
  float v = *p;
  for (int z = 1; z < splits; ++z) v += p[(size_t)z * zstride];
  return v;
}

// TAPS > 0: that many taps, inputs and weights in registers; 0: any number, inputs read again for every tap.
// NP pairs of neighbouring channels per lane (2 or 1), whose addresses allow accesses of 16 (8) bytes; 0: one pair, any
// addresses, either pairing.
template <typename T, int TAPS, int NP>
__global__ void __launch_bounds__(CH_WARPS * 32, 4)
conv_heads_kernel(const ConvJob j) {
  pdl_launch_dependents();
  extern __shared__ float held_all[];
  constexpr int NR = NP > 0 ? NP : 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = j.tile_seq[blockIdx.x], q0 = j.tile_q0[blockIdx.x];      // the step's own arrays: here before any kernel of the step
  const int tok0 = j.cu_q[seq], qlen = j.cu_q[seq + 1] - tok0;
  const int nt = min(CH_TILE, qlen - q0);
  pdl_wait();
  if (nt <= 0) return;
  const int row0 = tok0 + q0;
  if ((int)blockIdx.y * CH_WARPS >= j.heads) {          // the last row of blocks: the scalars of every head
    for (int e = threadIdx.x; e < nt * j.n_scalar; e += blockDim.x) {
      const int t = e / j.n_scalar, h = e - t * j.n_scalar;
      const size_t row = (size_t)(row0 + t);
      const float sp = conv_softplus(summed_at(j.a + row * j.ld + h, j.splits, j.zstride) + j.dt_bias[h]);
      j.decay[row * j.n_scalar + h] = -expf(j.a_log[h]) * sp;
      j.step[row * j.n_scalar + h] = j.scalars == 2 ? sp : 1.0f / (1.0f + expf(-summed_at(j.b + row * j.ld + h, j.splits, j.zstride)));
    }
    return;
  }
  // where the tile's tokens go, worked out once per block
  __shared__ int tok_pos[CH_TILE], tok_page[CH_TILE], tok_off[CH_TILE];
  if (threadIdx.x < nt && (j.cos_t || j.slots)) {
    const int t = threadIdx.x, slot = j.slots ? j.slots[row0 + t] : -1, pos = j.positions[row0 + t];
    tok_pos[t] = pos < 0 ? 0 : (pos >= j.n_table_pos ? j.n_table_pos - 1 : pos);      // the host refuses such positions
    tok_page[t] = slot < 0 ? -1 : slot / j.page_size;
    tok_off[t] = slot < 0 ? 0 : slot % j.page_size;
  }
  __syncthreads();
  const int head_all = blockIdx.y * CH_WARPS + warp;
  if (head_all >= j.heads) return;
  int si = 0;
  while (si + 1 < j.n_seg && head_all >= j.seg[si + 1].first_head) ++si;
  const ConvSegment g = j.seg[si];
  const int page_heads = g.dest == 2 ? g.n / g.d : 0;
  const int head = head_all - g.first_head;
  const int d = min(g.d, g.n - head * g.d);             // channels of this head
  const int ch0 = g.c0 + head * g.d;                    // its first channel
  const int taps = TAPS > 0 ? TAPS : j.taps;
  const int rot = g.finish == 2 ? j.rot_dims : 0, half = rot >> 1;
  float* tail = j.tail + (size_t)j.state_slots[seq] * j.slot_stride + ch0;
  const float* src = j.src + (size_t)tok0 * j.ld + ch0;
  float* held = held_all + (size_t)warp * CH_TILE * j.smem_head;

  // NR pairs of channels at a time: channel e0 and e1 of pair r, a place `p` (floats) at which channel e0 of the first lies
  auto read = [&](const float* p, int e0, int e1, float2 (&v)[NR]) {
    if constexpr (NP == 2) {
      const float4 x = *reinterpret_cast<const float4*>(p + e0);
      v[0] = make_float2(x.x, x.y);
      v[1] = make_float2(x.z, x.w);
    } else if constexpr (NP == 1) {
      v[0] = *reinterpret_cast<const float2*>(p + e0);
    } else {
      v[0] = make_float2(p[e0], p[e1]);
    }
  };
  const int units = (d + 2 * NR - 1) / (2 * NR);        // of 2 NR channels
  for (int p = lane; p < units; p += 32) {
    int e0 = 2 * NR * p, e1 = e0 + 1;
    if (NP == 0 && !j.neighbours && p < half) {         // (i, i + rot/2); the channels that do not turn follow in twos
      e0 = p;
      e1 = p + half;
    }
    const bool two = NP > 0 || e1 < d;
    const int f1 = two ? e1 : e0;                       // a channel that exists
    float2 ib[NR], ob[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) ib[r] = ob[r] = make_float2(0.f, 0.f);
    if (j.in_bias) read(j.in_bias + ch0, e0, f1, ib);
    if (j.out_bias) read(j.out_bias + ch0, e0, f1, ob);
    // the inputs of row `at` of this request's portion (negative: carried from before the step)
    auto fetch = [&](int at, float2 (&v)[NR]) {
      if (at < 0) {
        read(tail + (size_t)(taps - 1 + at) * j.C, e0, f1, v);
        return;
      }
      const float* x = src + (size_t)at * j.ld;
      read(x, e0, f1, v);
      for (int z = 1; z < j.splits; ++z) {
        float2 y[NR];
        read(x + (size_t)z * j.zstride, e0, f1, y);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          v[r].x += y[r].x;
          v[r].y += y[r].y;
        }
      }
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        v[r].x += ib[r].x;
        v[r].y += ib[r].y;
      }
    };
    constexpr int W = TAPS > 0 ? TAPS : 1;
    float2 win[W][NR], k[W][NR];
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < TAPS; ++i) {
        read(j.kern + (size_t)i * j.C + ch0, e0, f1, k[i]);
        if (i > 0) fetch(q0 - TAPS + i, win[i]);        // inputs before the tile; every token shifts them down by one
      }
    }
    constexpr int AHEAD = 4;                            // tokens whose inputs are asked for together
#pragma unroll 1
    for (int t0 = 0; t0 < nt; t0 += AHEAD) {
      float2 in[AHEAD][NR];
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) fetch(q0 + min(t0 + u, nt - 1), in[u]);
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const int t = t0 + u;
        if (t >= nt) break;
        float2 y[NR];
#pragma unroll
        for (int r = 0; r < NR; ++r) y[r] = make_float2(0.f, 0.f);
        if constexpr (TAPS > 0) {
#pragma unroll
          for (int r = 0; r < NR; ++r) {
#pragma unroll
            for (int i = 0; i + 1 < TAPS; ++i) win[i][r] = win[i + 1][r];
            win[TAPS - 1][r] = in[u][r];
#pragma unroll
            for (int i = 0; i < TAPS; ++i) {
              y[r].x = fmaf(k[i][r].x, win[i][r].x, y[r].x);
              y[r].y = fmaf(k[i][r].y, win[i][r].y, y[r].y);
            }
          }
        } else {
          for (int i = 0; i < taps; ++i) {
            float2 x[NR], kk[NR];
            fetch(q0 + t - (taps - 1) + i, x);
            read(j.kern + (size_t)i * j.C + ch0, e0, f1, kk);
#pragma unroll
            for (int r = 0; r < NR; ++r) {
              y[r].x = fmaf(kk[r].x, x[r].x, y[r].x);
              y[r].y = fmaf(kk[r].y, x[r].y, y[r].y);
            }
          }
        }
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          y[r].x += ob[r].x;
          y[r].y += ob[r].y;
          if (j.act == 1) {
            y[r].x = conv_silu(y[r].x);
            y[r].y = conv_silu(y[r].y);
          }
          if (NR * p + r < half) {
            const size_t at = (size_t)tok_pos[t] * half + NR * p + r;
            rotate_pair(y[r].x, y[r].y, j.cos_t[at], j.sin_t[at]);
          }
        }
        if (g.finish == 1) {
#pragma unroll
          for (int r = 0; r < NR; ++r) {
            held[t * j.smem_head + e0 + 2 * r] = y[r].x;
            if (two) held[t * j.smem_head + e1 + 2 * r] = y[r].y;
          }
          continue;
        }
        // where it goes
        const size_t row = (size_t)(row0 + t);
        if (g.dest == 0) {
          float* o = static_cast<float*>(g.out) + row * g.ldo + (size_t)head * g.d;
          if constexpr (NP == 2) {
            *reinterpret_cast<float4*>(o + e0) = make_float4(y[0].x, y[0].y, y[1].x, y[1].y);
          } else if constexpr (NP == 1) {
            *reinterpret_cast<float2*>(o + e0) = y[0];
          } else {
            o[e0] = y[0].x;
            if (two) o[e1] = y[0].y;
          }
          continue;
        }
        T* o;
        if (g.dest == 1) {
          o = static_cast<T*>(g.out) + row * g.ldo + (size_t)head * g.d;
        } else {
          if (tok_page[t] < 0) continue;                // a row that pads a captured batch
          o = static_cast<T*>(g.out) + (((size_t)tok_page[t] * page_heads + head) * j.page_size + tok_off[t]) * g.d;
        }
        if constexpr (NP > 0 && sizeof(T) == 2) {
          __nv_bfloat162 b[NR];
#pragma unroll
          for (int r = 0; r < NR; ++r) b[r] = __floats2bfloat162_rn(y[r].x, y[r].y);
          if constexpr (NP == 2) *reinterpret_cast<uint2*>(o + e0) = make_uint2(*reinterpret_cast<uint32_t*>(&b[0]), *reinterpret_cast<uint32_t*>(&b[1]));
          else *reinterpret_cast<__nv_bfloat162*>(o + e0) = b[0];
        } else {
#pragma unroll
          for (int r = 0; r < NR; ++r) {
            o[e0 + 2 * r] = from_f32<T>(y[r].x);
            if (two) o[e1 + 2 * r] = from_f32<T>(y[r].y);
          }
        }
      }
    }
    if (q0 == 0) {                                      // the inputs that the next step finds; ascending rows overwrite in place
      for (int i = 0; i < taps - 1; ++i) {
        float2 u[NR];
        fetch(qlen - (taps - 1) + i, u);                // from before this step: row i + qlen of the old tail
        float* o = tail + (size_t)i * j.C;
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          o[e0 + 2 * r] = u[r].x;
          if (two) o[e1 + 2 * r] = u[r].y;
        }
      }
    }
  }
  if (g.finish == 1) {
    __syncwarp();
    for (int t = 0; t < nt; ++t) {
      const float* x = held + t * j.smem_head;
      float ss = 0.f;
      for (int e = lane; e < d; e += 32) ss = fmaf(x[e], x[e], ss);
      const float inv = g.scale / sqrtf(warp_sum(ss) + j.unit_eps);
      const size_t at = (size_t)(row0 + t) * g.ldo + (size_t)head * g.d;
      for (int e = lane; e < d; e += 32) {
        if (g.dest == 0) static_cast<float*>(g.out)[at + e] = x[e] * inv;
        else static_cast<T*>(g.out)[at + e] = from_f32<T>(x[e] * inv);
      }
    }
  }
}
}  // namespace

extern "C" int zi_conv_heads_tile() { return CH_TILE; }

// segs: n_seg rows of 5 ints (channels, channels per head, finish, dest, row pitch), seg_out their places.
extern "C" int zi_conv_heads(const float* src, int ld, int splits, long long zstride, int T, int C, int taps, const float* kern,
                             const float* in_bias, const float* out_bias, int act, float* tail, long long slot_stride, int n_seg,
                             const int* segs, void* const* seg_out, const float* seg_scale, int out_dtype, float unit_eps,
                             const float* cos_t, const float* sin_t, int n_table_pos, int rot_dims, int neighbours,
                             const int* positions, const int* slots, int page_size, int scalars, int n_scalar, const float* a,
                             const float* b, const float* a_log, const float* dt_bias, float* decay, float* step,
                             const int* tile_seq, const int* tile_q0, int n_tiles, int tile_rows, const int* cu_q,
                             const int* state_slots, cudaStream_t stream) {
  if (T <= 0 || n_tiles <= 0) return 0;
  // a tile behind a request's first must not reach the carried inputs, which the first tile's blocks move on
  if (taps < 1 || taps > CH_TILE + 1) return zi_refuse("conv_heads: %d taps (1 to %d)", taps, CH_TILE + 1);
  if (n_seg < 1 || n_seg > CH_SEGMENTS) return zi_refuse("conv_heads: %d segments", n_seg);
  if (tile_rows != CH_TILE) return zi_refuse("conv_heads: tiles of %d tokens (takes %d)", tile_rows, CH_TILE);
  if (splits < 1 || !src || !kern || (taps > 1 && !tail)) return zi_refuse("conv_heads: needs rows, weights and carried inputs");
  if (rot_dims < 0 || rot_dims % 2 || (cos_t == nullptr) != (sin_t == nullptr)) return zi_refuse("conv_heads: %d rotated dimensions", rot_dims);
  if (scalars < 0 || scalars > 2 || (scalars && (n_scalar <= 0 || !a || !a_log || !dt_bias || !decay || !step || (scalars == 1 && !b))))
    return zi_refuse("conv_heads: steps and decays need their operands");
  ConvJob j = {};
  j.n_seg = n_seg;
  int c = 0, heads = 0, widest = 0;
  auto al = [](const void* p, size_t n) { return p == nullptr || ((uintptr_t)p & (n - 1)) == 0; };
  auto fits = [&](int n) {       // accesses of n floats
    return ld % n == 0 && zstride % n == 0 && C % n == 0 && slot_stride % n == 0 && al(src, 4 * n) && al(tail, 4 * n) && al(kern, 4 * n) &&
           al(in_bias, 4 * n) && al(out_bias, 4 * n);
  };
  int np = fits(4) ? 2 : (fits(2) ? 1 : 0);      // pairs of channels per lane
  for (int i = 0; i < n_seg; ++i) {
    ConvSegment& g = j.seg[i];
    g.c0 = c;
    g.n = segs[5 * i];
    g.d = segs[5 * i + 1];
    g.finish = segs[5 * i + 2];
    g.dest = segs[5 * i + 3];
    g.ldo = segs[5 * i + 4];
    g.scale = seg_scale[i];
    g.out = seg_out[i];
    g.first_head = heads;
    if (g.n <= 0 || g.d <= 0 || !g.out || g.finish < 0 || g.finish > 2 || g.dest < 0 || g.dest > 2)
      return zi_refuse("conv_heads: segment %d of %d channels in heads of %d", i, g.n, g.d);
    if ((g.finish || g.dest == 2) && g.n % g.d) return zi_refuse("conv_heads: %d channels do not form heads of %d", g.n, g.d);
    if (g.finish == 2 && (!cos_t || rot_dims > g.d)) return zi_refuse("conv_heads: %d rotated dimensions of a head of %d", rot_dims, g.d);
    if (g.dest == 2 && (!slots || page_size <= 0)) return zi_refuse("conv_heads: pages need slots");
    if (g.finish == 1 && g.d > widest) widest = g.d;
    if (g.finish == 1 && g.dest == 2) return zi_refuse("conv_heads: unit vectors go to rows");
    const size_t wide = g.dest == 0 ? 4 : (out_dtype == ZI_BF16 ? 2 : 4);
    while (np > 0 && (g.d % (2 * np) || g.n % (2 * np) || g.ldo % (2 * np) || !al(g.out, 2 * np * wide) || (g.finish == 2 && !neighbours))) --np;
    c += g.n;
    heads += (g.n + g.d - 1) / g.d;
  }
  if (c != C) return zi_refuse("conv_heads: segments of %d channels for %d", c, C);
  j.heads = heads;
  j.src = src; j.ld = ld; j.splits = splits; j.zstride = zstride;
  j.in_bias = in_bias; j.kern = kern; j.out_bias = out_bias; j.act = act;
  j.tail = tail; j.slot_stride = slot_stride; j.C = C; j.taps = taps; j.unit_eps = unit_eps;
  j.cos_t = cos_t; j.sin_t = sin_t; j.n_table_pos = n_table_pos; j.rot_dims = rot_dims; j.neighbours = neighbours;
  j.positions = positions; j.slots = slots; j.page_size = page_size;
  j.tile_seq = tile_seq; j.tile_q0 = tile_q0; j.cu_q = cu_q; j.state_slots = state_slots;
  j.smem_head = (widest + 1) & ~1;
  j.scalars = scalars; j.n_scalar = n_scalar; j.a = a; j.b = b; j.a_log = a_log; j.dt_bias = dt_bias; j.decay = decay; j.step = step;
  const size_t smem = (size_t)CH_WARPS * CH_TILE * j.smem_head * sizeof(float);
  if (smem > 200 * 1024) return zi_refuse("conv_heads: unit vectors of %d values are more than this kernel holds", widest);
  const int rows_of_blocks = (heads + CH_WARPS - 1) / CH_WARPS + (scalars ? 1 : 0);
  if (rows_of_blocks > 65535) return zi_refuse("conv_heads: %d heads", heads);
  dim3 grid(n_tiles, rows_of_blocks), block(CH_WARPS * 32);
#define ZI_CH(TT, TAPS, NP)                                                                                               \
  do {                                                                                                                    \
    auto kern_fn = conv_heads_kernel<TT, TAPS, NP>;                                                                       \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern_fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
      return zi_refuse("conv_heads: cannot get %zu bytes of shared memory", smem);                                        \
    zi_launch(kern_fn, grid, block, smem, stream, j);                                                                     \
  } while (0)
#define ZI_CH_TAPS(TT, NP)                             \
  do {                                                 \
    switch (taps) {                                    \
      case 2: ZI_CH(TT, 2, NP); break;                 \
      case 3: ZI_CH(TT, 3, NP); break;                 \
      case 4: ZI_CH(TT, 4, NP); break;                 \
      default: ZI_CH(TT, 0, NP); break;                \
    }                                                  \
  } while (0)
  ZI_DISPATCH_DTYPE(out_dtype, TT, { if (np == 2) ZI_CH_TAPS(TT, 2); else if (np == 1) ZI_CH_TAPS(TT, 1); else ZI_CH_TAPS(TT, 0); });
#undef ZI_CH_TAPS
#undef ZI_CH
  return zi_check_launch("conv_heads");
}

ZI_TRACE_SETTER(conv_heads)
