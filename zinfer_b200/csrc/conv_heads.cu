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
// keeps the running inputs of its two channels in registers while it walks the tile, so every input is read once (plus
// taps-1 before the tile).  A lane's two channels are those of a rotated pair: neighbours (2i, 2i+1), or (i, i + rot/2).
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
// PAIRS: a lane's two channels are neighbours whose addresses allow 8-byte accesses.
template <typename T, int TAPS, bool PAIRS>
__global__ void __launch_bounds__(CH_WARPS * 32)
conv_heads_kernel(const ConvJob j) {
  pdl_launch_dependents();
  extern __shared__ float held_all[];
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
  float* tail = j.tail + (size_t)j.state_slots[seq] * j.slot_stride;
  float* held = held_all + (size_t)warp * CH_TILE * j.smem_head;

  // an input of the convolution: row `at` of this request's portion (negative: carried from before the step)
  auto input = [&](int at, int e, float bias) {
    if (at < 0) return tail[(size_t)(taps - 1 + at) * j.C + ch0 + e];
    return summed_at(j.src + (size_t)(tok0 + at) * j.ld + ch0 + e, j.splits, j.zstride) + bias;
  };
  auto input2 = [&](int at, int e, float2 bias) {
    const float* p = at < 0 ? tail + (size_t)(taps - 1 + at) * j.C + ch0 + e : j.src + (size_t)(tok0 + at) * j.ld + ch0 + e;
    float2 v = *reinterpret_cast<const float2*>(p);
    if (at < 0) return v;
    for (int z = 1; z < j.splits; ++z) {
      const float2 u = *reinterpret_cast<const float2*>(p + (size_t)z * j.zstride);
      v.x += u.x;
      v.y += u.y;
    }
    return make_float2(v.x + bias.x, v.y + bias.y);
  };
  // where a finished value goes
  auto put = [&](int t, int e0, int e1, float y0, float y1, bool two) {
    const size_t row = (size_t)(row0 + t);
    if (g.dest == 0) {
      float* o = static_cast<float*>(g.out) + row * g.ldo + (size_t)head * g.d;
      if (PAIRS && two) {
        *reinterpret_cast<float2*>(o + e0) = make_float2(y0, y1);
      } else {
        o[e0] = y0;
        if (two) o[e1] = y1;
      }
      return;
    }
    T* o;
    if (g.dest == 1) {
      o = static_cast<T*>(g.out) + row * g.ldo + (size_t)head * g.d;
    } else {
      const int page = tok_page[t];
      if (page < 0) return;                             // a row that pads a captured batch
      o = static_cast<T*>(g.out) + (((size_t)page * page_heads + head) * j.page_size + tok_off[t]) * g.d;
    }
    if constexpr (PAIRS && sizeof(T) == 2) {
      if (two) {
        *reinterpret_cast<__nv_bfloat162*>(o + e0) = __floats2bfloat162_rn(y0, y1);
        return;
      }
    }
    o[e0] = from_f32<T>(y0);
    if (two) o[e1] = from_f32<T>(y1);
  };

  const int np = (d + 1) >> 1;
  for (int p = lane; p < np; p += 32) {
    int e0 = 2 * p, e1 = 2 * p + 1;
    if (!PAIRS && !j.neighbours && p < half) {          // (i, i + rot/2); the channels that do not turn follow in twos
      e0 = p;
      e1 = p + half;
    }
    const bool two = e1 < d;
    const int f1 = two ? e1 : e0;                       // a channel that exists
    float2 ib = make_float2(0.f, 0.f), ob = ib;
    if (j.in_bias) ib = make_float2(j.in_bias[ch0 + e0], j.in_bias[ch0 + f1]);
    if (j.out_bias) ob = make_float2(j.out_bias[ch0 + e0], j.out_bias[ch0 + f1]);
    auto fetch = [&](int at) {
      if (PAIRS) return input2(at, e0, ib);
      return make_float2(input(at, e0, ib.x), input(at, f1, ib.y));
    };
    constexpr int W = TAPS > 0 ? TAPS : 1;
    float2 win[W], k[W];
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < TAPS; ++i) {
        k[i] = make_float2(j.kern[(size_t)i * j.C + ch0 + e0], j.kern[(size_t)i * j.C + ch0 + f1]);
        if (i > 0) win[i] = fetch(q0 - TAPS + i);       // inputs before the tile; every token shifts them down by one
      }
    }
    constexpr int AHEAD = 4;                            // tokens whose inputs are asked for together
#pragma unroll 1
    for (int t0 = 0; t0 < nt; t0 += AHEAD) {
      float2 in[AHEAD];
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) in[u] = t0 + u < nt ? fetch(q0 + t0 + u) : make_float2(0.f, 0.f);
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const int t = t0 + u;
        if (t >= nt) break;
        float2 acc = make_float2(0.f, 0.f);
        if constexpr (TAPS > 0) {
#pragma unroll
          for (int i = 0; i + 1 < TAPS; ++i) win[i] = win[i + 1];
          win[TAPS - 1] = in[u];
#pragma unroll
          for (int i = 0; i < TAPS; ++i) {
            acc.x = fmaf(k[i].x, win[i].x, acc.x);
            acc.y = fmaf(k[i].y, win[i].y, acc.y);
          }
        } else {
          for (int i = 0; i < taps; ++i) {
            const float2 x = fetch(q0 + t - (taps - 1) + i);
            acc.x = fmaf(j.kern[(size_t)i * j.C + ch0 + e0], x.x, acc.x);
            acc.y = fmaf(j.kern[(size_t)i * j.C + ch0 + f1], x.y, acc.y);
          }
        }
        float y0 = acc.x + ob.x, y1 = acc.y + ob.y;
        if (j.act == 1) {
          y0 = conv_silu(y0);
          y1 = conv_silu(y1);
        }
        if (g.finish == 1) {
          held[t * j.smem_head + e0] = y0;
          if (two) held[t * j.smem_head + e1] = y1;
          continue;
        }
        if (p < half) {
          const size_t at = (size_t)tok_pos[t] * half + p;
          rotate_pair(y0, y1, j.cos_t[at], j.sin_t[at]);
        }
        put(t, e0, e1, y0, y1, two);
      }
    }
    if (q0 == 0) {                                      // the inputs that the next step finds; ascending rows overwrite in place
      for (int r = 0; r < taps - 1; ++r) {
        const float2 u = fetch(qlen - (taps - 1) + r);  // from before this step: row r + qlen of the old tail
        float* o = tail + (size_t)r * j.C + ch0;
        o[e0] = u.x;
        if (two) o[e1] = u.y;
      }
    }
  }
  if (g.finish == 1) {
    for (int t = 0; t < nt; ++t) {                      // a lane reads its own values only
      const float* x = held + t * j.smem_head;
      float ss = 0.f;
      for (int p = lane; p < np; p += 32) {
        ss = fmaf(x[2 * p], x[2 * p], ss);
        if (2 * p + 1 < d) ss = fmaf(x[2 * p + 1], x[2 * p + 1], ss);
      }
      const float inv = g.scale / sqrtf(warp_sum(ss) + j.unit_eps);
      for (int p = lane; p < np; p += 32) {
        const bool two = 2 * p + 1 < d;
        put(t, 2 * p, 2 * p + 1, x[2 * p] * inv, two ? x[2 * p + 1] * inv : 0.f, two);
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
  bool pairs = ld % 2 == 0 && zstride % 2 == 0 && C % 2 == 0 && slot_stride % 2 == 0 && al(src, 8) && al(tail, 8);
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
    pairs = pairs && g.d % 2 == 0 && g.n % 2 == 0 && g.ldo % 2 == 0 && al(g.out, 8) && (g.finish != 2 || neighbours);
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
#define ZI_CH(TT, TAPS, PAIRS)                                                                                            \
  do {                                                                                                                    \
    auto kern_fn = conv_heads_kernel<TT, TAPS, PAIRS>;                                                                    \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern_fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
      return zi_refuse("conv_heads: cannot get %zu bytes of shared memory", smem);                                        \
    zi_launch(kern_fn, grid, block, smem, stream, j);                                                                     \
  } while (0)
#define ZI_CH_TAPS(TT, PAIRS)                          \
  do {                                                 \
    switch (taps) {                                    \
      case 2: ZI_CH(TT, 2, PAIRS); break;              \
      case 3: ZI_CH(TT, 3, PAIRS); break;              \
      case 4: ZI_CH(TT, 4, PAIRS); break;              \
      default: ZI_CH(TT, 0, PAIRS); break;             \
    }                                                  \
  } while (0)
  ZI_DISPATCH_DTYPE(out_dtype, TT, { if (pairs) ZI_CH_TAPS(TT, true); else ZI_CH_TAPS(TT, false); });
#undef ZI_CH_TAPS
#undef ZI_CH
  return zi_check_launch("conv_heads");
}

ZI_TRACE_SETTER(conv_heads)
