// The seam between two sublayers of a block that norms a sublayer's input AND its output:
//   y = N_post(scale * a) * w_post     (or y = scale * a without a post norm; nothing without an update)
//   h = h + y                          (32-bit residual stream, in place)
//   x = N_pre(h) * w_pre               (what the next sublayer reads, in the activations' type)
// in one pass: the update and the stream are read once, the row stays in registers in between.  Each norm is one of
//   0  RMS norm     v / sqrt(mean(v^2) + eps)
//   1  layer norm   (v - mean) / sqrt(mean((v - mean)^2) + eps)
// The update comes whole (float32 or bfloat16) or as split-K partial sums [splits][T][H] that are added in order.  With
// `rows` the picked rows' x is made and h is left as it is.  One block per row, 32-bit throughout.
//
// A layer norm's mean and squared deviations come from ONE exchange between the threads: every thread takes the count,
// mean and squared deviations of its own values, and these meet pairwise (Chan, Golub, LeVeque, "Updating Formulae and
// a Pairwise Algorithm for Computing Sample Variances", 1979), so no large mean is ever cancelled against.
#include "api.h"
#include "common.cuh"

namespace {
struct Moments {
  float n, mean, m2;
};

__device__ __forceinline__ Moments merge(const Moments& a, const Moments& b) {
  Moments r;
  r.n = a.n + b.n;
  const float d = b.mean - a.mean, wb = r.n > 0.f ? b.n / r.n : 0.f;
  r.mean = fmaf(d, wb, a.mean);
  r.m2 = a.m2 + b.m2 + d * d * a.n * wb;
  return r;
}

__device__ __forceinline__ Moments shuffled(const Moments& a, int o) {
  return {__shfl_xor_sync(0xffffffffu, a.n, o), __shfl_xor_sync(0xffffffffu, a.mean, o), __shfl_xor_sync(0xffffffffu, a.m2, o)};
}

// (mean, 1 / sqrt(spread + eps)) of the row whose values the block holds, n_own of them in this thread's v[0 .. cap).
// scratch: 3 * 32 floats that no other call of the kernel uses.
template <int CAP>
__device__ __forceinline__ float2 row_moments(const float (&v)[CAP], int n_own, int H, int kind, float eps, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  if (kind == 0) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < CAP; ++i) ss = fmaf(v[i], v[i], ss);         // places beyond the row hold zeros
    ss = warp_sum(ss);
    if (lane == 0) scratch[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < n_warps ? scratch[lane] : 0.f);
    return make_float2(0.f, 1.0f / sqrtf(ss / (float)H + eps));
  }
  Moments m = {(float)n_own, 0.f, 0.f};
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < CAP; ++i) sum += v[i];
  if (H == (int)blockDim.x * CAP) {
    // every thread holds as many values as every other (the common case): the pairs that meet have equal counts
    m.mean = sum * (1.0f / CAP);
#pragma unroll
    for (int i = 0; i < CAP; ++i) {
      const float d = v[i] - m.mean;
      m.m2 = fmaf(d, d, m.m2);
    }
    float half = 0.5f * CAP;                                         // half the count of either side
#pragma unroll
    for (int o = 1; o < 32; o <<= 1, half *= 2.f) {
      const float other = __shfl_xor_sync(0xffffffffu, m.mean, o), d = other - m.mean;
      m.m2 = fmaf(d * d, half, m.m2 + __shfl_xor_sync(0xffffffffu, m.m2, o));
      m.mean = 0.5f * (m.mean + other);
    }
    if (lane == 0) {
      scratch[warp] = m.mean;
      scratch[32 + warp] = m.m2;
    }
    __syncthreads();
    m.mean = scratch[lane & (n_warps - 1)];                          // a power of two of warps
    m.m2 = scratch[32 + (lane & (n_warps - 1))];
    for (int o = 1; o < n_warps; o <<= 1, half *= 2.f) {
      const float other = __shfl_xor_sync(0xffffffffu, m.mean, o), d = other - m.mean;
      m.m2 = fmaf(d * d, half, m.m2 + __shfl_xor_sync(0xffffffffu, m.m2, o));
      m.mean = 0.5f * (m.mean + other);
    }
    return make_float2(m.mean, 1.0f / sqrtf(m.m2 / (float)H + eps));
  }
  if (n_own > 0) m.mean = sum / (float)n_own;
#pragma unroll
  for (int i = 0; i < CAP; ++i) {
    const float d = v[i] - m.mean;
    if (i < n_own) m.m2 = fmaf(d, d, m.m2);
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const Moments other = shuffled(m, o);
    m = (lane & o) ? merge(other, m) : merge(m, other);              // the same order on both sides
  }
  if (lane == 0) {
    scratch[warp] = m.n;
    scratch[32 + warp] = m.mean;
    scratch[64 + warp] = m.m2;
  }
  __syncthreads();
  m = lane < n_warps ? Moments{scratch[lane], scratch[32 + lane], scratch[64 + lane]} : Moments{0.f, 0.f, 0.f};
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    if (o >= n_warps) break;
    const Moments other = shuffled(m, o);
    m = (lane & o) ? merge(other, m) : merge(m, other);
  }
  return make_float2(__shfl_sync(0xffffffffu, m.mean, 0), 1.0f / sqrtf(__shfl_sync(0xffffffffu, m.m2, 0) / (float)H + eps));
}

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float* v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// NV pieces of W values (4: 16-byte accesses; 1: any width and alignment) per thread.
template <typename TA, typename TO, int NV, int W>
__global__ void __launch_bounds__(NV <= 2 ? 1024 : 512)
sandwich_norm_kernel(float* __restrict__ h, const TA* __restrict__ a, const float* __restrict__ part, int splits, size_t zstride,
                     float scale, const float* __restrict__ w_post, int post_kind, float post_eps,
                     const float* __restrict__ w_pre, int pre_kind, float pre_eps, TO* __restrict__ x_out,
                     const int* __restrict__ rows, int H) {
  pdl_launch_dependents();
  __shared__ float scratch[2][96];
  constexpr int CAP = NV * W;
  const int step = blockDim.x * W, c0 = threadIdx.x * W;
  // few values per thread (a decode step's rows): the first norm's weights, which come from no kernel of the step, are
  // fetched before the wait; else they are read where they are used and cost no registers
  constexpr bool EARLY = NV <= 2;
  float wp[EARLY ? CAP : W];
  auto fetch_w = [&](float* to, int c) {
    if constexpr (W == 4) *reinterpret_cast<float4*>(to) = load4(w_post + c);
    else *to = w_post[c];
  };
  if (EARLY && w_post) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (c0 + i * step < H) fetch_w(wp + i * W, c0 + i * step);
  }
  pdl_wait();
  const size_t src = (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * H;
  float y[CAP], v[CAP];
  int n_own = 0;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    const bool in = c < H;
    n_own += in ? W : 0;
#pragma unroll
    for (int u = 0; u < W; ++u) y[i * W + u] = v[i * W + u] = 0.f;
    if (!in) continue;
    if constexpr (W == 4) {
      *reinterpret_cast<float4*>(v + i * 4) = load4(h + src + c);
      if (part) {
        float4 s = load4(part + src + c);
        for (int z = 1; z < splits; ++z) {
          const float4 p = load4(part + (size_t)z * zstride + src + c);
          s.x += p.x; s.y += p.y; s.z += p.z; s.w += p.w;
        }
        *reinterpret_cast<float4*>(y + i * 4) = s;
      } else if (a) {
        *reinterpret_cast<float4*>(y + i * 4) = load4(a + src + c);
      }
    } else {
      v[i] = h[src + c];
      if (part) {
        float s = part[src + c];
        for (int z = 1; z < splits; ++z) s += part[(size_t)z * zstride + src + c];
        y[i] = s;
      } else if (a) {
        y[i] = to_f32(a[src + c]);
      }
    }
  }
  if (a || part) {
#pragma unroll
    for (int i = 0; i < CAP; ++i) y[i] *= scale;
    if (w_post) {
      const float2 st = row_moments(y, n_own, H, post_kind, post_eps, scratch[0]);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        if (c >= H) continue;
        if (!EARLY) fetch_w(wp, c);
#pragma unroll
        for (int u = 0; u < W; ++u) y[i * W + u] = (y[i * W + u] - st.x) * st.y * wp[(EARLY ? i * W : 0) + u];
      }
    }
#pragma unroll
    for (int i = 0; i < CAP; ++i)
      if (i < n_own) v[i] += y[i];
    if (!rows) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        if (c >= H) continue;
        if constexpr (W == 4) store4(h + src + c, v + i * 4);
        else h[src + c] = v[i];
      }
    }
  }
  if (!w_pre) return;
  const float2 st = row_moments(v, n_own, H, pre_kind, pre_eps, scratch[1]);
  const size_t dst = (size_t)blockIdx.x * H;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    if (c >= H) continue;
    if constexpr (W == 4) {
      const float4 w = load4(w_pre + c);
      const float o[4] = {(v[i * 4] - st.x) * st.y * w.x, (v[i * 4 + 1] - st.x) * st.y * w.y, (v[i * 4 + 2] - st.x) * st.y * w.z,
                          (v[i * 4 + 3] - st.x) * st.y * w.w};
      store4(x_out + dst + c, o);
    } else {
      x_out[dst + c] = from_f32<TO>((v[i] - st.x) * st.y * w_pre[c]);
    }
  }
}
}  // namespace

extern "C" int zi_sandwich_norm(float* h, const void* a, int a_dtype, const float* part, int splits, long long zstride, float scale,
                                const float* w_post, int post_kind, float post_eps, const float* w_pre, int pre_kind,
                                float pre_eps, void* x_out, int out_dtype, const int* rows, int n_rows, int H,
                                cudaStream_t stream) {
  if (n_rows <= 0 || H <= 0) return 0;
  if (a && part) return zi_refuse("sandwich_norm: give the update either whole or as partial sums");
  if (part && splits < 1) return zi_refuse("sandwich_norm: %d partial sums", splits);
  if ((w_pre == nullptr) != (x_out == nullptr)) return zi_refuse("sandwich_norm: the second norm and its output go together");
  if (rows && !w_pre) return zi_refuse("sandwich_norm: picked rows without a second norm");
  for (int k : {post_kind, pre_kind})
    if (k != 0 && k != 1) return zi_refuse("sandwich_norm: unknown norm %d", k);
  auto al16 = [](const void* p) { return p == nullptr || ((uintptr_t)p & 15) == 0; };
  const bool vec = H % 4 == 0 && al16(h) && al16(a) && al16(part) && zstride % 4 == 0 && al16(w_post) && al16(w_pre) && al16(x_out);
  const int pieces = vec ? H / 4 : H;
  // Few rows (a decode step) spread a row over as many threads as it has pieces; many rows fill the GPU with small
  // blocks.  The 32-bit path keeps one block size per width, so that its sums' order depends on nothing but the row.
  const bool few = out_dtype == ZI_BF16 && n_rows <= 512;
  int threads = few ? 1024 : 256;
  while (threads > 32 && threads / 2 >= pieces) threads /= 2;
  int nv = (pieces + threads - 1) / threads;
  while (nv > 8 && threads < 512) {
    threads *= 2;
    nv = (pieces + threads - 1) / threads;
  }
  while (nv > 2 && threads > 512) {       // the forms of more pieces per thread take blocks of up to 512
    threads /= 2;
    nv = (pieces + threads - 1) / threads;
  }
  if (nv > 8) return zi_refuse("sandwich_norm: rows of %d values are more than this kernel holds", H);
#define ZI_SN(TA, TO, NV, W)                                                                                              \
  zi_launch(sandwich_norm_kernel<TA, TO, NV, W>, dim3(n_rows), dim3(threads), 0, stream, h, (const TA*)a, part, splits,   \
            (size_t)zstride, scale, w_post, post_kind, post_eps, w_pre, pre_kind, pre_eps, (TO*)x_out, rows, H)
#define ZI_SN_W(TA, TO, NV) do { if (vec) ZI_SN(TA, TO, NV, 4); else ZI_SN(TA, TO, NV, 1); } while (0)
#define ZI_SN_NV(TA, TO)                                   \
  do {                                                     \
    if (nv <= 1) ZI_SN_W(TA, TO, 1);                       \
    else if (nv <= 2) ZI_SN_W(TA, TO, 2);                  \
    else if (nv <= 4) ZI_SN_W(TA, TO, 4);                  \
    else ZI_SN_W(TA, TO, 8);                               \
  } while (0)
  ZI_DISPATCH_DTYPE(a ? a_dtype : ZI_F32, TA, ZI_DISPATCH_DTYPE(out_dtype, TO, ZI_SN_NV(TA, TO)));
#undef ZI_SN_NV
#undef ZI_SN_W
#undef ZI_SN
  return zi_check_launch("sandwich_norm");
}

ZI_TRACE_SETTER(sandwich_norm)
