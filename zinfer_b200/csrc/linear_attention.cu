// Kernels of mixers that keep a matrix-valued state per head instead of keys (linear attention
// with a decay per key channel, with or without the delta rule), and of the short convolutions and
// the gated per-head norm around them.
//
// The recurrence, per head, with S [D key channels, V value channels] carried per request:
//     S <- diag(g_t) S                      the decay acts on the rows that belong to key channels
//     u_t = v_t, or beta_t v_t              plain form, without or with a step size per token and head
//     u_t = beta_t (v_t - S^T k_t)          delta rule
//     S <- S + k_t u_t^T ;  o_t = S^T (q_scale q_t)
// In a third form (HGRN2: "HGRN2: Gated Linear RNNs with State Expansion", Qin et al., 2024) a write is
// what the decay leaves room for: g = l + (1 - l) sigmoid(z + b) with a lower bound l per channel, k = 1 - g, u_t = v_t, q = silu(raw q).
// The kernel makes g, k and q from the projections as it stages them.
// Everything here is 32-bit arithmetic.  A request's tokens of this step are rows cu_q[s] ..
// cu_q[s+1]-1 of the flat batch and continue the request from slot state_slots[s].  Each column of S
// is visited by one group of lanes, token after token, in an order that depends on D alone, so a
// result depends neither on how the request was cut into steps nor on the batch.
#include "api.h"
#include "common.cuh"

namespace {

__device__ __forceinline__ float softplus_f32(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ int seq_of_token(const int* __restrict__ cu_q, int n_seqs, int t) {
  int s = 0, hi = n_seqs - 1;          // cu_q[s] <= t < cu_q[s+1]
  while (s < hi) {
    const int mid = (s + hi + 1) >> 1;
    if (cu_q[mid] <= t) s = mid; else hi = mid - 1;
  }
  return s;
}

// ------------------------------------------------------------------ short causal convolution
// y[t, c] = act(sum_j kern[c, j] * x[t - (taps-1-j), c]), inputs before the step's first token from the
// carried rows tail[slot][taps-1][C] (oldest first), one thread per (token, channel).
template <typename T>
__global__ void short_conv_kernel(float* __restrict__ y, int ldy, const T* __restrict__ x, int ldx,
                                  const float* __restrict__ kern, const float* __restrict__ tail,
                                  long long slot_stride, int C, int taps, int act, const int* __restrict__ cu_q,
                                  const int* __restrict__ state_slots, int n_seqs) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int s = seq_of_token(cu_q, n_seqs, t);
  const int tok0 = cu_q[s], tl = t - tok0;
  const float* st = tail + (size_t)state_slots[s] * slot_stride;
  float acc = 0.f;
  for (int j = 0; j < taps; ++j) {
    const int src = tl - (taps - 1 - j);
    float v;
    if (src >= 0) v = to_f32(x[(size_t)(tok0 + src) * ldx + c]);
    else v = st[(size_t)(taps - 1 + src) * C + c];      // src = -1: the newest carried input, row taps-2
    acc = fmaf(kern[(size_t)c * taps + j], v, acc);
  }
  if (act == 1) acc = acc * sigmoid_f32(acc);
  y[(size_t)t * ldy + c] = acc;
}

// The carried rows after the step: the last taps-1 inputs of each request, one thread per (request, channel).
// Row r takes an index above r, so ascending r may overwrite in place.
template <typename T>
__global__ void short_conv_carry_kernel(float* __restrict__ tail, long long slot_stride, const T* __restrict__ x, int ldx,
                                        int C, int taps, const int* __restrict__ cu_q,
                                        const int* __restrict__ state_slots, int n_seqs) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C || s >= n_seqs) return;
  const int tok0 = cu_q[s], qlen = cu_q[s + 1] - tok0;
  if (qlen <= 0) return;
  float* st = tail + (size_t)state_slots[s] * slot_stride;
  for (int r = 0; r < taps - 1; ++r) {
    const int src = qlen - (taps - 1) + r;
    st[(size_t)r * C + c] = src >= 0 ? to_f32(x[(size_t)(tok0 + src) * ldx + c]) : st[(size_t)(r + qlen) * C + c];
  }
}

// ------------------------------------------------------------------------------- decays
// mode 0: g = sigmoid(z + bias)^(inv_tau) = exp(log_sigmoid(z + bias) * inv_tau)
// mode 1: g = exp(-exp(a_log[head]) * softplus(z + bias)), head = column / D
__global__ void decay_kernel(float* __restrict__ z, size_t total, int N, int D, const float* __restrict__ bias,
                             const float* __restrict__ a_log, float inv_tau, int mode) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const int c = (int)(idx % N);
  const float x = z[idx] + (bias ? bias[c] : 0.f);
  z[idx] = mode == 0 ? expf(log_sigmoid_f32(x) * inv_tau) : expf(-expf(a_log[c / D]) * softplus_f32(x));
}

// x[t, head, :] <- scale * x / sqrt(sum(x^2) + eps), one warp per (token, head), in place
__global__ void unit_norm_kernel(float* __restrict__ x, int ld, int T, int heads, int d, float eps, float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int w = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= T * heads) return;
  float* p = x + (size_t)(w / heads) * ld + (size_t)(w % heads) * d;
  float ss = 0.f;
  for (int i = lane; i < d; i += 32) ss = fmaf(p[i], p[i], ss);
  ss = warp_sum(ss);
  const float r = scale / sqrtf(ss + eps);
  for (int i = lane; i < d; i += 32) p[i] *= r;
}

template <typename T>
__global__ void sigmoid_rows_kernel(float* __restrict__ out, int ldo, const T* __restrict__ x, int ldx, int rows, int W) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (size_t)rows * W) return;
  const int r = (int)(idx / W), c = (int)(idx % W);
  out[(size_t)r * ldo + c] = sigmoid_f32(to_f32(x[(size_t)r * ldx + c]));
}

// --------------------------------------------------------------------------- the recurrence
// Block: one request, one head, CB neighbouring value channels; 8 warps.  A column of S (D key channels of one
// value channel) belongs to P neighbouring lanes of one warp, R = 8 (or 16) rows each, in registers, and every
// lane works on NC = 2 columns at once (two independent chains of arithmetic per lane); the sums over a column's
// rows meet by a butterfly of shuffles over those P lanes (a fixed order), so nothing in the loop over tokens
// waits for another warp.  q, k and the decays of TB tokens at a time are staged in shared memory for the whole
// block, laid out so that the lanes' 16-byte reads fall into different banks; the next TB tokens are fetched
// into registers while these are worked on and stored afterwards (one barrier per TB tokens).
constexpr int LR_WARPS = 8, LR_THREADS = LR_WARPS * 32, TB = 16, NC = 2;

// What the third form (GATE) makes its gate from: `k` of the kernel is the raw forget projection z.  With splits > 1
// q, z and v are split-K partial sums, zstride apart, added in order as they are fetched.
struct ForgetGate {
  const float* lower;      // [H * D]
  const float* bias;       // [H * D] or null
  int splits;
  long long zstride;
};
__device__ __forceinline__ void forget_gate(float z, float lower, float& g, float& k) {
  const float e = expf(-fabsf(z)), r = 1.0f / (1.0f + e);      // sigmoid(|z|) = r, sigmoid(-|z|) = e r
  const float up = z >= 0.f ? r : e * r, down = z >= 0.f ? e * r : r;
  g = fmaf(1.0f - lower, up, lower);
  k = (1.0f - lower) * down;                                   // 1 - g without cancellation
}

// A long portion in tiles of `rows` tokens that run side by side, in three passes (CHUNK of the kernel): 1 every tile but a
// request's last makes the state it would leave if it began from zero, and the product of its decays; a small kernel
// then walks a request's tiles in order, S <- P S + L, and leaves each tile the state it begins with; 2 every tile runs
// the recurrence from that state.  0: a request's tokens in one walk.
struct RecurrenceTiles {
  const int* tile_seq;     // request of each tile
  const int* tile_q0;      // its first token within the request's portion
  int rows;
  float* states;           // [tiles][H][D][V]: L, then the state each tile begins with
  float* decays;           // [tiles][H][D]: P
  int only_single;         // CHUNK 0: leave out requests that bring more than one token
};

// MADE: the third form's q and gate come ready made (q, `decay`) and what is written is 1 - gate; there is no `k`.
// (The third form is held to the registers that let several blocks share an SM.)
template <typename TQ, typename TV, int R, bool DELTA, bool GATE = false, int CHUNK = 0, bool MADE = false>
__global__ void __launch_bounds__(LR_THREADS, MADE ? (R > 8 ? 3 : 4) : (GATE && R <= 8 ? 2 : 1))
linear_recurrence_kernel(float* __restrict__ out, int ldo, const TQ* __restrict__ q, int ldq, const TQ* __restrict__ k,
                         int ldk, const TV* __restrict__ v, int ldv, const float* __restrict__ decay, int ldg,
                         const float* __restrict__ beta, int ldb, float q_scale, float* __restrict__ state,
                         long long slot_stride, int H, int G, int D, int V, int P, const int* __restrict__ cu_q,
                         const int* __restrict__ state_slots, const ForgetGate fgate, const RecurrenceTiles tiles, int gh, int gi) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int DP = P * R;                           // key channels rounded up to whole parts
  const int CW = (32 / P) * NC, CB = LR_WARPS * CW;   // columns per warp and per block
  constexpr int PLANES = MADE ? 2 : 3;
  const int GO = (PLANES - 1) * TB * DP, VO = PLANES * TB * DP;
  const int BUF = VO + TB * CB + TB;     // one staging buffer: q, k (not MADE), g [TB][DP], v [TB][CB], beta [TB]
  const int s = CHUNK ? tiles.tile_seq[blockIdx.x] : blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * CB;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int p = lane % P, cw = lane / P;
  const int cb = warp * CW + cw * NC, col = j0 + cb;   // this lane's first column within the block, and of the head
  const int kvh = h / (H / G);
  const int q0 = CHUNK ? tiles.tile_q0[blockIdx.x] : 0;
  const int tok0 = cu_q[s] + q0, left = cu_q[s + 1] - tok0;
  const int qlen = CHUNK ? min(tiles.rows, left) : left;
  const bool last = qlen == left;
  if (qlen <= 0 || (CHUNK == 1 && last) || (CHUNK == 0 && tiles.only_single && qlen != 1)) return;
  float* S = state + (size_t)state_slots[s] * slot_stride + (size_t)h * D * V;
  float* ST = CHUNK ? tiles.states + ((size_t)blockIdx.x * H + h) * D * V : S;      // where this walk begins
  float Sr[NC][R];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = p * R + r;
      Sr[c][r] = (CHUNK != 1 && i < D && col + c < V) ? ST[(size_t)i * V + col + c] : 0.f;
    }
  const bool makes_decays = CHUNK == 1 && warp == 0 && blockIdx.z == 0;
  float Pr[CHUNK == 1 ? R : 1];
#pragma unroll
  for (int r = 0; r < (CHUNK == 1 ? R : 1); ++r) Pr[r] = 1.f;
  // DP and CB are powers of two: shifts instead of divisions
  const int lgDP = 31 - __clz(DP), lgCB = 31 - __clz(CB), lgP = 31 - __clz(P);
  // Key channel i = p R + 4 r4 + x lies at ((r4 P + p) 4 + x) of its token's row: for one r4 the P lanes of a column
  // read neighbouring 16-byte pieces.
  constexpr int LGR = R == 8 ? 3 : 4;
  auto place = [&](int i) { return ((((i >> 2) & (R / 4 - 1)) << lgP) + (i >> LGR)) * 4 + (i & 3); };
  // Staging in two halves: fetch() takes the first NPF elements per thread of q, k and the decays (all of them
  // while DP <= 128) and the first two of v into registers as they are stored; put() widens and stores them, and
  // fetches and stores whatever is left beyond them.
  constexpr int NPF = 8, NPV = 2;
  TQ fq[NPF], fk[NPF];
  TV fv[NPV];
  float fg[NPF], fb = 1.f;
  auto fetch = [&](int t0, int nt) {
    const int total = nt << lgDP;
#pragma unroll
    for (int u = 0; u < NPF; ++u) {
      const int e = tid + u * LR_THREADS;
      const int tt = e >> lgDP, i = e & (DP - 1);
      if (e < total && i < D) {
        const size_t row = (size_t)(tok0 + t0 + tt);
        if (CHUNK != 1) fq[u] = q[row * ldq + (size_t)kvh * D + i];
        if (!MADE) fk[u] = k[row * ldk + (size_t)kvh * D + i];
        if (!GATE) fg[u] = gi ? decay[row * ldg + (size_t)h * gh + i] : expf(decay[row * ldg + h]);
      } else {
        fq[u] = from_f32<TQ>(0.f);
        fk[u] = from_f32<TQ>(0.f);
        fg[u] = MADE ? 1.f : 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < NPV; ++u) {
      const int e = tid + u * LR_THREADS;
      const int c = j0 + (e & (CB - 1));
      fv[u] = (e < (nt << lgCB) && c < V) ? v[(size_t)(tok0 + t0 + (e >> lgCB)) * ldv + (size_t)h * V + c] : from_f32<TV>(0.f);
    }
    if (!GATE && !MADE && beta && tid < nt) fb = beta[(size_t)(tok0 + t0 + tid) * ldb + h];
    if constexpr (GATE) {
      for (int z = 1; z < fgate.splits; ++z) {
        const size_t zo = (size_t)z * fgate.zstride;
#pragma unroll
        for (int u = 0; u < NPF; ++u) {
          const int e = tid + u * LR_THREADS;
          const int tt = e >> lgDP, i = e & (DP - 1);
          if (e < total && i < D) {
            const size_t row = (size_t)(tok0 + t0 + tt);
            if (CHUNK != 1) fq[u] += q[zo + row * ldq + (size_t)kvh * D + i];
            fk[u] += k[zo + row * ldk + (size_t)kvh * D + i];
          }
        }
#pragma unroll
        for (int u = 0; u < NPV; ++u) {
          const int e = tid + u * LR_THREADS;
          const int c = j0 + (e & (CB - 1));
          if (e < (nt << lgCB) && c < V) fv[u] += v[zo + (size_t)(tok0 + t0 + (e >> lgCB)) * ldv + (size_t)h * V + c];
        }
      }
    }
  };
  // element i of a token's q, k and g into the staging buffer at `at`
  auto stage = [&](float* buf, int at, int i, float qv, float kv, float gv) {
    if constexpr (GATE) {
      if (i < D) {
        const int ch = h * D + i;
        forget_gate(kv + (fgate.bias ? fgate.bias[ch] : 0.f), fgate.lower[ch], gv, kv);
        if (CHUNK != 1) qv = qv * sigmoid_f32(qv);
      } else {
        kv = gv = 0.f;
      }
    }
    if (CHUNK != 1) buf[at] = qv * q_scale;
    if (!MADE) buf[TB * DP + at] = kv;
    buf[GO + at] = gv;
  };
  // a value that was not fetched into a register: whole, or the sum of its partial sums
  auto whole = [&](const auto* p) {
    float x = to_f32(*p);
    if constexpr (GATE)
      for (int z = 1; z < fgate.splits; ++z) x += to_f32(p[(size_t)z * fgate.zstride]);
    return x;
  };
  auto put = [&](int t0, int nt, float* buf) {
    const int total = nt << lgDP;
#pragma unroll
    for (int u = 0; u < NPF; ++u) {
      const int e = tid + u * LR_THREADS;
      if (e < total) {
        stage(buf, (e & ~(DP - 1)) + place(e & (DP - 1)), e & (DP - 1), to_f32(fq[u]), MADE ? 0.f : to_f32(fk[u]), GATE ? 0.f : fg[u]);
      }
    }
    for (int e = tid + NPF * LR_THREADS; e < total; e += LR_THREADS) {      // beyond the registers (DP > 128)
      const int tt = e >> lgDP, i = e & (DP - 1);
      const size_t row = (size_t)(tok0 + t0 + tt);
      const bool in = i < D;
      stage(buf, (e & ~(DP - 1)) + place(i), i, in ? whole(q + row * ldq + (size_t)kvh * D + i) : 0.f,
            in && !MADE ? whole(k + row * ldk + (size_t)kvh * D + i) : 0.f,
            in && !GATE ? (gi ? decay[row * ldg + (size_t)h * gh + i] : expf(decay[row * ldg + h])) : (MADE ? 1.f : 0.f));
    }
#pragma unroll
    for (int u = 0; u < NPV; ++u) {
      const int e = tid + u * LR_THREADS;
      if (e < (nt << lgCB)) buf[VO + e] = to_f32(fv[u]);
    }
    for (int e = tid + NPV * LR_THREADS; e < (nt << lgCB); e += LR_THREADS) {
      const int c = j0 + (e & (CB - 1));
      buf[VO + e] = c < V ? whole(v + (size_t)(tok0 + t0 + (e >> lgCB)) * ldv + (size_t)h * V + c) : 0.f;
    }
    if (tid < nt) buf[VO + TB * CB + tid] = fb;
  };
  fetch(0, min(TB, qlen));
  put(0, min(TB, qlen), sm);
  __syncthreads();
  int cur = 0;
  for (int t0 = 0; t0 < qlen; t0 += TB) {
    const int nt = min(TB, qlen - t0);
    const float* buf = sm + cur * BUF;
    // the next batch's loads go out now and land in the other buffer after this batch's work; nobody reads that
    // buffer before the barrier at the end of this iteration
    const bool more = t0 + TB < qlen;
    if (more) fetch(t0 + TB, min(TB, qlen - t0 - TB));
    const float* vs = buf + VO;
    const float* bs = vs + TB * CB;
    if constexpr (CHUNK == 1) {        // the state alone: no read-out
      for (int tt = 0; tt < nt; ++tt) {
        const float4* kt = reinterpret_cast<const float4*>(buf + TB * DP + tt * DP) + p;
        const float4* gt = reinterpret_cast<const float4*>(buf + GO + tt * DP) + p;
        float vj[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) vj[c] = vs[tt * CB + cb + c];
#pragma unroll
        for (int r4 = 0; r4 < R / 4; ++r4) {
          const float4 g4 = gt[r4 << lgP], k4 = MADE ? make_float4(1.f - g4.x, 1.f - g4.y, 1.f - g4.z, 1.f - g4.w) : kt[r4 << lgP];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            float* sr = Sr[c] + 4 * r4;
            sr[0] = fmaf(g4.x, sr[0], k4.x * vj[c]);
            sr[1] = fmaf(g4.y, sr[1], k4.y * vj[c]);
            sr[2] = fmaf(g4.z, sr[2], k4.z * vj[c]);
            sr[3] = fmaf(g4.w, sr[3], k4.w * vj[c]);
          }
          if (makes_decays) {
            Pr[4 * r4] *= g4.x; Pr[4 * r4 + 1] *= g4.y; Pr[4 * r4 + 2] *= g4.z; Pr[4 * r4 + 3] *= g4.w;
          }
        }
      }
    }
    if constexpr ((GATE || MADE) && CHUNK != 1) {       // what is written does not depend on the state: write, then read out
      for (int tt = 0; tt < nt; ++tt) {
        const float4* qt = reinterpret_cast<const float4*>(buf + tt * DP) + p;
        const float4* kt = reinterpret_cast<const float4*>(buf + TB * DP + tt * DP) + p;
        const float4* gt = reinterpret_cast<const float4*>(buf + GO + tt * DP) + p;
        float vj[NC], b[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          vj[c] = vs[tt * CB + cb + c];
          b[c] = 0.f;
        }
#pragma unroll
        for (int r4 = 0; r4 < R / 4; ++r4) {
          const float4 g4 = gt[r4 << lgP], q4 = qt[r4 << lgP];
          const float4 k4 = MADE ? make_float4(1.f - g4.x, 1.f - g4.y, 1.f - g4.z, 1.f - g4.w) : kt[r4 << lgP];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            float* sr = Sr[c] + 4 * r4;
            sr[0] = fmaf(g4.x, sr[0], k4.x * vj[c]);
            sr[1] = fmaf(g4.y, sr[1], k4.y * vj[c]);
            sr[2] = fmaf(g4.z, sr[2], k4.z * vj[c]);
            sr[3] = fmaf(g4.w, sr[3], k4.w * vj[c]);
            b[c] = fmaf(sr[0], q4.x, fmaf(sr[1], q4.y, fmaf(sr[2], q4.z, fmaf(sr[3], q4.w, b[c]))));
          }
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          if (o < P) {
#pragma unroll
            for (int c = 0; c < NC; ++c) b[c] += __shfl_xor_sync(0xffffffffu, b[c], o);
          }
        }
        float* po = out + (size_t)(tok0 + t0 + tt) * ldo + (size_t)h * V + col;
#pragma unroll
        for (int c = 0; c < NC; ++c)
          if (p == 0 && col + c < V) po[c] = b[c];
      }
    }
    for (int tt = 0; !GATE && !MADE && CHUNK != 1 && tt < nt; ++tt) {
      const float4* qt = reinterpret_cast<const float4*>(buf + tt * DP) + p;
      const float4* kt = reinterpret_cast<const float4*>(buf + TB * DP + tt * DP) + p;
      const float4* gt = reinterpret_cast<const float4*>(buf + 2 * TB * DP + tt * DP) + p;
      float a[NC], b[NC], kq = 0.f;      // (g S)^T k and (g S)^T q per column, k . q, over this lane's rows
#pragma unroll
      for (int c = 0; c < NC; ++c) a[c] = b[c] = 0.f;
      float kr[R];
#pragma unroll
      for (int r4 = 0; r4 < R / 4; ++r4) {
        const float4 g4 = gt[r4 << lgP], k4 = kt[r4 << lgP], q4 = qt[r4 << lgP];
        kr[4 * r4] = k4.x; kr[4 * r4 + 1] = k4.y; kr[4 * r4 + 2] = k4.z; kr[4 * r4 + 3] = k4.w;
        kq = fmaf(k4.x, q4.x, fmaf(k4.y, q4.y, fmaf(k4.z, q4.z, fmaf(k4.w, q4.w, kq))));
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float* sr = Sr[c] + 4 * r4;
          sr[0] *= g4.x; sr[1] *= g4.y; sr[2] *= g4.z; sr[3] *= g4.w;
          if (DELTA) a[c] = fmaf(sr[0], k4.x, fmaf(sr[1], k4.y, fmaf(sr[2], k4.z, fmaf(sr[3], k4.w, a[c]))));
          b[c] = fmaf(sr[0], q4.x, fmaf(sr[1], q4.y, fmaf(sr[2], q4.z, fmaf(sr[3], q4.w, b[c]))));
        }
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {       // the column's P lanes are neighbours: every lane ends with the sums
        if (o < P) {
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            if (DELTA) a[c] += __shfl_xor_sync(0xffffffffu, a[c], o);
            b[c] += __shfl_xor_sync(0xffffffffu, b[c], o);
          }
          kq += __shfl_xor_sync(0xffffffffu, kq, o);
        }
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const float vj = vs[tt * CB + cb + c];
        const float u = bs[tt] * (DELTA ? vj - a[c] : vj);
#pragma unroll
        for (int r = 0; r < R; ++r) Sr[c][r] = fmaf(kr[r], u, Sr[c][r]);
        if (p == 0 && col + c < V) out[(size_t)(tok0 + t0 + tt) * ldo + (size_t)h * V + col + c] = fmaf(u, kq, b[c]);
      }
    }
    if (more) put(t0 + TB, min(TB, qlen - t0 - TB), sm + (cur ^ 1) * BUF);
    __syncthreads();     // the other buffer is filled, and this one is free for the batch after it
    cur ^= 1;
  }
  if (CHUNK == 2 && !last) return;               // the next tile has its own
  float* SE = CHUNK == 1 ? ST : S;
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = p * R + r;
      if (i < D && col + c < V) SE[(size_t)i * V + col + c] = Sr[c][r];
    }
  if (makes_decays && cw == 0) {
#pragma unroll
    for (int r = 0; r < (CHUNK == 1 ? R : 1); ++r) {
      const int i = p * R + r;
      if (i < D) tiles.decays[((size_t)blockIdx.x * H + h) * D + i] = Pr[r];
    }
  }
}

// The third form's q and gate of every token and channel, made once for both passes over a long portion's tiles.
__global__ void make_gates_kernel(float* __restrict__ qs, float* __restrict__ gs, const float* __restrict__ q, int ldq,
                                  const float* __restrict__ z, int ldz, const float* __restrict__ bias,
                                  const float* __restrict__ lower, int W, size_t total) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const size_t row = idx / W;
  const int c = (int)(idx - row * W);
  const float x = q[row * ldq + c];
  float g, k;
  forget_gate(z[row * ldz + c] + (bias ? bias[c] : 0.f), lower[c], g, k);
  qs[idx] = x * sigmoid_f32(x);
  gs[idx] = g;
}

// Between the two passes over a long portion's tiles: one thread per element of a head's state walks its request's tiles
// in order.  A request's tiles may stand anywhere in the list, so each block first finds their places.
constexpr int SCAN_THREADS = 256, SCAN_TILES = 1024;

__global__ void __launch_bounds__(SCAN_THREADS)
recurrence_scan_kernel(const RecurrenceTiles tiles, int n_tiles, const float* __restrict__ state, long long slot_stride, int H, int D,
                       int V, const int* __restrict__ cu_q, const int* __restrict__ state_slots) {
  pdl_launch_dependents();
  __shared__ int at[SCAN_TILES];
  const int s = blockIdx.x, h = blockIdx.y, e = blockIdx.z * SCAN_THREADS + threadIdx.x;
  const int qlen = cu_q[s + 1] - cu_q[s];        // the step's own arrays: here before any kernel of the step
  const int n = min((qlen + tiles.rows - 1) / tiles.rows, SCAN_TILES);
  for (int t = threadIdx.x; t < n_tiles; t += SCAN_THREADS) {
    const int c = tiles.tile_q0[t] / tiles.rows;
    if (tiles.tile_seq[t] == s && c < n) at[c] = t;
  }
  __syncthreads();
  pdl_wait();
  if (qlen <= 1 || e >= D * V) return;           // single tokens have no tiles
  float S = state[(size_t)state_slots[s] * slot_stride + (size_t)h * D * V + e];
  const int i = e / V;
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < n; c0 += AHEAD) {
    float L[AHEAD], P[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int c = c0 + u;
      L[u] = P[u] = 0.f;
      if (c < n - 1) {
        L[u] = tiles.states[((size_t)at[c] * H + h) * D * V + e];
        P[u] = tiles.decays[((size_t)at[c] * H + h) * D + i];
      }
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      if (c0 + u >= n) break;
      tiles.states[((size_t)at[c0 + u] * H + h) * D * V + e] = S;
      S = fmaf(P[u], S, L[u]);
    }
  }
}

// ------------------------------------------- one token per request: the third form with the head norm, in one kernel
// A block takes one request's token and one head, whole.  A row of S (the value channels of one key channel) belongs to
// LPR neighbouring lanes, NCV 16-byte pieces each, so the state is read and written in whole lines; a thread's first RD
// rows are asked for before the kernel waits for the projection (nothing of this step has written this state: a
// request's state is touched by one kernel a step, and a step's kernels start after the copy of the step's arrays, which
// waits for the step before).  o is summed over rows per thread, then over threads in a fixed order, normed over the
// head's value channels, multiplied by w and written in the activations' type.
constexpr int GD_THREADS = 512, GD_RD = 8;

template <typename TO, int NCV>
__global__ void __launch_bounds__(GD_THREADS)
gated_decode_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ q, int ldq, const float* __restrict__ z, int ldz,
                    const float* __restrict__ v, int ldv, float* __restrict__ state, long long slot_stride, int D, int V, int LPR,
                    const int* __restrict__ cu_q, const int* __restrict__ state_slots, const ForgetGate fgate,
                    const float* __restrict__ w, float eps) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float gd[];
  __shared__ float scratch[33];
  float* qs = gd;                    // [D] q, gate and what is written, then v [V], then the partial sums [slots][V]
  float* gs = qs + D;
  float* ks = gs + D;
  float* vs = gd + ((3 * D + 3) & ~3);
  float* red = vs + V;
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int slots = GD_THREADS / LPR, slot = tid / LPR, l = tid % LPR;
  const int row = cu_q[s];
  float* S = state + (size_t)state_slots[s] * slot_stride + (size_t)h * D * V;
  float4 st[GD_RD][NCV];
  auto col = [&](int c) { return (c * LPR + l) * 4; };
  auto load = [&](int r0) {
#pragma unroll
    for (int u = 0; u < GD_RD; ++u) {
      const int i = r0 + u * slots;
#pragma unroll
      for (int c = 0; c < NCV; ++c)
        st[u][c] = i < D && col(c) < V ? *reinterpret_cast<const float4*>(S + (size_t)i * V + col(c)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(slot);
  pdl_wait();
  auto summed = [&](const float* p) {
    float x = *p;
    for (int k = 1; k < fgate.splits; ++k) x += p[(size_t)k * fgate.zstride];
    return x;
  };
  for (int e = tid; e < D + V; e += GD_THREADS) {
    if (e < D) {
      const int ch = h * D + e;
      const float x = summed(q + (size_t)row * ldq + ch);
      float g, k;
      forget_gate(summed(z + (size_t)row * ldz + ch) + (fgate.bias ? fgate.bias[ch] : 0.f), fgate.lower[ch], g, k);
      qs[e] = x * sigmoid_f32(x);
      gs[e] = g;
      ks[e] = k;
    } else {
      vs[e - D] = summed(v + (size_t)row * ldv + (size_t)h * V + e - D);
    }
  }
  __syncthreads();
  float4 acc[NCV], vv[NCV];
#pragma unroll
  for (int c = 0; c < NCV; ++c) {
    acc[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    vv[c] = col(c) < V ? *reinterpret_cast<const float4*>(vs + col(c)) : acc[c];
  }
  for (int r0 = slot; r0 < D; r0 += GD_RD * slots) {
    if (r0 != slot) load(r0);
#pragma unroll
    for (int u = 0; u < GD_RD; ++u) {
      const int i = r0 + u * slots;
      if (i >= D) break;
      const float g = gs[i], k = ks[i], x = qs[i];
#pragma unroll
      for (int c = 0; c < NCV; ++c) {
        float4& t = st[u][c];
        t.x = fmaf(g, t.x, k * vv[c].x);
        t.y = fmaf(g, t.y, k * vv[c].y);
        t.z = fmaf(g, t.z, k * vv[c].z);
        t.w = fmaf(g, t.w, k * vv[c].w);
        acc[c].x = fmaf(x, t.x, acc[c].x);
        acc[c].y = fmaf(x, t.y, acc[c].y);
        acc[c].z = fmaf(x, t.z, acc[c].z);
        acc[c].w = fmaf(x, t.w, acc[c].w);
        if (col(c) < V) *reinterpret_cast<float4*>(S + (size_t)i * V + col(c)) = t;
      }
    }
  }
#pragma unroll
  for (int c = 0; c < NCV; ++c)
    if (col(c) < V) *reinterpret_cast<float4*>(red + (size_t)slot * V + col(c)) = acc[c];
  __syncthreads();
  float o = 0.f;                     // V <= GD_THREADS: one value channel per thread
  if (tid < V)
    for (int k = 0; k < slots; ++k) o += red[(size_t)k * V + tid];
  const float inv = 1.0f / sqrtf(block_sum(o * o, scratch) / (float)V + eps);
  if (tid < V) out[(size_t)row * ldo + (size_t)h * V + tid] = from_f32<TO>(o * inv * w[tid]);
}

// ------------------------------- one token per request: a decay and a step per head, with the head norm and its gate
// A block takes one request's token and one head; the whole head's state lies in the registers of its HD_THREADS threads
// (rows of S in 16-byte pieces: LPR neighbouring lanes a row, HD_RD rows a thread), asked for before the kernel waits for the
// one before it (nothing of this step has written it).  Both read-outs, S^T k and S^T q, come from one pass over the old
// state:  o = g S^T q + (k . q) u,  u = beta (v - g S^T k) (DELTA) or beta v;  then S <- g S + k u^T is written.
// With norm_w: o / sqrt(mean(o^2) + eps) * norm_w * silu(gate) in the activations' type; else o as it is.
constexpr int HD_THREADS = 512, HD_RD = 8;

template <typename TO, int NCV, bool DELTA>
__global__ void __launch_bounds__(HD_THREADS)
head_decay_decode_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk,
                         const float* __restrict__ v, int ldv, const float* __restrict__ logg, const float* __restrict__ beta,
                         float* __restrict__ state, long long slot_stride, int H, int G, int D, int V, int LPR,
                         const int* __restrict__ cu_q, const int* __restrict__ state_slots, const float* __restrict__ norm_w, float eps,
                         const float* __restrict__ gate, int ldgate, int gsplits, long long gz) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float hd[];
  __shared__ float scratch[33];
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, kvh = h / (H / G);
  const int slots = HD_THREADS / LPR, slot = tid / LPR, l = tid % LPR;
  float* qs = hd;                    // [D] q and k, [V] u, then the partial sums [2][slots][V]
  float* ks = qs + D;
  float* us = hd + ((2 * D + 3) & ~3);
  float* ra = us + V;
  float* rb = ra + slots * V;
  const int row = cu_q[s];
  float* S = state + (size_t)state_slots[s] * slot_stride + (size_t)h * D * V;
  float4 st[HD_RD][NCV];
  auto col = [&](int c) { return (c * LPR + l) * 4; };
#pragma unroll
  for (int u = 0; u < HD_RD; ++u) {
    const int i = slot + u * slots;
#pragma unroll
    for (int c = 0; c < NCV; ++c)
      st[u][c] = i < D && col(c) < V ? *reinterpret_cast<const float4*>(S + (size_t)i * V + col(c)) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  for (int e = tid; e < 2 * D; e += HD_THREADS) {
    if (e < D) qs[e] = q[(size_t)row * ldq + (size_t)kvh * D + e];
    else ks[e - D] = k[(size_t)row * ldk + (size_t)kvh * D + e - D];
  }
  float vj = 0.f, gt = 0.f;
  if (tid < V) {
    vj = v[(size_t)row * ldv + (size_t)h * V + tid];
    if (gate) {
      const float* pg = gate + (size_t)row * ldgate + (size_t)h * V + tid;
      gt = *pg;
      for (int z = 1; z < gsplits; ++z) gt += pg[(size_t)z * gz];
    }
  }
  const float g = expf(logg[(size_t)row * H + h]), b = beta[(size_t)row * H + h];
  __syncthreads();
  float kq = 0.f;                    // every warp makes it for itself, in the same order
  for (int i = tid & 31; i < D; i += 32) kq = fmaf(ks[i], qs[i], kq);
  kq = warp_sum(kq);
  float4 a[NCV], o4[NCV];
#pragma unroll
  for (int c = 0; c < NCV; ++c) a[c] = o4[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int u = 0; u < HD_RD; ++u) {
    const int i = slot + u * slots;
    if (i >= D) break;
    const float ki = ks[i], qi = qs[i];
#pragma unroll
    for (int c = 0; c < NCV; ++c) {
      const float4 t = st[u][c];
      if (DELTA) {
        a[c].x = fmaf(ki, t.x, a[c].x);
        a[c].y = fmaf(ki, t.y, a[c].y);
        a[c].z = fmaf(ki, t.z, a[c].z);
        a[c].w = fmaf(ki, t.w, a[c].w);
      }
      o4[c].x = fmaf(qi, t.x, o4[c].x);
      o4[c].y = fmaf(qi, t.y, o4[c].y);
      o4[c].z = fmaf(qi, t.z, o4[c].z);
      o4[c].w = fmaf(qi, t.w, o4[c].w);
    }
  }
#pragma unroll
  for (int c = 0; c < NCV; ++c)
    if (col(c) < V) {
      if (DELTA) *reinterpret_cast<float4*>(ra + (size_t)slot * V + col(c)) = a[c];
      *reinterpret_cast<float4*>(rb + (size_t)slot * V + col(c)) = o4[c];
    }
  __syncthreads();
  float o = 0.f;
  if (tid < V) {                     // V <= HD_THREADS: one value channel per thread
    float sa = 0.f;
    for (int z = 0; z < slots; ++z) {
      if (DELTA) sa += ra[(size_t)z * V + tid];
      o += rb[(size_t)z * V + tid];
    }
    const float u = b * (DELTA ? vj - g * sa : vj);
    us[tid] = u;
    o = fmaf(u, kq, g * o);
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < HD_RD; ++u) {
    const int i = slot + u * slots;
    if (i >= D) break;
    const float ki = ks[i];
#pragma unroll
    for (int c = 0; c < NCV; ++c) {
      if (col(c) >= V) continue;
      const float4 u4 = *reinterpret_cast<const float4*>(us + col(c)), t = st[u][c];
      *reinterpret_cast<float4*>(S + (size_t)i * V + col(c)) =
          make_float4(fmaf(g, t.x, ki * u4.x), fmaf(g, t.y, ki * u4.y), fmaf(g, t.z, ki * u4.z), fmaf(g, t.w, ki * u4.w));
    }
  }
  if (norm_w) {                      // uniform
    const float inv = 1.0f / sqrtf(block_sum(o * o, scratch) / (float)V + eps);
    if (tid < V) o = o * inv * norm_w[tid] * (gt * sigmoid_f32(gt));
  }
  if (tid < V) out[(size_t)row * ldo + (size_t)h * V + tid] = from_f32<TO>(o);
}

// ----------------------------------------------------------------------- gated per-head norm
// out[t, head, :] = o / sqrt(mean(o^2) + eps) * w * act(gate[t, head, :]); act: 0 silu, 1 sigmoid, 2 no gate.
// The gate may come as split-K partial sums (float32, gz apart), added in order.  One warp per (token, head).
template <typename TG, typename TO>
__global__ void head_norm_gate_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ o, int ldi,
                                      const float* __restrict__ w, float eps, const TG* __restrict__ gate, int ldgate,
                                      int gsplits, long long gz, int act, int T, int heads, int V) {
  pdl_launch_dependents();
  pdl_wait();
  const int wi = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (wi >= T * heads) return;
  const int t = wi / heads, h = wi % heads;
  const float* p = o + (size_t)t * ldi + (size_t)h * V;
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) ss = fmaf(p[i], p[i], ss);
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)V + eps);
  for (int i = lane; i < V; i += 32) {
    float g = 1.f;
    if (act != 2) {
      const TG* pg = gate + (size_t)t * ldgate + (size_t)h * V + i;
      g = to_f32(*pg);
      for (int z = 1; z < gsplits; ++z) g += to_f32(pg[(size_t)z * gz]);
    }
    const float a = act == 2 ? 1.f : (act == 0 ? g * sigmoid_f32(g) : sigmoid_f32(g));
    out[(size_t)t * ldo + (size_t)h * V + i] = from_f32<TO>(p[i] * inv * w[i] * a);
  }
}
}  // namespace

extern "C" int zi_short_conv(float* y, int ldy, const void* x, int ldx, int dtype, const float* kern, const float* tail,
                             long long slot_stride, int C, int taps, int act, const int* cu_q, const int* state_slots,
                             int n_seqs, int T, cudaStream_t stream) {
  if (T <= 0 || C <= 0) return 0;
  if (taps < 1 || taps > 64) return zi_refuse("short_conv: %d taps", taps);
  dim3 grid((C + 127) / 128, T);
  ZI_DISPATCH_DTYPE(dtype, TT, zi_launch(short_conv_kernel<TT>, dim3(grid), dim3(128), 0, stream, y, ldy, (const TT*)x, ldx,
                                         kern, tail, slot_stride, C, taps, act, cu_q, state_slots, n_seqs));
  return zi_check_launch("short_conv");
}

extern "C" int zi_short_conv_carry(float* tail, long long slot_stride, const void* x, int ldx, int dtype, int C, int taps,
                                   const int* cu_q, const int* state_slots, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0 || C <= 0 || taps <= 1) return 0;
  dim3 grid((C + 127) / 128, n_seqs);
  ZI_DISPATCH_DTYPE(dtype, TT, zi_launch(short_conv_carry_kernel<TT>, dim3(grid), dim3(128), 0, stream, tail, slot_stride,
                                         (const TT*)x, ldx, C, taps, cu_q, state_slots, n_seqs));
  return zi_check_launch("short_conv_carry");
}

extern "C" int zi_decay(float* z, long long rows, int N, int D, const float* bias, const float* a_log, float inv_tau,
                        int mode, cudaStream_t stream) {
  const size_t total = (size_t)rows * N;
  if (total == 0) return 0;
  if (mode != 0 && mode != 1) return zi_refuse("decay: unknown mode %d", mode);
  if (mode == 1 && (!a_log || D <= 0 || N % D)) return zi_refuse("decay: the per-head form needs a_log and whole heads");
  zi_launch(decay_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, z, total, N, D, bias, a_log, inv_tau, mode);
  return zi_check_launch("decay");
}

extern "C" int zi_unit_norm(float* x, int ld, int T, int heads, int d, float eps, float scale, cudaStream_t stream) {
  if (T <= 0 || heads <= 0) return 0;
  const int warps = 4;
  zi_launch(unit_norm_kernel, dim3((unsigned)((T * heads + warps - 1) / warps)), dim3(warps * 32), 0, stream, x, ld, T, heads, d,
            eps, scale);
  return zi_check_launch("unit_norm");
}

extern "C" int zi_sigmoid_rows(float* out, int ldo, const void* x, int ldx, int dtype, int rows, int W, cudaStream_t stream) {
  const size_t total = (size_t)rows * W;
  if (total == 0) return 0;
  ZI_DISPATCH_DTYPE(dtype, TT, zi_launch(sigmoid_rows_kernel<TT>, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream,
                                         out, ldo, (const TT*)x, ldx, rows, W));
  return zi_check_launch("sigmoid_rows");
}

extern "C" int zi_linear_recurrence(float* out, int ldo, const void* q, int ldq, const void* k, int ldk, int qk_dtype,
                                    const void* v, int ldv, int v_dtype, const float* decay, int ldg, const float* beta,
                                    int ldb, float q_scale, float* state, long long slot_stride, int H, int G, int D,
                                    int V, int delta, int head_decay, int only_single, const int* cu_q, const int* state_slots,
                                    int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const int gh = head_decay ? 1 : D, gi = head_decay ? 0 : 1;      // one decay per head (its logarithm), or one per key channel
  RecurrenceTiles walk = {};
  walk.only_single = only_single;
  if (H <= 0 || G <= 0 || H % G) return zi_refuse("linear_recurrence: %d heads do not divide into %d key heads", H, G);
  if (D <= 0 || D > 512 || V <= 0) return zi_refuse("linear_recurrence: %d key channels (1..512), %d value channels", D, V);
  if (delta && !beta) return zi_refuse("linear_recurrence: the delta rule needs beta");
  // R rows of a column per lane, P lanes per column (a power of two: the sums meet by a butterfly of shuffles)
  const int R = D <= 256 ? 8 : 16;
  int P = 1;
  while (P * R < D) P <<= 1;
  const int CB = LR_WARPS * (32 / P) * NC;
  const size_t smem = (size_t)2 * (3 * TB * P * R + TB * CB + TB) * sizeof(float);
  dim3 grid(n_seqs, H, (V + CB - 1) / CB), block(LR_THREADS);
#define ZI_LR(TQ, TV, RR, DD)                                                                                          \
  do {                                                                                                                 \
    auto kern = linear_recurrence_kernel<TQ, TV, RR, DD>;                                                              \
    if (smem > 48 * 1024) {                                                                                            \
      if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)           \
        return zi_refuse("linear_recurrence: cannot get %zu bytes of shared memory", smem);                            \
    }                                                                                                                  \
    zi_launch(kern, dim3(grid), dim3(block), smem, stream, out, ldo, (const TQ*)q, ldq, (const TQ*)k, ldk, (const TV*)v, \
              ldv, decay, ldg, beta, ldb, q_scale, state, slot_stride, H, G, D, V, P, cu_q, state_slots, ForgetGate{}, \
              walk, gh, gi);                                                                                           \
  } while (0)
#define ZI_LR_R(TQ, TV)                                          \
  do {                                                           \
    if (R == 8) { if (delta) ZI_LR(TQ, TV, 8, true); else ZI_LR(TQ, TV, 8, false); } \
    else { if (delta) ZI_LR(TQ, TV, 16, true); else ZI_LR(TQ, TV, 16, false); }         \
  } while (0)
  if (qk_dtype == ZI_F32 && v_dtype == ZI_F32) ZI_LR_R(float, float);
  else if (qk_dtype == ZI_BF16 && v_dtype == ZI_BF16) ZI_LR_R(__nv_bfloat16, __nv_bfloat16);
  else if (qk_dtype == ZI_F32 && v_dtype == ZI_BF16) ZI_LR_R(float, __nv_bfloat16);
  else return zi_refuse("linear_recurrence: operand types %d and %d", qk_dtype, v_dtype);
#undef ZI_LR_R
#undef ZI_LR
  return zi_check_launch("linear_recurrence");
}

// The third form: q, z and v are float32 projections (rows may be views of wider rows), whole or split-K partial sums.
extern "C" int zi_linear_recurrence_gated(float* out, int ldo, const float* q, int ldq, const float* z, int ldz, const float* v,
                                          int ldv, int splits, long long zstride, const float* f_bias, const float* lower,
                                          float* state, long long slot_stride, int H, int D, int V, const int* cu_q,
                                          const int* state_slots, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (H <= 0 || H > 65535) return zi_refuse("linear_recurrence_gated: %d heads", H);
  if (D <= 0 || D > 512 || V <= 0) return zi_refuse("linear_recurrence_gated: %d key channels (1..512), %d value channels", D, V);
  if (!lower || splits < 1) return zi_refuse("linear_recurrence_gated: needs the gate's lower bound and whole rows or partial sums");
  const int R = D <= 256 ? 8 : 16;
  int P = 1;
  while (P * R < D) P <<= 1;
  const int CB = LR_WARPS * (32 / P) * NC;
  const size_t smem = (size_t)2 * (3 * TB * P * R + TB * CB + TB) * sizeof(float);
  dim3 grid(n_seqs, H, (V + CB - 1) / CB), block(LR_THREADS);
  const ForgetGate gate = {lower, f_bias, splits, zstride};
  auto kern = R == 8 ? linear_recurrence_kernel<float, float, 8, false, true> : linear_recurrence_kernel<float, float, 16, false, true>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return zi_refuse("linear_recurrence_gated: cannot get %zu bytes of shared memory", smem);
  zi_launch(kern, grid, block, smem, stream, out, ldo, q, ldq, z, ldz, v, ldv, (const float*)nullptr, 0, (const float*)nullptr, 0, 1.0f,
            state, slot_stride, H, H, D, V, P, cu_q, state_slots, gate, RecurrenceTiles{}, D, 1);
  return zi_check_launch("linear_recurrence_gated");
}

// Floats of workspace that the form with tiles needs: q and the gates of T tokens, the tiles' states, their decays.
extern "C" long long zi_linear_recurrence_tiles_floats(int T, int n_tiles, int H, int D, int V) {
  return 2ll * T * H * D + (long long)n_tiles * H * D * (V + 1);
}
extern "C" int zi_linear_recurrence_tiles_supported(int n_tiles, int max_q_len, int rows, int D) {
  return n_tiles > 0 && rows > 0 && D > 0 && D <= 512 && (max_q_len + rows - 1) / rows <= SCAN_TILES;
}

// The same with the long portions cut into tiles of `rows` tokens that run side by side (tile_seq, tile_q0: the step's list
// over the requests that bring more than one token; n_single requests bring exactly one).
extern "C" int zi_linear_recurrence_gated_tiles(float* out, int ldo, const float* q, int ldq, const float* z, int ldz, const float* v,
                                                int ldv, int splits, long long zstride, const float* f_bias, const float* lower,
                                                float* state, long long slot_stride, int T, int H, int D, int V, const int* cu_q,
                                                const int* state_slots, int n_seqs, const int* tile_seq, const int* tile_q0,
                                                int n_tiles, int rows, int max_q_len, int n_single, float* workspace,
                                                cudaStream_t stream) {
  if (n_seqs <= 0 || T <= 0) return 0;
  if (H <= 0 || H > 65535 || V <= 0 || !zi_linear_recurrence_tiles_supported(n_tiles, max_q_len, rows, D))
    return zi_refuse("linear_recurrence_gated_tiles: %d tiles of %d tokens, %d key channels", n_tiles, rows, D);
  if (!lower || splits != 1 || !workspace) return zi_refuse("linear_recurrence_gated_tiles: needs whole rows, the gate's lower bound and a workspace");
  constexpr int R = 16;      // more rows per lane than the one-walk form: fewer lanes share a column, so fewer sums between lanes
  int P = 1;
  while (P * R < D) P <<= 1;
  const int CB = LR_WARPS * (32 / P) * NC;
  const size_t smem = (size_t)2 * (2 * TB * P * R + TB * CB + TB) * sizeof(float);
  const ForgetGate gate = {};
  float* qs = workspace;                                  // q and the gates, made once
  float* gs = qs + (size_t)T * H * D;
  float* ts = gs + (size_t)T * H * D;
  RecurrenceTiles tiles = {tile_seq, tile_q0, rows, ts, ts + (size_t)n_tiles * H * D * V, 0};
  const size_t total = (size_t)T * H * D;
  zi_launch(make_gates_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, qs, gs, q, ldq, z, ldz, f_bias, lower, H * D, total);
  int rc = zi_check_launch("linear_recurrence_gated_tiles (gates)");
  if (rc) return rc;
  auto run = [&](auto kern, int blocks) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return zi_refuse("linear_recurrence_gated_tiles: cannot get %zu bytes of shared memory", smem);
    zi_launch(kern, dim3(blocks, H, (V + CB - 1) / CB), dim3(LR_THREADS), smem, stream, out, ldo, (const float*)qs, H * D,
              (const float*)nullptr, 0, v, ldv, (const float*)gs, H * D, (const float*)nullptr, 0, 1.0f, state, slot_stride, H, H, D, V, P, cu_q, state_slots, gate, tiles, D, 1);
    return zi_check_launch("linear_recurrence_gated_tiles");
  };
  rc = run(linear_recurrence_kernel<float, float, R, false, false, 1, true>, n_tiles);
  if (rc) return rc;
  zi_launch(recurrence_scan_kernel, dim3(n_seqs, H, (D * V + SCAN_THREADS - 1) / SCAN_THREADS), dim3(SCAN_THREADS), 0, stream, tiles, n_tiles,
            (const float*)state, slot_stride, H, D, V, cu_q, state_slots);
  rc = zi_check_launch("linear_recurrence_gated_tiles (scan)");
  if (rc) return rc;
  rc = run(linear_recurrence_kernel<float, float, R, false, false, 2, true>, n_tiles);
  if (rc || n_single <= 0) return rc;
  tiles.only_single = 1;
  return run(linear_recurrence_kernel<float, float, R, false, false, 0, true>, n_seqs);
}

// Whether the one-kernel form for single tokens takes these sizes.
extern "C" int zi_gated_decode_supported(int D, int V) { return D > 0 && D <= 512 && V > 0 && V <= 256 && V % 4 == 0; }

// Every request brings one token: the third form and the head norm in one kernel; out [T, H * V] in the activations' type.
extern "C" int zi_gated_decode(void* out, int out_dtype, int ldo, const float* q, int ldq, const float* z, int ldz, const float* v,
                               int ldv, int splits, long long zstride, const float* f_bias, const float* lower, float* state,
                               long long slot_stride, int H, int D, int V, const float* norm_w, float eps, const int* cu_q,
                               const int* state_slots, int n_seqs, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (!zi_gated_decode_supported(D, V)) return zi_refuse("gated_decode: %d key channels, %d value channels", D, V);
  if (H <= 0 || H > 65535 || !lower || splits < 1 || !norm_w) return zi_refuse("gated_decode: %d heads, %d splits", H, splits);
  if (slot_stride % 4 || ((uintptr_t)state & 15)) return zi_refuse("gated_decode: the state must be 16-byte aligned");
  int LPR = 8;
  while (LPR < 32 && LPR * 4 < V) LPR <<= 1;
  const ForgetGate gate = {lower, f_bias, splits, zstride};
  const size_t smem = (size_t)(((3 * D + 3) & ~3) + V + GD_THREADS / LPR * V) * sizeof(float);
  dim3 grid(n_seqs, H), block(GD_THREADS);
  ZI_DISPATCH_DTYPE(out_dtype, TO, {
    auto kern = V <= 128 ? gated_decode_kernel<TO, 1> : gated_decode_kernel<TO, 2>;
    zi_launch(kern, grid, block, smem, stream, (TO*)out, ldo, q, ldq, z, ldz, v, ldv, state, slot_stride, D, V, LPR, cu_q, state_slots,
              gate, norm_w, eps);
  });
  return zi_check_launch("gated_decode");
}

static int head_decay_lanes(int V) {
  int lpr = 8;
  while (lpr < 32 && lpr * 4 < V) lpr <<= 1;
  return lpr;
}
// Whether a head's state fits the registers of one block.
extern "C" int zi_head_decay_decode_supported(int D, int V) {
  return D > 0 && V > 0 && V <= 256 && V % 4 == 0 && D <= HD_RD * (HD_THREADS / head_decay_lanes(V));
}

// Every request brings one token: the recurrence with one decay and one step per head, read-out included; with norm_w the
// head norm and its silu gate (float32 columns, whole or split-K partial sums) as well, in the activations' type.
extern "C" int zi_head_decay_decode(void* out, int out_dtype, int ldo, const float* q, int ldq, const float* k, int ldk, const float* v,
                                    int ldv, const float* logg, const float* beta, float* state, long long slot_stride, int H, int G,
                                    int D, int V, int delta, const float* norm_w, float eps, const float* gate, int ldgate,
                                    int gate_splits, long long gate_zstride, const int* cu_q, const int* state_slots, int n_seqs,
                                    cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (!zi_head_decay_decode_supported(D, V)) return zi_refuse("head_decay_decode: %d key channels, %d value channels", D, V);
  if (H <= 0 || H > 65535 || G <= 0 || H % G || !logg || !beta) return zi_refuse("head_decay_decode: %d heads, %d of keys", H, G);
  if ((norm_w == nullptr) != (gate == nullptr)) return zi_refuse("head_decay_decode: a norm goes with its gate");
  if (slot_stride % 4 || ((uintptr_t)state & 15)) return zi_refuse("head_decay_decode: the state must be 16-byte aligned");
  const int LPR = head_decay_lanes(V);
  const size_t smem = (size_t)(((2 * D + 3) & ~3) + V + 2 * (HD_THREADS / LPR) * V) * sizeof(float);
  dim3 grid(n_seqs, H), block(HD_THREADS);
  ZI_DISPATCH_DTYPE(out_dtype, TO, {
    auto kern = V <= 128 ? (delta ? head_decay_decode_kernel<TO, 1, true> : head_decay_decode_kernel<TO, 1, false>)
                         : (delta ? head_decay_decode_kernel<TO, 2, true> : head_decay_decode_kernel<TO, 2, false>);
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return zi_refuse("head_decay_decode: cannot get %zu bytes of shared memory", smem);
    zi_launch(kern, grid, block, smem, stream, (TO*)out, ldo, q, ldq, k, ldk, v, ldv, logg, beta, state, slot_stride, H, G, D, V, LPR, cu_q,
              state_slots, norm_w, eps, gate, ldgate, gate_splits, gate_zstride);
  });
  return zi_check_launch("head_decay_decode");
}

extern "C" int zi_head_norm_gate(void* out, int out_dtype, int ldo, const float* o, int ldi, const float* w, float eps,
                                 const void* gate, int gate_dtype, int ldgate, int gate_splits, long long gate_zstride, int act,
                                 int T, int heads, int V, cudaStream_t stream) {
  if (T <= 0 || heads <= 0) return 0;
  if (act < 0 || act > 2 || (act != 2 && !gate)) return zi_refuse("head_norm_gate: unknown gate %d", act);
  const int warps = 4;
  dim3 grid((unsigned)(((size_t)T * heads + warps - 1) / warps));
  ZI_DISPATCH_DTYPE(gate_dtype, TG, ZI_DISPATCH_DTYPE(out_dtype, TO,
      zi_launch(head_norm_gate_kernel<TG, TO>, dim3(grid), dim3(warps * 32), 0, stream, (TO*)out, ldo, o, ldi, w, eps,
                (const TG*)gate, ldgate, gate_splits, gate_zstride, act, T, heads, V)));
  return zi_check_launch("head_norm_gate");
}

// ------------------------------------------------------------------ gated norm of a row's parts
// y' = (y + skip[c / V] * x) * silu(z); each of `parts` equal parts of the row is divided by its own root mean square and
// multiplied by w.  skip and x may be absent; z may come as split-K partial sums.  One block per (token, part).
namespace {
template <typename TO>
__global__ void __launch_bounds__(512)
gated_part_norm_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ y, int ldy, const float* __restrict__ x, int ldx,
                       const float* __restrict__ skip, int V, const float* __restrict__ z, int ldz, int splits, long long zstride,
                       const float* __restrict__ w, float eps, int n) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float part[];
  __shared__ float scratch[33];
  const size_t t = blockIdx.x;
  const int c0 = blockIdx.y * n;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int c = c0 + i;
    float v = y[t * ldy + c];
    if (skip) v = fmaf(skip[c / V], x[t * ldx + c], v);
    float g = z[t * ldz + c];
    for (int k = 1; k < splits; ++k) g += z[(size_t)k * zstride + t * ldz + c];
    v *= g * sigmoid_f32(g);
    part[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) out[t * ldo + c0 + i] = from_f32<TO>(part[i] * inv * w[c0 + i]);
}

// The same in 16-byte pieces, a part's values in registers (parts of up to 4,096 values).
template <typename TO>
__global__ void __launch_bounds__(256)
gated_part_norm_vec_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ y, int ldy, const float* __restrict__ x, int ldx,
                           const float* __restrict__ skip, int V, const float* __restrict__ z, int ldz, int splits, long long zstride,
                           const float* __restrict__ w, float eps, int n) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[33];
  constexpr int MAXV = 4;
  const size_t t = blockIdx.x;
  const int c0 = blockIdx.y * n;
  auto at = [](const float* p) { return *reinterpret_cast<const float4*>(p); };
  float4 v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < MAXV; ++u) {
    const int i = (u * blockDim.x + threadIdx.x) * 4, c = c0 + i;
    v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < n) {
      v[u] = at(y + t * ldy + c);
      if (skip) {
        const float4 xv = at(x + t * ldx + c);
        const float s = skip[c / V];
        v[u] = make_float4(fmaf(s, xv.x, v[u].x), fmaf(s, xv.y, v[u].y), fmaf(s, xv.z, v[u].z), fmaf(s, xv.w, v[u].w));
      }
      float4 g = at(z + t * ldz + c);
      for (int k = 1; k < splits; ++k) {
        const float4 h = at(z + (size_t)k * zstride + t * ldz + c);
        g = make_float4(g.x + h.x, g.y + h.y, g.z + h.z, g.w + h.w);
      }
      v[u] = make_float4(v[u].x * g.x * sigmoid_f32(g.x), v[u].y * g.y * sigmoid_f32(g.y), v[u].z * g.z * sigmoid_f32(g.z),
                         v[u].w * g.w * sigmoid_f32(g.w));
      ss = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, ss))));
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
#pragma unroll
  for (int u = 0; u < MAXV; ++u) {
    const int i = (u * blockDim.x + threadIdx.x) * 4, c = c0 + i;
    if (i >= n) continue;
    const float4 wv = at(w + c);
    const float o[4] = {v[u].x * inv * wv.x, v[u].y * inv * wv.y, v[u].z * inv * wv.z, v[u].w * inv * wv.w};
    TO* po = out + t * ldo + c;
    if constexpr (sizeof(TO) == 4) {
      *reinterpret_cast<float4*>(po) = make_float4(o[0], o[1], o[2], o[3]);
    } else {
      __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1]), b = __floats2bfloat162_rn(o[2], o[3]);
      *reinterpret_cast<uint2*>(po) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
  }
}
}  // namespace

extern "C" int zi_gated_part_norm(void* out, int out_dtype, int ldo, const float* y, int ldy, const float* x, int ldx, const float* skip,
                                  int V, const float* z, int ldz, int splits, long long zstride, const float* w, float eps, int T,
                                  int width, int parts, cudaStream_t stream) {
  if (T <= 0 || width <= 0) return 0;
  if (parts <= 0 || width % parts || parts > 65535) return zi_refuse("gated_part_norm: %d columns in %d parts", width, parts);
  if (skip && (!x || V <= 0)) return zi_refuse("gated_part_norm: a skip needs what it multiplies");
  if (!z || splits < 1) return zi_refuse("gated_part_norm: needs its gate");
  const int n = width / parts;
  const size_t smem = (size_t)n * sizeof(float);
  if (smem > 200 * 1024) return zi_refuse("gated_part_norm: parts of %d values are more than this kernel holds", n);
  const int threads = n >= 1024 ? 512 : (n >= 256 ? 256 : 128);
  auto al16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (n % 4 == 0 && n <= 4096 && ldo % 4 == 0 && ldy % 4 == 0 && ldz % 4 == 0 && zstride % 4 == 0 && al16(out) && al16(y) && al16(z) && al16(w) &&
      (!skip || (V % 4 == 0 && ldx % 4 == 0 && al16(x)))) {
    ZI_DISPATCH_DTYPE(out_dtype, TO, zi_launch(gated_part_norm_vec_kernel<TO>, dim3(T, parts), dim3(n > 2048 ? 256 : (n > 512 ? 128 : 64)), 0,
                                               stream, (TO*)out, ldo, y, ldy, x, ldx, skip, V, z, ldz, splits, zstride, w, eps, n));
    return zi_check_launch("gated_part_norm");
  }
  ZI_DISPATCH_DTYPE(out_dtype, TO, {
    auto kern = gated_part_norm_kernel<TO>;
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return zi_refuse("gated_part_norm: cannot get %zu bytes of shared memory", smem);
    zi_launch(kern, dim3(T, parts), dim3(threads), smem, stream, (TO*)out, ldo, y, ldy, x, ldx, skip, V, z, ldz, splits, zstride, w, eps, n);
  });
  return zi_check_launch("gated_part_norm");
}

ZI_TRACE_SETTER(linear_attention)
