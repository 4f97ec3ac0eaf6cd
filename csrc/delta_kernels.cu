// Gated delta rules: short causal convolutions over time, unit-norm keys and queries, decays, and the recurrence
//
//     S <- g * S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          (per head, S is dim x vdim)
//
// over a ragged batch.  Everything that enters the recurrence is fp32, and so is the state.  Three orders of rows:
//   causal  a sequence's rows follow one another and its state advances (prompt portions, decoded tokens);
//   tree    every node continues its parent's state (packed ancestor bits, parents before children), nothing is stored:
//           each root-to-leaf path is walked from the stored state;
//   path    the stored state advances along chosen rows (the accepted nodes of a tree), nothing is read out.
// A sequence whose committed length is 0 starts from zeros whatever its state slot holds.
//
// Retention is the same walk with u = v and one constant decay per head (js_retention_seq).
//
// The convolutions' last inputs are a ring per state slot: the un-convolved row of position p is entry p % taps, so a
// decode step writes an entry that no reader of the same step looks at.
#include "common.cuh"

#include <limits.h>
#include <math.h>

namespace js {

JS_DEVICE float dl_ld(const float* p) { return *p; }
JS_DEVICE float dl_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
JS_DEVICE void dl_st(float* p, float v) { *p = v; }
JS_DEVICE void dl_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
JS_DEVICE float dl_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
JS_DEVICE float dl_silu(float z) { return z / (1.f + expf(-z)); }
JS_DEVICE float dl_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

JS_DEVICE int dl_find_seq(const int* cu_q, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

constexpr int kMaxTaps = 17;

struct DeltaShape {
  int H, G, D, V, taps;
  int channel;      // one decay per (head, key channel) instead of one per head
  const float* decay;       // retention: the heads' constant decays (H)
};

// ---------------------------------------------------------------- inputs of the recurrence
// One warp per (row, unit): G query heads, G key heads, H value heads, H units of decays and step size.
// q (T, G, D) includes the 1/sqrt(D); gl (T, H or H*D) are logarithms of the decays.
template <typename E>
__global__ void __launch_bounds__(256)
delta_prep_kernel(DeltaShape s, const E* pre, int ldp, const float* z, int ldz, const float* b, int ldb, const E* taps, const E* A_log,
                  const E* dt_bias, const E* conv, const int* rows, const int* cu_q, const int* past_lens, const int* mask_bits,
                  int W, int B, int T, float* q, float* k, float* v, float* gl, float* beta) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (unit >= 2 * s.G + 2 * s.H) return;
  if (unit >= 2 * s.G + s.H) {
    const int h = unit - 2 * s.G - s.H;
    const float a = expf(dl_ld(A_log + h));
    if (s.channel) {
      for (int d = lane; d < s.D; d += 32) {
        const int c = h * s.D + d;
        gl[static_cast<size_t>(t) * s.H * s.D + c] = -a * dl_softplus(z[static_cast<size_t>(t) * ldz + c] + dl_ld(dt_bias + c));
      }
    } else if (lane == 0) {
      gl[static_cast<size_t>(t) * s.H + h] = -a * dl_softplus(z[static_cast<size_t>(t) * ldz + h] + dl_ld(dt_bias + h));
    }
    if (lane == 0) beta[static_cast<size_t>(t) * s.H + h] = dl_sigmoid(b[static_cast<size_t>(t) * ldb + h]);
    return;
  }
  const int sq = dl_find_seq(cu_q, B, t);
  const int q0 = cu_q[sq], i = t - q0, past = past_lens[sq];
  const int C = 2 * s.G * s.D + s.H * s.V;
  const E* cs = conv + static_cast<size_t>(rows[sq]) * s.taps * C;
  // sources of the taps, newest first: rows of this batch (>= 0), ring entries (-1 - entry), or nothing (INT_MIN)
  int src[kMaxTaps];
  int have = 0;                         // rows of this batch found so far
  if (mask_bits == nullptr) {
    for (int m = 0; m < s.taps; ++m) {
      if (m <= i) { src[m] = t - m; ++have; }
    }
  } else {
    for (int w = W - 1; w >= 0 && have < s.taps; --w) {
      unsigned bits = static_cast<unsigned>(mask_bits[static_cast<size_t>(t) * W + w]);
      if (32 * w > i) bits = 0u;
      else if (32 * w + 31 > i) bits &= (2u << (i & 31)) - 1u;
      while (bits != 0u && have < s.taps) {
        const int hi = 31 - __clz(bits);
        src[have++] = q0 + 32 * w + hi;
        bits &= ~(1u << hi);
      }
    }
  }
  for (int m = have; m < s.taps; ++m) {
    const int pos = past - 1 - (m - have);
    src[m] = pos >= 0 ? -1 - pos % s.taps : INT_MIN;
  }
  const bool is_v = unit >= 2 * s.G;
  const int n = is_v ? s.V : s.D;
  const int c0 = is_v ? 2 * s.G * s.D + (unit - 2 * s.G) * s.V : unit * s.D;     // q heads, then k heads, then v heads
  float* dst = is_v ? v + (static_cast<size_t>(t) * s.H + unit - 2 * s.G) * s.V
             : unit < s.G ? q + (static_cast<size_t>(t) * s.G + unit) * s.D
                          : k + (static_cast<size_t>(t) * s.G + unit - s.G) * s.D;
  float keep[8], ss = 0.f;              // dim <= 256
  for (int j = 0; j * 32 < n; ++j) {
    const int d = j * 32 + lane;
    float y = 0.f;
    if (d < n) {
      const int c = c0 + d;
      for (int m = s.taps - 1; m >= 0; --m) {
        float in = 0.f;
        if (src[m] >= 0) in = dl_ld(pre + static_cast<size_t>(src[m]) * ldp + c);
        else if (src[m] != INT_MIN) in = dl_ld(cs + static_cast<size_t>(-1 - src[m]) * C + c);
        y += in * dl_ld(taps + static_cast<size_t>(c) * s.taps + s.taps - 1 - m);
      }
      y = dl_silu(y);
    }
    if (is_v) {
      if (d < n) dst[d] = y;
    } else {
      if (j < 8) keep[j] = y;
      ss += y * y;
    }
  }
  if (is_v) return;
  ss = warp_sum(ss);
  const float r = (unit < s.G ? 1.f / sqrtf(static_cast<float>(s.D)) : 1.f) / sqrtf(ss + 1e-6f);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int d = j * 32 + lane;
    if (d < n) dst[d] = keep[j] * r;
  }
}

// ---------------------------------------------------------------- the recurrence, row by row
struct DeltaSeqParams {
  DeltaShape s;
  const float *q, *k, *v, *gl, *beta;
  float* state;                 // (slots, H, D, V)
  const int *rows, *cu_q, *past_lens;
  int B;
  const int* mask_bits;         // tree mode: (T, W)
  int W, leaf_groups;
  const int *path, *path_len;   // path mode: rows of the (only) sequence to advance along
  float* out;                   // (T, H, V); null in path mode
  const void* pre;              // un-convolved rows, for the stored convolution inputs
  int ldp, pre_bf16;
  void* conv;                   // (slots, taps, C) ring
};

enum : int { kDeltaCausal = 0, kDeltaTree = 1, kDeltaPath = 2 };
constexpr int kDeltaCols = 32;      // value columns per CTA
constexpr int kDeltaMaxPath = 256;

// channel c of the ring: the inputs of the walk's last rows (path: their indices), the first of which has position `past`
template <typename E>
JS_DEVICE void delta_store_conv(const DeltaShape& s, void* conv, const void* pre, int ldp, int q0, const int* path, int n, int past,
                                int slot, int c) {
  const int C = 2 * s.G * s.D + s.H * s.V;
  E* cs = static_cast<E*>(conv) + static_cast<size_t>(slot) * s.taps * C + c;
  const E* src = static_cast<const E*>(pre) + c;
  for (int i = max(0, n - s.taps + 1); i < n; ++i)
    cs[static_cast<size_t>((past + i) % s.taps) * C] = src[static_cast<size_t>(q0 + (path != nullptr ? path[i] : i)) * ldp];
}

// ... for every channel that belongs to the value columns [v0, v0 + vn) of head h (and to its group's q and k, once)
JS_DEVICE void delta_store_conv_head(const DeltaShape& s, void* conv, const void* pre, int ldp, int bf16, int q0, const int* path, int n,
                                     int past, int slot, int h, int v0, int vn) {
  if (s.taps < 2) return;
  const int g = h / (s.H / s.G);
  const int qk = v0 == 0 && h % (s.H / s.G) == 0 ? 2 * s.D : 0;
  for (int c = threadIdx.x; c < vn + qk; c += blockDim.x) {
    const int x = c - vn;
    const int ch = c < vn ? 2 * s.G * s.D + h * s.V + v0 + c : x < s.D ? g * s.D + x : (s.G + g) * s.D + x - s.D;
    if (c < vn && v0 + c >= s.V) continue;
    if (bf16) delta_store_conv<__nv_bfloat16>(s, conv, pre, ldp, q0, path, n, past, slot, ch);
    else delta_store_conv<float>(s, conv, pre, ldp, q0, path, n, past, slot, ch);
  }
}

// kinds of recurrence: delta rule with a decay per head or per key channel, retention
enum : int { kRecHead = 0, kRecChannel = 1, kRecRetention = 2 };

// R lanes share a column: lane r holds the rows 4 (i R + r) .. + 3.  DP: dim rounded up (32, 64, 128, 256).
template <int DP, int R, int TB, int REC, int MODE>
__global__ void __launch_bounds__(kDeltaCols* R)
delta_seq_kernel(DeltaSeqParams p) {
  constexpr int NT = kDeltaCols * R, NI = DP / (4 * R);
  constexpr bool CH = REC == kRecChannel, RET = REC == kRecRetention;
  __shared__ __align__(16) float sq[2][TB][DP], sk[2][TB][DP], sg[2][TB][CH ? DP : 1];
  __shared__ float sv[2][TB][kDeltaCols], sb[2][TB];
  __shared__ int spath[kDeltaMaxPath];
  __shared__ unsigned inner[8];
  pdl_launch_dependents();
  pdl_wait();
  const DeltaShape s = p.s;
  const int h = blockIdx.x, sqi = blockIdx.y, tid = threadIdx.x;
  const int slices = (s.V + kDeltaCols - 1) / kDeltaCols;
  const int slice = MODE == kDeltaTree ? blockIdx.z % slices : blockIdx.z;
  const int col = slice * kDeltaCols + tid / R, r = tid % R;
  const int g = h / (s.H / s.G), slot = p.rows[sqi];
  const int q0 = p.cu_q[sqi], n_rows = p.cu_q[sqi + 1] - q0;
  const bool fresh = MODE != kDeltaPath && p.past_lens[sqi] == 0;      // a tree always has a committed prefix
  if (n_rows <= 0) return;
  float* st = p.state + (static_cast<size_t>(slot) * s.H + h) * s.D * s.V;
  const bool cv = col < s.V;

  auto load_state = [&](float (&S)[NI][4]) {
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 4 * (i * R + r) + e;
        S[i][e] = (!fresh && cv && d < s.D) ? st[static_cast<size_t>(d) * s.V + col] : 0.f;
      }
  };
  // stage rows [t0, t0 + TB) of the walk (their indices in spath, or consecutive) into buffer `buf`
  auto stage = [&](int buf, int t0, int n) {
    for (int x = tid; x < TB * DP; x += NT) {
      const int j = x / DP, d = x % DP;
      float qv = 0.f, kv = 0.f, gv = 1.f;
      if (t0 + j < n && d < s.D) {
        const size_t t = q0 + (MODE == kDeltaCausal ? t0 + j : spath[t0 + j]);
        if (MODE != kDeltaPath) qv = p.q[(t * s.G + g) * s.D + d];
        kv = p.k[(t * s.G + g) * s.D + d];
        if (CH) gv = expf(p.gl[(t * s.H + h) * s.D + d]);
      }
      sq[buf][j][d] = qv;
      sk[buf][j][d] = kv;
      if (CH) sg[buf][j][d] = gv;
    }
    for (int x = tid; x < TB * kDeltaCols; x += NT) {
      const int j = x / kDeltaCols, c = slice * kDeltaCols + x % kDeltaCols;
      const bool ok = t0 + j < n && c < s.V;
      const size_t t = q0 + (ok ? (MODE == kDeltaCausal ? t0 + j : spath[t0 + j]) : 0);
      sv[buf][j][x % kDeltaCols] = ok ? p.v[(t * s.H + h) * s.V + c] : 0.f;
    }
    for (int j = tid; j < TB; j += NT) {
      const bool ok = t0 + j < n;
      const size_t t = q0 + (ok ? (MODE == kDeltaCausal ? t0 + j : spath[t0 + j]) : 0);
      sb[buf][j] = ok && !RET ? p.beta[t * s.H + h] : 0.f;
      if (!CH) sg[buf][j][0] = !ok ? 1.f : RET ? s.decay[h] : expf(p.gl[t * s.H + h]);
    }
  };
  auto walk = [&](float (&S)[NI][4], int n) {
    int buf = 0;
    stage(0, 0, n);
    __syncthreads();
    for (int t0 = 0; t0 < n; t0 += TB, buf ^= 1) {
      if (t0 + TB < n) stage(buf ^ 1, t0 + TB, n);
      const int m = n - t0 < TB ? n - t0 : TB;
      for (int j = 0; j < m; ++j) {
        const float4* k4 = reinterpret_cast<const float4*>(sk[buf][j]);
        const float4* q4 = reinterpret_cast<const float4*>(sq[buf][j]);
        const float4* g4 = reinterpret_cast<const float4*>(sg[buf][j]);
        const float gs = CH ? 1.f : sg[buf][j][0];
        float4 kk[NI];
        float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          kk[i] = k4[i * R + r];
          const float4 gg = CH ? g4[i * R + r] : make_float4(gs, gs, gs, gs);
          S[i][0] *= gg.x; S[i][1] *= gg.y; S[i][2] *= gg.z; S[i][3] *= gg.w;
          if (!RET) {
            d0 += S[i][0] * kk[i].x; d1 += S[i][1] * kk[i].y; d2 += S[i][2] * kk[i].z; d3 += S[i][3] * kk[i].w;
          }
        }
        float d = (d0 + d1) + (d2 + d3), u = sv[buf][j][tid / R];
        if (!RET) {
#pragma unroll
          for (int o = R / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
          u = sb[buf][j] * (u - d);
        }
        d0 = d1 = d2 = d3 = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          S[i][0] += kk[i].x * u; S[i][1] += kk[i].y * u; S[i][2] += kk[i].z * u; S[i][3] += kk[i].w * u;
          if (MODE != kDeltaPath) {
            const float4 qq = q4[i * R + r];
            d0 += S[i][0] * qq.x; d1 += S[i][1] * qq.y; d2 += S[i][2] * qq.z; d3 += S[i][3] * qq.w;
          }
        }
        if (MODE != kDeltaPath) {
          d = (d0 + d1) + (d2 + d3);
#pragma unroll
          for (int o = R / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
          if (r == 0 && cv) {
            const size_t t = q0 + (MODE == kDeltaCausal ? t0 + j : spath[t0 + j]);
            p.out[(t * s.H + h) * s.V + col] = d;
          }
        }
      }
      __syncthreads();
    }
  };

  if (MODE == kDeltaTree) {
    // leaves: nodes that are nobody's proper ancestor.  Every leaf's path is walked; nodes shared by several paths are
    // written by each of them with the same value.
    if (tid < 8) inner[tid] = 0u;
    __syncthreads();
    const int words = p.W < 8 ? p.W : 8;
    for (int x = tid; x < n_rows * words; x += NT) {
      const int i = x / words, w = x % words;
      unsigned bits = static_cast<unsigned>(p.mask_bits[static_cast<size_t>(q0 + i) * p.W + w]);
      if ((i >> 5) == w) bits &= ~(1u << (i & 31));
      if (bits != 0u) atomicOr(&inner[w], bits);
    }
    __syncthreads();
    const int group = blockIdx.z / slices;
    int seen = 0;
    for (int leaf = 0; leaf < n_rows; ++leaf) {
      if ((inner[leaf >> 5] >> (leaf & 31)) & 1u) continue;
      if (seen++ % p.leaf_groups != group) continue;
      int n = 0;                        // every thread counts, thread 0 writes
      for (int w = 0; w < words; ++w) {
        unsigned bits = static_cast<unsigned>(p.mask_bits[static_cast<size_t>(q0 + leaf) * p.W + w]);
        while (bits != 0u) {
          const int lo = __ffs(bits) - 1;
          if (tid == 0) spath[n] = 32 * w + lo;
          ++n;
          bits &= bits - 1u;
        }
      }
      __syncthreads();
      float S[NI][4];
      load_state(S);
      walk(S, n);
      __syncthreads();
    }
    return;
  }

  int n = n_rows;
  if (MODE == kDeltaPath) {
    n = *p.path_len;
    n = n < 0 ? 0 : (n > kDeltaMaxPath ? kDeltaMaxPath : n);
    for (int x = tid; x < n; x += NT) {
      int i = p.path[x];
      spath[x] = i < 0 ? 0 : (i >= n_rows ? n_rows - 1 : i);
    }
    __syncthreads();
    if (n == 0) return;
  }
  float S[NI][4];
  load_state(S);
  walk(S, n);
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 4 * (i * R + r) + e;
      if (cv && d < s.D) st[static_cast<size_t>(d) * s.V + col] = S[i][e];
    }
  // in path mode past_lens is the committed length behind the path
  delta_store_conv_head(s, p.conv, p.pre, p.ldp, p.pre_bf16, q0, MODE == kDeltaPath ? spath : nullptr, n,
                        p.past_lens[sqi] - (MODE == kDeltaPath ? n : 0), slot, h, slice * kDeltaCols, kDeltaCols);
}

template <int DP, int R, int TB>
static int launch_delta_seq(const DeltaSeqParams& p, int mode, int pdl, cudaStream_t stream) {
  const int slices = (p.s.V + kDeltaCols - 1) / kDeltaCols;
  cudaLaunchConfig_t c = {};
  c.gridDim = dim3(p.s.H, p.B, slices * (mode == kDeltaTree ? p.leaf_groups : 1));
  c.blockDim = dim3(kDeltaCols * R);
  c.stream = stream;
  cudaLaunchAttribute a;
  a.id = cudaLaunchAttributeProgrammaticStreamSerialization;
  a.val.programmaticStreamSerializationAllowed = 1;
  c.attrs = &a;
  c.numAttrs = pdl ? 1 : 0;
  auto pick = [&](auto causal, auto tree, auto path) {
    return mode == kDeltaCausal ? cudaLaunchKernelEx(&c, causal, p) : mode == kDeltaTree ? cudaLaunchKernelEx(&c, tree, p) : cudaLaunchKernelEx(&c, path, p);
  };
#define JS_WALK(REC) \
  pick(delta_seq_kernel<DP, R, TB, REC, kDeltaCausal>, delta_seq_kernel<DP, R, TB, REC, kDeltaTree>, delta_seq_kernel<DP, R, TB, REC, kDeltaPath>)
  const cudaError_t e = p.s.decay != nullptr ? JS_WALK(kRecRetention) : p.s.channel ? JS_WALK(kRecChannel) : JS_WALK(kRecHead);
#undef JS_WALK
  return e == cudaSuccess ? 0 : -4;
}

static int launch_walk(const DeltaSeqParams& p, int mode, int pdl, cudaStream_t stream) {
  if (p.s.D <= 32) return launch_delta_seq<32, 4, 8>(p, mode, pdl, stream);
  if (p.s.D <= 64) return launch_delta_seq<64, 4, 8>(p, mode, pdl, stream);
  if (p.s.D <= 128) return launch_delta_seq<128, 4, 8>(p, mode, pdl, stream);
  return launch_delta_seq<256, 8, 4>(p, mode, pdl, stream);
}

// ---------------------------------------------------------------- read-out
// out = o / rms(o) * w * act(gate), one warp per (row, head)
template <typename E>
__global__ void __launch_bounds__(256)
gated_head_norm_kernel(const float* o, const E* w, const E* gate, int ldg, E* out, int ldo, int T, int H, int V, int Vp, int silu, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= T * H) return;
  const int t = u / H, h = u % H;
  const float* src = o + static_cast<size_t>(u) * V;
  float ss = 0.f;
  for (int d = lane; d < V; d += 32) ss += src[d] * src[d];
  const float r = 1.f / sqrtf(warp_sum(ss) / V + eps);
  for (int d = lane; d < Vp; d += 32) {
    float y = 0.f;
    if (d < V) {
      const float z = dl_ld(gate + static_cast<size_t>(t) * ldg + h * V + d);
      y = src[d] * r * (w != nullptr ? dl_ld(w + d) : 1.f) * (silu ? dl_silu(z) : dl_sigmoid(z));
    }
    dl_st(out + static_cast<size_t>(t) * ldo + h * Vp + d, y);
  }
}

// the same for V a multiple of 4 up to 256 and Vp = V, four columns a lane and one pass over memory
__global__ void __launch_bounds__(256)
gated_head_norm_vec_kernel(const float* o, const __nv_bfloat16* w, const __nv_bfloat16* gate, int ldg, __nv_bfloat16* out, int ldo, int T, int H,
                           int V, int silu, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= T * H) return;
  const int t = u / H, h = u % H;
  const float4* src = reinterpret_cast<const float4*>(o + static_cast<size_t>(u) * V);
  float4 y[2];
  uint2 zr[2];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int d = 4 * (lane + 32 * j);
    y[j] = d < V ? src[d / 4] : make_float4(0.f, 0.f, 0.f, 0.f);
    zr[j] = d < V ? *reinterpret_cast<const uint2*>(gate + static_cast<size_t>(t) * ldg + h * V + d) : make_uint2(0u, 0u);
  }
#pragma unroll
  for (int j = 0; j < 2; ++j) ss += y[j].x * y[j].x + y[j].y * y[j].y + y[j].z * y[j].z + y[j].w * y[j].w;
  const float r = 1.f / sqrtf(warp_sum(ss) / V + eps);
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int d = 4 * (lane + 32 * j);
    if (d >= V) continue;
    const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&zr[j]);
    const uint2 wr = w != nullptr ? *reinterpret_cast<const uint2*>(w + d) : make_uint2(0x3f803f80u, 0x3f803f80u);      // bf16 ones
    const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&wr);
    const float2 za = __bfloat1622float2(z2[0]), zb = __bfloat1622float2(z2[1]);
    const float2 wa = __bfloat1622float2(w2[0]), wb = __bfloat1622float2(w2[1]);
    auto act = [&](float z) { return silu ? dl_silu(z) : dl_sigmoid(z); };
    uint2 pk;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&pk);
    o2[0] = __floats2bfloat162_rn(y[j].x * r * wa.x * act(za.x), y[j].y * r * wa.y * act(za.y));
    o2[1] = __floats2bfloat162_rn(y[j].z * r * wb.x * act(zb.x), y[j].w * r * wb.y * act(zb.y));
    *reinterpret_cast<uint2*>(out + static_cast<size_t>(t) * ldo + h * V + d) = pk;
  }
}

struct DeltaLaunch {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a;
  DeltaLaunch(dim3 grid, dim3 block, cudaStream_t stream, int pdl) {
    c.gridDim = grid;
    c.blockDim = block;
    c.stream = stream;
    a.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    a.val.programmaticStreamSerializationAllowed = 1;
    c.attrs = &a;
    c.numAttrs = pdl ? 1 : 0;
  }
};

static bool delta_shape_ok(int H, int G, int D, int V, int taps) {
  return H > 0 && G > 0 && H % G == 0 && D > 0 && D <= 256 && V > 0 && taps >= 1 && taps <= kMaxTaps;
}

}  // namespace js

// pre (T, ldp) un-convolved q | k | v rows, taps (C, n), conv (slots, n, C) ring, A_log (H), dt_bias (H or H*D): bf16 or fp32;
// z (T, ldz), b (T, ldb) fp32.  Outputs fp32: q, k (T, G, D), v (T, H, V), gl (T, H or H*D), beta (T, H).  mask_bits (T, W)
// for token trees, else null.
extern "C" int js_delta_prep(int H, int G, int D, int V, int ntaps, int channel, const void* pre, int ldp, const float* z, int ldz,
                             const float* b, int ldb, const void* taps, const void* A_log, const void* dt_bias, const void* conv,
                             const int* rows, const int* cu_q, const int* past_lens, const int* mask_bits, int W, int B, int T,
                             float* q, float* k, float* v, float* gl, float* beta, int bf16, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || B <= 0) return 0;
  if (!delta_shape_ok(H, G, D, V, ntaps)) return -10;
  const DeltaShape s{H, G, D, V, ntaps, channel, nullptr};
  DeltaLaunch l(dim3(T, (2 * G + 2 * H + 7) / 8), dim3(256), stream, pdl);
  using bf = __nv_bfloat16;
  const cudaError_t e =
      bf16 ? cudaLaunchKernelEx(&l.c, delta_prep_kernel<bf>, s, (const bf*)pre, ldp, z, ldz, b, ldb, (const bf*)taps, (const bf*)A_log,
                                (const bf*)dt_bias, (const bf*)conv, rows, cu_q, past_lens, mask_bits, W, B, T, q, k, v, gl, beta)
           : cudaLaunchKernelEx(&l.c, delta_prep_kernel<float>, s, (const float*)pre, ldp, z, ldz, b, ldb, (const float*)taps,
                                (const float*)A_log, (const float*)dt_bias, (const float*)conv, rows, cu_q, past_lens, mask_bits, W,
                                B, T, q, k, v, gl, beta);
  return e == cudaSuccess ? 0 : -4;
}

// The recurrence over prepared inputs.  mode 0 causal, 1 tree (W <= 8, at most 256 nodes), 2 path (B = 1; path_len on the
// device, at most 256; past_lens is then the committed length behind the path).  state (slots, H, D, V) fp32; out (T, H, V) fp32.
extern "C" int js_delta_seq(int mode, int H, int G, int D, int V, int ntaps, int channel, const float* q, const float* k, const float* v,
                            const float* gl, const float* beta, float* state, const int* rows, const int* cu_q, const int* past_lens,
                            int B, const int* mask_bits, int W, int leaf_groups, const int* path, const int* path_len, float* out,
                            const void* pre, int ldp, void* conv, int bf16, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0) return 0;
  if (!delta_shape_ok(H, G, D, V, ntaps) || mode < 0 || mode > 2) return -10;
  if (mode == kDeltaTree && (mask_bits == nullptr || W < 1 || W > 8 || leaf_groups < 1)) return -13;
  if (mode == kDeltaPath && (path == nullptr || path_len == nullptr || B != 1)) return -13;
  if (mode != kDeltaPath && out == nullptr) return -13;
  DeltaSeqParams p{};
  p.s = DeltaShape{H, G, D, V, ntaps, channel, nullptr};
  p.q = q; p.k = k; p.v = v; p.gl = gl; p.beta = beta; p.state = state;
  p.rows = rows; p.cu_q = cu_q; p.past_lens = past_lens; p.B = B;
  p.mask_bits = mask_bits; p.W = W; p.leaf_groups = leaf_groups; p.path = path; p.path_len = path_len;
  p.out = out; p.pre = pre; p.ldp = ldp; p.pre_bf16 = bf16; p.conv = conv;
  return launch_walk(p, mode, pdl, stream);
}

// Retention over prepared fp32 rows q, k (T, H, D), v (T, H, V) with the heads' decays (H); modes and the rest as above.
extern "C" int js_retention_seq(int mode, int H, int D, int V, const float* q, const float* k, const float* v, const float* decay,
                                float* state, const int* rows, const int* cu_q, const int* past_lens, int B, const int* mask_bits, int W,
                                int leaf_groups, const int* path, const int* path_len, float* out, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0) return 0;
  if (!delta_shape_ok(H, H, D, V, 1) || mode < 0 || mode > 2 || decay == nullptr) return -10;
  if (mode == kDeltaTree && (mask_bits == nullptr || W < 1 || W > 8 || leaf_groups < 1)) return -13;
  if (mode == kDeltaPath && (path == nullptr || path_len == nullptr || B != 1)) return -13;
  if (mode != kDeltaPath && out == nullptr) return -13;
  DeltaSeqParams p{};
  p.s = DeltaShape{H, H, D, V, 1, 0, decay};
  p.q = q; p.k = k; p.v = v; p.state = state;
  p.rows = rows; p.cu_q = cu_q; p.past_lens = past_lens; p.B = B;
  p.mask_bits = mask_bits; p.W = W; p.leaf_groups = leaf_groups; p.path = path; p.path_len = path_len;
  p.out = out;
  return launch_walk(p, mode, pdl, stream);
}

// o (T, H, V) fp32 -> out (T, ldo) with head h at h * Vp (columns past V zero): o / rms * w * (silu or sigmoid)(gate (T, ldg)).
extern "C" int js_gated_head_norm(const float* o, const void* w, const void* gate, int ldg, void* out, int ldo, int T, int H, int V, int Vp,
                                  int silu, float eps, int bf16, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  DeltaLaunch l(dim3((T * H + 7) / 8), dim3(256), stream, pdl);
  using bf = __nv_bfloat16;
  const bool aligned = !((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 7) &&
                       !(reinterpret_cast<uintptr_t>(o) & 15);
  if (bf16 && V == Vp && V % 4 == 0 && V <= 256 && ldg % 4 == 0 && ldo % 4 == 0 && aligned)
    return cudaLaunchKernelEx(&l.c, gated_head_norm_vec_kernel, o, (const bf*)w, (const bf*)gate, ldg, (bf*)out, ldo, T, H, V, silu, eps) == cudaSuccess ? 0 : -4;
  const cudaError_t e =
      bf16 ? cudaLaunchKernelEx(&l.c, gated_head_norm_kernel<bf>, o, (const bf*)w, (const bf*)gate, ldg, (bf*)out, ldo, T, H, V, Vp, silu, eps)
           : cudaLaunchKernelEx(&l.c, gated_head_norm_kernel<float>, o, (const float*)w, (const float*)gate, ldg, (float*)out, ldo, T, H, V,
                                Vp, silu, eps);
  return e == cudaSuccess ? 0 : -4;
}
