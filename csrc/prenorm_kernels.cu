// Steps between the GEMMs of pre-norm decoders with mixed mixers: scaled embedding (with learned positions) with the first norm
// and the step's rotary tables, RMS norm of the fp32 residual stream, the residual step of sublayers whose output is normed
// (with a weighted average over the depth), what follows an attention's input projections (biases, norms over whole
// projections, general rotations, cache scatter), and the unfused forms.  Math is fp32; the residual stream is fp32.
//
// Rotations: entry pairs (i, i + n) ("half") or (2i, 2i + 1) ("next") of a head's first 2n entries.  The fused steps read
// (amp cos, amp sin) of every token from a table the embedding kernel makes once per forward for all layers.
#include "common.cuh"

#include <math.h>

namespace js {

JS_DEVICE float pn_ld(const float* p) { return *p; }
JS_DEVICE float pn_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
JS_DEVICE void pn_st(float* p, float v) { *p = v; }
JS_DEVICE void pn_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

struct PrenormLaunch {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a;
  PrenormLaunch(dim3 grid, dim3 block, cudaStream_t stream, int pdl, size_t smem = 0) {
    c.gridDim = grid;
    c.blockDim = block;
    c.stream = stream;
    c.dynamicSmemBytes = smem;
    a.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    a.val.programmaticStreamSerializationAllowed = 1;
    c.attrs = &a;
    c.numAttrs = pdl ? 1 : 0;
  }
};

// sum over a CTA of NT threads; every thread gets the result
template <int NT>
JS_DEVICE float pn_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) s += red[i];
  __syncthreads();
  return s;
}

static int pn_grid(size_t n) {
  const size_t b = (n + 255) / 256;
  return static_cast<int>(b > 1184 ? 1184 : b);
}

// ---------------------------------------------------------------- unfused forms
template <typename E>
__global__ void gelu_erf_kernel(const E* x, E* out, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const float z = pn_ld(x + i);
    pn_st(out + i, 0.5f * z * (1.f + erff(z * 0.7071067811865476f)));        // 1 / sqrt(2)
  }
}

template <typename E>
__global__ void xielu_kernel(const E* x, E* out, size_t n, float up, float down) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const float z = pn_ld(x + i);
    pn_st(out + i, 0.5f * z + (z > 0.f ? up * z * z : down * (expm1f(z) - z)));
  }
}

// out = sum_j w[j] hist_j, the terms given by address
constexpr int kDepthTerms = 64;
struct DepthTerms {
  const float* x[kDepthTerms];
};
__global__ void depth_average_kernel(DepthTerms h, int terms, const float* w, int first, float* out, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    float acc = first ? 0.f : out[i];
    for (int j = 0; j < terms; ++j) acc += w[j] * h.x[j][i];
    out[i] = acc;
  }
}

// out (T, H, V) = y * sigmoid(logits[t, h])
template <typename E>
__global__ void head_gate_kernel(const E* y, const float* logits, int ldz, E* out, size_t n, int H, int V) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t u = i / V;
    pn_st(out + i, pn_ld(y + i) / (1.f + expf(-logits[u / H * ldz + u % H])));
  }
}

// one thread per pair or passed-through entry of x (T, heads, D)
template <typename E, typename O>
__global__ void rotate_kernel(const E* x, O* out, const int* positions, size_t units, int heads, int D, int n, int next, const float* freq,
                              float amp) {
  const int items = D - n;
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < units * items; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t u = i / items;
    const int e = static_cast<int>(i % items);
    const E* src = x + u * D;
    O* dst = out + u * D;
    if (e >= n) {
      pn_st(dst + n + e, pn_ld(src + n + e));
      continue;
    }
    const int a = next ? 2 * e : e, b = next ? 2 * e + 1 : e + n;
    float sn, cs;
    sincosf(static_cast<float>(positions[u / heads]) * freq[e], &sn, &cs);
    const float p = pn_ld(src + a), q = pn_ld(src + b);
    cs *= amp;
    sn *= amp;
    pn_st(dst + a, p * cs - q * sn);
    pn_st(dst + b, q * cs + p * sn);
  }
}

// ---------------------------------------------------------------- embedding, first norm, rotary tables
constexpr int kRowThreads = 256;
constexpr int kRowKeep = 8;              // float4s a thread holds on to (rows up to 8192 wide); the rest is read twice

// x[t] = scale * table[ids[t]] (+ pos_table[positions[t]], its last row past the end), h[t] = bf16(x / rms(x) * w), rot[t] = (amp cos, amp sin) of the nf concatenated frequencies.
// Rows are ld long (a multiple of 4), zero past W; w too.
__global__ void __launch_bounds__(kRowThreads)
embed_rms_kernel(const int* ids, const __nv_bfloat16* table, int V, int ldt, float scale, const float* w, float eps, float* x,
                 __nv_bfloat16* h, int ld, int W, const int* positions, const __nv_bfloat16* pos_table, int n_pos, const float* freq,
                 const float* amp, int nf, float2* rot) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, W4 = ld / 4;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  const uint2* src = reinterpret_cast<const uint2*>(table + static_cast<size_t>(id) * ldt);
  float4* xr = reinterpret_cast<float4*>(x + static_cast<size_t>(t) * ld);
  const uint2* add = nullptr;
  if (pos_table != nullptr) {
    const int at = positions[t];
    add = reinterpret_cast<const uint2*>(pos_table + static_cast<size_t>(at < 0 ? 0 : (at >= n_pos ? n_pos - 1 : at)) * ldt);
  }
  auto load = [&](int c) {
    const uint2 raw = src[c];
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    float4 v = make_float4(lo.x * scale, lo.y * scale, hi.x * scale, hi.y * scale);
    if (add != nullptr) {
      const uint2 more = add[c];
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&more.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&more.y));
      v.x += a.x;
      v.y += a.y;
      v.z += b.x;
      v.w += b.y;
    }
    return v;
  };
  float ss = 0.f;
  for (int c = tid; c < W4; c += kRowThreads) {
    const float4 v = load(c);
    xr[c] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float r = 1.f / sqrtf(pn_sum<kRowThreads>(ss, red) / W + eps);
  uint2* hr = reinterpret_cast<uint2*>(h + static_cast<size_t>(t) * ld);
  for (int c = tid; c < W4; c += kRowThreads) {
    const float4 v = load(c), g = reinterpret_cast<const float4*>(w)[c];
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x * r * g.x, v.y * r * g.y), b = __floats2bfloat162_rn(v.z * r * g.z, v.w * r * g.w);
    hr[c] = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
  const float pos = static_cast<float>(positions[t]);
  for (int i = tid; i < nf; i += kRowThreads) {
    float sn, cs;
    sincosf(pos * freq[i], &sn, &cs);
    rot[static_cast<size_t>(t) * nf + i] = make_float2(amp[i] * cs, amp[i] * sn);
  }
}

// h[t] = bf16(x / rms(x) * w); tap[t] = bf16(x) where wanted
__global__ void __launch_bounds__(kRowThreads)
rms_rows_kernel(const float* x, const float* w, float eps, __nv_bfloat16* h, int ld, int W, __nv_bfloat16* tap, int ldt) {
  __shared__ float red[kRowThreads / 32];
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, W4 = ld / 4;
  const float4* w4 = reinterpret_cast<const float4*>(w);
  float4 g[kRowKeep];                    // weights do not depend on the kernel before
#pragma unroll
  for (int j = 0; j < kRowKeep; ++j) {
    const int c = tid + j * kRowThreads;
    g[j] = c < W4 ? w4[c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  const float4* xr = reinterpret_cast<const float4*>(x + static_cast<size_t>(t) * ld);
  float4 v[kRowKeep];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kRowKeep; ++j) {
    const int c = tid + j * kRowThreads;
    v[j] = c < W4 ? xr[c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int j = 0; j < kRowKeep; ++j) ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
  for (int c = tid + kRowKeep * kRowThreads; c < W4; c += kRowThreads) {
    const float4 u = xr[c];
    ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
  }
  const float r = 1.f / sqrtf(pn_sum<kRowThreads>(ss, red) / W + eps);
  uint2* hr = reinterpret_cast<uint2*>(h + static_cast<size_t>(t) * ld);
  auto put = [&](int c, float4 u, float4 k) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(u.x * r * k.x, u.y * r * k.y), b = __floats2bfloat162_rn(u.z * r * k.z, u.w * r * k.w);
    hr[c] = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    if (tap != nullptr) {
      const float e[4] = {u.x, u.y, u.z, u.w};
      for (int i = 0; i < 4; ++i)
        if (4 * c + i < W) tap[static_cast<size_t>(t) * ldt + 4 * c + i] = __float2bfloat16_rn(e[i]);
    }
  };
#pragma unroll
  for (int j = 0; j < kRowKeep; ++j) {
    const int c = tid + j * kRowThreads;
    if (c < W4) put(c, v[j], g[j]);
  }
  for (int c = tid + kRowKeep * kRowThreads; c < W4; c += kRowThreads) put(c, xr[c], w4[c]);
}

// ---------------------------------------------------------------- the residual step of a sublayer whose output is normed
// v = src + y / rms(y) * w.  Within a layer x = v.  At a layer's end (d set) v is the layer's result: it goes to hist slot `terms`
// and x = sum_{j < terms} d[j] hist[j] + d[terms] v.  h = bf16(x / rms(x) * fw), tap = bf16(x).  Rows are ld long (a multiple of
// 4) and zero past W, weights too.
struct SandwichParams {
  const __nv_bfloat16* y;
  const float *src, *w, *fw, *d;
  float *hist, *x;
  __nv_bfloat16 *h, *tap;
  size_t hist_stride;
  int ldy, ld, ldt, W, terms;
  float eps;
};

template <int NT, int KEEP>
__global__ void __launch_bounds__(NT) sandwich_kernel(SandwichParams p) {
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, W4 = p.ld / 4;
  const size_t row = static_cast<size_t>(t) * p.ld;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_wait();
  float4 v[KEEP], s[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = tid + j * NT;
    v[j] = s[j] = zero;
    if (c < W4) {
      const uint2 raw = *reinterpret_cast<const uint2*>(p.y + static_cast<size_t>(t) * p.ldy + 4 * c);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
      v[j] = make_float4(a.x, a.y, b.x, b.y);
      s[j] = reinterpret_cast<const float4*>(p.src + row)[c];
    }
    ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
  }
  // the history is on its way while the sum is made
  float4 acc[KEEP];
#pragma unroll
  for (int j = 0; j < KEEP; ++j) acc[j] = zero;
  for (int i = 0; i < p.terms; ++i) {
    const float di = __ldg(p.d + i);
    const float4* hr = reinterpret_cast<const float4*>(p.hist + i * p.hist_stride + row);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int c = tid + j * NT;
      if (c < W4) {
        const float4 u = hr[c];
        acc[j].x += di * u.x;
        acc[j].y += di * u.y;
        acc[j].z += di * u.z;
        acc[j].w += di * u.w;
      }
    }
  }
  const float r = 1.f / sqrtf(pn_sum<NT>(ss, red) / p.W + p.eps);
  const float dl = p.d != nullptr ? __ldg(p.d + p.terms) : 1.f;
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = tid + j * NT;
    if (c >= W4) continue;
    const float4 g = reinterpret_cast<const float4*>(p.w)[c];
    float4 u = make_float4(s[j].x + v[j].x * r * g.x, s[j].y + v[j].y * r * g.y, s[j].z + v[j].z * r * g.z, s[j].w + v[j].w * r * g.w);
    if (p.d != nullptr) {
      reinterpret_cast<float4*>(p.hist + p.terms * p.hist_stride + row)[c] = u;
      u = make_float4(acc[j].x + dl * u.x, acc[j].y + dl * u.y, acc[j].z + dl * u.z, acc[j].w + dl * u.w);
    }
    reinterpret_cast<float4*>(p.x + row)[c] = u;
    if (p.tap != nullptr) {
      const float e[4] = {u.x, u.y, u.z, u.w};
      for (int i = 0; i < 4; ++i)
        if (4 * c + i < p.W) p.tap[static_cast<size_t>(t) * p.ldt + 4 * c + i] = __float2bfloat16_rn(e[i]);
    }
    v[j] = u;
    ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
  }
  const float rf = 1.f / sqrtf(pn_sum<NT>(ss, red) / p.W + p.eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = tid + j * NT;
    if (c >= W4) continue;
    const float4 g = reinterpret_cast<const float4*>(p.fw)[c];
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[j].x * rf * g.x, v[j].y * rf * g.y);
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[j].z * rf * g.z, v[j].w * rf * g.w);
    reinterpret_cast<uint2*>(p.h + row)[c] = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
}

// ---------------------------------------------------------------- behind the input projections of a K/V attention
// proj (T, ldp): [q heads | k heads | v heads].  grid y: 0 = q to qout (T, G, Gp, Dq) (each group of H/G heads padded to Gp heads,
// which stay zero), 1 = k and 2 = v to their pool rows (G, S, Dp) and (G, S, Vp).  Biases are added, q and k optionally
// divided by the root mean square of the WHOLE projection (times its weights), then rotated.
struct AttnPostParams {
  const __nv_bfloat16* proj;
  const float *bias, *qw, *kw;           // bias of [q | k | v] or null; norm weights (H D), (G D) or null
  const float2* rot;                     // (T, ldr), this layer's n pairs
  const int* slots;
  __nv_bfloat16 *qout, *kpool, *vpool;
  int* status;
  int ldp, H, G, Gp, D, V, Dq, Dp, Vp, n, next, ldr, S;
  float eps;
};

constexpr int kPostThreads = 512;

__global__ void __launch_bounds__(kPostThreads) attn_post_kernel(AttnPostParams p) {
  extern __shared__ float sv[];          // the unit's values with their bias
  __shared__ float red[kPostThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, unit = blockIdx.y, tid = threadIdx.x;
  const __nv_bfloat16* row = p.proj + static_cast<size_t>(t) * p.ldp;
  int slot = 0;
  if (unit > 0) {
    slot = p.slots[t];
    if (slot < 0 || slot >= p.S) {
      if (tid == 0) report(p.status, kBadSlot);
      return;
    }
  }
  if (unit == 2) {
    const int c0 = (p.H + p.G) * p.D;
    for (int i = tid; i < p.G * p.Vp; i += kPostThreads) {
      const int g = i / p.Vp, d = i % p.Vp, c = c0 + g * p.V + d;
      const float v = d < p.V ? __bfloat162float(row[c]) + (p.bias != nullptr ? p.bias[c] : 0.f) : 0.f;
      p.vpool[(static_cast<size_t>(g) * p.S + slot) * p.Vp + d] = __float2bfloat16_rn(v);
    }
    return;
  }
  const bool is_q = unit == 0;
  const int heads = is_q ? p.H : p.G, c0 = is_q ? 0 : p.H * p.D, N = heads * p.D, width = is_q ? p.Dq : p.Dp, n = p.n;
  const float* w = is_q ? p.qw : p.kw;
  float ss = 0.f;
  for (int i = tid; i < N; i += kPostThreads) {
    const float v = __bfloat162float(row[c0 + i]) + (p.bias != nullptr ? p.bias[c0 + i] : 0.f);
    sv[i] = w != nullptr ? v * w[i] : v;
    ss += v * v;
  }
  const float total = pn_sum<kPostThreads>(ss, red);      // its barriers also publish sv
  const float r = w != nullptr ? 1.f / sqrtf(total / N + p.eps) : 1.f;
  const float2* rot = p.rot + static_cast<size_t>(t) * p.ldr;
  for (int i = tid; i < heads * width; i += kPostThreads) {
    const int hh = i / width, e = i % width;
    const float* v = sv + hh * p.D;
    float y = 0.f;
    if (e < 2 * n) {
      const int pair = p.next ? e >> 1 : (e < n ? e : e - n);
      const bool second = p.next ? (e & 1) != 0 : e >= n;
      const float2 cs = rot[pair];
      const float a = v[p.next ? 2 * pair : pair], b = v[p.next ? 2 * pair + 1 : pair + n];
      y = (second ? b * cs.x + a * cs.y : a * cs.x - b * cs.y) * r;
    } else if (e < p.D) {
      y = v[e] * r;
    }
    if (is_q) {
      const int g = p.H / p.G;
      p.qout[(static_cast<size_t>(t) * p.G * p.Gp + (hh / g) * p.Gp + hh % g) * width + e] = __float2bfloat16_rn(y);
    } else {
      p.kpool[(static_cast<size_t>(hh) * p.S + slot) * width + e] = __float2bfloat16_rn(y);
    }
  }
}

// The same with a token's q, k and v in one CTA and everything between load and store in registers.  An item is a group of
// rotated entries ("half": 2 + 2 of them, "next": 2), 2 that pass, or 2 of padding.  Needs even D, V and widths, an even n
// for "half", and at most kPostItems items of q and half as many of k a thread.
constexpr int kPostItems = 4;

struct PostItem {
  float2 a, b;             // b: the partners of a rotated "half" group
  float4 cs;               // (cos, sin) of one pair ("next") or two ("half")
  int head, e, kind;       // first entry; 0 nothing, 1 rotated "half", 2 rotated "next", 3 passes, 4 padding
};

// quotient of small non-negative integers by a divisor whose reciprocal is given
JS_DEVICE int small_div(int x, float inv) { return static_cast<int>((x + 0.5f) * inv); }

JS_DEVICE PostItem post_load(const AttnPostParams& p, const __nv_bfloat16* row, const float2* rot, int c0, const float* w, int heads, int width,
                             float inv_per, int idx, float& ss) {
  PostItem it{};
  const int n = p.n, groups = p.next ? n : n / 2, per = groups + (width - 2 * n) / 2;
  if (idx >= heads * per) return it;
  it.head = small_div(idx, inv_per);
  const int g = idx - it.head * per;
  it.kind = g < groups ? (p.next ? 2 : 1) : 2 * n + 2 * (g - groups) < p.D ? 3 : 4;
  it.e = g < groups ? 2 * g : 2 * n + 2 * (g - groups);
  if (it.kind == 4) return it;
  auto load = [&](int c) {
    float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + c0 + c));
    if (p.bias != nullptr) {
      const float2 b = *reinterpret_cast<const float2*>(p.bias + c0 + c);
      v.x += b.x;
      v.y += b.y;
    }
    ss += v.x * v.x + v.y * v.y;
    if (w != nullptr) {
      const float2 g2 = *reinterpret_cast<const float2*>(w + c);
      v.x *= g2.x;
      v.y *= g2.y;
    }
    return v;
  };
  if (it.kind == 1) it.cs = *reinterpret_cast<const float4*>(rot + it.e);
  if (it.kind == 2) {
    const float2 c = rot[it.e >> 1];
    it.cs = make_float4(c.x, c.y, 0.f, 0.f);
  }
  it.a = load(it.head * p.D + it.e);
  if (it.kind == 1) it.b = load(it.head * p.D + it.e + n);
  return it;
}

JS_DEVICE void post_store(const AttnPostParams& p, const PostItem& it, float r, __nv_bfloat16* dst) {
  if (it.kind == 0) return;
  float2 a = it.a;
  const float4 cs = it.cs;
  if (it.kind == 1) {
    a = make_float2(it.a.x * cs.x - it.b.x * cs.y, it.a.y * cs.z - it.b.y * cs.w);
    const float2 b = make_float2(it.b.x * cs.x + it.a.x * cs.y, it.b.y * cs.z + it.a.y * cs.w);
    *reinterpret_cast<__nv_bfloat162*>(dst + it.e + p.n) = __floats2bfloat162_rn(b.x * r, b.y * r);
  } else if (it.kind == 2) {
    a = make_float2(it.a.x * cs.x - it.a.y * cs.y, it.a.y * cs.x + it.a.x * cs.y);
  }
  *reinterpret_cast<__nv_bfloat162*>(dst + it.e) = __floats2bfloat162_rn(a.x * r, a.y * r);
}

template <int QI>
__global__ void __launch_bounds__(kPostThreads, QI <= 2 ? 2 : 1)
attn_post_vec_kernel(AttnPostParams p, float inv_q, float inv_k, float inv_v, float inv_group) {
  constexpr int KI = QI > 1 ? QI / 2 : 1, NW = kPostThreads / 32;
  __shared__ float red[2 * NW];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
  const __nv_bfloat16* row = p.proj + static_cast<size_t>(t) * p.ldp;
  const float2* rot = p.rot + static_cast<size_t>(t) * p.ldr;
  const int slot = p.slots[t], kc = p.H * p.D, vc = kc + p.G * p.D;
  PostItem q[QI], k[KI];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int j = 0; j < QI; ++j) q[j] = post_load(p, row, rot, 0, p.qw, p.H, p.Dq, inv_q, tid + j * kPostThreads, sq);
#pragma unroll
  for (int j = 0; j < KI; ++j) k[j] = post_load(p, row, rot, kc, p.kw, p.G, p.Dp, inv_k, tid + j * kPostThreads, sk);
  const bool ok = slot >= 0 && slot < p.S;
  if (!ok && tid == 0) report(p.status, kBadSlot);
  if (ok) {
    const int half = p.Vp / 2;
    for (int i = tid; i < p.G * half; i += kPostThreads) {
      const int g = small_div(i, inv_v), d = 2 * (i - g * half), c = vc + g * p.V + d;
      float2 v = make_float2(0.f, 0.f);
      if (d < p.V) {
        v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + c));
        if (p.bias != nullptr) {
          const float2 b = *reinterpret_cast<const float2*>(p.bias + c);
          v.x += b.x;
          v.y += b.y;
        }
      }
      *reinterpret_cast<__nv_bfloat162*>(p.vpool + (static_cast<size_t>(g) * p.S + slot) * p.Vp + d) = __floats2bfloat162_rn(v.x, v.y);
    }
  }
  float rq = 1.f, rk = 1.f;
  if (p.qw != nullptr) {
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { red[tid >> 5] = sq; red[NW + (tid >> 5)] = sk; }
    __syncthreads();
    static_assert(NW == 16, "one load a lane: q's sums in the lower half of the warp, k's in the upper");
    float s = red[lane];
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    rq = 1.f / sqrtf(__shfl_sync(0xffffffffu, s, 0) / (p.H * p.D) + p.eps);
    rk = 1.f / sqrtf(__shfl_sync(0xffffffffu, s, 16) / (p.G * p.D) + p.eps);
  }
  const int group = p.H / p.G;
#pragma unroll
  for (int j = 0; j < QI; ++j) {
    int hp = q[j].head;
    if (p.Gp != group) {
      const int g = small_div(hp, inv_group);
      hp = g * p.Gp + hp - g * group;
    }
    post_store(p, q[j], rq, p.qout + (static_cast<size_t>(t) * p.G * p.Gp + hp) * p.Dq);
  }
  if (!ok) return;
#pragma unroll
  for (int j = 0; j < KI; ++j) post_store(p, k[j], rk, p.kpool + (static_cast<size_t>(k[j].head) * p.S + slot) * p.Dp);
}

// ---------------------------------------------------------------- behind the input projections of a latent attention
// grid y: 0 = the cache row: raw (T, ldw) fp32 [latent | rotated key part] -> [latent / rms * w | rotated | zeros] at the token's pool
// row; 1 = the rotated part of every query head, in place: q (T, ldq) with heads dq apart, entries [dim, dim + 2n).
__global__ void __launch_bounds__(256)
latent_rot_post_kernel(const float* raw, int ldw, int rank, int n, const float* w, float eps, __nv_bfloat16* pool, int Rp, int S, const int* slots,
                       __nv_bfloat16* q, int ldq, int H, int dq, int dim, const float2* rot, int ldr, int* status) {
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const float2* rt = rot + static_cast<size_t>(t) * ldr;
  if (blockIdx.y == 1) {
    __nv_bfloat16* qr = q + static_cast<size_t>(t) * ldq + dim;
    for (int i = tid; i < H * n; i += 256) {
      __nv_bfloat16* e = qr + (i / n) * dq + 2 * (i % n);
      const float2 cs = rt[i % n];
      const float a = __bfloat162float(e[0]), b = __bfloat162float(e[1]);
      e[0] = __float2bfloat16_rn(a * cs.x - b * cs.y);
      e[1] = __float2bfloat16_rn(b * cs.x + a * cs.y);
    }
    return;
  }
  const int slot = slots[t];
  if (slot < 0 || slot >= S) {
    if (tid == 0) report(status, kBadSlot);
    return;
  }
  const float* src = raw + static_cast<size_t>(t) * ldw;
  __nv_bfloat16* dst = pool + static_cast<size_t>(slot) * Rp;
  constexpr int KEEP = 4;
  float v[KEEP], ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = tid + j * 256;
    v[j] = i < rank ? src[i] : 0.f;
    ss += v[j] * v[j];
  }
  for (int i = tid + KEEP * 256; i < rank; i += 256) ss += src[i] * src[i];
  const float r = 1.f / sqrtf(pn_sum<256>(ss, red) / rank + eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = tid + j * 256;
    if (i < rank) dst[i] = __float2bfloat16_rn(v[j] * r * w[i]);
  }
  for (int i = tid + KEEP * 256; i < rank; i += 256) dst[i] = __float2bfloat16_rn(src[i] * r * w[i]);
  for (int i = tid; i < n; i += 256) {
    const float2 cs = rt[i];
    const float a = src[rank + 2 * i], b = src[rank + 2 * i + 1];
    dst[rank + 2 * i] = __float2bfloat16_rn(a * cs.x - b * cs.y);
    dst[rank + 2 * i + 1] = __float2bfloat16_rn(b * cs.x + a * cs.y);
  }
  for (int i = rank + 2 * n + tid; i < Rp; i += 256) dst[i] = __float2bfloat16_rn(0.f);
}

}  // namespace js

extern "C" int js_gelu_erf(const void* x, void* out, long long n, int bf16, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  if (n <= 0) return 0;
  if (bf16) gelu_erf_kernel<bf><<<pn_grid(n), 256, 0, stream>>>((const bf*)x, (bf*)out, n);
  else gelu_erf_kernel<float><<<pn_grid(n), 256, 0, stream>>>((const float*)x, (float*)out, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// y, out (T, H * V) contiguous; logits (T, ldz) fp32
extern "C" int js_head_gate(const void* y, const float* logits, int ldz, void* out, int T, int H, int V, int bf16, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  const size_t n = static_cast<size_t>(T) * H * V;
  if (T <= 0 || H <= 0 || V <= 0) return 0;
  if (bf16) head_gate_kernel<bf><<<pn_grid(n), 256, 0, stream>>>((const bf*)y, logits, ldz, (bf*)out, n, H, V);
  else head_gate_kernel<float><<<pn_grid(n), 256, 0, stream>>>((const float*)y, logits, ldz, (float*)out, n, H, V);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// x, out (T, heads, D) contiguous; freq (dims / 2) fp32; next: pairs (2i, 2i + 1), else (i, i + dims / 2)
extern "C" int js_rotate(const void* x, int x_bf16, void* out, int o_bf16, const int* positions, int T, int heads, int D, int dims, int next,
                         const float* freq, float amp, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  if (T <= 0 || heads <= 0 || D <= 0) return 0;
  if (dims < 0 || (dims & 1) || dims > D) return -10;
  const int n = dims / 2;
  const size_t units = static_cast<size_t>(T) * heads;
  const int g = pn_grid(units * (D - n));
  if (x_bf16 && o_bf16) rotate_kernel<bf, bf><<<g, 256, 0, stream>>>((const bf*)x, (bf*)out, positions, units, heads, D, n, next, freq, amp);
  else if (x_bf16) rotate_kernel<bf, float><<<g, 256, 0, stream>>>((const bf*)x, (float*)out, positions, units, heads, D, n, next, freq, amp);
  else if (o_bf16) rotate_kernel<float, bf><<<g, 256, 0, stream>>>((const float*)x, (bf*)out, positions, units, heads, D, n, next, freq, amp);
  else rotate_kernel<float, float><<<g, 256, 0, stream>>>((const float*)x, (float*)out, positions, units, heads, D, n, next, freq, amp);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// table (V, ldt) bf16, x (T, ld) fp32, h (T, ld) bf16, w (ld) fp32; ld and ldt multiples of 4, at least W; rot (T, nf) float2.
// pos_table (n_pos, ldt) bf16 or null.
extern "C" int js_embed_rms(const int* ids, const void* table, int V, int ldt, float scale, const float* w, float eps, float* x, void* h, int ld,
                            int T, int W, const int* positions, const void* pos_table, int n_pos, const float* freq, const float* amp, int nf,
                            void* rot, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if ((ld % 4) || (ldt % 4) || ldt < ld || W < 1 || W > ld) return -10;
  PrenormLaunch l(dim3(T), dim3(kRowThreads), stream, pdl);
  return cudaLaunchKernelEx(&l.c, embed_rms_kernel, ids, (const __nv_bfloat16*)table, V, ldt, scale, w, eps, x, (__nv_bfloat16*)h, ld, W, positions,
                            (const __nv_bfloat16*)pos_table, n_pos, freq, amp, nf, (float2*)rot) == cudaSuccess ? 0 : -4;
}

extern "C" int js_xielu(const void* x, void* out, long long n, float up, float down, int bf16, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  if (n <= 0) return 0;
  if (bf16) xielu_kernel<bf><<<pn_grid(n), 256, 0, stream>>>((const bf*)x, (bf*)out, n, up, down);
  else xielu_kernel<float><<<pn_grid(n), 256, 0, stream>>>((const float*)x, (float*)out, n, up, down);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// out (n) = sum over `terms` of w[j] times the n floats at addr[j] (host array of device addresses)
extern "C" int js_depth_average(const unsigned long long* addr, int terms, const float* w, float* out, long long n, cudaStream_t stream) {
  using namespace js;
  if (n <= 0 || terms <= 0) return 0;
  for (int j0 = 0; j0 < terms; j0 += kDepthTerms) {
    DepthTerms h{};
    const int m = terms - j0 < kDepthTerms ? terms - j0 : kDepthTerms;
    for (int j = 0; j < m; ++j) h.x[j] = reinterpret_cast<const float*>(addr[j0 + j]);
    depth_average_kernel<<<pn_grid(n), 256, 0, stream>>>(h, m, w + j0, j0 == 0, out, n);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// See sandwich_kernel.  d: null within a layer, else terms + 1 weights on the device; hist (layers + 1, T, ld) with hist_stride
// elements between layers.  ld a multiple of 4, at most 32768; ldy a multiple of 4, at least ld.
extern "C" int js_sandwich(const void* y, int ldy, const float* src, const float* w, const float* d, int terms, float* hist,
                           long long hist_stride, float* x, const float* fw, float eps, void* h, int ld, void* tap, int ldt, int T, int W,
                           int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if ((ld % 4) || (ldy % 4) || ldy < ld || W < 1 || W > ld || ld > 32768 || terms < 0 || (d != nullptr) != (hist != nullptr) || (d == nullptr && terms)) return -10;
  SandwichParams p{(const __nv_bfloat16*)y, src, w, fw, d, hist, x, (__nv_bfloat16*)h, (__nv_bfloat16*)tap, (size_t)hist_stride,
                   ldy, ld, ldt, W, terms, eps};
  const int w4 = ld / 4;
  // few rows (decode) want many threads a row, many rows several float4 a thread
  const bool few = T <= 296;
  int nt = 256;
  auto kern = sandwich_kernel<256, 1>;
  if (w4 <= 256) {}
  else if (w4 <= 512 && !few) kern = sandwich_kernel<256, 2>;
  else if (w4 <= 512) { kern = sandwich_kernel<512, 1>; nt = 512; }
  else if (w4 <= 1024 && !few) kern = sandwich_kernel<256, 4>;
  else if (w4 <= 1024) { kern = sandwich_kernel<1024, 1>; nt = 1024; }
  else if (w4 <= 2048) { kern = sandwich_kernel<512, 4>; nt = 512; }
  else if (w4 <= 4096) { kern = sandwich_kernel<1024, 4>; nt = 1024; }
  else { kern = sandwich_kernel<1024, 8>; nt = 1024; }
  PrenormLaunch l(dim3(T), dim3(nt), stream, pdl);
  return cudaLaunchKernelEx(&l.c, kern, p) == cudaSuccess ? 0 : -4;
}

// x (T, ld) fp32 -> h (T, ld) bf16, w (ld) fp32, ld a multiple of 4; tap (T, ldt) bf16 gets the first W columns of x, or is null.
extern "C" int js_rms_rows(const float* x, const float* w, float eps, void* h, int ld, int T, int W, void* tap, int ldt, int pdl,
                           cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if ((ld % 4) || W < 1 || W > ld) return -10;
  PrenormLaunch l(dim3(T), dim3(kRowThreads), stream, pdl);
  return cudaLaunchKernelEx(&l.c, rms_rows_kernel, x, w, eps, (__nv_bfloat16*)h, ld, W, (__nv_bfloat16*)tap, ldt) == cudaSuccess ? 0 : -4;
}

// See attn_post_kernel.  H * D at most 24576.
extern "C" int js_attn_post(const void* proj, int ldp, const float* bias, const float* qw, const float* kw, int H, int G, int Gp, int D, int V,
                            int Dq, int Dp, int Vp, int dims, int next, const void* rot, int ldr, float eps, const int* slots, int S, int T,
                            void* qout, void* kpool, void* vpool, int* status, int pdl, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  if (T <= 0) return 0;
  if (H < 1 || G < 1 || H % G || Gp < H / G || D > Dq || D > Dp || V > Vp || dims > D || (dims & 1) || ldr < dims / 2 || H * D > 24576) return -10;
  AttnPostParams p{(const bf*)proj, bias, qw, kw, (const float2*)rot, slots, (bf*)qout, (bf*)kpool, (bf*)vpool, status,
                   ldp, H, G, Gp, D, V, Dq, Dp, Vp, dims / 2, next, ldr, S, eps};
  const int n = dims / 2, rot_items = next ? n : n / 2;
  const bool even = !((D | V | Dq | Dp | Vp | ldp | ldr) & 1) && (next || !(n & 1)) && !(reinterpret_cast<uintptr_t>(rot) & 15) && (qw == nullptr) == (kw == nullptr);
  const int qi = H * (rot_items + (Dq - 2 * n) / 2), ki = G * (rot_items + (Dp - 2 * n) / 2);
  auto fits = [&](int items) { return qi <= items * kPostThreads && ki <= (items > 1 ? items / 2 : 1) * kPostThreads; };
  if (even && fits(kPostItems)) {
    PrenormLaunch l(dim3(T), dim3(kPostThreads), stream, pdl);
    auto kern = fits(1) ? attn_post_vec_kernel<1> : fits(2) ? attn_post_vec_kernel<2> : attn_post_vec_kernel<kPostItems>;
    auto inv = [](int x) { return x > 0 ? 1.f / static_cast<float>(x) : 0.f; };
    return cudaLaunchKernelEx(&l.c, kern, p, inv(qi / H), inv(ki / G), inv(Vp / 2), inv(H / G)) == cudaSuccess ? 0 : -4;
  }
  const int smem = H * D * 4;
  static int configured[kMaxDevicesCached] = {};
  if (smem > 40 * 1024 && ensure_dyn_smem(attn_post_kernel, smem, configured) != 0) return -3;
  PrenormLaunch l(dim3(T, 3), dim3(kPostThreads), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, attn_post_kernel, p) == cudaSuccess ? 0 : -4;
}

// See latent_rot_post_kernel; dims = 2n rotated entries.
extern "C" int js_latent_rot_post(const float* raw, int ldw, int rank, int dims, const float* w, float eps, void* pool, int Rp, int S,
                                  const int* slots, void* q, int ldq, int H, int dq, int dim, const void* rot, int ldr, int T, int* status,
                                  int pdl, cudaStream_t stream) {
  using namespace js;
  using bf = __nv_bfloat16;
  if (T <= 0) return 0;
  if (rank < 1 || dims < 0 || (dims & 1) || rank + dims > Rp || ldw < rank + dims || dim + dims > dq || H * dq > ldq || ldr < dims / 2) return -10;
  PrenormLaunch l(dim3(T, dims > 0 ? 2 : 1), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, latent_rot_post_kernel, raw, ldw, rank, dims / 2, w, eps, (bf*)pool, Rp, S, slots, (bf*)q, ldq, H, dq, dim,
                            (const float2*)rot, ldr, status) == cudaSuccess ? 0 : -4;
}
