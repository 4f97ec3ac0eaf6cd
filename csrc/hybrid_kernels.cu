// Kernels around window attention, post-norm sublayers and table-routed experts: rotation + norm of q and k with the
// cache scatter, window attention on the plain cores (32-bit path, and heads the tensor-core kernel does not take), the
// residual step behind a sublayer (norms of its output, sum of experts, next input, final norm), and the permutation of
// (token, expert) pairs when a table of token ids names the experts.  Math is fp32; the residual stream is fp32.
#include "common.cuh"

#include <math.h>

namespace js {

JS_DEVICE float hk_ld(const float* p) { return *p; }
JS_DEVICE float hk_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
JS_DEVICE void hk_st(float* p, float v) { *p = v; }
JS_DEVICE void hk_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

struct HybridLaunch {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a;
  HybridLaunch(dim3 grid, dim3 block, cudaStream_t stream, int pdl, size_t smem = 0) {
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
JS_DEVICE float cta_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) s += red[i];
  __syncthreads();
  return s;
}

// ---------------------------------------------------------------- unfused forms
template <typename TW>
__global__ void __launch_bounds__(256) rmsnorm_f32_kernel(const float* x, int ldx, const TW* w, float* out, int W, float eps) {
  __shared__ float red[8];
  const float* xr = x + static_cast<size_t>(blockIdx.x) * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += 256) ss += xr[c] * xr[c];
  const float r = 1.f / sqrtf(cta_sum<256>(ss, red) / W + eps);
  for (int c = threadIdx.x; c < W; c += 256) out[static_cast<size_t>(blockIdx.x) * W + c] = xr[c] * r * hk_ld(w + c);
}

// One head vector per warp: rotate the pairs (2i, 2i+1) of the first `dims` entries, optionally divide by the root mean
// square, store `width` entries (zeros past D).  Lane l holds the pairs l, l + 32, ...
template <typename E, typename EB>
JS_DEVICE void head_rotate_norm(const E* src, const EB* bias, E* dst, int D, int width, int dims, const float* freq, float pos,
                                bool norm, float eps, float factor = 1.f) {
  constexpr int NP = 8;                // up to 512 entries
  const int lane = threadIdx.x & 31;
  float a[NP], b[NP], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int e = 2 * (lane + 32 * i);
    a[i] = b[i] = 0.f;
    if (e < D) a[i] = hk_ld(src + e) + (bias != nullptr ? hk_ld(bias + e) : 0.f);
    if (e + 1 < D) b[i] = hk_ld(src + e + 1) + (bias != nullptr ? hk_ld(bias + e + 1) : 0.f);
    if (e + 1 < dims) {
      float sn, cs;
      sincosf(pos * freq[e >> 1], &sn, &cs);
      const float u = a[i], v = b[i];
      a[i] = u * cs - v * sn;
      b[i] = v * cs + u * sn;
    }
    ss += a[i] * a[i] + b[i] * b[i];
  }
  const float r = (norm ? 1.f / sqrtf(warp_sum(ss) / D + eps) : 1.f) * factor;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int e = 2 * (lane + 32 * i);
    if (e < width) hk_st(dst + e, a[i] * r);
    if (e + 1 < width) hk_st(dst + e + 1, b[i] * r);
  }
}

template <typename E>
__global__ void __launch_bounds__(256)
rotate_norm_kernel(const E* x, E* out, const int* positions, int T, int heads, int D, int dims, const float* freq, int norm, float eps) {
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (u >= T * heads) return;
  head_rotate_norm<E, E>(x + static_cast<size_t>(u) * D, nullptr, out + static_cast<size_t>(u) * D, D, D, dims, freq,
                         static_cast<float>(positions[u / heads]), norm != 0, eps);
}

// ---------------------------------------------------------------- fused: biases, rotation, norm, temperature, cache scatter
// proj (T, ldp): [q heads | k heads | v heads]; q goes to qout (T, G, Gp, maps, Dq) (each group of H/G heads padded to Gp heads,
// which stay zero), k and v to their pool rows (G, S, Dp) and (G, S, Vp), the keys of a head's maps side by side.  Values come
// from column vcol of proj on (the keys' own column: they are the keys as projected).  Without kv there are queries only.
struct WindowPostParams {
  const __nv_bfloat16* proj;
  const float *bias, *freq;
  const int *positions, *slots;
  __nv_bfloat16 *qout, *kpool, *vpool;
  int* status;
  int ldp, H, G, Gp, maps, D, V, Dq, Dp, Vp, dims, norm, S, vcol, kv, temp_every;
  float eps, temp_coef;
};

__global__ void __launch_bounds__(256) window_post_kernel(WindowPostParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, u = blockIdx.y * 8 + (threadIdx.x >> 5);
  const int nq = p.H * p.maps, nk = p.kv ? p.G * p.maps : 0, nv = p.kv ? p.G : 0;
  if (u >= nq + nk + nv) return;
  const __nv_bfloat16* row = p.proj + static_cast<size_t>(t) * p.ldp;
  const int ipos = p.positions[t];
  const float pos = static_cast<float>(ipos);
  if (u < nq) {
    const int h = u / p.maps, group = p.H / p.G, hp = (h / group) * p.Gp + h % group;
    const float f = p.temp_every > 0 ? 1.f + p.temp_coef * logf(static_cast<float>((ipos + 1) / p.temp_every + 1)) : 1.f;
    head_rotate_norm<__nv_bfloat16, float>(row + u * p.D, p.bias != nullptr ? p.bias + u * p.D : nullptr,
                                           p.qout + ((static_cast<size_t>(t) * p.G * p.Gp + hp) * p.maps + u % p.maps) * p.Dq, p.D, p.Dq, p.dims,
                                           p.freq, pos, p.norm != 0, p.eps, f);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0 || slot >= p.S) {
    if (lane == 0) report(p.status, kBadSlot);
    return;
  }
  if (u < nq + nk) {
    const int c = u * p.D, i = u - nq, share = p.Dp / p.maps;
    head_rotate_norm<__nv_bfloat16, float>(row + c, p.bias != nullptr ? p.bias + c : nullptr,
                                           p.kpool + (static_cast<size_t>(i / p.maps) * p.S + slot) * p.Dp + (i % p.maps) * share, p.D, share, p.dims,
                                           p.freq, pos, p.norm != 0, p.eps);
    return;
  }
  const int g = u - nq - nk, c = p.vcol + g * p.V;
  __nv_bfloat16* dst = p.vpool + (static_cast<size_t>(g) * p.S + slot) * p.Vp;
  for (int d = lane; d < p.Vp; d += 32)
    dst[d] = __float2bfloat16_rn(d < p.V ? __bfloat162float(row[c + d]) + (p.bias != nullptr ? p.bias[c + d] : 0.f) : 0.f);
}

// The same without rotation, 8 entries a thread: 2^lp neighbouring lanes make a head vector, 2^lpv a value row.  With tied values
// the key's lanes store the value row too.  D, V, the widths, ldp and vcol multiples of 8.
__global__ void __launch_bounds__(256) window_post_vec_kernel(WindowPostParams p, int lp, int lpv, int tied) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, idx = blockIdx.y * 256 + threadIdx.x;
  const int nq = p.H * p.maps, nk = p.kv ? p.G * p.maps : 0, nv = p.kv && !tied ? p.G : 0;
  const int vectors = (nq + nk) << lp, share = p.Dp / p.maps;
  const __nv_bfloat16* row = p.proj + static_cast<size_t>(t) * p.ldp;
  const bool head = idx < vectors, value = !head && idx - vectors < nv << lpv;
  const int u = head ? idx >> lp : (idx - vectors) >> lpv;
  const int e = 8 * (head ? idx & ((1 << lp) - 1) : (idx - vectors) & ((1 << lpv) - 1));
  const int col = (head ? u * p.D : p.vcol + u * p.V) + e;
  float v[8] = {}, ss = 0.f;
  if ((head || value) && e < (head ? p.D : p.V)) {
    const uint4 raw = *reinterpret_cast<const uint4*>(row + col);
    const __nv_bfloat162* r2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(r2[j]);
      v[2 * j] = f.x;
      v[2 * j + 1] = f.y;
    }
    if (p.bias != nullptr) {
      const float4 a = *reinterpret_cast<const float4*>(p.bias + col), b = *reinterpret_cast<const float4*>(p.bias + col + 4);
      v[0] += a.x; v[1] += a.y; v[2] += a.z; v[3] += a.w;
      v[4] += b.x; v[5] += b.y; v[6] += b.z; v[7] += b.w;
    }
  }
  auto store = [&](__nv_bfloat16* dst, float f) {
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int j = 0; j < 4; ++j) o2[j] = __floats2bfloat162_rn(v[2 * j] * f, v[2 * j + 1] * f);
    *reinterpret_cast<uint4*>(dst) = out;
  };
  float f = 1.f;
  if (p.norm) {                              // every lane takes part
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
    for (int o = 1; o < 1 << lp; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    f = 1.f / sqrtf(ss / p.D + p.eps);
  }
  if (!head && !value) return;
  if (head && u < nq) {
    if (e >= p.Dq) return;
    if (p.temp_every > 0) f *= 1.f + p.temp_coef * logf(static_cast<float>((p.positions[t] + 1) / p.temp_every + 1));
    const int h = u / p.maps, group = p.H / p.G, hp = (h / group) * p.Gp + h % group;
    store(p.qout + ((static_cast<size_t>(t) * p.G * p.Gp + hp) * p.maps + u % p.maps) * p.Dq + e, f);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0 || slot >= p.S) {
    if (e == 0) report(p.status, kBadSlot);
    return;
  }
  if (head) {
    const int i = u - nq;
    if (e < share) store(p.kpool + (static_cast<size_t>(i / p.maps) * p.S + slot) * p.Dp + (i % p.maps) * share + e, f);
    if (tied && e < p.Vp) store(p.vpool + (static_cast<size_t>(i) * p.S + slot) * p.Vp + e, 1.f);
  } else if (e < p.Vp) {
    store(p.vpool + (static_cast<size_t>(u) * p.S + slot) * p.Vp + e, 1.f);
  }
}

// ---------------------------------------------------------------- pooled blocks
// Means of the cached keys and values of the blocks of P tokens whose last token is among the new ones.  One CTA per (block, head).
// New tokens of sequence b: positions past .. past + n - 1 with n = cu[b + 1] - cu[b]; with counts instead n = counts[b] positions
// that END at past (per_seq blocks are looked at then).
struct PoolBlocks {
  const void *kp, *vp;
  void *kb, *vb;
  const int *block_map, *slot_map, *seq_rows, *cu_q, *past_lens, *counts;
  int* status;
  int S, rows, Kw, Vw, max_blocks, P, max_len, per_seq, B;
};

// Row of the block candidate c stands for, and where its tokens' slots are; false: no such block.
JS_DEVICE bool block_of(const PoolBlocks& p, int c, int& dst, const int*& slots) {
  int b, j, past, n;
  if (p.counts != nullptr) {
    b = c / p.per_seq;
    j = c % p.per_seq;
    n = p.counts[b];
    past = p.past_lens[b] - n;
  } else {
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu_q[mid] / p.P + mid <= c) lo = mid; else hi = mid - 1;
    }
    b = lo;
    j = c - (p.cu_q[b] / p.P + b);
    n = p.cu_q[b + 1] - p.cu_q[b];
    past = p.past_lens[b];
  }
  const int blk = past / p.P + j;
  if (blk >= (past + n) / p.P) return false;
  const int row = p.seq_rows[b];
  dst = blk < p.max_blocks ? p.block_map[static_cast<size_t>(row) * p.max_blocks + blk] : -1;
  if (dst < 0 || dst >= p.rows) {
    if (threadIdx.x == 0) report(p.status, kBadSlot);
    return false;
  }
  slots = p.slot_map + static_cast<size_t>(row) * p.max_len + static_cast<size_t>(blk) * p.P;
  return true;
}

template <typename E>
__global__ void __launch_bounds__(128) pool_blocks_kernel(PoolBlocks p) {
  pdl_launch_dependents();
  pdl_wait();
  const int g = blockIdx.y;
  int dst;
  const int* slots;
  if (!block_of(p, blockIdx.x, dst, slots)) return;
  const float inv = 1.f / p.P;
  for (int e = threadIdx.x; e < p.Kw + p.Vw; e += blockDim.x) {
    const bool k = e < p.Kw;
    const int w = k ? p.Kw : p.Vw, col = k ? e : e - p.Kw;
    const E* src = reinterpret_cast<const E*>(k ? p.kp : p.vp) + static_cast<size_t>(g) * p.S * w + col;
    float acc = 0.f;
#pragma unroll 4
    for (int i = 0; i < p.P; ++i) {
      const int slot = slots[i];
      if (slot >= 0 && slot < p.S) acc += hk_ld(src + static_cast<size_t>(slot) * w);
      else report(p.status, kBadSlot);
    }
    hk_st(reinterpret_cast<E*>(k ? p.kb : p.vb) + (static_cast<size_t>(g) * p.rows + dst) * w + col, acc * inv);
  }
}

// bf16 rows of Kw + Vw <= 256 columns, multiples of 8: 8 warps take every eighth token each, a lane 8 columns
__global__ void __launch_bounds__(256) pool_blocks_vec_kernel(PoolBlocks p) {
  __shared__ float part[8][256];
  pdl_launch_dependents();
  pdl_wait();
  const int g = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int dst;
  const int* slots;
  if (!block_of(p, blockIdx.x, dst, slots)) return;
  const int e = lane * 8, all = p.Kw + p.Vw;
  const bool k = e < p.Kw;
  const int w = k ? p.Kw : p.Vw, col = k ? e : e - p.Kw;
  const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(k ? p.kp : p.vp) + static_cast<size_t>(g) * p.S * w + col;
  float acc[8] = {};
  if (e < all) {
#pragma unroll 4
    for (int i = warp; i < p.P; i += 8) {
      int slot = slots[i];
      if (slot < 0 || slot >= p.S) { report(p.status, kBadSlot); slot = 0; }
      const uint4 raw = *reinterpret_cast<const uint4*>(src + static_cast<size_t>(slot) * w);
      const __nv_bfloat162* r2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(r2[j]);
        acc[2 * j] += f.x;
        acc[2 * j + 1] += f.y;
      }
    }
    *reinterpret_cast<float4*>(&part[warp][e]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    *reinterpret_cast<float4*>(&part[warp][e + 4]) = make_float4(acc[4], acc[5], acc[6], acc[7]);
  }
  __syncthreads();
  const int c = threadIdx.x;
  if (c >= all) return;
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) sum += part[i][c];
  const bool ck = c < p.Kw;
  reinterpret_cast<__nv_bfloat16*>(ck ? p.kb : p.vb)[(static_cast<size_t>(g) * p.rows + dst) * (ck ? p.Kw : p.Vw) + (ck ? c : c - p.Kw)] =
      __float2bfloat16_rn(sum / p.P);
}

// ---------------------------------------------------------------- window attention on the plain cores
// One CTA per (token, head); four warps take every fourth visible key each and merge at the end.  The row sees the last
// `window` tokens of its own path (0: all) and the positions below `keep`; the sink is a key without a value whose score is sinks[h]
// (or 0).  With `gate` (T, ldg) the head's output is multiplied by the sigmoid of its logit.  softcap > 0 caps the scores.
// Pooled blocks of P positions that end before the window are keys too, read from their rows or, where they reach into a token
// tree, averaged over the row's path.  MAPS = 2: two queries a head against the two halves of a key row, outputs combined to
// share * (o1 - lam o2) / rms over Vn columns (the rest of V is padding).
struct WindowSimt {
  const void *q, *kpool, *vpool, *kblocks, *vblocks;
  void* out;
  const int *slot_map, *seq_rows, *cu_q, *past_lens, *mask_bits, *block_map;
  const float *sinks, *gate, *lam;
  int* status;
  long long q_tok;
  int Dp, Vp, ldo, B, H, G, D, V, S, max_len, W, causal, window, sink, keep, ldg, P, block_rows, max_blocks, Vn;
  float scale, softcap, share, eps;
};

template <typename E, int NPL, int MAPS>
__global__ void __launch_bounds__(128) window_attn_simt_kernel(WindowSimt p) {
  pdl_launch_dependents();
  pdl_wait();
  const E *kpool = reinterpret_cast<const E*>(p.kpool), *vpool = reinterpret_cast<const E*>(p.vpool);
  const int t = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G), D = p.D, V = p.V, W = p.W;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kmap = p.Dp / MAPS;
  int lo = 0, hi = p.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const bool causal = p.causal != 0;
  const int i = t - p.cu_q[lo], past = p.past_lens[lo], n_b = p.cu_q[lo + 1] - p.cu_q[lo];
  const int* slots = p.slot_map + static_cast<size_t>(p.seq_rows[lo]) * p.max_len;
  const int* bits = causal ? nullptr : p.mask_bits + static_cast<size_t>(t) * W;
  int pos = past + i;
  if (!causal) {
    int cnt = 0;
    for (int w = 0; w < W; ++w) cnt += __popc(static_cast<unsigned>(bits[w]));
    pos = past + cnt - 1;
  }
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int last = causal ? past + i : past + n_b - 1;
  float qv[MAPS][NPL], acc[MAPS][NPL], m[MAPS], l[MAPS];
#pragma unroll
  for (int u = 0; u < MAPS; ++u) {
#pragma unroll
    for (int e = 0; e < NPL; ++e) {
      const int c = lane + 32 * e;
      qv[u][e] = c < D ? hk_ld(reinterpret_cast<const E*>(p.q) + t * p.q_tok + static_cast<size_t>(h * MAPS + u) * D + c) * p.scale : 0.f;
      acc[u][e] = 0.f;
    }
    m[u] = -INFINITY;
    l[u] = 0.f;
    if (p.sink && warp == 0) { m[u] = p.sinks != nullptr ? p.sinks[h] : 0.f; l[u] = 1.f; }
  }
  auto dot = [&](const E* kr, int u) {
    float d = 0.f;
#pragma unroll
    for (int e = 0; e < NPL; ++e) {
      const int c = lane + 32 * e;
      if (c < D) d += qv[u][e] * hk_ld(kr + u * kmap + c);
    }
    return warp_sum(d);
  };
  // one more key of score d (map u) and value v(c)
  auto add = [&](float d, int u, auto v) {
    if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
    const float mn = fmaxf(m[u], d), a = expf(m[u] - mn), w = expf(d - mn);
    l[u] = l[u] * a + w;
#pragma unroll
    for (int e = 0; e < NPL; ++e) {
      const int c = lane + 32 * e;
      acc[u][e] = acc[u][e] * a + (c < V ? w * v(c) : 0.f);
    }
    m[u] = mn;
  };
  auto slot_of = [&](int j) {
    int slot = slots[j];
    if (slot < 0 || slot >= p.S) { if (lane == 0) report(p.status, kBadSlot); slot = 0; }
    return static_cast<size_t>(slot);
  };
  const int first_j = causal ? first : min(first, past), kept = min(p.keep, first_j);      // two ranges: [0, kept) and [first_j, last]
  for (int x = warp; x < kept + last - first_j + 1; x += 4) {
    const int j = x < kept ? x : first_j + x - kept;
    if (j < past) {
      if (j < first && j >= p.keep) continue;
    } else if (!causal) {
      const int n = j - past;
      if (!((bits[n >> 5] >> (n & 31)) & 1)) continue;
      int depth = 0;                       // proper ancestors of node n, which are those of this row below n
      for (int w = 0; w < (n >> 5); ++w) depth += __popc(static_cast<unsigned>(bits[w]));
      depth += __popc(static_cast<unsigned>(bits[n >> 5]) & ((1u << (n & 31)) - 1u));
      if (past + depth < first && past + depth >= p.keep) continue;
    }
    const size_t slot = slot_of(j);
    const E* kr = kpool + (static_cast<size_t>(g) * p.S + slot) * p.Dp;
    const E* vr = vpool + (static_cast<size_t>(g) * p.S + slot) * p.Vp;
#pragma unroll
    for (int u = 0; u < MAPS; ++u) add(dot(kr, u), u, [&](int c) { return hk_ld(vr + c); });
  }
  if (p.P > 0) {
    const int blocks = pos - p.window >= 0 ? (pos - p.window + 1) / p.P : 0, stored = causal ? blocks : past / p.P;
    // slot of position j of this row's own path
    auto path_slot = [&](int j) {
      if (j < past) return slot_of(j);
      int left = j - past, w = 0;
      while (w < W && left >= __popc(static_cast<unsigned>(bits[w]))) left -= __popc(static_cast<unsigned>(bits[w++]));
      if (w >= W) { if (lane == 0) report(p.status, kBadNode); return slot_of(past); }
      unsigned word = static_cast<unsigned>(bits[w]);
      for (; left > 0; --left) word &= word - 1u;
      return slot_of(past + 32 * w + __ffs(static_cast<int>(word)) - 1);
    };
    for (int b = warp; b < blocks; b += 4) {
      if (b < stored) {
        int r = b < p.max_blocks ? p.block_map[static_cast<size_t>(p.seq_rows[lo]) * p.max_blocks + b] : -1;
        if (r < 0 || r >= p.block_rows) { if (lane == 0) report(p.status, kBadSlot); r = 0; }
        const E* kr = reinterpret_cast<const E*>(p.kblocks) + (static_cast<size_t>(g) * p.block_rows + r) * p.Dp;
        const E* vr = reinterpret_cast<const E*>(p.vblocks) + (static_cast<size_t>(g) * p.block_rows + r) * p.Vp;
#pragma unroll
        for (int u = 0; u < MAPS; ++u) add(dot(kr, u), u, [&](int c) { return hk_ld(vr + c); });
        continue;
      }
      const float inv = 1.f / p.P;
      float d[MAPS] = {}, mean[NPL] = {};
      for (int j = b * p.P; j < (b + 1) * p.P; ++j) {
        const size_t slot = path_slot(j);
#pragma unroll
        for (int u = 0; u < MAPS; ++u) d[u] += dot(kpool + (static_cast<size_t>(g) * p.S + slot) * p.Dp, u);
#pragma unroll
        for (int e = 0; e < NPL; ++e)
          if (lane + 32 * e < V) mean[e] += hk_ld(vpool + (static_cast<size_t>(g) * p.S + slot) * p.Vp + lane + 32 * e);
      }
#pragma unroll
      for (int u = 0; u < MAPS; ++u) add(d[u] * inv, u, [&](int c) { return mean[(c - lane) / 32] * inv; });
    }
  }
  __shared__ float sm[MAPS][4], sl[MAPS][4], red[4];
  extern __shared__ float so[];            // MAPS x 4 x V
#pragma unroll
  for (int u = 0; u < MAPS; ++u) {
    if (lane == 0) { sm[u][warp] = m[u]; sl[u][warp] = l[u]; }
#pragma unroll
    for (int e = 0; e < NPL; ++e)
      if (lane + 32 * e < V) so[(u * 4 + warp) * V + lane + 32 * e] = acc[u][e];
  }
  __syncthreads();
  float f[MAPS][4];
#pragma unroll
  for (int u = 0; u < MAPS; ++u) {
    const float mm = fmaxf(fmaxf(sm[u][0], sm[u][1]), fmaxf(sm[u][2], sm[u][3]));
    float tot = 0.f;
#pragma unroll
    for (int w2 = 0; w2 < 4; ++w2) {
      f[u][w2] = sm[u][w2] == -INFINITY ? 0.f : expf(sm[u][w2] - mm);
      tot += sl[u][w2] * f[u][w2];
    }
    const float inv = tot > 0.f ? 1.f / tot : 0.f;
#pragma unroll
    for (int w2 = 0; w2 < 4; ++w2) f[u][w2] *= inv;
  }
  auto read = [&](int u, int c) {
    const float* o = so + u * 4 * V + c;
    return o[0] * f[u][0] + o[V] * f[u][1] + o[2 * V] * f[u][2] + o[3 * V] * f[u][3];
  };
  E* out = reinterpret_cast<E*>(p.out) + static_cast<size_t>(t) * p.ldo + h * V;
  if constexpr (MAPS == 1) {
    const float gate = p.gate != nullptr ? 1.f / (1.f + expf(-p.gate[static_cast<size_t>(t) * p.ldg + h])) : 1.f;
    for (int c = threadIdx.x; c < V; c += blockDim.x) hk_st(out + c, read(0, c) * gate);
  } else {
    const float lam = *p.lam;
    float o[(NPL + 3) / 4], ss = 0.f;      // a thread's columns: threadIdx.x, + 128, ...
#pragma unroll
    for (int e = 0; e < (NPL + 3) / 4; ++e) {
      const int c = threadIdx.x + 128 * e;
      o[e] = c < V ? read(0, c) - lam * read(1, c) : 0.f;
      ss += o[e] * o[e];
    }
    const float r = p.share / sqrtf(cta_sum<128>(ss, red) / p.Vn + p.eps);
#pragma unroll
    for (int e = 0; e < (NPL + 3) / 4; ++e) {
      const int c = threadIdx.x + 128 * e;
      if (c < V) hk_st(out + c, o[e] * r);
    }
  }
}

template <typename E, int MAPS>
static int launch_window_simt(const WindowSimt& p, int T, int pdl, cudaStream_t stream) {
  HybridLaunch l(dim3(T, p.H), dim3(128), stream, pdl, MAPS * 4 * p.V * sizeof(float));
  const int n = p.D > p.V ? p.D : p.V;
  auto kern = n <= 64 ? window_attn_simt_kernel<E, 2, MAPS> : n <= 128 ? window_attn_simt_kernel<E, 4, MAPS>
            : n <= 256 ? window_attn_simt_kernel<E, 8, MAPS> : window_attn_simt_kernel<E, 16, MAPS>;
  return cudaLaunchKernelEx(&l.c, kern, p) == cudaSuccess ? 0 : -4;
}

// ---------------------------------------------------------------- the residual step behind a sublayer
// y = one of
//   pair    0.5 (a / rms(a) * wa + b / rms(b) * wb),  a = ya + bias
//   single  ya + bias
//   experts (sum_j ys[inv[t k + j]]) / k + sh
// then x += y / rms(y) * w.  h = bf16(x), or with fw (the model's last norm) h = bf16(x / rms(x) * fw) and tap = bf16(x).
struct ResidParams {
  const __nv_bfloat16 *ya, *yb;
  const float *bias, *wa, *wb;
  int lda, ldb;
  const __nv_bfloat16 *ys, *sh;
  const int* inv;
  int ldy, lds, k;
  const float *w, *fw;
  float eps;
  float* x;
  __nv_bfloat16 *h, *tap;
  int ld, ldt, W;
};

constexpr int kResidThreads = 512;      // few rows (decode) want many threads a row

__global__ void __launch_bounds__(kResidThreads) resid_norm_kernel(ResidParams p) {
  extern __shared__ float ry[];            // W
  __shared__ float red[kResidThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, W = p.W, tid = threadIdx.x;
  float ss = 0.f;
  if (p.ya == nullptr) {
    const float wt = p.k > 0 ? 1.f / p.k : 0.f;
    for (int c = tid * 4; c < W; c += kResidThreads * 4) {        // rows are padded to multiples of 4
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      auto add = [&](const __nv_bfloat16* row) {
        const uint2 raw = *reinterpret_cast<const uint2*>(row + c);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        acc[0] += lo.x; acc[1] += lo.y; acc[2] += hi.x; acc[3] += hi.y;
      };
#pragma unroll 4
      for (int j = 0; j < p.k; ++j) add(p.ys + static_cast<size_t>(p.inv[t * p.k + j]) * p.ldy);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] *= wt;
      if (p.sh != nullptr) add(p.sh + static_cast<size_t>(t) * p.lds);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < W) { ry[c + e] = acc[e]; ss += acc[e] * acc[e]; }
    }
  } else {
    const __nv_bfloat16* a = p.ya + static_cast<size_t>(t) * p.lda;
    const __nv_bfloat16* b = p.yb != nullptr ? p.yb + static_cast<size_t>(t) * p.ldb : nullptr;
    auto load_a = [&](int c) {             // rows are padded to even length
      float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(a + c));
      if (p.bias != nullptr) { v.x += p.bias[c]; v.y += c + 1 < W ? p.bias[c + 1] : 0.f; }
      if (c + 1 >= W) v.y = 0.f;
      return v;
    };
    auto put = [&](int c, float2 v) {
      ry[c] = v.x;
      if (c + 1 < W) ry[c + 1] = v.y;
    };
    if (b != nullptr) {
      float sa = 0.f, sb = 0.f;
      for (int c = tid * 2; c < W; c += kResidThreads * 2) {
        const float2 v = load_a(c);
        put(c, v);
        sa += v.x * v.x + v.y * v.y;
        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(b + c));
        sb += u.x * u.x + (c + 1 < W ? u.y * u.y : 0.f);
      }
      const float ra = 0.5f / sqrtf(cta_sum<kResidThreads>(sa, red) / W + p.eps);
      const float rb = 0.5f / sqrtf(cta_sum<kResidThreads>(sb, red) / W + p.eps);
      for (int c = tid * 2; c < W; c += kResidThreads * 2) {
        const bool two = c + 1 < W;
        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(b + c));
        const float2 v = make_float2(ry[c] * ra * p.wa[c] + u.x * rb * p.wb[c],
                                     two ? ry[c + 1] * ra * p.wa[c + 1] + u.y * rb * p.wb[c + 1] : 0.f);
        put(c, v);
        ss += v.x * v.x + v.y * v.y;
      }
    } else {
      for (int c = tid * 2; c < W; c += kResidThreads * 2) {
        const float2 v = load_a(c);
        put(c, v);
        ss += v.x * v.x + v.y * v.y;
      }
    }
  }
  const float r = 1.f / sqrtf(cta_sum<kResidThreads>(ss, red) / W + p.eps);     // its barriers also publish ry
  float* x = p.x + static_cast<size_t>(t) * p.ld;
  __nv_bfloat16* h = p.h + static_cast<size_t>(t) * p.ld;
  ss = 0.f;
  for (int c = tid; c < W; c += kResidThreads) {
    const float v = x[c] + ry[c] * r * p.w[c];
    x[c] = v;
    if (p.tap != nullptr) p.tap[static_cast<size_t>(t) * p.ldt + c] = __float2bfloat16_rn(v);
    if (p.fw == nullptr) h[c] = __float2bfloat16_rn(v);
    else { ry[c] = v; ss += v * v; }
  }
  if (p.fw == nullptr) return;
  const float rf = 1.f / sqrtf(cta_sum<kResidThreads>(ss, red) / W + p.eps);
  for (int c = tid; c < W; c += kResidThreads) h[c] = __float2bfloat16_rn(ry[c] * rf * p.fw[c]);
}

// x[t] = table[ids[t]] in fp32, h[t] the same in bf16
__global__ void __launch_bounds__(256)
embed_f32_kernel(const int* ids, const __nv_bfloat16* table, int V, int ldt, float* x, __nv_bfloat16* h, int ld, int W) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const __nv_bfloat16 v = table[static_cast<size_t>(id) * ldt + c];
    x[static_cast<size_t>(t) * ld + c] = __bfloat162float(v);
    h[static_cast<size_t>(t) * ld + c] = v;
  }
}

// ---------------------------------------------------------------- permutation of table-routed pairs
// One CTA per (layer, pass): pairs (token, choice) of rows [t0, t0 + n) sorted by expert, stably.  All layers' permutations
// depend on the token ids alone, so one launch at the start of a forward makes them all.
struct TableLayer {
  const int* table;      // (V, top)
  int top, E;
  int off_tok;           // where this layer's outputs start in `out`: per pass [tok | inv | group offsets]
};

constexpr int kTableWarps = 32;

__global__ void __launch_bounds__(32 * kTableWarps)
table_sort_kernel(const TableLayer* layers, const int* ids, int T, int rows_per_pass, int V, int* out) {
  extern __shared__ int sh[];
  __shared__ int warp_tot[kTableWarps];
  pdl_launch_dependents();
  pdl_wait();
  const TableLayer L = layers[blockIdx.x];
  const int t0 = blockIdx.y * rows_per_pass;
  const int n = min(rows_per_pass, T - t0);
  if (n <= 0) return;
  const int P = n * L.top, E = L.E, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int* cnt = sh;                 // (warps, E): pairs of the warp's chunk per expert, then where the warp's next one goes
  unsigned short* key = reinterpret_cast<unsigned short*>(sh + kTableWarps * E);      // P
  int* tok = out + L.off_tok + static_cast<size_t>(t0) * 2 * L.top + static_cast<size_t>(blockIdx.y) * (E + 1);
  int* inv = tok + P;
  int* goff = inv + P;
  for (int i = tid; i < kTableWarps * E; i += blockDim.x) cnt[i] = 0;
  __syncthreads();
  // every warp takes a consecutive chunk of the pairs, so that the order within an expert is the pairs' own
  const int chunk = ((P + kTableWarps - 1) / kTableWarps + 31) / 32 * 32;
  const int p0 = warp * chunk, p1 = min(P, p0 + chunk);
  int* mine = cnt + warp * E;
  for (int p = p0 + lane; p < p1; p += 32) {
    int id = ids[t0 + p / L.top];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    const int e = L.table[static_cast<size_t>(id) * L.top + p % L.top];
    key[p] = static_cast<unsigned short>(e);
    atomicAdd(&mine[e], 1);
  }
  __syncthreads();
  // exclusive scan over (expert, warp): thread e owns expert e (E <= 1024)
  int total = 0;
  if (tid < E)
    for (int w = 0; w < kTableWarps; ++w) total += cnt[w * E + tid];
  int inc = total;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += v;
  }
  if (lane == 31) warp_tot[warp] = inc;
  __syncthreads();
  int base = inc - total;
  for (int w = 0; w < warp; ++w) base += warp_tot[w];
  if (tid < E) {
    goff[tid] = base;
    for (int w = 0; w < kTableWarps; ++w) {
      const int c = cnt[w * E + tid];
      cnt[w * E + tid] = base;
      base += c;
    }
  }
  if (tid == 0) goff[E] = P;
  __syncthreads();
  for (int pb = p0; pb < p1; pb += 32) {
    const int p = pb + lane;
    const int e = p < p1 ? key[p] : -1;
    const unsigned same = __match_any_sync(0xffffffffu, e);
    const int rank = __popc(same & ((1u << lane) - 1u));
    const int at = e >= 0 ? mine[e] + rank : 0;
    __syncwarp();
    if (e >= 0) {
      tok[at] = t0 + p / L.top;
      inv[p] = at;
      if (rank == 0) mine[e] += __popc(same);
    }
    __syncwarp();
  }
}

}  // namespace js

extern "C" int js_rmsnorm_f32(const float* x, int ldx, const void* w, int w_bf16, float* out, int T, int W, float eps, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (w_bf16) rmsnorm_f32_kernel<__nv_bfloat16><<<T, 256, 0, stream>>>(x, ldx, (const __nv_bfloat16*)w, out, W, eps);
  else rmsnorm_f32_kernel<float><<<T, 256, 0, stream>>>(x, ldx, (const float*)w, out, W, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// x, out (T, heads, D) contiguous; D at most 512, freq (dims / 2) fp32.
extern "C" int js_rotate_norm(const void* x, void* out, const int* positions, int T, int heads, int D, int dims, const float* freq,
                              int norm, float eps, int bf16, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (D > 512 || dims > D || (dims & 1)) return -10;
  const int g = (T * heads + 7) / 8;
  if (bf16) rotate_norm_kernel<__nv_bfloat16><<<g, 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)out, positions, T, heads, D, dims, freq, norm, eps);
  else rotate_norm_kernel<float><<<g, 256, 0, stream>>>((const float*)x, (float*)out, positions, T, heads, D, dims, freq, norm, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// See window_post_kernel.
extern "C" int js_window_post(const void* proj, int ldp, const float* bias, int H, int G, int Gp, int maps, int D, int V, int Dq, int Dp, int Vp,
                              int dims, const float* freq, int norm, float eps, int temp_every, float temp_coef, int vcol, int kv,
                              const int* positions, const int* slots, int S, int T, void* qout, void* kpool, void* vpool, int* status,
                              int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (maps < 1 || H % G || Dp > 512 * maps || Dp % maps || Dq > 512 || D > Dq || D > Dp / maps || V > Vp || dims > D || (dims & 1) || Gp < H / G) return -10;
  using bf = __nv_bfloat16;
  WindowPostParams p{(const bf*)proj, bias, freq, positions, slots, (bf*)qout, (bf*)kpool, (bf*)vpool, status,
                     ldp, H, G, Gp, maps, D, V, Dq, Dp, Vp, dims, norm, S, vcol, kv, temp_every, eps, temp_coef};
  const int share = Dp / maps, wide = Dq > share ? Dq : share;
  const bool tied = kv && maps == 1 && vcol == H * D && V == D && Vp <= wide;
  if (dims == 0 && ((D | V | Dq | share | Vp | ldp | vcol) & 7) == 0 && wide <= 256 && Vp <= 256 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0 &&
      (reinterpret_cast<uintptr_t>(bias) & 15) == 0) {
    int lp = 0, lpv = 0;
    while (8 << lp < wide) ++lp;
    while (8 << lpv < Vp) ++lpv;
    const int n = ((H * maps + (kv ? G * maps : 0)) << lp) + (kv && !tied ? G << lpv : 0);
    HybridLaunch l(dim3(T, (n + 255) / 256), dim3(256), stream, pdl);
    return cudaLaunchKernelEx(&l.c, window_post_vec_kernel, p, lp, lpv, static_cast<int>(tied)) == cudaSuccess ? 0 : -4;
  }
  HybridLaunch l(dim3(T, (H * maps + (kv ? G * (maps + 1) : 0) + 7) / 8), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, window_post_kernel, p) == cudaSuccess ? 0 : -4;
}

// Pools (G, S, Kw) and (G, S, Vw), block rows (G, rows, Kw) and (G, rows, Vw); see pool_blocks_kernel.  T bounds the new tokens of
// all sequences; with counts, per_seq bounds a sequence's blocks.
extern "C" int js_pool_blocks(const void* kp, const void* vp, void* kb, void* vb, int G, int S, int rows, int Kw, int Vw, const int* block_map,
                              int max_blocks, int P, const int* slot_map, int max_len, const int* seq_rows, const int* cu_q,
                              const int* past_lens, const int* counts, int per_seq, int B, int T, int bf16, int* status, int pdl,
                              cudaStream_t stream) {
  using namespace js;
  if (B <= 0 || (counts == nullptr && T <= 0)) return 0;
  if (P < 1 || G < 1 || (counts == nullptr ? cu_q == nullptr : per_seq < 1)) return -10;
  PoolBlocks p{kp, vp, kb, vb, block_map, slot_map, seq_rows, cu_q, past_lens, counts, status, S, rows, Kw, Vw, max_blocks, P, max_len, per_seq, B};
  const bool vec = bf16 && Kw % 8 == 0 && Vw % 8 == 0 && Kw + Vw <= 256;
  HybridLaunch l(dim3(counts != nullptr ? B * per_seq : T / P + B, G), dim3(vec ? 256 : 128), stream, pdl);
  auto kern = vec ? pool_blocks_vec_kernel : bf16 ? pool_blocks_kernel<__nv_bfloat16> : pool_blocks_kernel<float>;
  return cudaLaunchKernelEx(&l.c, kern, p) == cudaSuccess ? 0 : -4;
}

// q: token t at t * q_tok, head h (map m) at (h * maps + m) * D; pools (G, S, Dp) and (G, S, Vp); out (T, ldo), head h at h * V.
// D, V at most 512.  sink: a valueless key of score sinks[h] (null: 0) takes part; keep: positions below it stay visible behind the
// window (0: no window); gate (T, ldg) fp32 logits or null; softcap 0: none; P > 0: pooled blocks in kb (G, block_rows, Dp), vb
// (G, block_rows, Vp) through block_map (rows, max_blocks); maps 2 combines with lam (device), share and eps, normed over the first Vn of V columns (the rest being zero).
extern "C" int js_window_attention_simt(const void* q, long long q_tok, const void* kp, const void* vp, int Dp, int Vp, const int* slot_map,
                                        const int* seq_rows, const int* cu_q, const int* past_lens, const int* mask_bits, void* out,
                                        int ldo, int B, int T, int H, int G, int D, int V, int S, int max_len, int W, int causal,
                                        float scale, int window, int sink, int keep, const float* sinks, const float* gate, int ldg,
                                        float softcap, int P, const void* kb, const void* vb, int block_rows, const int* block_map,
                                        int max_blocks, int maps, const float* lam, float share, float eps, int Vn, int bf16, int* status, int pdl,
                                        cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || B <= 0) return 0;
  if (maps < 1 || maps > 2 || H % G || D > 512 || V > 512 || Dp % maps || D > Dp / maps || V > Vp || window < 0 || keep < 0 || P < 0) return -10;
  if (!causal && (mask_bits == nullptr || W < 1)) return -13;
  if ((P > 0 && (window < 1 || kb == nullptr || vb == nullptr || block_map == nullptr)) || (maps == 2 && (lam == nullptr || Vn < 1 || Vn > V))) return -13;
  WindowSimt p{q, kp, vp, kb, vb, out, slot_map, seq_rows, cu_q, past_lens, mask_bits, block_map, sinks, gate, lam, status, q_tok,
               Dp, Vp, ldo, B, H, G, D, V, S, max_len, W, causal, window, sink, keep, ldg, P, block_rows, max_blocks, Vn,
               scale, softcap, share, eps};
  if (bf16) return maps == 2 ? launch_window_simt<__nv_bfloat16, 2>(p, T, pdl, stream) : launch_window_simt<__nv_bfloat16, 1>(p, T, pdl, stream);
  return maps == 2 ? launch_window_simt<float, 2>(p, T, pdl, stream) : launch_window_simt<float, 1>(p, T, pdl, stream);
}

// Either ya (with yb, wa, wb for a pair; bias optional) or ys / inv / k and sh, all bf16 rows whose
// length is a multiple of 2 (ys, sh: 4) and >= W.  W at most 24576.
extern "C" int js_resid_norm(const void* ya, int lda, const float* bias, const float* wa, const void* yb, int ldb, const float* wb,
                             const void* ys, int ldy, const int* inv, int k, const void* sh, int lds, const float* w, const float* fw,
                             float eps, float* x, void* h, int ld, void* tap, int ldt, int T, int W, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (W < 1 || W > 24576 || ((lda | ldb) & 1) || ((ldy | lds) & 3)) return -10;
  if (ya == nullptr && ys == nullptr && sh == nullptr) return -13;
  if (yb != nullptr && (wa == nullptr || wb == nullptr)) return -13;
  using bf = __nv_bfloat16;
  ResidParams p{(const bf*)ya, (const bf*)yb, bias, wa, wb, lda, ldb, (const bf*)ys, (const bf*)sh, inv, ldy, lds, ys != nullptr ? k : 0, w, fw, eps, x,
                (bf*)h, (bf*)tap, ld, ldt, W};
  const int smem = W * 4;
  static int configured[kMaxDevicesCached] = {};
  if (smem > 40 * 1024 && ensure_dyn_smem(resid_norm_kernel, smem, configured) != 0) return -3;
  HybridLaunch l(dim3(T), dim3(kResidThreads), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, resid_norm_kernel, p) == cudaSuccess ? 0 : -4;
}

extern "C" int js_embed_f32(const int* ids, const void* table, int V, int ldt, float* x, void* h, int ld, int T, int W, int pdl,
                            cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  HybridLaunch l(dim3(T), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, embed_f32_kernel, ids, (const __nv_bfloat16*)table, V, ldt, x, (__nv_bfloat16*)h, ld, W) == cudaSuccess ? 0 : -4;
}

// layers: n_layers TableLayer records in device memory.  rows_per_pass * max_top at most 16384, max_E at most 1024.
extern "C" int js_table_sort(const void* layers, int n_layers, const int* ids, int T, int rows_per_pass, int V, int max_top, int max_E,
                             int* out, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || n_layers <= 0) return 0;
  if (rows_per_pass < 1 || max_top < 1 || rows_per_pass * max_top > 16384 || max_E < 1 || max_E > 1024) return -10;
  const int rows = T < rows_per_pass ? T : rows_per_pass;
  const int smem = kTableWarps * max_E * 4 + rows * max_top * 2;
  static int configured[kMaxDevicesCached] = {};
  if (ensure_dyn_smem(table_sort_kernel, smem, configured) != 0) return -3;
  HybridLaunch l(dim3(n_layers, (T + rows_per_pass - 1) / rows_per_pass), dim3(32 * kTableWarps), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, table_sort_kernel, (const TableLayer*)layers, ids, T, rows_per_pass, V, out) == cudaSuccess ? 0 : -4;
}
