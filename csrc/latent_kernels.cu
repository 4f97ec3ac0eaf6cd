// Small kernels of latent-attention decoders with Dynamic Tanh norms and sigmoid-routed experts: the steps between the
// tensor-core GEMMs (embedding + first norm, latent norms + cache scatter, routing, combine + next norm) and their
// unfused forms.  Math is fp32 throughout; the residual stream is fp32.  Kernels that the 32-bit path needs as well are
// templates over the element type.
#include "common.cuh"

#include <math.h>

namespace js {

JS_DEVICE float ld_f(const float* p) { return *p; }
JS_DEVICE float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
JS_DEVICE void st_f(float* p, float v) { *p = v; }
JS_DEVICE void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

JS_DEVICE float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));   // sqrt(2 / pi)
}

// sum over the CTA (blockDim.x a multiple of 32, at most 1024); every thread gets the result
JS_DEVICE float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) s += red[i];
  __syncthreads();
  return s;
}

// ---------------------------------------------------------------- unfused forms
template <typename TW, typename TO>
__global__ void dynamic_tanh_kernel(const float* x, int ldx, const TW* alpha, const TW* w, const TW* b, TO* out, int ldo,
                                    int T, int W) {
  const size_t n = static_cast<size_t>(T) * W;
  const float a = ld_f(alpha);
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t t = i / W, c = i % W;
    st_f(out + t * ldo + c, tanhf(a * x[t * ldx + c]) * ld_f(w + c) + ld_f(b + c));
  }
}

template <typename E>
__global__ void gelu_tanh_mul_kernel(const E* g, const E* u, E* out, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x)
    st_f(out + i, gelu_tanh_f(ld_f(g + i)) * ld_f(u + i));
}

template <typename E>
__global__ void relu_squared_kernel(const E* x, E* out, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const float r = fmaxf(ld_f(x + i), 0.f);
    st_f(out + i, r * r);
  }
}

template <typename E>
__global__ void latent_scatter_kernel(const E* c, int ldc, int R, E* pool, int Rp, int S, const int* slots, int T, int* status) {
  const int t = blockIdx.x;
  if (t >= T) return;
  const int slot = slots[t];
  if (slot < 0 || slot >= S) {
    if (threadIdx.x == 0) report(status, kBadSlot);
    return;
  }
  for (int i = threadIdx.x; i < Rp; i += blockDim.x)
    st_f(pool + static_cast<size_t>(slot) * Rp + i, i < R ? ld_f(c + static_cast<size_t>(t) * ldc + i) : 0.f);
}

// ---------------------------------------------------------------- fused steps
// x[t] = table[ids[t]] (fp32), emb[t] = the same in bf16 (kept for the loop passes), h[t] = Dynamic Tanh of x.
__global__ void __launch_bounds__(256)
embed_dyt_kernel(const int* ids, const __nv_bfloat16* table, int V, int ldt, float* x, __nv_bfloat16* emb, __nv_bfloat16* h, int ld,
                 const float* w, const float* b, float alpha, int W) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  const __nv_bfloat16* src = table + static_cast<size_t>(id) * ldt;
  const size_t o = static_cast<size_t>(t) * ld;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float v = __bfloat162float(src[c]);
    x[o + c] = v;
    if (emb != nullptr) emb[o + c] = src[c];
    h[o + c] = __float2bfloat16_rn(tanhf(alpha * v) * w[c] + b[c]);
  }
}

// RMS norms of the two latents of one token, from the fp32 input projection [q latent | kv latent | ...]: the query
// latent goes to cq (T, qp), the kv latent to its pool row; columns past the ranks are zeroed.
__global__ void __launch_bounds__(256)
latent_post_kernel(const float* proj, int ldp, int q_rank, int kv_rank, const __nv_bfloat16* qw, const __nv_bfloat16* kw, float eps,
                   __nv_bfloat16* cq, int qp, __nv_bfloat16* pool, int Rp, int S, const int* slots, int* status) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const bool is_q = blockIdx.y == 0;
  const int n = is_q ? q_rank : kv_rank, width = is_q ? qp : Rp;
  const float* src = proj + static_cast<size_t>(t) * ldp + (is_q ? 0 : q_rank);
  const __nv_bfloat16* w = is_q ? qw : kw;
  size_t row = t;
  if (!is_q) {
    const int slot = slots[t];
    if (slot < 0 || slot >= S) {
      if (threadIdx.x == 0) report(status, kBadSlot);
      return;
    }
    row = slot;
  }
  constexpr int KEEP = 8;                    // values a thread holds on to (latents up to 2048 wide); the rest is read twice
  float v[KEEP], ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = threadIdx.x + j * 256;
    v[j] = i < n ? src[i] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < KEEP; ++j) ss += v[j] * v[j];
  for (int i = threadIdx.x + KEEP * 256; i < n; i += 256) ss += src[i] * src[i];
  const float inv = 1.f / sqrtf(block_sum(ss, red) / n + eps);
  __nv_bfloat16* dst = (is_q ? cq : pool) + row * width;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = threadIdx.x + j * 256;
    if (i < width) dst[i] = __float2bfloat16_rn(i < n ? v[j] * inv * __bfloat162float(w[i]) : 0.f);
  }
  for (int i = threadIdx.x + KEEP * 256; i < width; i += 256)
    dst[i] = __float2bfloat16_rn(i < n ? src[i] * inv * __bfloat162float(w[i]) : 0.f);
}

// Sigmoid routing, one warp per token: scores s = sigmoid(z), the k largest s + correction are chosen (ties: lower
// expert), weights s / (sum of the chosen s + 1e-20) * scale.  With `act`, the warp also scales the token's shared-expert
// activations by sigmoid(z[gate_col]).
template <int PL>     // experts per lane
__global__ void __launch_bounds__(256)
sigmoid_route_kernel(const float* z, int ldz, const float* corr, int T, int E, int k, float scale, float* wts, int* idx,
                     int gate_col, __nv_bfloat16* act, int lda, int act_cols) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* zr = z + static_cast<size_t>(t) * ldz;
  float s[PL], c[PL];
#pragma unroll
  for (int i = 0; i < PL; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < E ? 1.f / (1.f + expf(-zr[e])) : 0.f;
    c[i] = e < E ? s[i] + corr[e] : -INFINITY;
  }
  float kept = 0.f, my_w = 0.f;
  int my_e = 0;
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int be = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PL; ++i)
      if (c[i] > best) { best = c[i]; be = lane + 32 * i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
    }
    float sw = 0.f;
#pragma unroll
    for (int i = 0; i < PL; ++i)
      if (lane + 32 * i == be) { sw = s[i]; c[i] = -INFINITY; }
    sw = warp_sum(sw);                        // only the winner's lane holds a value
    kept += sw;
    if (lane == j) { my_w = sw; my_e = be < E ? be : 0; }
  }
  if (lane < k) {
    wts[static_cast<size_t>(t) * k + lane] = my_w / (kept + 1e-20f) * scale;
    idx[static_cast<size_t>(t) * k + lane] = my_e;
  }
  if (act != nullptr) {
    const float g = 1.f / (1.f + expf(-zr[gate_col]));
    __nv_bfloat16* a = act + static_cast<size_t>(t) * lda;
    for (int i = 2 * lane; i < act_cols; i += 64) {
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(a + i));
      *reinterpret_cast<__nv_bfloat162*>(a + i) = __floats2bfloat162_rn(v.x * g, v.y * g);
    }
  }
}

// x[t] += sum_j row_weight[r] * ys[r] (r = inv[t*k + j], choice order) + emb[t]; h[t] = Dynamic Tanh of the new x.
// `ys`, `emb`, `h` may be null (a layer without experts, no loop pass ahead, no norm behind).
__global__ void __launch_bounds__(256)
combine_dyt_kernel(const __nv_bfloat16* ys, int ldy, const int* inv, const float* row_weight, int k, const __nv_bfloat16* emb,
                   float* x, __nv_bfloat16* h, int ld, const float* w, const float* b, float alpha, int W) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const size_t o = static_cast<size_t>(t) * ld;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < W; c += gridDim.y * blockDim.x * 4) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (ys != nullptr) {
      for (int j = 0; j < k; ++j) {
        const int r = inv[t * k + j];
        const float wt = row_weight[r];
        const uint2 raw = *reinterpret_cast<const uint2*>(ys + static_cast<size_t>(r) * ldy + c);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 f = __bfloat1622float2(h2[e]);
          acc[2 * e] += wt * f.x;
          acc[2 * e + 1] += wt * f.y;
        }
      }
    }
    const float4 xv = *reinterpret_cast<const float4*>(x + o + c);
    float v[4] = {xv.x + acc[0], xv.y + acc[1], xv.z + acc[2], xv.w + acc[3]};
    if (emb != nullptr) {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] += __bfloat162float(emb[o + c + e]);
    }
    *reinterpret_cast<float4*>(x + o + c) = make_float4(v[0], v[1], v[2], v[3]);
    if (h != nullptr) {
#pragma unroll
      for (int e = 0; e < 4; ++e) h[o + c + e] = __float2bfloat16_rn(tanhf(alpha * v[e]) * w[c + e] + b[c + e]);
    }
  }
}

// dst[i] = bf16(x[i, :W])  (a tapped residual row for the draft head)
__global__ void tap_rows_kernel(const float* x, int ld, __nv_bfloat16* dst, int ldd, int W) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    dst[static_cast<size_t>(t) * ldd + c] = __float2bfloat16_rn(x[static_cast<size_t>(t) * ld + c]);
}

// ---------------------------------------------------------------- latent attention on the plain cores
// One CTA per (token, head) row of absorbed queries: scores q . c over the sequence's cached latent rows, softmax, and
// the weighted sum of the same rows.  Four warps take every fourth key each and merge at the end.  This is the 32-bit
// path, and the bf16 path of rows the tensor-core kernel does not take.  sinks (H): a valueless key's score (unscaled) per
// head; gate (T, ldg): logits whose sigmoid multiplies a head's output; both may be null.
template <typename E, int NPL>
__global__ void __launch_bounds__(128)
latent_attn_simt_kernel(const E* q, const E* pool, const int* slot_map, const int* seq_rows, const int* cu_q, const int* past_lens,
                        const int* mask_bits, E* out, int B, int H, int Rp, int S, int max_len, int W, int causal, float scale,
                        const float* sinks, const float* gate, int ldg, int* status) {
  const int row = blockIdx.x, t = row / H;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int i = t - cu_q[lo], past = past_lens[lo], n_b = cu_q[lo + 1] - cu_q[lo];
  const int* slots = slot_map + static_cast<size_t>(seq_rows[lo]) * max_len;
  const int L = causal ? past + i + 1 : past + n_b;
  float qv[NPL], acc[NPL];
#pragma unroll
  for (int e = 0; e < NPL; ++e) {
    const int c = lane + 32 * e;
    qv[e] = c < Rp ? ld_f(q + static_cast<size_t>(row) * Rp + c) * scale : 0.f;
    acc[e] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  if (sinks != nullptr && warp == 0) { m = sinks[row % H]; l = 1.f; }
  for (int j = warp; j < L; j += 4) {
    if (!causal && j >= past) {
      const int n = j - past;
      if (!((mask_bits[static_cast<size_t>(t) * W + (n >> 5)] >> (n & 31)) & 1)) continue;
    }
    int slot = slots[j];
    if (slot < 0 || slot >= S) { if (lane == 0) report(status, kBadSlot); slot = 0; }
    const E* kr = pool + static_cast<size_t>(slot) * Rp;
    float kv[NPL], d = 0.f;
#pragma unroll
    for (int e = 0; e < NPL; ++e) {
      const int c = lane + 32 * e;
      kv[e] = c < Rp ? ld_f(kr + c) : 0.f;
      d += qv[e] * kv[e];
    }
    d = warp_sum(d);
    const float mn = fmaxf(m, d), a = expf(m - mn), p = expf(d - mn);
    l = l * a + p;
#pragma unroll
    for (int e = 0; e < NPL; ++e) acc[e] = acc[e] * a + p * kv[e];
    m = mn;
  }
  __shared__ float sm[4], sl[4];
  extern __shared__ float so[];            // 4 x Rp
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
  for (int e = 0; e < NPL; ++e)
    if (lane + 32 * e < Rp) so[warp * Rp + lane + 32 * e] = acc[e];
  __syncthreads();
  const float mm = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  float f[4], tot = 0.f;
#pragma unroll
  for (int w2 = 0; w2 < 4; ++w2) {
    f[w2] = sm[w2] == -INFINITY ? 0.f : expf(sm[w2] - mm);
    tot += sl[w2] * f[w2];
  }
  float inv = tot > 0.f ? 1.f / tot : 0.f;
  if (gate != nullptr) inv /= 1.f + expf(-gate[static_cast<size_t>(t) * ldg + row % H]);
  for (int c = threadIdx.x; c < Rp; c += blockDim.x)
    st_f(out + static_cast<size_t>(row) * Rp + c,
         (so[c] * f[0] + so[Rp + c] * f[1] + so[2 * Rp + c] * f[2] + so[3 * Rp + c] * f[3]) * inv);
}

template <typename E>
static int launch_simt(const void* q, const void* pool, const int* slot_map, const int* seq_rows, const int* cu_q,
                       const int* past_lens, const int* mask_bits, void* out, int B, int T, int H, int Rp, int S, int max_len,
                       int W, int causal, float scale, const float* sinks, const float* gate, int ldg, int* status,
                       cudaStream_t stream) {
  const int smem = 4 * Rp * 4;
#define JS_SIMT(N)                                                                                                        \
  if (Rp <= 32 * N) {                                                                                                     \
    latent_attn_simt_kernel<E, N><<<T * H, 128, smem, stream>>>(static_cast<const E*>(q), static_cast<const E*>(pool),    \
        slot_map, seq_rows, cu_q, past_lens, mask_bits, static_cast<E*>(out), B, H, Rp, S, max_len, W, causal, scale, \
        sinks, gate, ldg, status);                                                                                        \
    return cudaGetLastError() == cudaSuccess ? 0 : -4;                                                                    \
  }
  JS_SIMT(2) JS_SIMT(4) JS_SIMT(8) JS_SIMT(16) JS_SIMT(32) JS_SIMT(64)
#undef JS_SIMT
  return -14;
}

// attributes of a launch that may start before its predecessor ends
struct LaunchCfg {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a;
  LaunchCfg(dim3 grid, dim3 block, cudaStream_t stream, int pdl, size_t smem = 0) {
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

static int grid_for(size_t n) {
  const size_t b = (n + 255) / 256;
  return static_cast<int>(b > 1184 ? 1184 : b);
}

}  // namespace js

// x (T, W) fp32 -> out (T, W); weights bf16 (w_bf16 = 1) or fp32, output bf16 (o_bf16 = 1) or fp32.
extern "C" int js_dynamic_tanh(const float* x, int ldx, const void* alpha, const void* w, const void* b, int w_bf16, void* out,
                               int ldo, int o_bf16, int T, int W, cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || W <= 0) return 0;
  const int g = grid_for(static_cast<size_t>(T) * W);
  using bf = __nv_bfloat16;
  if (w_bf16 && o_bf16)
    dynamic_tanh_kernel<bf, bf><<<g, 256, 0, stream>>>(x, ldx, (const bf*)alpha, (const bf*)w, (const bf*)b, (bf*)out, ldo, T, W);
  else if (w_bf16)
    dynamic_tanh_kernel<bf, float><<<g, 256, 0, stream>>>(x, ldx, (const bf*)alpha, (const bf*)w, (const bf*)b, (float*)out, ldo, T, W);
  else if (o_bf16)
    dynamic_tanh_kernel<float, bf><<<g, 256, 0, stream>>>(x, ldx, (const float*)alpha, (const float*)w, (const float*)b, (bf*)out, ldo, T, W);
  else
    dynamic_tanh_kernel<float, float><<<g, 256, 0, stream>>>(x, ldx, (const float*)alpha, (const float*)w, (const float*)b, (float*)out, ldo, T, W);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int js_gelu_tanh_mul(const void* g, const void* u, void* out, long long n, int bf16, cudaStream_t stream) {
  using namespace js;
  if (n <= 0) return 0;
  if (bf16)
    gelu_tanh_mul_kernel<__nv_bfloat16><<<grid_for(n), 256, 0, stream>>>((const __nv_bfloat16*)g, (const __nv_bfloat16*)u, (__nv_bfloat16*)out, n);
  else
    gelu_tanh_mul_kernel<float><<<grid_for(n), 256, 0, stream>>>((const float*)g, (const float*)u, (float*)out, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int js_relu_squared(const void* x, void* out, long long n, int bf16, cudaStream_t stream) {
  using namespace js;
  if (n <= 0) return 0;
  if (bf16)
    relu_squared_kernel<__nv_bfloat16><<<grid_for(n), 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)out, n);
  else
    relu_squared_kernel<float><<<grid_for(n), 256, 0, stream>>>((const float*)x, (float*)out, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int js_latent_scatter(const void* c, int ldc, int R, void* pool, int Rp, int S, const int* slots, int T, int bf16,
                                 int* status, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (bf16)
    latent_scatter_kernel<__nv_bfloat16><<<T, 128, 0, stream>>>((const __nv_bfloat16*)c, ldc, R, (__nv_bfloat16*)pool, Rp, S, slots, T, status);
  else
    latent_scatter_kernel<float><<<T, 128, 0, stream>>>((const float*)c, ldc, R, (float*)pool, Rp, S, slots, T, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// q, out (T*H, Rp); pool (S, Rp); Rp at most 2048.
extern "C" int js_latent_attention_simt(const void* q, const void* pool, const int* slot_map, const int* seq_rows, const int* cu_q,
                                        const int* past_lens, const int* mask_bits, void* out, int B, int T, int H, int Rp, int S,
                                        int max_len, int W, int causal, float scale, const float* sinks, const float* gate, int ldg,
                                        int bf16, int* status, cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || B <= 0) return 0;
  if (!causal && (mask_bits == nullptr || W < 1)) return -13;
  return bf16 ? launch_simt<__nv_bfloat16>(q, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, out, B, T, H, Rp, S, max_len, W, causal, scale, sinks, gate, ldg, status, stream)
              : launch_simt<float>(q, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, out, B, T, H, Rp, S, max_len, W, causal, scale, sinks, gate, ldg, status, stream);
}

// table (V, ldt) bf16; x fp32, emb (may be null) and h bf16 with leading dimension ld; w, b fp32 (W).
extern "C" int js_embed_dyt(const int* ids, const void* table, int V, int ldt, float* x, void* emb, void* h, int ld, const float* w,
                            const float* b, float alpha, int T, int W, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  LaunchCfg l(dim3(T), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, embed_dyt_kernel, ids, (const __nv_bfloat16*)table, V, ldt, x, (__nv_bfloat16*)emb,
                            (__nv_bfloat16*)h, ld, w, b, alpha, W) == cudaSuccess ? 0 : -4;
}

// proj (T, ldp) fp32, columns [0, q_rank) and [q_rank, q_rank + kv_rank); cq (T, qp) bf16; pool (S, Rp) bf16.
extern "C" int js_latent_post(const float* proj, int ldp, int q_rank, int kv_rank, const void* qw, const void* kw, float eps, void* cq,
                              int qp, void* pool, int Rp, int S, const int* slots, int T, int* status, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  LaunchCfg l(dim3(T, 2), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, latent_post_kernel, proj, ldp, q_rank, kv_rank, (const __nv_bfloat16*)qw, (const __nv_bfloat16*)kw,
                            eps, (__nv_bfloat16*)cq, qp, (__nv_bfloat16*)pool, Rp, S, slots, status) == cudaSuccess ? 0 : -4;
}

// z (T, ldz) fp32 router logits -> wts (T, k) fp32, idx (T, k) int32.  E <= 1024, k <= min(32, E).  act (optional): bf16
// rows of act_cols columns (even) scaled in place by sigmoid(z[:, gate_col]).
extern "C" int js_sigmoid_route(const float* z, int ldz, const float* corr, int T, int E, int k, float scale, float* wts, int* idx,
                                int gate_col, void* act, int lda, int act_cols, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (E < 1 || E > 1024 || k < 1 || k > 32 || k > E || (act_cols & 1) || (lda & 1)) return -10;
  LaunchCfg l(dim3((T + 7) / 8), dim3(256), stream, pdl);
  auto kern = E <= 64 ? sigmoid_route_kernel<2> : E <= 256 ? sigmoid_route_kernel<8> : sigmoid_route_kernel<32>;
  return cudaLaunchKernelEx(&l.c, kern, z, ldz, corr, T, E, k, scale, wts, idx, gate_col, (__nv_bfloat16*)act, lda,
                            act_cols) == cudaSuccess ? 0 : -4;
}

// W a multiple of 4; rows of x, h, emb with leading dimension ld (a multiple of 4), ys (rows, ldy), ldy a multiple of 4.
extern "C" int js_combine_dyt(const void* ys, int ldy, const int* inv, const float* row_weight, int k, const void* emb, float* x, void* h,
                              int ld, const float* w, const float* b, float alpha, int T, int W, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if ((W % 4) || (ld % 4) || (ldy % 4)) return -10;
  const int gy = T >= 148 ? 1 : (W + 1023) / 1024;
  LaunchCfg l(dim3(T, gy), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, combine_dyt_kernel, (const __nv_bfloat16*)ys, ldy, inv, row_weight, k, (const __nv_bfloat16*)emb, x,
                            (__nv_bfloat16*)h, ld, w, b, alpha, W) == cudaSuccess ? 0 : -4;
}

extern "C" int js_tap_rows(const float* x, int ld, void* dst, int ldd, int T, int W, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  LaunchCfg l(dim3(T), dim3(256), stream, pdl);
  return cudaLaunchKernelEx(&l.c, tap_rows_kernel, x, ld, (__nv_bfloat16*)dst, ldd, W) == cudaSuccess ? 0 : -4;
}
