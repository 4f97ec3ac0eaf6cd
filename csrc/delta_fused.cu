// Fused forms of the gated delta rule (equations and state layout: delta_kernels.cu).
//
//   step   one row per sequence (decode): convolution, unit norms, decays, recurrence, per-head norm and gate in ONE kernel,
//          the head's whole state in registers, read once and written once;
//   block  prompt portions: rows go in blocks of 8.  With c the logarithms of the decays accumulated inside a block, c_N at its
//          end, M_ij = beta_i sum_d k_i k_j e^(c_i - c_j) below the diagonal, P the same with q and the diagonal, T = (1 + M)^-1:
//
//              w_i = beta_i v_i - (beta_i e^(c_i) k_i)^T S          everything is read from the state BEFORE the block, so
//              o_i = (e^(c_i) q_i)^T S + sum_m (P T)_im w_m         the only chain left is one matrix product per block
//              S  <- e^(c_N) S + sum_m (sum_j T_jm e^(c_N - c_j) k_j) w_m^T
//
//          A first kernel makes the bracketed rows of all blocks in parallel (with the convolutions and norms), in fp32; a
//          second one walks the blocks with the state in registers.  Its products run on the tensor cores as three tf32
//          products of split operands each, which keeps 32-bit accuracy; sums are fp32.  No exponent is ever positive.
#include "tf32_split.cuh"

#include <math.h>

namespace js {

JS_DEVICE float df_ld(const float* p) { return *p; }
JS_DEVICE float df_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
JS_DEVICE float df_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
JS_DEVICE float df_silu(float z) { return z / (1.f + expf(-z)); }
// the activation behind a convolution: its input is a bf16 projection, so the fast exponential's error does not show
JS_DEVICE float df_silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }
JS_DEVICE float df_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

constexpr int kBlk = 8;
constexpr int kBlkMaxTaps = 17;

struct DeltaIn {
  int H, G, D, V, taps, channel;
  const __nv_bfloat16* pre;            // (T, ldp) un-convolved q | k | v
  const float *z, *b;                  // (T, ldz), (T, ldb)
  int ldp, ldz, ldb;
  const __nv_bfloat16 *wt, *A_log, *dt_bias;     // taps (C, n), (H), (H or H*D)
  __nv_bfloat16* conv;                 // (slots, taps, C) ring
  const int *rows, *cu_q, *past_lens;
  int B;
};

// silu of the convolution of channel c at local row i of a sequence (rows q0 .., committed length past, ring cs)
// un-convolved input of channel c at local row i of a sequence (rows q0 .., committed length past, ring cs)
JS_DEVICE float conv_in(const DeltaIn& p, const __nv_bfloat16* cs, int C, int q0, int past, int i, int c) {
  if (i >= 0) return __bfloat162float(p.pre[static_cast<size_t>(q0 + i) * p.ldp + c]);
  return past + i >= 0 ? __bfloat162float(cs[static_cast<size_t>((past + i) % p.taps) * C + c]) : 0.f;
}

// silu of the convolution of channel c at local row i
JS_DEVICE float conv_at(const DeltaIn& p, const __nv_bfloat16* cs, int C, int q0, int past, int i, int c) {
  float y = 0.f;
  const __nv_bfloat16* w = p.wt + static_cast<size_t>(c) * p.taps;
  for (int m = p.taps - 1; m >= 0; --m) y += conv_in(p, cs, C, q0, past, i - m, c) * __bfloat162float(w[p.taps - 1 - m]);
  return df_silu_fast(y);
}

// the same for rows i0 .. i0 + n - 1 (n <= kBlk; the others give 0), every input loaded once; TP >= taps
template <int TP>
JS_DEVICE void conv_rows(const DeltaIn& p, const __nv_bfloat16* cs, int C, int q0, int past, int i0, int n, int c, float (&y)[kBlk]) {
  float w[TP], x[kBlk + TP - 1];
  const int skip = TP - p.taps;                 // leading taps of weight 0
#pragma unroll
  for (int j = 0; j < TP; ++j) w[j] = j >= skip ? __bfloat162float(p.wt[static_cast<size_t>(c) * p.taps + j - skip]) : 0.f;
  if (i0 >= TP - 1) {
    // all rows belong to this batch: plain loads that overlap (rows past the end repeat the last one and are dropped below)
    const __nv_bfloat16* src = p.pre + static_cast<size_t>(q0 + i0 - (TP - 1)) * p.ldp + c;
    const int last = TP - 2 + max(n, 1);
#pragma unroll
    for (int j = 0; j < kBlk + TP - 1; ++j) x[j] = __bfloat162float(src[static_cast<size_t>(min(j, last)) * p.ldp]);
  } else {
#pragma unroll
    for (int j = 0; j < kBlk + TP - 1; ++j) {
      const int i = i0 + j - (TP - 1);
      x[j] = (j >= skip && i < i0 + n) ? conv_in(p, cs, C, q0, past, i, c) : 0.f;
    }
  }
#pragma unroll
  for (int i = 0; i < kBlk; ++i) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < TP; ++j) s += x[i + j] * w[j];
    y[i] = i < n ? df_silu_fast(s) : 0.f;
  }
}

// ================================================================ one row per sequence
struct DeltaStepParams {
  DeltaIn in;
  float* state;                        // (slots, H, D, V)
  const __nv_bfloat16 *gate, *norm_w;  // (T, ldg), (V)
  __nv_bfloat16* out;                  // (T, ldo)
  int ldg, ldo, silu;
  float eps;
};

constexpr int kStepThreads = 256;

// VG column groups of 4 (a power of two, 4 VG >= V); thread (rl, cg) holds rows rl, rl + RL, ... (NR of them)
template <int NR>
__global__ void __launch_bounds__(kStepThreads, 1) delta_step_kernel(DeltaStepParams p, int VG) {
  __shared__ float sq[256], sk[256], sg[256], sv[256], su[256];
  __shared__ float red[8 * 256], scal[4];
  const DeltaIn& in = p.in;
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = in.D, V = in.V, g = h / (in.H / in.G);
  const int C = 2 * in.G * D + in.H * V;
  const int RL = kStepThreads / VG, cg = tid % VG, rl = tid / VG, col = 4 * cg;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = in.rows[t], past = in.past_lens[t];
  float* st = p.state + (static_cast<size_t>(slot) * in.H + h) * D * V;
  float4 S[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = rl + j * RL;
    S[j] = (past > 0 && d < D && col < V) ? *reinterpret_cast<const float4*>(st + static_cast<size_t>(d) * V + col) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const __nv_bfloat16* cs = in.conv + static_cast<size_t>(slot) * in.taps * C;
  for (int x = tid; x < 2 * D + V; x += kStepThreads) {
    const int c = x < D ? g * D + x : x < 2 * D ? (in.G + g) * D + x - D : 2 * in.G * D + h * V + x - 2 * D;
    const float y = conv_at(in, cs, C, t, past, 0, c);
    if (x < D) sq[x] = y; else if (x < 2 * D) sk[x - D] = y; else sv[x - 2 * D] = y;
  }
  const float a = expf(__bfloat162float(in.A_log[h]));
  if (in.channel) {
    for (int d = tid; d < D; d += kStepThreads)
      sg[d] = expf(-a * df_softplus(in.z[static_cast<size_t>(t) * in.ldz + h * D + d] + __bfloat162float(in.dt_bias[h * D + d])));
  } else {
    const float gs = expf(-a * df_softplus(in.z[static_cast<size_t>(t) * in.ldz + h] + __bfloat162float(in.dt_bias[h])));
    for (int d = tid; d < D; d += kStepThreads) sg[d] = gs;
  }
  const float beta = df_sigmoid(in.b[static_cast<size_t>(t) * in.ldb + h]);
  __syncthreads();
  if (warp < 2) {                       // unit norms of q (with 1/sqrt(D)) and k
    const float* src = warp == 0 ? sq : sk;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += src[d] * src[d];
    ss = warp_sum(ss);
    if (lane == 0) scal[warp] = (warp == 0 ? 1.f / sqrtf(static_cast<float>(D)) : 1.f) / sqrtf(ss + 1e-6f);
  }
  // the ring entry of this position: no CTA of this launch reads it
  if (in.taps > 1) {
    __nv_bfloat16* dst = in.conv + (static_cast<size_t>(slot) * in.taps + past % in.taps) * C;
    const __nv_bfloat16* src = in.pre + static_cast<size_t>(t) * in.ldp;
    for (int c = tid; c < V; c += kStepThreads) dst[2 * in.G * D + h * V + c] = src[2 * in.G * D + h * V + c];
    if (h % (in.H / in.G) == 0)
      for (int c = tid; c < 2 * D; c += kStepThreads) {
        const int ch = c < D ? g * D + c : (in.G + g) * D + c - D;
        dst[ch] = src[ch];
      }
  }
  __syncthreads();
  const float nq = scal[0], nk = scal[1];
  // sum over the rows of a per-thread partial, for every column; the result lands in dst[0 .. 4 VG)
  auto column_sum = [&](float4 v, float* dst) {
    for (int o = VG; o < 32; o <<= 1) {
      v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
      v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
      v.z += __shfl_xor_sync(0xffffffffu, v.z, o);
      v.w += __shfl_xor_sync(0xffffffffu, v.w, o);
    }
    const int sets = VG <= 32 ? 8 : kStepThreads / VG, set = VG <= 32 ? warp : rl;
    if (VG > 32 || lane < VG) *reinterpret_cast<float4*>(red + set * 256 + col) = v;
    __syncthreads();
    for (int c = tid; c < 4 * VG; c += kStepThreads) {
      float s = 0.f;
      for (int i = 0; i < sets; ++i) s += red[i * 256 + c];
      dst[c] = s;
    }
    __syncthreads();
  };
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = rl + j * RL;
    if (d < D) {
      const float gd = sg[d], kd = sk[d] * nk;
      S[j].x *= gd; S[j].y *= gd; S[j].z *= gd; S[j].w *= gd;
      acc.x += S[j].x * kd; acc.y += S[j].y * kd; acc.z += S[j].z * kd; acc.w += S[j].w * kd;
    }
  }
  column_sum(acc, su);
  float4 u;
  u.x = beta * ((col < V ? sv[col] : 0.f) - su[col]);
  u.y = beta * ((col + 1 < V ? sv[col + 1] : 0.f) - su[col + 1]);
  u.z = beta * ((col + 2 < V ? sv[col + 2] : 0.f) - su[col + 2]);
  u.w = beta * ((col + 3 < V ? sv[col + 3] : 0.f) - su[col + 3]);
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = rl + j * RL;
    if (d < D) {
      const float kd = sk[d] * nk, qd = sq[d] * nq;
      S[j].x += kd * u.x; S[j].y += kd * u.y; S[j].z += kd * u.z; S[j].w += kd * u.w;
      acc.x += S[j].x * qd; acc.y += S[j].y * qd; acc.z += S[j].z * qd; acc.w += S[j].w * qd;
      if (col < V) *reinterpret_cast<float4*>(st + static_cast<size_t>(d) * V + col) = S[j];
    }
  }
  __syncthreads();                      // su has been read by everyone
  column_sum(acc, su);
  if (warp == 0) {
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) ss += su[c] * su[c];
    ss = warp_sum(ss);
    if (lane == 0) scal[2] = 1.f / sqrtf(ss / V + p.eps);
  }
  __syncthreads();
  const float r = scal[2];
  for (int c = tid; c < V; c += kStepThreads) {
    const float zg = __bfloat162float(p.gate[static_cast<size_t>(t) * p.ldg + h * V + c]);
    p.out[static_cast<size_t>(t) * p.ldo + h * V + c] =
        __float2bfloat16_rn(su[c] * r * __bfloat162float(p.norm_w[c]) * (p.silu ? df_silu(zg) : df_sigmoid(zg)));
  }
}

// ================================================================ blocks of 8 rows
// Sequence s owns the blocks cu_q[s] / 8 + s, ...; padded row = 8 block + row of the block.  All arrays are per head.
struct DeltaBlocks {
  float *kt, *qt, *kh;                 // (H, R, DP): beta e^c k, e^c q, T^T e^(c_N - c) k
  float *bv;                           // (H, R, V): beta v
  float *pt;                           // (H, R, 8): P T
  float *ge;                           // (H, R / 8, DP): e^(c_N)
  int R;
};

// sums over the warp of N values, halving what every lane keeps: N = 64 leaves entries 2 l and 2 l + 1 in v[0], v[1] of lane l,
// N = 16 entry l / 2 in v[0]
template <int N>
JS_DEVICE void warp_transpose_sum(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int b = 16, half = N / 2; b > 0; b >>= 1, half >>= 1) {
    const bool hi = (lane & b) != 0;
    if (half > 0) {
#pragma unroll
      for (int j = 0; j < half; ++j) {
        const float send = hi ? v[j] : v[j + half];
        const float keep = hi ? v[j + half] : v[j];
        v[j] = keep + __shfl_xor_sync(0xffffffffu, send, b);
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], b);
    }
  }
}

template <int DP, bool CH, int TP>
__global__ void __launch_bounds__(DP, TP <= 4 ? 640 / DP : 1) delta_block_prep_kernel(DeltaIn in, DeltaBlocks o) {
  constexpr int NW = DP / 32;
  __shared__ float part[NW][64], G[64], Tm[64], nrm[NW][16], inv_norm[16], sbeta[kBlk], sg[kBlk];
  // no early start of the walk behind: its few long CTAs would pile up on the SMs that empty first
  pdl_wait();
  const int h = blockIdx.y, tile = blockIdx.x, d = threadIdx.x, warp = d >> 5, lane = d & 31;
  int lo = 0, hi = in.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (in.cu_q[mid] / kBlk + mid <= tile) lo = mid; else hi = mid - 1;
  }
  const int q0 = in.cu_q[lo], n = in.cu_q[lo + 1] - q0, r0 = (tile - (q0 / kBlk + lo)) * kBlk;
  if (r0 >= n) return;
  const int past = in.past_lens[lo], m_rows = min(kBlk, n - r0);
  const int D = in.D, V = in.V, g = h / (in.H / in.G), C = 2 * in.G * D + in.H * V;
  const __nv_bfloat16* cs = in.conv + static_cast<size_t>(in.rows[lo]) * in.taps * C;
  const float a = expf(__bfloat162float(in.A_log[h]));
  if (d < kBlk) {
    const bool ok = d < m_rows;
    const size_t t = q0 + r0 + (ok ? d : 0);
    sbeta[d] = ok ? df_sigmoid(in.b[t * in.ldb + h]) : 0.f;
    if (!CH) sg[d] = ok ? expf(-a * df_softplus(in.z[t * in.ldz + h] + __bfloat162float(in.dt_bias[h]))) : 1.f;
  }
  float q[kBlk], k[kBlk], v[kBlk], gd[kBlk];
  const int dc = min(d, D - 1), rows_d = d < D ? m_rows : 0;
  conv_rows<TP>(in, cs, C, q0, past, r0, rows_d, g * D + dc, q);
  conv_rows<TP>(in, cs, C, q0, past, r0, rows_d, (in.G + g) * D + dc, k);
  conv_rows<TP>(in, cs, C, q0, past, r0, d < V ? m_rows : 0, 2 * in.G * D + h * V + min(d, V - 1), v);
  if (CH) {
#pragma unroll
    for (int i = 0; i < kBlk; ++i) gd[i] = in.z[static_cast<size_t>(q0 + r0 + min(i, m_rows - 1)) * in.ldz + h * D + dc];
    const float dt = __bfloat162float(in.dt_bias[h * D + dc]);
#pragma unroll
    for (int i = 0; i < kBlk; ++i) gd[i] = (d < D && i < m_rows) ? expf(-a * df_softplus(gd[i] + dt)) : 1.f;
  }
  {
    float ss[16];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) { ss[i] = q[i] * q[i]; ss[8 + i] = k[i] * k[i]; }
    warp_transpose_sum<16>(ss);         // lane l: sum l / 2
    if ((lane & 1) == 0) nrm[warp][lane >> 1] = ss[0];
  }
  __syncthreads();
  if (d < 16) {                         // q's includes the 1/sqrt(D)
    float s = 1e-6f;
#pragma unroll
    for (int w = 0; w < NW; ++w) s += nrm[w][d];
    inv_norm[d] = 1.f / sqrtf(d < 8 ? static_cast<float>(D) * s : s);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kBlk; ++i) {
    q[i] *= inv_norm[i];
    k[i] *= inv_norm[8 + i];
    if (!CH) gd[i] = sg[i];
  }
  // pair sums: P_ij (j <= i) at [i][j], the strict K K^T part (j < i) at [j][i]; kd[j] = k_j decayed from row j to row i
  {
    float s[64], kd[kBlk];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) {
      if (i > 0) {
#pragma unroll
        for (int j = 0; j < i; ++j) kd[j] *= gd[i];
      }
      kd[i] = k[i];
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        s[i * 8 + j] = q[i] * kd[j];
        if (j < i) s[j * 8 + i] = k[i] * kd[j];
      }
    }
    warp_transpose_sum<64>(s);          // lane l: sums 2 l and 2 l + 1
    part[warp][2 * lane] = s[0];
    part[warp][2 * lane + 1] = s[1];
  }
  // what does not need T: decayed q and k, beta v
  const size_t row = static_cast<size_t>(h) * o.R + static_cast<size_t>(tile) * kBlk;
  float e[kBlk], run = 1.f;
#pragma unroll
  for (int i = 0; i < kBlk; ++i) {
    run *= gd[i];
    o.kt[(row + i) * DP + d] = sbeta[i] * run * k[i];
    o.qt[(row + i) * DP + d] = run * q[i];
  }
  o.ge[(static_cast<size_t>(h) * (o.R / kBlk) + tile) * DP + d] = run;
  run = 1.f;
#pragma unroll
  for (int i = kBlk - 1; i >= 0; --i) {
    e[i] = run * k[i];
    run *= gd[i];
  }
  if (d < V) {
#pragma unroll
    for (int i = 0; i < kBlk; ++i) o.bv[(row + i) * V + d] = sbeta[i] * v[i];
  }
  for (int vc = d + DP; vc < V; vc += DP) {
    conv_rows<TP>(in, cs, C, q0, past, r0, m_rows, 2 * in.G * D + h * V + vc, v);
#pragma unroll
    for (int i = 0; i < kBlk; ++i) o.bv[(row + i) * V + vc] = sbeta[i] * v[i];
  }
  __syncthreads();
  for (int x = d; x < 64; x += DP) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) s += part[w][x];
    G[x] = s;
  }
  __syncthreads();
  if (d < kBlk) {                       // column d of T = (1 + M)^-1
    float col[kBlk];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) {
      float s = i == d ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j)
        if (j >= d) s -= sbeta[i] * G[j * 8 + i] * col[j];
      col[i] = i < d ? 0.f : s;
      Tm[i * 8 + d] = col[i];
    }
  }
  __syncthreads();
  for (int x = d; x < 64; x += DP) {
    const int i = x >> 3, m = x & 7;
    float s = 0.f;
    for (int j = m; j <= i; ++j) s += G[i * 8 + j] * Tm[j * 8 + m];
    o.pt[row * 8 + x] = s;
  }
#pragma unroll
  for (int m = 0; m < kBlk; ++m) {
    float s = 0.f;
#pragma unroll
    for (int j = m; j < kBlk; ++j) s += Tm[j * 8 + m] * e[j];
    o.kh[(row + m) * DP + d] = s;
  }
}

JS_DEVICE void df_cp16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
JS_DEVICE void df_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
JS_DEVICE void df_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int kBlkStages = 6;

// The walk over the blocks of one (sequence, head): a CTA holds 16 NV value columns of the state, KW warps an equal part of
// the key dimension each.  A warp keeps its piece TRANSPOSED as the accumulators of 16 (values) x 8 (keys) tiles.  The column
// order of an accumulator tile differs from the one an A operand wants, but as long as the B operand takes its rows in the
// same order the sum over them is the same, so the state feeds the next product straight from the accumulators:
//
//   per block   [K part | Q part] (values x 8 rows) = S^T [kt | qt]^T   partial sums over the warp's keys, added across warps
//               W^T = bv^T - K part;  O^T = Q part + W^T pt^T;  S^T = S^T ge + W^T kh
template <int DP, int NV, int KW>
__global__ void __launch_bounds__(32 * KW * NV)
delta_block_kernel(DeltaIn in, DeltaBlocks o, float* state, float* out) {
  constexpr int NT = DP / (8 * KW);             // key tiles of 8 a warp holds
  constexpr int LK = DP + 8, LH = DP + 4, LV = 16 * NV + 4;       // row strides without bank conflicts for their readers
  constexpr int THREADS = 32 * KW * NV, HALF = NV * KW * 64;
  struct __align__(16) Stage {
    float kt[kBlk][LK], qt[kBlk][LK], kh[kBlk][LH], ge[DP], bv[kBlk][LV], pt[64];
  };
  extern __shared__ __align__(16) uint8_t raw[];
  Stage* sm = reinterpret_cast<Stage*>(raw);
  float4* part = reinterpret_cast<float4*>(raw + sizeof(Stage) * kBlkStages);      // [2][NV][KW][K, Q][32]
  pdl_launch_dependents();
  pdl_wait();
  const int slice = blockIdx.x, h = blockIdx.y, sq = blockIdx.z, tid = threadIdx.x, lane = tid & 31;
  const int kw = (tid >> 5) % KW, vt = (tid >> 5) / KW;
  const int gr = lane >> 2, qd = lane & 3;
  const int q0 = in.cu_q[sq], n = in.cu_q[sq + 1] - q0;
  if (n <= 0) return;
  const int D = in.D, V = in.V, past = in.past_lens[sq], slot = in.rows[sq];
  const int tile0 = q0 / kBlk + sq, nb = (n + kBlk - 1) / kBlk;
  const size_t row0 = static_cast<size_t>(h) * o.R + static_cast<size_t>(tile0) * kBlk;
  float* st = state + (static_cast<size_t>(slot) * in.H + h) * D * V;
  const int v0 = slice * 16 * NV + vt * 16 + gr;          // this lane's value columns: v0 and v0 + 8
  const int dw = kw * (DP / KW);                          // first key of the warp

  auto stage_in = [&](int b) {
    Stage& s = sm[b % kBlkStages];
    const size_t row = row0 + static_cast<size_t>(b) * kBlk;
    constexpr int CH = DP / 4;                            // 16-byte chunks of a row
    for (int x = tid; x < kBlk * CH; x += THREADS) {
      const int i = x / CH, c = x % CH * 4;
      df_cp16(&s.kt[i][c], o.kt + (row + i) * DP + c);
      df_cp16(&s.qt[i][c], o.qt + (row + i) * DP + c);
      df_cp16(&s.kh[i][c], o.kh + (row + i) * DP + c);
    }
    const float* ge = o.ge + (static_cast<size_t>(h) * (o.R / kBlk) + tile0 + b) * DP;
    if (tid < CH) df_cp16(s.ge + 4 * tid, ge + 4 * tid);
    else if (tid >= 64 && tid < 80) df_cp16(s.pt + 4 * (tid - 64), o.pt + row * 8 + 4 * (tid - 64));
    else if (tid >= 96 && tid < 128) {
      for (int x = tid - 96; x < kBlk * 4 * NV; x += 32) {
        const int i = x / (4 * NV), c = x % (4 * NV) * 4;
        if (slice * 16 * NV + c < V) df_cp16(&s.bv[i][c], o.bv + (row + i) * V + slice * 16 * NV + c);
      }
    }
  };
  for (int b = 0; b < kBlkStages - 1; ++b) {
    if (b < nb) stage_in(b);
    df_commit();
  }
  float S[NT][4];                       // (v0, d), (v0, d + 1), (v0 + 8, d), (v0 + 8, d + 1), d = dw + 8 nt + 2 qd
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = dw + 8 * nt + 2 * qd + (e & 1), v = v0 + (e >> 1) * 8;
      S[nt][e] = (past > 0 && d < D && v < V) ? st[static_cast<size_t>(d) * V + v] : 0.f;
    }
  // three accumulators, not one: the chain of dependent products is what a block waits for
  auto fold = [](const float (&x)[3][4]) {
    return make_float4(x[0][0] + (x[1][0] + x[2][0]), x[0][1] + (x[1][1] + x[2][1]), x[0][2] + (x[1][2] + x[2][2]),
                       x[0][3] + (x[1][3] + x[2][3]));
  };
  // (P T) of block b as a B operand: read while the block's stage is still there, used one block later
  float4* pmine = part + vt * KW * 64 + kw * 64 + lane;
  auto gather = [&](const float4* pb) {         // sum of a part over the warps, in warp order
    float4 t = pb[0];
#pragma unroll
    for (int w = 1; w < KW; ++w) {
      const float4 x = pb[w * 64];
      t = make_float4(t.x + x.x, t.y + x.y, t.z + x.z, t.w + x.w);
    }
    return t;
  };
  uint32_t wh[4] = {}, wl[4] = {};      // W^T of the block before, split, as an A operand
  float2 pt_prev = make_float2(0.f, 0.f);
  // the read-outs of a block: its Q parts were exchanged at the barrier behind it; the warps take turns
  auto read_out = [&](int b) {
    if (kw != (b & (KW - 1))) return;
    const float4 q4 = gather(part + ((b + 1) & 1) * HALF + vt * KW * 64 + 32 + lane);
    float O[4] = {q4.x, q4.y, q4.z, q4.w};
    uint32_t h0, l0, h1, l1;
    tf32_split(pt_prev.x, h0, l0);
    tf32_split(pt_prev.y, h1, l1);
    float low[4];
    mma_tf32_first(low, wh, l0, l1);
    mma_tf32(low, wl, h0, h1);
    mma_tf32(O, wh, h0, h1);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = b * kBlk + 2 * qd + (e & 1), v = v0 + (e >> 1) * 8;
      if (i < n && v < V) out[(static_cast<size_t>(q0 + i) * in.H + h) * V + v] = O[e] + low[e];
    }
  };
  df_wait<kBlkStages - 2>();
  __syncthreads();
  for (int b = 0; b < nb; ++b) {
    const Stage& s = sm[b % kBlkStages];
    // ---- K part of block b, on the way to the barrier
    uint32_t sh[NT][4], sl[NT][4];
    {
      float ak[3][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const float2 kv = *reinterpret_cast<const float2*>(&s.kt[gr][dw + 8 * nt + 2 * qd]);
        tf32_split(S[nt][0], sh[nt][0], sl[nt][0]);
        tf32_split(S[nt][2], sh[nt][1], sl[nt][1]);
        tf32_split(S[nt][1], sh[nt][2], sl[nt][2]);
        tf32_split(S[nt][3], sh[nt][3], sl[nt][3]);
        uint32_t h0, l0, h1, l1;
        tf32_split(kv.x, h0, l0);
        tf32_split(kv.y, h1, l1);
        if (nt == 0) {
          mma_tf32_first(ak[0], sh[nt], h0, h1);
          mma_tf32_first(ak[1], sh[nt], l0, l1);
          mma_tf32_first(ak[2], sl[nt], h0, h1);
        } else {
          mma_tf32(ak[0], sh[nt], h0, h1);
          mma_tf32(ak[1], sh[nt], l0, l1);
          mma_tf32(ak[2], sl[nt], h0, h1);
        }
      }
      pmine[(b & 1) * HALF] = fold(ak);
    }
    df_wait<kBlkStages - 3>();          // block b + 1 is here too
    __syncthreads();                    // ... for everyone, with all K parts of block b and all Q parts of block b - 1
    const float4 k4 = gather(part + (b & 1) * HALF + vt * KW * 64 + lane);
    // ---- Q part of block b from the state before it; exchanged at the next barrier
    {
      float aq[3][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const float2 qv = *reinterpret_cast<const float2*>(&s.qt[gr][dw + 8 * nt + 2 * qd]);
        uint32_t h0, l0, h1, l1;
        tf32_split(qv.x, h0, l0);
        tf32_split(qv.y, h1, l1);
        if (nt == 0) {
          mma_tf32_first(aq[0], sh[nt], h0, h1);
          mma_tf32_first(aq[1], sh[nt], l0, l1);
          mma_tf32_first(aq[2], sl[nt], h0, h1);
        } else {
          mma_tf32(aq[0], sh[nt], h0, h1);
          mma_tf32(aq[1], sh[nt], l0, l1);
          mma_tf32(aq[2], sl[nt], h0, h1);
        }
      }
      if (b > 0) read_out(b - 1);       // reads the Q parts of block b - 1 from the other half of `part`
      pmine[((b + 1) & 1) * HALF + 32] = fold(aq);
    }
    // ---- W and the state's step
    {
      const int c = vt * 16 + gr;
      tf32_split(s.bv[2 * qd][c] - k4.x, wh[0], wl[0]);
      tf32_split(s.bv[2 * qd][c + 8] - k4.z, wh[1], wl[1]);
      tf32_split(s.bv[2 * qd + 1][c] - k4.y, wh[2], wl[2]);
      tf32_split(s.bv[2 * qd + 1][c + 8] - k4.w, wh[3], wl[3]);
    }
    pt_prev = *reinterpret_cast<const float2*>(&s.pt[gr * 8 + 2 * qd]);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int d = dw + 8 * nt;
      const float2 gv = *reinterpret_cast<const float2*>(&s.ge[d + 2 * qd]);
      uint32_t h0, l0, h1, l1;
      tf32_split(s.kh[2 * qd][d + gr], h0, l0);
      tf32_split(s.kh[2 * qd + 1][d + gr], h1, l1);
      float low[4];
      mma_tf32_first(low, wh, l0, l1);
      mma_tf32(low, wl, h0, h1);
#pragma unroll
      for (int e = 0; e < 4; ++e) S[nt][e] = fmaf(S[nt][e], (e & 1) ? gv.y : gv.x, low[e]);
      mma_tf32(S[nt], wh, h0, h1);
    }
    // the buffer of block b - 1 is free: everyone passed this block's barrier
    if (b + kBlkStages - 1 < nb) stage_in(b + kBlkStages - 1);
    df_commit();
  }
  __syncthreads();
  read_out(nb - 1);
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = dw + 8 * nt + 2 * qd + (e & 1), v = v0 + (e >> 1) * 8;
      if (d < D && v < V) st[static_cast<size_t>(d) * V + v] = S[nt][e];
    }
  // the last rows' convolution inputs; every reader of the ring ran in the kernel before
  if (in.taps > 1) {
    constexpr int NCOL = 16 * NV;
    const int C = 2 * in.G * D + in.H * V, g = h / (in.H / in.G);
    const int qk = slice == 0 && h % (in.H / in.G) == 0 ? 2 * D : 0;
    __nv_bfloat16* ring = in.conv + static_cast<size_t>(slot) * in.taps * C;
    for (int x = tid; x < NCOL + qk; x += THREADS) {
      if (x < NCOL && slice * NCOL + x >= V) continue;
      const int y = x - NCOL;
      const int c = x < NCOL ? 2 * in.G * D + h * V + slice * NCOL + x : y < D ? g * D + y : (in.G + g) * D + y - D;
      for (int i = max(0, n - in.taps + 1); i < n; ++i)
        ring[static_cast<size_t>((past + i) % in.taps) * C + c] = in.pre[static_cast<size_t>(q0 + i) * in.ldp + c];
    }
  }
}

struct FusedLaunch {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a;
  FusedLaunch(dim3 grid, dim3 block, cudaStream_t stream, int pdl, size_t smem = 0) {
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

template <int DP, int NV, int KW>
static int launch_blocks(const DeltaIn& in, const DeltaBlocks& o, float* state, float* out, int pdl, cudaStream_t stream) {
  constexpr int smem = kBlkStages * (kBlk * (3 * DP + 20 + 16 * NV + 4) + DP + 64) * 4 + 2 * NV * KW * 64 * 16;
  static int configured[kMaxDevicesCached] = {};
  auto kern = delta_block_kernel<DP, NV, KW>;
  if (ensure_dyn_smem(kern, smem, configured) != 0) return -3;
  FusedLaunch l(dim3((in.V + 16 * NV - 1) / (16 * NV), in.H, in.B), dim3(32 * KW * NV), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, kern, in, o, state, out) == cudaSuccess ? 0 : -4;
}

template <int DP>
static int launch_block_prep(const DeltaIn& in, const DeltaBlocks& o, int tiles, int pdl, cudaStream_t stream) {
  FusedLaunch l(dim3(tiles, in.H), dim3(DP), stream, pdl);
  auto kern = in.channel ? (in.taps <= 4 ? delta_block_prep_kernel<DP, true, 4> : delta_block_prep_kernel<DP, true, kBlkMaxTaps>)
                         : (in.taps <= 4 ? delta_block_prep_kernel<DP, false, 4> : delta_block_prep_kernel<DP, false, kBlkMaxTaps>);
  return cudaLaunchKernelEx(&l.c, kern, in, o) == cudaSuccess ? 0 : -4;
}

static bool fused_shape_ok(int H, int G, int D, int V, int taps) {
  return H > 0 && G > 0 && H % G == 0 && D > 0 && V > 0 && V % 4 == 0 && taps >= 1 && taps <= kBlkMaxTaps;
}

}  // namespace js

// One row per sequence, bf16: T = B rows.  Needs V % 4 == 0, V <= 256 and D * (V rounded up to a power of two) <= 16384 (D is
// covered by at most 16 rows a thread).  gate (T, ldg), norm_w (V), out (T, ldo) bf16.
extern "C" int js_delta_step(int H, int G, int D, int V, int ntaps, int channel, const void* pre, int ldp, const float* z, int ldz,
                             const float* b, int ldb, const void* taps, const void* A_log, const void* dt_bias, void* conv, float* state,
                             const int* rows, const int* cu_q, const int* past_lens, int B, const void* gate, int ldg, const void* norm_w,
                             int silu, float eps, void* out, int ldo, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0) return 0;
  if (!fused_shape_ok(H, G, D, V, ntaps) || V > 256 || D > 256) return -10;
  int VG = 1;
  while (4 * VG < V) VG *= 2;
  const int RL = kStepThreads / VG, NR = (D + RL - 1) / RL;
  using bf = __nv_bfloat16;
  DeltaStepParams p{};
  p.in = DeltaIn{H, G, D, V, ntaps, channel, (const bf*)pre, z, b, ldp, ldz, ldb, (const bf*)taps, (const bf*)A_log, (const bf*)dt_bias,
                 (bf*)conv, rows, cu_q, past_lens, B};
  p.state = state; p.gate = (const bf*)gate; p.norm_w = (const bf*)norm_w; p.out = (bf*)out;
  p.ldg = ldg; p.ldo = ldo; p.silu = silu; p.eps = eps;
  FusedLaunch l(dim3(H, B), dim3(kStepThreads), stream, pdl);
  if (NR > 16) return -10;
  auto kern = NR <= 4 ? delta_step_kernel<4> : NR <= 8 ? delta_step_kernel<8> : delta_step_kernel<16>;
  return cudaLaunchKernelEx(&l.c, kern, p, VG) == cudaSuccess ? 0 : -4;
}

// Prompt portions in blocks of 8 rows, bf16 inputs; D <= 128, V % 4 == 0.  R = 8 * (T / 8 + B) padded rows; kt, qt, kh (H, R, DP),
// ge (H, R / 8, DP) with DP = 64 or 128; bv (H, R, V); pt (H, R, 8); out (T, H, V) fp32.  wide: 32 value columns a CTA, not 16.
extern "C" int js_delta_blocks(int H, int G, int D, int V, int ntaps, int channel, const void* pre, int ldp, const float* z, int ldz,
                               const float* b, int ldb, const void* taps, const void* A_log, const void* dt_bias, void* conv, float* state,
                               const int* rows, const int* cu_q, const int* past_lens, int B, int T, float* kt, float* qt, float* kh,
                               float* bv, float* pt, float* ge, float* out, int wide, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || B <= 0) return 0;
  if (!fused_shape_ok(H, G, D, V, ntaps) || D > 128) return -10;
  using bf = __nv_bfloat16;
  const DeltaIn in{H, G, D, V, ntaps, channel, (const bf*)pre, z, b, ldp, ldz, ldb, (const bf*)taps, (const bf*)A_log, (const bf*)dt_bias,
                   (bf*)conv, rows, cu_q, past_lens, B};
  const int tiles = T / kBlk + B;
  const DeltaBlocks o{kt, qt, kh, bv, pt, ge, tiles * kBlk};
  if (D <= 64) {
    if (int rc = launch_block_prep<64>(in, o, tiles, pdl, stream)) return rc;
    return launch_blocks<64, 1, 4>(in, o, state, out, pdl, stream);
  }
  if (int rc = launch_block_prep<128>(in, o, tiles, pdl, stream)) return rc;
  return wide ? launch_blocks<128, 2, 4>(in, o, state, out, pdl, stream) : launch_blocks<128, 1, 4>(in, o, state, out, pdl, stream);
}
