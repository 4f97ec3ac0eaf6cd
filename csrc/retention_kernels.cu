// Retention: linear attention with one fixed decay per head,  S <- d S + k v^T,  o = S^T q  (per head, S is dim x vdim, fp32),
// from bf16 projections [q | k | v | gate] with rotary q and k, followed by a per-head norm without a weight and a silu gate.
// Everything that enters the recurrence is fp32.  With a fixed decay nothing but the state links rows that are far apart:
//
//   step    one row per sequence (decode): rotation to gated norm in one kernel, the state read once and written once; the CTAs of
//           a cluster share a head's value columns and add up the norm's sum of squares;
//   chunks  portions, in chunks of 128 rows.  With i, j counted inside a chunk of n rows and S the state before it:
//             U   = sum_j d^(n-1-j) k_j v_j^T                                  every chunk on its own      (retention_update)
//             S_c = d^n S_(c-1) + U_c                                          elementwise over the chunks (retention_scan)
//             o_i = d^(i+1) S^T q_i + sum_(j<=i) d^(i-j) (q_i k_j) v_j         every 64 rows on their own  (retention_rows)
//           the last kernel holds all value columns of its rows, so the norm and the gate are its epilogue;
//   tree    retention_rows alone: the sum runs over a node's ancestors (packed bits), powers count the path between them, the
//           stored state stays as it is; retention_path then advances it along the accepted nodes.
//
// Products run on the tensor cores from split tf32 operands (tf32_split.cuh): three per product of two fp32 numbers, two where
// one factor is a value row, which bf16 makes exact.  Powers of the decays come from a table made in double precision.
#include "tf32_split.cuh"

#include <math.h>

namespace js {

constexpr int kRetTile = 64;             // rows per CTA of retention_rows
constexpr int kRetChunk = 128;           // rows between stored states
constexpr int kRetPow = 257;             // powers 0 .. 256 of every head's decay
constexpr int kRetThreads = 256;

struct RetIn {
  int H, D, V, n;                        // n rotated pairs (i, i + n)
  const __nv_bfloat16* act;              // (T, ldp): q heads at column 0, k at kc, v at vc, gate at gc
  int ldp, kc, vc, gc;
  const float2* rot;                     // (T, ldr): this layer's (cos, sin)
  int ldr;
  const float* pw;                       // (H, kRetPow)
  const int *rows, *cu_q, *past_lens;
  int B;
  float k_scale;
};

JS_DEVICE float ret_silu(float z) { return z / (1.f + expf(-z)); }

// One warp: a head's row, rotated and scaled, to dst[0 .. DP); entries past D are zero.  A row that does not exist gives zeros.
template <int DP>
JS_DEVICE void ret_load_row(const RetIn& p, const __nv_bfloat16* src, const float2* rot, float scale, bool valid, float* dst) {
  const int lane = threadIdx.x & 31, n = p.n, D = p.D;
  if (!valid) {
    for (int e = lane; e < DP; e += 32) dst[e] = 0.f;
    return;
  }
  if (((n | D | p.ldp | p.ldr) & 1) == 0) {
    for (int e = 2 * lane; e < n; e += 64) {
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e + n));
      const float4 cs = *reinterpret_cast<const float4*>(rot + e);
      *reinterpret_cast<float2*>(dst + e) = make_float2((a.x * cs.x - b.x * cs.y) * scale, (a.y * cs.z - b.y * cs.w) * scale);
      *reinterpret_cast<float2*>(dst + e + n) = make_float2((b.x * cs.x + a.x * cs.y) * scale, (b.y * cs.z + a.y * cs.w) * scale);
    }
  } else {
    for (int e = lane; e < n; e += 32) {
      const float a = __bfloat162float(src[e]), b = __bfloat162float(src[e + n]);
      const float2 cs = rot[e];
      dst[e] = (a * cs.x - b * cs.y) * scale;
      dst[e + n] = (b * cs.x + a * cs.y) * scale;
    }
  }
  for (int e = 2 * n + lane; e < DP; e += 32) dst[e] = e < D ? __bfloat162float(src[e]) * scale : 0.f;
}

JS_DEVICE void ret_cp16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
JS_DEVICE void ret_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
JS_DEVICE void ret_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// The whole CTA: ROWS rows from token t0 on of the head whose columns start at col, rotated and times scale(row), to dst[row][LD];
// rows from `rows` on are zero.  A warp takes every eighth row, four at a time, so that their loads overlap.
template <int DP, int LD, int ROWS, typename F>
JS_DEVICE void ret_load_rows(const RetIn& p, int col, size_t t0, int rows, F scale, float* dst) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = p.n, D = p.D, e = 2 * lane;
  if (((n | D | p.ldp | p.ldr) & 1) != 0) {
    for (int r = warp; r < ROWS; r += 8) {
      const bool ok = r < rows;
      const size_t t = t0 + (ok ? r : 0);
      ret_load_row<DP>(p, p.act + t * p.ldp + col, p.rot + t * p.ldr, ok ? scale(r) : 0.f, ok, dst + r * LD);
    }
    return;
  }
  constexpr int BATCH = 4;
  static_assert(DP <= 128 && ROWS % (8 * BATCH) == 0, "a lane covers a row's pairs at once");
  for (int r0 = warp; r0 < ROWS; r0 += 8 * BATCH) {
    uint32_t a[BATCH] = {}, b[BATCH] = {}, c[BATCH][2] = {};
    float4 cs[BATCH];
    float f[BATCH];
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int r = r0 + 8 * i;
      const bool ok = r < rows;
      const size_t t = t0 + (ok ? r : 0);
      const __nv_bfloat16* src = p.act + t * p.ldp + col;
      cs[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok && e < n) {
        a[i] = *reinterpret_cast<const uint32_t*>(src + e);
        b[i] = *reinterpret_cast<const uint32_t*>(src + e + n);
        cs[i] = *reinterpret_cast<const float4*>(p.rot + t * p.ldr + e);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (ok && 2 * n + e + 64 * j < D) c[i][j] = *reinterpret_cast<const uint32_t*>(src + 2 * n + e + 64 * j);
      f[i] = ok ? scale(r) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      float* out = dst + (r0 + 8 * i) * LD;
      if (e < n) {
        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[i])), v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&b[i]));
        *reinterpret_cast<float2*>(out + e) = make_float2((u.x * cs[i].x - v.x * cs[i].y) * f[i], (u.y * cs[i].z - v.y * cs[i].w) * f[i]);
        *reinterpret_cast<float2*>(out + e + n) = make_float2((v.x * cs[i].x + u.x * cs[i].y) * f[i], (v.y * cs[i].z + u.y * cs[i].w) * f[i]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (2 * n + e + 64 * j < DP) {       // entries past D are zero
          const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&c[i][j]));
          *reinterpret_cast<float2*>(out + 2 * n + e + 64 * j) = make_float2(u.x * f[i], u.y * f[i]);
        }
    }
  }
}

// ROWS value rows of a head (columns [v0, v0 + VT)) to dst[row][LV], zeros where they do not exist; the caller waits for the copies
template <int VT, int LV, int ROWS>
JS_DEVICE void ret_load_values(const RetIn& p, const __nv_bfloat16* src, int rows, int v0, __nv_bfloat16* dst) {
  if (((p.V | p.ldp | v0) & 7) == 0) {
    for (int x = threadIdx.x; x < ROWS * (VT / 8); x += kRetThreads) {
      const int r = x / (VT / 8), c = x % (VT / 8) * 8;
      const bool ok = r < rows && v0 + c < p.V;
      ret_cp16(dst + r * LV + c, ok ? src + static_cast<size_t>(r) * p.ldp + v0 + c : src, ok);
    }
  } else {
    for (int x = threadIdx.x; x < ROWS * VT; x += kRetThreads) {
      const int r = x / VT, c = x % VT;
      dst[r * LV + c] = r < rows && v0 + c < p.V ? src[static_cast<size_t>(r) * p.ldp + v0 + c] : __float2bfloat16_rn(0.f);
    }
  }
  ret_commit();
}

// sequence of a tile when sequence s starts at tile cu_q[s] / size + s
JS_DEVICE int ret_find(const int* cu_q, int B, int tile, int size) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] / size + mid <= tile) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// Value columns are dealt to accumulator tiles in pairs: column 2 gr of a group of 16 goes to the even tile and 2 gr + 1 to the odd
// one, so a lane reads both tiles' operands with one load and holds four consecutive columns 4 qd .. 4 qd + 3 of the result.
JS_DEVICE void ret_values(const __nv_bfloat16* base, uint32_t& even, uint32_t& odd) {
  const uint32_t w = *reinterpret_cast<const uint32_t*>(base);
  even = w << 16;
  odd = w & 0xffff0000u;
}

// ================================================================ U of every chunk
// grid (chunks, H, ceil(V / VT)).  U (chunks, H, D, V) fp32.
template <int DP, int VT>
__global__ void __launch_bounds__(kRetThreads, 2) retention_update_kernel(RetIn p, float* U) {
  constexpr int MW = DP / 16, NG = 8 / MW, NT = VT / NG / 8, LK = DP + 8, LV = VT + 16;
  extern __shared__ __align__(16) uint8_t raw[];
  float* sK = reinterpret_cast<float*>(raw);                               // [128][LK]
  __nv_bfloat16* sV = reinterpret_cast<__nv_bfloat16*>(sK + kRetChunk * LK);   // [128][LV]
  pdl_launch_dependents();
  pdl_wait();
  const int tile = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gr = lane >> 2, qd = lane & 3;
  const int s = ret_find(p.cu_q, p.B, tile, kRetChunk);
  const int q0 = p.cu_q[s], n_seq = p.cu_q[s + 1] - q0, r0 = (tile - (q0 / kRetChunk + s)) * kRetChunk;
  if (r0 >= n_seq) return;
  const int n = min(kRetChunk, n_seq - r0);
  const float* pw = p.pw + h * kRetPow;
  const int d0 = (warp % MW) * 16, c0 = (warp / MW) * (VT / NG);
  float acc[NT][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
  const size_t t0 = q0 + r0;
  ret_load_values<VT, LV, kRetChunk>(p, p.act + t0 * p.ldp + p.vc + h * p.V, n, v0, sV);
  ret_load_rows<DP, LK, kRetChunk>(p, p.kc + h * p.D, t0, n, [&](int r) { return p.k_scale * pw[n - 1 - r]; }, sK);
  ret_wait<0>();
  __syncthreads();
#pragma unroll 2
  for (int j = 0; j < kRetChunk; j += 8) {
    if (j >= n) break;
    uint32_t ah[4], al[4];
    tf32_split(sK[(j + qd) * LK + d0 + gr], ah[0], al[0]);
    tf32_split(sK[(j + qd) * LK + d0 + gr + 8], ah[1], al[1]);
    tf32_split(sK[(j + qd + 4) * LK + d0 + gr], ah[2], al[2]);
    tf32_split(sK[(j + qd + 4) * LK + d0 + gr + 8], ah[3], al[3]);
#pragma unroll
    for (int t = 0; t < NT; t += 2) {
      uint32_t e0, o0, e1, o1;
      const __nv_bfloat16* b = sV + (j + qd) * LV + c0 + 8 * t + 2 * gr;
      ret_values(b, e0, o0);
      ret_values(b + 4 * LV, e1, o1);
      mma_tf32(acc[t], al, e0, e1);
      mma_tf32(acc[t], ah, e0, e1);
      mma_tf32(acc[t + 1], al, o0, o1);
      mma_tf32(acc[t + 1], ah, o0, o1);
    }
  }
  float* dst = U + (static_cast<size_t>(tile) * p.H + h) * p.D * p.V;
#pragma unroll
  for (int t = 0; t < NT; t += 2)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int d = d0 + gr + 8 * half, c = v0 + c0 + 8 * t + 4 * qd;
      if (d >= p.D) continue;
      const float v[4] = {acc[t][2 * half], acc[t + 1][2 * half], acc[t][2 * half + 1], acc[t + 1][2 * half + 1]};
      float* o = dst + static_cast<size_t>(d) * p.V + c;
      if ((p.V & 3) == 0) {
        if (c < p.V) *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]);
      } else {
        for (int e = 0; e < 4; ++e)
          if (c + e < p.V) o[e] = v[e];
      }
    }
}

// ================================================================ the states before every chunk (in place of U), and the last one
__global__ void __launch_bounds__(kRetThreads) retention_scan_kernel(RetIn p, float* U, float* state) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, s = blockIdx.z, N = p.D * p.V;
  const int x = (blockIdx.x * kRetThreads + threadIdx.x) * 4;
  const int q0 = p.cu_q[s], n_seq = p.cu_q[s + 1] - q0;
  if (n_seq <= 0 || x >= N) return;
  const int chunks = (n_seq + kRetChunk - 1) / kRetChunk;
  const float* pw = p.pw + h * kRetPow;
  float* st = state + (static_cast<size_t>(p.rows[s]) * p.H + h) * N + x;
  float* u = U + (static_cast<size_t>(q0 / kRetChunk + s) * p.H + h) * N + x;
  const size_t step = static_cast<size_t>(p.H) * N;
  const bool fresh = p.past_lens[s] == 0;
  const float full = pw[kRetChunk], tail = pw[n_seq - (chunks - 1) * kRetChunk];
  if ((N & 3) == 0) {
    float4 S = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
    constexpr int BATCH = 8;             // loads in flight
    for (int c0 = 0; c0 < chunks; c0 += BATCH) {
      float4 a[BATCH];
#pragma unroll
      for (int i = 0; i < BATCH; ++i)
        if (c0 + i < chunks) a[i] = *reinterpret_cast<const float4*>(u + (c0 + i) * step);
#pragma unroll
      for (int i = 0; i < BATCH; ++i) {
        if (c0 + i >= chunks) break;
        const float d = c0 + i + 1 < chunks ? full : tail;
        *reinterpret_cast<float4*>(u + (c0 + i) * step) = S;
        S = make_float4(fmaf(d, S.x, a[i].x), fmaf(d, S.y, a[i].y), fmaf(d, S.z, a[i].z), fmaf(d, S.w, a[i].w));
      }
    }
    *reinterpret_cast<float4*>(st) = S;
  } else {
    for (int e = 0; e < 4 && x + e < N; ++e) {
      float S = fresh ? 0.f : st[e];
      for (int c = 0; c < chunks; ++c) {
        const float a = u[c * step + e];
        u[c * step + e] = S;
        S = fmaf(c + 1 < chunks ? full : tail, S, a);
      }
      st[e] = S;
    }
  }
}

// ================================================================ the rows
// grid (tiles of 64 rows, H).  prefix: states before the chunks (chunks, H, D, V); with mask_bits (T, W) a token tree, whose prefix is
// the sequence's own state (slots, H, D, V).  out (T, ldo) bf16, head h at column h * V.
template <int DP, int VP>
__global__ void __launch_bounds__(kRetThreads, VP >= 128 ? 2 : 3)
retention_rows_kernel(RetIn p, const float* prefix, const int* mask_bits, int W, float eps, __nv_bfloat16* out, int ldo) {
  constexpr int NT = VP / 16, LQ = DP + 4, LP = kRetTile + 4, LV = VP + 16, LS = VP + 8;
  constexpr int SROWS = DP <= 64 && VP >= 256 ? 16 : 32;      // state rows per slab
  extern __shared__ __align__(16) uint8_t raw[];
  float* sQ = reinterpret_cast<float*>(raw);                               // [64][LQ]
  float* sK = sQ + kRetTile * LQ;                                          // [64][LQ], later the weights [64][LP]
  __nv_bfloat16* sV = reinterpret_cast<__nv_bfloat16*>(sK + kRetTile * LQ);    // [64][LV]
  float* sS = sK;                                                          // two slabs [SROWS][LS], before the first key tile
  __shared__ float spw[kRetPow], ssum[kRetTile][2];
  __shared__ unsigned smask[kRetTile][8];
  __shared__ int sdep[256];
  static_assert(LP <= LQ, "the weights fit the keys' place");
  static_assert(2 * SROWS * LS * 4 <= kRetTile * (LQ * 4 + LV * 2), "two slabs fit the keys' and values' place");
  pdl_launch_dependents();
  pdl_wait();
  const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gr = lane >> 2, qd = lane & 3, rg = (warp & 3) * 16, ch = warp >> 2, D = p.D, V = p.V;
  const int s = ret_find(p.cu_q, p.B, tile, kRetTile);
  const int q0 = p.cu_q[s], n_seq = p.cu_q[s + 1] - q0, lt = tile - (q0 / kRetTile + s), r0 = lt * kRetTile;
  if (r0 >= n_seq) return;
  const bool tree = mask_bits != nullptr;
  const int past = p.past_lens[s], n = min(kRetTile, n_seq - r0);
  const int chunk = r0 / kRetChunk, first = tree ? 0 : chunk * kRetChunk;       // first key row
  const float* S = tree ? prefix + (static_cast<size_t>(p.rows[s]) * p.H + h) * D * V
                        : prefix + (static_cast<size_t>(q0 / kRetChunk + s + chunk) * p.H + h) * D * V;
  const bool has_state = past > 0 || (!tree && chunk > 0);
  for (int x = tid; x < kRetPow; x += kRetThreads) spw[x] = p.pw[h * kRetPow + x];
  if (tree) {
    for (int x = tid; x < min(n_seq, 256); x += kRetThreads) {
      int c = 0;
      for (int w = 0; w < W; ++w) c += __popc(static_cast<unsigned>(mask_bits[static_cast<size_t>(q0 + x) * W + w]));
      sdep[x] = max(0, min(c, 256) - 1);
    }
    for (int x = tid; x < kRetTile * 8; x += kRetThreads) {
      const int r = x >> 3, w = x & 7;
      smask[r][w] = r < n && w < W ? static_cast<unsigned>(mask_bits[static_cast<size_t>(q0 + r0 + r) * W + w]) : 0u;
    }
  }
  auto load_slab = [&](int d0, float* dst) {
    if ((V & 3) == 0) {
      for (int x = tid; x < SROWS * (VP / 4); x += kRetThreads) {
        const int r = x / (VP / 4), c = x % (VP / 4) * 4;
        const bool ok = d0 + r < D && c < V;
        ret_cp16(dst + r * LS + c, ok ? S + static_cast<size_t>(d0 + r) * V + c : S, ok);
      }
    } else {
      for (int x = tid; x < SROWS * VP; x += kRetThreads) {
        const int r = x / VP, c = x % VP;
        dst[r * LS + c] = d0 + r < D && c < V ? S[static_cast<size_t>(d0 + r) * V + c] : 0.f;
      }
    }
    ret_commit();
  };
  if (has_state) load_slab(0, sS);
  ret_load_rows<DP, LQ, kRetTile>(p, h * D, q0 + r0, n, [](int) { return 1.f; }, sQ);
  float acc[NT][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
  const int cw = ch * (VP / 2);          // first value column of the warp
  // ---- the state before the chunk
  if (has_state) {
    for (int d0 = 0, i = 0; d0 < D; d0 += SROWS, ++i) {
      if (i > 0) __syncthreads();        // the slab before has been read: its place takes the next one
      if (d0 + SROWS < D) {
        load_slab(d0 + SROWS, sS + ((i + 1) & 1) * SROWS * LS);
        ret_wait<1>();
      } else {
        ret_wait<0>();
      }
      __syncthreads();
      const float* slab = sS + (i & 1) * SROWS * LS;
#pragma unroll
      for (int k = 0; k < SROWS; k += 8) {
        uint32_t ah[4], al[4];
        tf32_split(sQ[(rg + gr) * LQ + d0 + k + qd], ah[0], al[0]);
        tf32_split(sQ[(rg + gr + 8) * LQ + d0 + k + qd], ah[1], al[1]);
        tf32_split(sQ[(rg + gr) * LQ + d0 + k + qd + 4], ah[2], al[2]);
        tf32_split(sQ[(rg + gr + 8) * LQ + d0 + k + qd + 4], ah[3], al[3]);
#pragma unroll
        for (int t = 0; t < NT; t += 2) {
          const float2 b0 = *reinterpret_cast<const float2*>(slab + (k + qd) * LS + cw + 8 * t + 2 * gr);
          const float2 b1 = *reinterpret_cast<const float2*>(slab + (k + qd + 4) * LS + cw + 8 * t + 2 * gr);
          uint32_t h0, l0, h1, l1;
          tf32_split(b0.x, h0, l0);
          tf32_split(b1.x, h1, l1);
          mma_tf32(acc[t], ah, l0, l1);
          mma_tf32(acc[t], al, h0, h1);
          mma_tf32(acc[t], ah, h0, h1);
          tf32_split(b0.y, h0, l0);
          tf32_split(b1.y, h1, l1);
          mma_tf32(acc[t + 1], ah, l0, l1);
          mma_tf32(acc[t + 1], al, h0, h1);
          mma_tf32(acc[t + 1], ah, h0, h1);
        }
      }
    }
    const int ra = rg + gr, rb = ra + 8;
    const float fa = ra < n ? spw[tree ? sdep[min(r0 + ra, 255)] + 1 : r0 + ra - first + 1] : 0.f;
    const float fb = rb < n ? spw[tree ? sdep[min(r0 + rb, 255)] + 1 : r0 + rb - first + 1] : 0.f;
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      acc[t][0] *= fa; acc[t][1] *= fa; acc[t][2] *= fb; acc[t][3] *= fb;
    }
  }
  // ---- keys of the chunk up to the tile's own rows
  for (int k0 = first; k0 <= r0; k0 += kRetTile) {
    const int nk = min(kRetTile, n_seq - k0);
    __syncthreads();
    ret_load_values<VP, LV, kRetTile>(p, p.act + static_cast<size_t>(q0 + k0) * p.ldp + p.vc + h * V, nk, 0, sV);
    ret_load_rows<DP, LQ, kRetTile>(p, p.kc + h * D, q0 + k0, nk, [&](int) { return p.k_scale; }, sK);
    __syncthreads();
    float w[4][4];                       // the warp's 16 rows against 32 of the keys
#pragma unroll
    for (int t = 0; t < 4; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) w[t][e] = 0.f;
#pragma unroll 2
    for (int k = 0; k < DP; k += 8) {
      uint32_t ah[4], al[4];
      tf32_split(sQ[(rg + gr) * LQ + k + qd], ah[0], al[0]);
      tf32_split(sQ[(rg + gr + 8) * LQ + k + qd], ah[1], al[1]);
      tf32_split(sQ[(rg + gr) * LQ + k + qd + 4], ah[2], al[2]);
      tf32_split(sQ[(rg + gr + 8) * LQ + k + qd + 4], ah[3], al[3]);
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        uint32_t h0, l0, h1, l1;
        const float* b = sK + (ch * 32 + 8 * t + gr) * LQ + k + qd;
        tf32_split(b[0], h0, l0);
        tf32_split(b[4], h1, l1);
        mma_tf32(w[t], ah, l0, l1);
        mma_tf32(w[t], al, h0, h1);
        mma_tf32(w[t], ah, h0, h1);
      }
    }
    __syncthreads();                     // the keys have been read
#pragma unroll
    for (int t = 0; t < 4; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = rg + gr + 8 * half, c = ch * 32 + 8 * t + 2 * qd;
        float f[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = r0 + r, j = k0 + c + e;
          if (tree) f[e] = r < n && j < n_seq && ((smask[r][(j >> 5) & 7] >> (j & 31)) & 1u) ? spw[max(0, sdep[min(i, 255)] - sdep[min(j, 255)])] : 0.f;
          else f[e] = r < n && j <= i ? spw[i - j] : 0.f;
        }
        *reinterpret_cast<float2*>(sK + r * LP + c) = make_float2(w[t][2 * half] * f[0], w[t][2 * half + 1] * f[1]);
      }
    ret_wait<0>();                       // the values
    __syncthreads();
#pragma unroll 2
    for (int j = 0; j < kRetTile; j += 8) {
      uint32_t ah[4], al[4];
      tf32_split(sK[(rg + gr) * LP + j + qd], ah[0], al[0]);
      tf32_split(sK[(rg + gr + 8) * LP + j + qd], ah[1], al[1]);
      tf32_split(sK[(rg + gr) * LP + j + qd + 4], ah[2], al[2]);
      tf32_split(sK[(rg + gr + 8) * LP + j + qd + 4], ah[3], al[3]);
#pragma unroll
      for (int t = 0; t < NT; t += 2) {
        uint32_t e0, o0, e1, o1;
        const __nv_bfloat16* b = sV + (j + qd) * LV + cw + 8 * t + 2 * gr;
        ret_values(b, e0, o0);
        ret_values(b + 4 * LV, e1, o1);
        mma_tf32(acc[t], al, e0, e1);
        mma_tf32(acc[t], ah, e0, e1);
        mma_tf32(acc[t + 1], al, o0, o1);
        mma_tf32(acc[t + 1], ah, o0, o1);
      }
    }
  }
  // ---- per-head norm and gate
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    sa += acc[t][0] * acc[t][0] + acc[t][1] * acc[t][1];
    sb += acc[t][2] * acc[t][2] + acc[t][3] * acc[t][3];
  }
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    sa += __shfl_xor_sync(0xffffffffu, sa, o);
    sb += __shfl_xor_sync(0xffffffffu, sb, o);
  }
  if (qd == 0) {
    ssum[rg + gr][ch] = sa;
    ssum[rg + gr + 8][ch] = sb;
  }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = rg + gr + 8 * half;
    if (r >= n) continue;
    const float inv = 1.f / sqrtf((ssum[r][0] + ssum[r][1]) / V + eps);
    const size_t t = q0 + r0 + r;
    const __nv_bfloat16* gate = p.act + t * p.ldp + p.gc + h * V;
    __nv_bfloat16* dst = out + t * ldo + h * V;
#pragma unroll
    for (int tt = 0; tt < NT; tt += 2) {
      const int c = cw + 8 * tt + 4 * qd;
      const float v[4] = {acc[tt][2 * half], acc[tt + 1][2 * half], acc[tt][2 * half + 1], acc[tt + 1][2 * half + 1]};
      if (((V | p.ldp | ldo) & 3) == 0) {
        if (c >= V) continue;
        const uint2 graw = *reinterpret_cast<const uint2*>(gate + c);
        const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.x));
        const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.y));
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0] * inv * ret_silu(g0.x), v[1] * inv * ret_silu(g0.y));
        const __nv_bfloat162 b = __floats2bfloat162_rn(v[2] * inv * ret_silu(g1.x), v[3] * inv * ret_silu(g1.y));
        *reinterpret_cast<uint2*>(dst + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
      } else {
        for (int e = 0; e < 4; ++e)
          if (c + e < V) dst[c + e] = __float2bfloat16_rn(v[e] * inv * ret_silu(__bfloat162float(gate[c + e])));
      }
    }
  }
}

// ================================================================ one row per sequence
// grid (CL * H, B), clusters of CL CTAs along x: CTA c of a cluster owns value columns [c VS, c VS + VS).  Thread (rl, cg): VEC columns
// from VEC cg on, state rows rl, rl + RL, ...
template <int VEC>
__global__ void __launch_bounds__(kRetThreads)
retention_step_kernel(RetIn p, float* state, float eps, __nv_bfloat16* out, int ldo, int CL, int VS, int VG) {
  __shared__ float sq[256], sk[256], sv[256], part[8];
  __shared__ __align__(16) float red[kRetThreads * VEC];
  pdl_launch_dependents();
  cluster_arrive();                      // waited for before the first store to a peer: it must have started by then
  pdl_wait();
  const int h = blockIdx.x / CL, rank = blockIdx.x % CL, t = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.D, V = p.V, v0 = rank * VS, vn = min(VS, V - v0);        // vn may be <= 0
  const int RL = kRetThreads / VG, cg = tid % VG, rl = tid / VG, col = VEC * cg;
  const int past = p.past_lens[t];
  const float d = p.pw[h * kRetPow + 1];
  const __nv_bfloat16* row = p.act + static_cast<size_t>(t) * p.ldp;
  if (warp < 2) ret_load_row<256>(p, row + (warp == 0 ? 0 : p.kc) + h * D, p.rot + static_cast<size_t>(t) * p.ldr, warp == 0 ? 1.f : p.k_scale, true, warp == 0 ? sq : sk);
  else
    for (int c = tid - 64; c < vn; c += kRetThreads - 64) sv[c] = __bfloat162float(row[p.vc + h * V + v0 + c]);
  __syncthreads();
  float o[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) o[e] = 0.f;
  if (col < vn) {
    float vv[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) vv[e] = sv[col + e];
    float* st = state + (static_cast<size_t>(p.rows[t]) * p.H + h) * D * V + v0 + col;
#pragma unroll 8
    for (int x = rl; x < D; x += RL) {
      float* sp = st + static_cast<size_t>(x) * V;
      float S[VEC];
      if constexpr (VEC == 4) {
        const float4 u = past > 0 ? *reinterpret_cast<const float4*>(sp) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[0] = u.x; S[1] = u.y; S[2] = u.z; S[3] = u.w;
      } else {
        S[0] = past > 0 ? *sp : 0.f;
      }
      const float kx = sk[x], qx = sq[x];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        S[e] = fmaf(d, S[e], kx * vv[e]);
        o[e] = fmaf(qx, S[e], o[e]);
      }
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(sp) = make_float4(S[0], S[1], S[2], S[3]);
      else *sp = S[0];
    }
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) red[rl * VG * VEC + col + e] = o[e];
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < vn; c += kRetThreads) {        // vn <= 256: at most one column a thread
    float x = 0.f;
    for (int i = 0; i < RL; ++i) x += red[i * VG * VEC + c];
    sv[c] = x;
    ss += x * x;
  }
  __syncthreads();
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  cluster_wait();
  if (tid < CL) {                        // the slice's sum to every CTA of the cluster
    float x = 0.f;
    for (int i = 0; i < kRetThreads / 32; ++i) x += red[i];
    st_dsmem_f32(map_to_cta(smem_u32(&part[rank]), tid), x);
  }
  __syncthreads();
  cluster_sync();
  float total = 0.f;
  for (int i = 0; i < CL; ++i) total += part[i];
  const float inv = 1.f / sqrtf(total / V + eps);
  for (int c = tid; c < vn; c += kRetThreads) {
    const float g = __bfloat162float(row[p.gc + h * V + v0 + c]);
    out[static_cast<size_t>(t) * ldo + h * V + v0 + c] = __float2bfloat16_rn(sv[c] * inv * ret_silu(g));
  }
}

// ================================================================ a state along the accepted nodes of a tree
// grid (H, ceil(V / 64)); path: rows of the only sequence, path_len of them; past_lens: the committed length behind the path.
__global__ void __launch_bounds__(kRetThreads) retention_path_kernel(RetIn p, float* state, const int* path, const int* path_len) {
  constexpr int PB = 16;
  __shared__ float sk[PB][256], sv[PB][64];
  __shared__ int sp[256];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, v0 = blockIdx.y * 64, tid = threadIdx.x, warp = tid >> 5, D = p.D, V = p.V;
  const int q0 = p.cu_q[0], n_rows = p.cu_q[1] - q0, n = max(0, min(*path_len, 256));
  if (n == 0 || n_rows <= 0) return;
  for (int x = tid; x < n; x += kRetThreads) sp[x] = max(0, min(path[x], n_rows - 1));
  const float* pw = p.pw + h * kRetPow;
  float* st = state + (static_cast<size_t>(p.rows[0]) * p.H + h) * D * V;
  const bool fresh = p.past_lens[0] - n <= 0;
  const int c = tid & 63, d0 = tid >> 6;                 // column c, state rows d0, d0 + 4, ...
  const bool cv = v0 + c < V;
  for (int b = 0; b < n; b += PB) {
    const int m = min(PB, n - b);
    __syncthreads();
    for (int r = warp; r < m; r += 8) {
      const size_t t = q0 + sp[b + r];
      ret_load_row<256>(p, p.act + t * p.ldp + p.kc + h * D, p.rot + t * p.ldr, p.k_scale * pw[m - 1 - r], true, sk[r]);
    }
    for (int x = tid; x < m * 64; x += kRetThreads) {
      const int r = x >> 6, cc = x & 63;
      sv[r][cc] = v0 + cc < V ? __bfloat162float(p.act[static_cast<size_t>(q0 + sp[b + r]) * p.ldp + p.vc + h * V + v0 + cc]) : 0.f;
    }
    __syncthreads();
    if (!cv) continue;
    const float f = pw[m];
    for (int d = d0; d < D; d += 4) {
      float* s = st + static_cast<size_t>(d) * V + v0 + c;
      float x = fresh && b == 0 ? 0.f : f * *s;
      for (int r = 0; r < m; ++r) x = fmaf(sk[r][d], sv[r][c], x);
      *s = x;
    }
  }
}

// ================================================================ rows for the row-by-row walk (delta_kernels.cu)
__global__ void __launch_bounds__(kRetThreads) retention_prep_kernel(RetIn p, float* q, float* k, float* v) {
  __shared__ float buf[8][256];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, u = blockIdx.y * 8 + warp;
  const __nv_bfloat16* row = p.act + static_cast<size_t>(t) * p.ldp;
  if (u >= 3 * p.H) return;
  const int h = u % p.H;
  if (u >= 2 * p.H) {
    for (int c = lane; c < p.V; c += 32) v[(static_cast<size_t>(t) * p.H + h) * p.V + c] = __bfloat162float(row[p.vc + h * p.V + c]);
    return;
  }
  const bool is_q = u < p.H;
  ret_load_row<256>(p, row + (is_q ? 0 : p.kc) + h * p.D, p.rot + static_cast<size_t>(t) * p.ldr, is_q ? 1.f : p.k_scale, true, buf[warp]);
  __syncwarp();
  float* dst = (is_q ? q : k) + (static_cast<size_t>(t) * p.H + h) * p.D;
  for (int d = lane; d < p.D; d += 32) dst[d] = buf[warp][d];
}

struct RetLaunch {
  cudaLaunchConfig_t c = {};
  cudaLaunchAttribute a[2];
  RetLaunch(dim3 grid, dim3 block, cudaStream_t stream, int pdl, size_t smem = 0, int cluster = 0) {
    c.gridDim = grid;
    c.blockDim = block;
    c.stream = stream;
    c.dynamicSmemBytes = smem;
    int n = 0;
    if (pdl) {
      a[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
      a[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 1) {
      a[n].id = cudaLaunchAttributeClusterDimension;
      a[n].val.clusterDim.x = cluster;
      a[n].val.clusterDim.y = 1;
      a[n++].val.clusterDim.z = 1;
    }
    c.attrs = a;
    c.numAttrs = n;
  }
};

static RetIn ret_in(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr, const float* pw,
                    const int* rows, const int* cu_q, const int* past_lens, int B) {
  return RetIn{H, D, V, dims / 2, (const __nv_bfloat16*)act, ldp, kc, vc, gc, (const float2*)rot, ldr, pw, rows, cu_q, past_lens, B,
               static_cast<float>(1.0 / sqrt(static_cast<double>(D)))};
}

static bool ret_ok(int H, int D, int V, int dims, int ldp, int kc, int vc, int gc, int ldr) {
  return H > 0 && D > 0 && D <= 256 && V > 0 && dims >= 0 && !(dims & 1) && dims <= D && ldr >= dims / 2 && kc >= H * D && vc >= kc + H * D &&
         gc >= vc + H * V && ldp >= gc + H * V && !((kc | vc | gc) & 7);
}

// vector loads start at row starts: the projections and the table's columns of a layer
static bool ret_aligned(const void* act, const void* rot) { return !((reinterpret_cast<uintptr_t>(act) | reinterpret_cast<uintptr_t>(rot)) & 15); }

template <int DP, int VT>
static int launch_update(const RetIn& p, float* U, int chunks, int pdl, cudaStream_t stream) {
  constexpr int smem = kRetChunk * ((DP + 8) * 4 + (VT + 16) * 2);
  static int configured[kMaxDevicesCached] = {};
  auto kern = retention_update_kernel<DP, VT>;
  if (ensure_dyn_smem(kern, smem, configured) != 0) return -3;
  RetLaunch l(dim3(chunks, p.H, (p.V + VT - 1) / VT), dim3(kRetThreads), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, kern, p, U) == cudaSuccess ? 0 : -4;
}

template <int DP, int VP>
static int launch_rows(const RetIn& p, const float* prefix, const int* mask_bits, int W, float eps, void* out, int ldo, int tiles, int pdl,
                       cudaStream_t stream) {
  constexpr int smem = kRetTile * (2 * (DP + 4) * 4 + (VP + 16) * 2);
  static int configured[kMaxDevicesCached] = {};
  auto kern = retention_rows_kernel<DP, VP>;
  if (ensure_dyn_smem(kern, smem, configured) != 0) return -3;
  RetLaunch l(dim3(tiles, p.H), dim3(kRetThreads), stream, pdl, smem);
  return cudaLaunchKernelEx(&l.c, kern, p, prefix, mask_bits, W, eps, (__nv_bfloat16*)out, ldo) == cudaSuccess ? 0 : -4;
}

static int launch_rows_for(const RetIn& p, const float* prefix, const int* mask_bits, int W, float eps, void* out, int ldo, int tiles, int pdl,
                           cudaStream_t stream) {
  if (p.D <= 64) {
    if (p.V <= 64) return launch_rows<64, 64>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
    if (p.V <= 128) return launch_rows<64, 128>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
    return launch_rows<64, 256>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
  }
  if (p.V <= 64) return launch_rows<128, 64>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
  if (p.V <= 128) return launch_rows<128, 128>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
  return launch_rows<128, 256>(p, prefix, mask_bits, W, eps, out, ldo, tiles, pdl, stream);
}

}  // namespace js

// Common arguments: act (T, ldp) bf16 with the q heads at column 0 and k, v, gate at columns kc, vc, gc (multiples of 8); rot (T, ldr)
// float2 from js_embed_rms at this layer's first frequency; pw (H, 257) powers of the decays; state (slots, H, D, V) fp32; a sequence
// whose committed length past_lens is 0 starts from zeros.

// One row per sequence, T = B rows; D <= 256, cl CTAs per head (1, 2, 4 or 8), V <= 256 cl.
extern "C" int js_retention_step(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr,
                                 const float* pw, const int* rows, const int* cu_q, const int* past_lens, int B, float* state, float eps,
                                 void* out, int ldo, int cl, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0) return 0;
  if (!ret_aligned(act, rot) || !ret_ok(H, D, V, dims, ldp, kc, vc, gc, ldr) || (cl != 1 && cl != 2 && cl != 4 && cl != 8) || B > 65535) return -10;
  const int vec = V % 4 == 0 ? 4 : 1;
  const int VS = ((V + cl - 1) / cl + vec - 1) / vec * vec;
  if (VS > 256) return -10;
  int VG = 1;
  while (VG * vec < VS) VG *= 2;
  const RetIn p = ret_in(H, D, V, dims, act, ldp, kc, vc, gc, rot, ldr, pw, rows, cu_q, past_lens, B);
  RetLaunch l(dim3(cl * H, B), dim3(kRetThreads), stream, pdl, 0, cl);
  const cudaError_t e = vec == 4 ? cudaLaunchKernelEx(&l.c, retention_step_kernel<4>, p, state, eps, (__nv_bfloat16*)out, ldo, cl, VS, VG)
                                 : cudaLaunchKernelEx(&l.c, retention_step_kernel<1>, p, state, eps, (__nv_bfloat16*)out, ldo, cl, VS, VG);
  return e == cudaSuccess ? 0 : -4;
}

// Portions; D <= 128, V <= 256.  U (T / 128 + B, H, D, V) fp32 is workspace.
extern "C" int js_retention_chunks(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr,
                                   const float* pw, const int* rows, const int* cu_q, const int* past_lens, int B, int T, float* state, float* U,
                                   float eps, void* out, int ldo, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0 || T <= 0) return 0;
  if (!ret_aligned(act, rot) || !ret_ok(H, D, V, dims, ldp, kc, vc, gc, ldr) || D > 128 || V > 256 || B > 65535) return -10;
  const RetIn p = ret_in(H, D, V, dims, act, ldp, kc, vc, gc, rot, ldr, pw, rows, cu_q, past_lens, B);
  const int chunks = T / kRetChunk + B, tiles = T / kRetTile + B;
  int rc = D <= 64 ? (V <= 64 ? launch_update<64, 64>(p, U, chunks, pdl, stream) : launch_update<64, 128>(p, U, chunks, pdl, stream))
                   : (V <= 64 ? launch_update<128, 64>(p, U, chunks, pdl, stream) : launch_update<128, 128>(p, U, chunks, pdl, stream));
  if (rc != 0) return rc;
  RetLaunch l(dim3((D * V + 4 * kRetThreads - 1) / (4 * kRetThreads), H, B), dim3(kRetThreads), stream, pdl);
  if (cudaLaunchKernelEx(&l.c, retention_scan_kernel, p, U, state) != cudaSuccess) return -4;
  return launch_rows_for(p, U, nullptr, 0, eps, out, ldo, tiles, pdl, stream);
}

// Token trees of up to 256 nodes (mask_bits (T, W), W <= 8): nothing is stored.  D <= 128, V <= 256.
extern "C" int js_retention_tree(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr,
                                 const float* pw, const int* rows, const int* cu_q, const int* past_lens, int B, int T, const float* state,
                                 const int* mask_bits, int W, float eps, void* out, int ldo, int pdl, cudaStream_t stream) {
  using namespace js;
  if (B <= 0 || T <= 0) return 0;
  if (!ret_aligned(act, rot) || !ret_ok(H, D, V, dims, ldp, kc, vc, gc, ldr) || D > 128 || V > 256) return -10;
  if (mask_bits == nullptr || W < 1 || W > 8) return -13;
  const RetIn p = ret_in(H, D, V, dims, act, ldp, kc, vc, gc, rot, ldr, pw, rows, cu_q, past_lens, B);
  return launch_rows_for(p, state, mask_bits, W, eps, out, ldo, T / kRetTile + B, pdl, stream);
}

// B = 1; path_len on the device, at most 256; past_lens is the committed length behind the path.
extern "C" int js_retention_path(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr,
                                 const float* pw, const int* rows, const int* cu_q, const int* past_lens, float* state, const int* path,
                                 const int* path_len, int pdl, cudaStream_t stream) {
  using namespace js;
  if (!ret_aligned(act, rot) || !ret_ok(H, D, V, dims, ldp, kc, vc, gc, ldr)) return -10;
  if (path == nullptr || path_len == nullptr) return -13;
  const RetIn p = ret_in(H, D, V, dims, act, ldp, kc, vc, gc, rot, ldr, pw, rows, cu_q, past_lens, 1);
  RetLaunch l(dim3(H, (V + 63) / 64), dim3(kRetThreads), stream, pdl);
  return cudaLaunchKernelEx(&l.c, retention_path_kernel, p, state, path, path_len) == cudaSuccess ? 0 : -4;
}

// Rotated fp32 rows q, k (T, H, D) and v (T, H, V) for js_retention_seq.
extern "C" int js_retention_prep(int H, int D, int V, int dims, const void* act, int ldp, int kc, int vc, int gc, const void* rot, int ldr,
                                 int T, float* q, float* k, float* v, int pdl, cudaStream_t stream) {
  using namespace js;
  if (T <= 0) return 0;
  if (!ret_aligned(act, rot) || !ret_ok(H, D, V, dims, ldp, kc, vc, gc, ldr)) return -10;
  const RetIn p = ret_in(H, D, V, dims, act, ldp, kc, vc, gc, rot, ldr, nullptr, nullptr, nullptr, nullptr, 0);
  RetLaunch l(dim3(T, (3 * H + 7) / 8), dim3(kRetThreads), stream, pdl);
  return cudaLaunchKernelEx(&l.c, retention_prep_kernel, p, q, k, v) == cudaSuccess ? 0 : -4;
}
