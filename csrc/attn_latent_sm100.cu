// Paged attention over cached latent rows (absorbed form) on the 5th-generation tensor cores.
//
// Every head of a token attends over the SAME cached row c per key: score = qa . c with qa = W_uk^T q, and the output is
// the weighted sum of the rows themselves (W_uv is applied afterwards).  So the heads are simply more query rows over one
// shared key/value matrix, and one gathered tile of latent rows serves as K (K-major operand) and as V (MN-major operand)
// of both MMAs: a cached byte is read once per (128 query rows, column group).
//
//   * rows: a sequence's (token, head) pairs in row-major order, 128 per CTA (64 for rows above 512 wide), any number of heads;
//   * S = QA C^T and O += P C are tcgen05.mma with M = 128; S (two buffers) and O (up to 256 columns) live in tensor
//     memory; outputs wider than 256 are covered by two column groups (grid y), each computing all scores and its own half
//     of the output columns; columns behind the latent (a rotated key part) enter the scores only;
//   * latent rows are gathered by slot with cp.async into 128-byte-swizzled tiles of 64 columns, TK keys each;
//   * with few query rows (decode) only RQ = 32 or 64 rows of Q and P are kept in shared memory: an MMA's other rows then
//     read whatever follows them, which only reaches accumulator rows nobody reads;
//   * softmax in fp32 with an integer running maximum (see attn_tc_sm100.cu); the probabilities are rounded to bf16 as MMA
//     operands and the denominator sums the rounded values;
//   * key splits go through a workspace and latent_attn_merge_kernel.
//
// Roles (416 threads): warps 0-3 softmax + epilogue, warp 4 MMA issuer / TMEM owner, warps 5-12 loaders.  Every wait is
// bounded (status word).
#include "common.cuh"

#include <math.h>

namespace js {

constexpr int LROWS = 128;
constexpr int LLOADERS = 256;
constexpr int LTHREADS = 160 + LLOADERS;
constexpr int LMAX_STAGES = 6;
constexpr int kLatentSmemMax = 227 * 1024;

struct LatentAttnParams {
  const __nv_bfloat16* q;      // (T*H, Rp) absorbed queries
  const __nv_bfloat16* pool;   // (S, Rp)
  const int* slot_map;         // (max_seqs, max_len)
  const int* seq_rows;         // (B)
  const int* cu_q;             // (B+1)
  const int* past_lens;        // (B)
  const int* mask_bits;        // (T, W) or null when causal
  __nv_bfloat16* out;          // (T*H, Rp)
  float* ws_o;                 // (splits, T*H, Rp)
  float* ws_ml;                // (splits, T*H, 2)
  int* status;
  int B, T, H, Rp, S, max_len, W, causal, splits;
  float scale_log2;
  const float* sinks;          // (H) a valueless key's score (unscaled) per head, counted by the last split; may be null
  const float* gate;           // (T, ldg) logits: head h's output is multiplied by sigmoid(gate[t, h]); may be null
  int ldg;
  int nk;                      // 64-column chunks of a latent row
  int nout;                    // leading chunks that are output
  int chunks0;                 // chunks of column group 0 (the rest belong to group 1)
  int trows;                   // query rows per CTA: 128 or 64
  int rq;                      // query rows kept in shared memory: 32, 64 or 128
  int stages;
};

JS_DEVICE void lat_cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
JS_DEVICE void lat_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
JS_DEVICE void lat_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

JS_DEVICE bool lat_mbar_wait(uint64_t* bar, uint32_t parity, int* status, int code) {
  for (uint32_t i = 0; i < (kSpinLimit >> 2); ++i) {
    if (mbar_test_wait(bar, parity)) return true;
    __nanosleep(20);
  }
  report(status, code);
  return false;
}
JS_DEVICE float lat_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
JS_DEVICE void lat_tmem_st(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
        "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
        "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
JS_DEVICE uint64_t lat_desc_mn(uint32_t smem_addr, uint32_t chunk_stride) {   // MN-major, 64-element chunks of 128-byte rows
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(chunk_stride >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}

// bytes of P: two buffers; with 32 keys both share one tile of 128-byte rows (64 bytes each)
__host__ __device__ inline int lat_p_bytes(int tk, int rq) { return (tk == 64 ? 2 : 1) * rq * 128; }
__host__ __device__ inline int lat_stage_bytes(int tk, int nk) { return nk * tk * 128; }

template <int TK>
__global__ void __launch_bounds__(LTHREADS, 1) latent_attn_tc_kernel(LatentAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int RQ = p.rq, nk = p.nk, NST = p.stages;
  const int q_chunk = RQ * 128;                       // bytes of one 64-column chunk of Q
  const int k_chunk = TK * 128, k_stage = lat_stage_bytes(TK, nk);
  uint8_t* sQ = smem;
  uint8_t* sP = sQ + nk * q_chunk;
  uint8_t* sK = sP + lat_p_bytes(TK, RQ);
  uint64_t* bars = reinterpret_cast<uint64_t*>(sK + NST * k_stage);
  uint64_t* q_full = bars;
  uint64_t* kv_full = bars + 1;
  uint64_t* kv_empty = kv_full + LMAX_STAGES;
  uint64_t* s_full = kv_empty + LMAX_STAGES;
  uint64_t* p_full = s_full + 2;
  uint64_t* pv_done = p_full + 2;
  uint64_t* o_done = pv_done + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int grp = blockIdx.y, split = blockIdx.z;
  const int v0 = grp == 0 ? 0 : p.chunks0;                       // first column chunk of this CTA's output
  const int nv = grp == 0 ? p.chunks0 : p.nout - p.chunks0;      // and how many (at most 4)

  pdl_launch_dependents();
  pdl_wait();

  int lo = 0, hi = p.B - 1;
  const int tile = blockIdx.x;
  while (lo < hi) {      // sequence b starts at tile cu_q[b]*H/trows + b
    const int mid = (lo + hi + 1) >> 1;
    if (static_cast<int>(static_cast<long long>(p.cu_q[mid]) * p.H / p.trows) + mid <= tile) lo = mid; else hi = mid - 1;
  }
  const int b = lo;
  const int q_begin = p.cu_q[b], n_b = p.cu_q[b + 1] - q_begin;
  const int row0 = (tile - (static_cast<int>(static_cast<long long>(q_begin) * p.H / p.trows) + b)) * p.trows;
  const int n_rows = min(p.trows, n_b * p.H - row0);
  if (n_rows <= 0) return;
  const int past = p.past_lens[b];
  const int* slots = p.slot_map + static_cast<size_t>(p.seq_rows[b]) * p.max_len;
  int L = past + n_b;
  if (p.causal) L = min(L, past + (row0 + n_rows - 1) / p.H + 1);
  const int n_tiles = (L + TK - 1) / TK;
  const int t_begin = static_cast<int>(static_cast<long long>(n_tiles) * split / p.splits);
  const int t_end = static_cast<int>(static_cast<long long>(n_tiles) * (split + 1) / p.splits);
  const int nt = t_end - t_begin;

  const int row = (warp & 3) * 32 + lane;              // softmax thread's row
  const bool row_valid = row < n_rows;
  const int node = (row0 + (row_valid ? row : 0)) / p.H;
  const size_t first_row = static_cast<size_t>(q_begin) * p.H + row0;
  const size_t out_row = first_row + (row_valid ? row : 0);

  if (nt <= 0) {
    if (warp < 4 && row_valid && p.splits > 1 && grp == 0) {
      float* ml = p.ws_ml + (static_cast<size_t>(split) * p.T * p.H + out_row) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }

  if (tid == 0) {
    mbar_init(q_full, LLOADERS);
    for (int s = 0; s < NST; ++s) { mbar_init(&kv_full[s], LLOADERS); mbar_init(&kv_empty[s], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 128); mbar_init(&pv_done[i], 1); }
    mbar_init(o_done, 1);
    fence_barrier_init();
  }
  const uint32_t tmem_cols = nv > 2 ? 512u : 256u;
  if (warp == 4) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 128;            // S buffers at columns [0, TK) and [64, 64 + TK)
  const uint32_t t_lane = static_cast<uint32_t>((warp & 3) * 32) << 16;

  if (warp >= 5) {
    // ================================================================ loaders
    const int lt = tid - 160;
    const int piece = lt & 7, r0 = lt >> 3;             // 16-byte piece of a 128-byte chunk row; rows r0, r0 + 32, ...
    const uint32_t q_addr = smem_u32(sQ);
    for (int ch = 0; ch < nk; ++ch) {
      for (int r = r0; r < RQ; r += 32) {
        const bool valid = r < n_rows;
        lat_cp16(q_addr + ch * q_chunk + r * 128 + ((piece ^ (r & 7)) << 4),
                 p.q + (first_row + (valid ? r : 0)) * p.Rp + ch * 64 + piece * 8, valid);
      }
    }
    lat_commit();
    constexpr int RPT = TK / 32;                        // key rows per thread and tile
    int slot_next[RPT];
#pragma unroll
    for (int j = 0; j < RPT; ++j) {
      const int kp = t_begin * TK + r0 + 32 * j;
      slot_next[j] = kp < L ? __ldg(slots + kp) : 0;
    }
    bool ok = true;
    int next_sig = -1;                                  // next group to publish (-1 = Q)
    auto publish_before = [&](int upto) {
      if (next_sig < upto) fence_proxy_async();
      for (; next_sig < upto; ++next_sig) {
        if (next_sig < 0) mbar_arrive(q_full); else mbar_arrive(&kv_full[next_sig % NST]);
      }
    };
    for (int i = 0; i < nt && ok; ++i) {
      const int s = i % NST;
      if (i >= NST) {
        const uint32_t par = ((i / NST) & 1) ^ 1;
        if (!mbar_test_wait(&kv_empty[s], par)) {
          lat_wait<0>();
          publish_before(i);
          ok = lat_mbar_wait(&kv_empty[s], par, p.status, kTimeoutEmpty);
        }
      }
      if (!ok) break;
      const int k0 = (t_begin + i) * TK;
      const uint32_t k_addr = smem_u32(sK + s * k_stage);
#pragma unroll
      for (int j = 0; j < RPT; ++j) {
        const int r = r0 + 32 * j;
        const bool valid = k0 + r < L;
        int slot = slot_next[j];
        const int kpn = k0 + TK + r;
        slot_next[j] = (i + 1 < nt && kpn < L) ? __ldg(slots + kpn) : 0;
        if (slot < 0 || slot >= p.S) { report(p.status, kBadSlot); slot = 0; }
        const __nv_bfloat16* src = p.pool + static_cast<size_t>(slot) * p.Rp + piece * 8;
        const uint32_t dst = k_addr + r * 128 + ((piece ^ (r & 7)) << 4);
        for (int ch = 0; ch < nk; ++ch) lat_cp16(dst + ch * k_chunk, src + ch * 64, valid);
      }
      lat_commit();
      // all but the newest NST - 1 tiles have landed: publish as early as the ring allows
      if (NST == 2) { lat_wait<1>(); publish_before(i); }
      else if (NST == 3) { lat_wait<2>(); publish_before(i - 1); }
      else { lat_wait<3>(); publish_before(i - 2); }
    }
    lat_wait<0>();                                      // on an error path too: no copy outlives the CTA
    if (ok) publish_before(nt);
  } else if (warp == 4) {
    // ================================================================ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = umma_idesc_bf16(LROWS, TK);
      const uint32_t idesc_pv = umma_idesc_bf16(LROWS, 0) | ((static_cast<uint32_t>(nv) * 64u >> 3) << 17) | (1u << 16);   // N = 64 nv, B MN-major
      bool ok = lat_mbar_wait(q_full, 0, p.status, kTimeoutFull);
      auto issue_pv = [&](int j) {
        const int s = j % NST, pb = j & 1;
        const uint32_t v_addr = smem_u32(sK + s * k_stage) + v0 * k_chunk;
        // 32 keys: buffer pb is bytes [64 pb, 64 pb + 64) of the shared tile's rows (+4 in 16-byte units)
        const uint64_t a_desc = TK == 64 ? umma_desc_sw128(smem_u32(sP) + pb * RQ * 128) : umma_desc_sw128(smem_u32(sP)) + 4 * pb;
#pragma unroll
        for (int k = 0; k < TK / 16; ++k)
          umma_f16(tmem_o, a_desc + 2 * k, lat_desc_mn(v_addr + k * 2048, k_chunk), idesc_pv, (j | k) != 0 ? 1u : 0u);
        umma_commit(&kv_empty[s]);
        umma_commit(&pv_done[pb]);
      };
      auto issue_qk = [&](int i) {
        const int s = i % NST, sb = i & 1;
        const uint32_t k_addr = smem_u32(sK + s * k_stage);
        for (int ch = 0; ch < nk; ++ch) {
          const uint64_t a = umma_desc_sw128(smem_u32(sQ) + ch * q_chunk), bd = umma_desc_sw128(k_addr + ch * k_chunk);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_f16(tmem_base + sb * 64, a + 2 * kk, bd + 2 * kk, idesc_qk, (ch | kk) != 0 ? 1u : 0u);
        }
        umma_commit(&s_full[sb]);
      };
      for (int i = 0; i < nt && ok; ++i) {
        // QK(i) needs tile i, PV(i-1) the probabilities of tile i-1; whichever is ready first goes first.  (With two
        // stages tile i cannot even be loaded before PV(i-2) is done, so PV must never queue behind a tile in flight.)
        bool qk = false, pv = i == 0;
        for (uint32_t it = 0; ok && !(qk && pv); ++it) {
          if (!qk && mbar_test_wait(&kv_full[i % NST], (i / NST) & 1)) {
            tc_fence_after();
            issue_qk(i);
            qk = true;
          }
          if (!pv && mbar_test_wait(&p_full[(i - 1) & 1], ((i - 1) >> 1) & 1)) {
            tc_fence_after();
            issue_pv(i - 1);
            pv = true;
          }
          if (qk && pv) break;
          __nanosleep(20);
          if (it >= kSpinLimit) {
            report(p.status, qk ? kTimeoutAccum : kTimeoutFull);
            ok = false;
          }
        }
      }
      if (ok) {
        ok = lat_mbar_wait(&p_full[(nt - 1) & 1], ((nt - 1) >> 1) & 1, p.status, kTimeoutAccum);
        if (ok) {
          tc_fence_after();
          issue_pv(nt - 1);
        }
      }
      umma_commit(o_done);     // also releases the epilogue on an error path
    }
  } else {
    // ================================================================ softmax + epilogue (one row per thread)
    int mw[8];
#pragma unroll
    for (int w = 0; w < 8; ++w)
      mw[w] = (!p.causal && row_valid && w < p.W) ? p.mask_bits[static_cast<size_t>(q_begin + node) * p.W + w] : 0;
    constexpr unsigned long long kAll = TK == 64 ? ~0ull : (1ull << (TK & 63)) - 1ull;
    float m_run = -INFINITY, l_run = 0.f;
    const int head = (row0 + (row_valid ? row : 0)) % p.H;
    if (p.sinks != nullptr && split == p.splits - 1) {   // the last split always has a tile
      const float s2 = p.sinks[head] * 1.4426950408889634f;
      m_run = ceilf(s2);
      l_run = exp2f(s2 - m_run);
    }
    bool ok = true;
    for (int i = 0; i < nt && ok; ++i) {
      const int sb = i & 1;
      ok = lat_mbar_wait(&s_full[sb], (i >> 1) & 1, p.status, kTimeoutAccum);
      if (!ok) break;
      tc_fence_after();
      uint32_t sr[TK];
      tmem_ld_32x32(tmem_base + t_lane + sb * 64, sr);
      if constexpr (TK == 64) tmem_ld_32x32(tmem_base + t_lane + sb * 64 + 32, sr + 32);
      tmem_ld_wait();
      const int k0 = (t_begin + i) * TK;
      const int jlo = k0 - past;                         // window index of the tile's first key (may be < 0)
      unsigned long long vm = 0ull;                      // bit c: key k0 + c is visible to this row
      if (row_valid) {
        if (jlo <= -TK) {
          vm = kAll;
        } else {
          if (jlo < 0) vm = (1ull << (-jlo)) - 1ull;
          if (p.causal) {
            const int cmax = node - jlo;
            if (cmax >= 63) vm = ~0ull; else if (cmax >= 0) vm |= (1ull << (cmax + 1)) - 1ull;
          } else {
#pragma unroll
            for (int w = 0; w < 8; ++w) {
              const int sh = 32 * w - jlo;
              const unsigned long long word = static_cast<unsigned int>(mw[w]);
              if (sh >= 0 && sh < 64) vm |= word << sh;
              else if (sh < 0 && sh > -32) vm |= word >> (-sh);
            }
          }
          vm &= kAll;
        }
        const int left = L - k0;
        if (left < 64) vm &= (left <= 0) ? 0ull : ((1ull << left) - 1ull);
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (vm == kAll) {
#pragma unroll
        for (int c = 0; c < TK; ++c) {
          const float x = __uint_as_float(sr[c]) * p.scale_log2;
          sr[c] = __float_as_uint(x);
          mx4[c & 3] = fmaxf(mx4[c & 3], x);
        }
      } else {
#pragma unroll
        for (int c = 0; c < TK; ++c) {
          const float x = ((vm >> c) & 1ull) ? __uint_as_float(sr[c]) * p.scale_log2 : -INFINITY;
          sr[c] = __float_as_uint(x);
          mx4[c & 3] = fmaxf(mx4[c & 3], x);
        }
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      const float m_new = fmaxf(m_run, ceilf(mx));
      const float m_safe = (m_new == -INFINITY) ? 0.f : m_new;
      const float alpha = exp2f(m_run - m_safe);
      const bool need = i > 0 && m_run != -INFINITY && alpha != 1.f;   // nothing accumulated yet: nothing to rescale
      m_run = m_new;
      if (i >= 2) ok = lat_mbar_wait(&pv_done[sb], ((i - 2) >> 1) & 1, p.status, kTimeoutAccum);
      if (!ok) break;
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t p_row = smem_u32(sP) + (TK == 64 ? sb * RQ * 128 : 0) + row * 128;
#pragma unroll
      for (int c8 = 0; c8 < TK / 8; ++c8) {
        uint32_t w4[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float p0 = lat_exp2(__uint_as_float(sr[c8 * 8 + 2 * e]) - m_safe);
          const float p1 = lat_exp2(__uint_as_float(sr[c8 * 8 + 2 * e + 1]) - m_safe);
          __nv_bfloat162 v = __floats2bfloat162_rn(p0, p1);
          const float2 pr = __bfloat1622float2(v);
          rs4[e] += pr.x + pr.y;
          w4[e] = *reinterpret_cast<uint32_t*>(&v);
        }
        const int chunk = TK == 64 ? c8 : c8 + 4 * sb;
        if (row < RQ)
          asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + ((chunk ^ (row & 7)) << 4)), "r"(w4[0]),
                       "r"(w4[1]), "r"(w4[2]), "r"(w4[3]) : "memory");
      }
      l_run = l_run * alpha + ((rs4[0] + rs4[1]) + (rs4[2] + rs4[3]));
      if (__any_sync(0xffffffffu, need)) {
        ok = lat_mbar_wait(&pv_done[(i - 1) & 1], ((i - 1) >> 1) & 1, p.status, kTimeoutAccum);
        if (!ok) break;
        tc_fence_after();
        const float f = need ? alpha : 1.f;
#pragma unroll 1
        for (int c0 = 0; c0 < nv * 64; c0 += 32) {
          uint32_t orr[32];
          tmem_ld_32x32(tmem_o + t_lane + c0, orr);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) orr[j] = __float_as_uint(__uint_as_float(orr[j]) * f);
          lat_tmem_st(tmem_o + t_lane + c0, orr);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(&p_full[sb]);
    }
    // ---- epilogue
    if (ok) ok = lat_mbar_wait(o_done, 0, p.status, kTimeoutAccum);
    tc_fence_after();
    if (ok) {
      float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      if (p.gate != nullptr) inv /= 1.f + expf(-p.gate[static_cast<size_t>(q_begin + node) * p.ldg + head]);
#pragma unroll 1
      for (int c0 = 0; c0 < nv * 64; c0 += 32) {
        uint32_t orr[32];
        tmem_ld_32x32(tmem_o + t_lane + c0, orr);
        tmem_ld_wait();
        if (!row_valid) continue;
        if (p.splits == 1) {
          uint4 pk[4];
          __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(pk);
#pragma unroll
          for (int j = 0; j < 16; ++j)
            o2[j] = __floats2bfloat162_rn(__uint_as_float(orr[2 * j]) * inv, __uint_as_float(orr[2 * j + 1]) * inv);
          uint4* dst = reinterpret_cast<uint4*>(p.out + out_row * p.Rp + v0 * 64 + c0);
#pragma unroll
          for (int j = 0; j < 4; ++j) dst[j] = pk[j];
        } else {
          float4* dst = reinterpret_cast<float4*>(p.ws_o + (static_cast<size_t>(split) * p.T * p.H + out_row) * p.Rp + v0 * 64 + c0);
#pragma unroll
          for (int j = 0; j < 8; ++j)
            dst[j] = make_float4(__uint_as_float(orr[4 * j]), __uint_as_float(orr[4 * j + 1]),
                                 __uint_as_float(orr[4 * j + 2]), __uint_as_float(orr[4 * j + 3]));
        }
      }
      if (p.splits > 1 && row_valid && grp == 0) {
        float* ml = p.ws_ml + (static_cast<size_t>(split) * p.T * p.H + out_row) * 2;
        ml[0] = m_run;
        ml[1] = l_run;
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

// one CTA per (token, head) row: merge the key splits (at most 16; four columns per thread)
constexpr int LMAX_SPLITS = 16;
__global__ void __launch_bounds__(128)
latent_attn_merge_kernel(const float* ws_o, const float* ws_ml, __nv_bfloat16* out, int rows, int H, int Rp, int cols, int splits,
                         const float* gate, int ldg) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, c = threadIdx.x * 4;
  __shared__ float w[LMAX_SPLITS];
  if (threadIdx.x < 32) {
    const int s = threadIdx.x;
    float2 ml = make_float2(-INFINITY, 0.f);
    if (s < splits) ml = *reinterpret_cast<const float2*>(ws_ml + (static_cast<size_t>(s) * rows + row) * 2);
    const float m = warp_max(ml.x);
    const float f = ml.x == -INFINITY ? 0.f : exp2f(ml.x - m);
    float l = warp_sum(ml.y * f);
    if (gate != nullptr) l *= 1.f + expf(-gate[static_cast<size_t>(row / H) * ldg + row % H]);
    if (s < LMAX_SPLITS) w[s] = l > 0.f ? f / l : 0.f;
  }
  __syncthreads();
  if (c >= cols) return;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
  for (int s = 0; s < splits; ++s) {
    const float f = w[s];
    if (f == 0.f) continue;                          // that split saw no visible key (its O may be unwritten)
    const float4 v = *reinterpret_cast<const float4*>(ws_o + (static_cast<size_t>(s) * rows + row) * Rp + c);
    acc[0] += v.x * f; acc[1] += v.y * f; acc[2] += v.z * f; acc[3] += v.w * f;
  }
  __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(out + static_cast<size_t>(row) * Rp + c);
  dst[0] = __floats2bfloat162_rn(acc[0], acc[1]);
  dst[1] = __floats2bfloat162_rn(acc[2], acc[3]);
}

template <int TK>
static int launch_latent(const LatentAttnParams& p, int q_tiles, int groups, int smem, bool pdl, cudaStream_t stream) {
  static int configured[kMaxDevicesCached] = {};
  auto kern = latent_attn_tc_kernel<TK>;
  if (ensure_dyn_smem(kern, smem, configured) != 0) return -3;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(q_tiles, groups, p.splits);
  cfg.blockDim = dim3(LTHREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, p) == cudaSuccess ? 0 : -4;
}

}  // namespace js

// q, out (T*H, Rp) bf16, pool (S, Rp) bf16, Rp a multiple of 64 up to 768, of which the first out_cols (at most 512) are values;
// sinks (H) and gate (T, ldg) fp32 or null; max_q = most query tokens of one sequence;
// masks of up to 8 words per token; tk_want = keys per tile (32, or 64 where it fits; 0 picks).  splits > 1 needs ws_o (splits, T*H, Rp) fp32 and ws_ml (splits, T*H, 2) fp32.
extern "C" int js_latent_attention_tc(const void* q, const void* pool, const int* slot_map, const int* seq_rows, const int* cu_q,
                                      const int* past_lens, const int* mask_bits, void* out, float* ws_o, float* ws_ml, int* status,
                                      int B, int T, int H, int Rp, int out_cols, int S, int max_len, int W, int causal, int splits, int max_q,
                                      float scale, const float* sinks, const float* gate, int ldg, int tk_want, int pdl,
                                      cudaStream_t stream) {
  using namespace js;
  if (T <= 0 || B <= 0) return 0;
  const int nout = (out_cols + 63) / 64;
  if (Rp % 64 || Rp < 64 || Rp > 768 || nout < 1 || nout > 8 || nout > Rp / 64 || H < 1) return -10;
  if (splits < 1 || splits > LMAX_SPLITS) return -11;
  if (splits > 1 && (ws_o == nullptr || ws_ml == nullptr)) return -12;
  if (!causal && (mask_bits == nullptr || W < 1 || W > 8)) return -13;
  const int nk = Rp / 64;
  const long long rows = static_cast<long long>(max_q < 1 ? T : max_q) * H;
  const int trows = Rp > 512 ? 64 : LROWS;        // a wide row leaves shared memory for 64 queries only
  const int rq = rows <= 32 ? 32 : rows <= 64 || trows == 64 ? 64 : 128;
  const int budget = kLatentSmemMax - 1024 - 256;
  int tk = 64, stages = (budget - nk * rq * 128 - lat_p_bytes(64, rq)) / lat_stage_bytes(64, nk);
  if (tk_want != 0 && tk_want != 32 && tk_want != 64) return -10;
  if (stages < 2 || tk_want == 32) {
    tk = 32;
    stages = (budget - nk * rq * 128 - lat_p_bytes(32, rq)) / lat_stage_bytes(32, nk);
  }
  if (stages < 2) return -18;
  if (stages > LMAX_STAGES) stages = LMAX_STAGES;
  const int chunks0 = nout <= 4 ? nout : (nout + 1) / 2;
  LatentAttnParams p{reinterpret_cast<const __nv_bfloat16*>(q), reinterpret_cast<const __nv_bfloat16*>(pool), slot_map, seq_rows, cu_q,
                     past_lens, mask_bits, reinterpret_cast<__nv_bfloat16*>(out), ws_o, ws_ml, status, B, T, H, Rp, S, max_len, W,
                     causal, splits, scale * 1.4426950408889634f, sinks, gate, ldg, nk, nout, chunks0, trows, rq, stages};
  int smem = 1024 + nk * rq * 128 + lat_p_bytes(tk, rq) + stages * lat_stage_bytes(tk, nk) + 256;
  // an MMA reads 128 rows from every Q chunk and P buffer: what follows them must reach at least that far
  const int after_p = stages * lat_stage_bytes(tk, nk) + rq * 128;
  if (after_p < LROWS * 128) return -18;
  const int q_tiles = static_cast<int>(static_cast<long long>(T) * H / trows) + B;
  const int groups = chunks0 < nout ? 2 : 1;
  const int rc = tk == 64 ? launch_latent<64>(p, q_tiles, groups, smem, pdl != 0, stream)
                          : launch_latent<32>(p, q_tiles, groups, smem, pdl != 0, stream);
  if (rc != 0 || splits == 1) return rc;
  cudaLaunchConfig_t c2 = {};
  c2.gridDim = dim3(T * H);
  c2.blockDim = dim3(128);
  c2.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  c2.attrs = attr;
  c2.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&c2, latent_attn_merge_kernel, static_cast<const float*>(ws_o), static_cast<const float*>(ws_ml),
                            reinterpret_cast<__nv_bfloat16*>(out), T * H, H, Rp, nout * 64, splits, gate, ldg) == cudaSuccess ? 0 : -5;
}
