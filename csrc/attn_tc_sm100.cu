// Paged tree-masked attention on the 5th-generation tensor cores (tcgen05 + tensor memory), head_dim 128.
// Reference twins: the Triton paged kernel jetspec/inference_engine/paged_tree_attn.py:55-367 (fp32 qq_bias, block tables)
// and the dense tree-attention kernel of the Hugging Face path, jetspec/core/tree_attention_kernel.py:63-216.
//
// Same contract as the mma.sync kernel in attn_sm100.cu (logical positions through a slot map, packed
// ancestor bits or causal window, GQA group packed into rows, optional key splits merged by
// attn_merge_kernel), different engine:
//
//   * one CTA = 128 query rows (128/G tree nodes x G query heads of one KV head) x one key split;
//   * S = Q K^T and O += P V are tcgen05.mma with M = 128; S (2 x 64 columns) and O (128 columns)
//     live in tensor memory, so the softmax threads own one ROW each (no shuffles): they read S with
//     tcgen05.ld, write P as bf16 into a swizzled shared-memory tile that feeds the second MMA, and
//     rescale O in tensor memory only when a row's integer running maximum grows;
//   * K/V rows are gathered by slot with cp.async into 128-byte-swizzled tiles (three stages) by four
//     loader warps; V is consumed as an MN-major operand, so no transpose is ever made;
//   * warp 4 issues all MMAs: QK(t+1) is issued before PV(t), so the tensor pipe works on the next
//     scores while the softmax of the current tile runs.
//
// Roles (416 threads): warps 0-3 softmax + epilogue (tensor-memory lane quadrant = warp id),
// warp 4 MMA issuer / TMEM owner, warps 5-12 loaders.  Every wait is bounded (status word).
//
// Forms (template parameter MODE):
//   * kPlain: the above, with an optional window, kept first tokens, sinks and gates;
//   * kPooled: scores may be capped, and tiles of pooled blocks (one key and value per P tokens, read through a block map)
//     stand ahead of the window's tiles;
//   * kDiff: two attention maps a head over the same values.  Query and key rows hold 64 columns for each map, so a tile's K
//     and V are gathered once and give two score tiles and two outputs (warps 0-3 and 4-7 own one map each, warp 8
//     issues, four loader warps); the epilogue (or the merge of the key splits) norms o1 - lam o2.
#include "common.cuh"

#include <math.h>
#include <type_traits>

namespace js {

constexpr int TD = 128;          // head dim
constexpr int TROWS = 128;       // query rows per CTA
constexpr int TKEYS = 64;        // keys per tile
constexpr int TSTAGES = 3;
constexpr int TTHREADS = 416;       // softmax threads of every map, one issuing warp, loaders
enum AttnMode : int { kPlain = 0, kPooled = 1, kDiff = 2 };
// loader threads (gather throughput grows with the copies in flight)
__host__ __device__ constexpr int loader_threads(int mode) { return TTHREADS - 32 - (mode == kDiff ? 256 : 128); }
__host__ __device__ constexpr int attn_maps(int mode) { return mode == kDiff ? 2 : 1; }
constexpr int kStageKV = 2 * TKEYS * 256;      // K then V, each 2 halves x 64 keys x 128 B
constexpr int kSmemQ = TROWS * 256;            // 2 halves x 128 rows x 128 B
constexpr int kSmemP = TROWS * 128;            // 128 rows x 64 keys bf16
constexpr int attn_tc_smem(int mode) { return kSmemQ + TSTAGES * kStageKV + 2 * attn_maps(mode) * kSmemP + 256 + 1024; }
// Key splits that merge inside a cluster (portable cluster size); the chunk receive area must fit the dead
// K/V stages + P buffers, the (max, sum) pairs the dead Q tile.
constexpr int kMaxClusterSplits = 8;
static_assert(kMaxClusterSplits * 16384 <= TSTAGES * kStageKV + 2 * kSmemP, "chunk receive area");
static_assert(3 * 2 * 16384 <= TSTAGES * kStageKV + 2 * kSmemP, "chunk receive area, 3 splits own 2 chunks each");
static_assert(kMaxClusterSplits * TROWS * 8 <= kSmemQ, "(max, sum) receive area");

struct AttnTcParams {
  const __nv_bfloat16* q;      // (T, Hq, 128)
  const __nv_bfloat16* k_pool; // (Hkv, S, 128)
  const __nv_bfloat16* v_pool;
  const int* slot_map;         // (max_seqs, max_len)
  const int* seq_rows;         // (B)
  const int* cu_q;             // (B+1)
  const int* past_lens;        // (B)
  const int* mask_bits;        // (T, W) or null when causal
  __nv_bfloat16* out;          // (T, Hq*128)
  float* ws_o;                 // (splits, T, Hq, 128) partial outputs
  float* ws_ml;                // (splits, T, Hq, 2)   partial (max, sum)
  int* status;
  int B, T, Hq, Hkv, S, max_len, W, causal, splits;
  float scale_log2;
  long long kv_head, kv_slot;  // elements between heads / slots of the pools (S*128 and 128 for a (Hkv, S, 128) pool)
  int ldo;                     // elements between tokens of `out`
  int window;                  // > 0: a row sees the last `window` tokens of its own path only
  int sink;                    // a valueless key takes part in the softmax (counted by the last split)
  int keep;                    // positions below it stay visible behind the window
  const float* sinks;          // (Hq) the valueless key's score (unscaled), null: 0
  const float* gate;           // (T, ldg) logits: head h's output is multiplied by sigmoid(gate[t, h]); may be null
  int ldg;
  int cluster_merge;           // the key splits of a tile form a cluster and merge through distributed shared memory
  // kPooled
  float cap_log2, cap_in;      // score cap in the log2 domain (0: none), 2 log2(e) scale / cap
  int P;                       // tokens to a block, 0 without blocks
  const __nv_bfloat16 *kb_pool, *vb_pool;      // (Hkv, block_rows, 128)
  const int* block_map;        // (max_seqs, max_blocks)
  int block_rows, max_blocks;
  // kDiff
  const float* lam;
  float share, eps;
  int V;                       // true width of a head's values
};

// cap tanh(s / cap) in the log2 domain, x = 2 log2(e) s / cap: absolute error below 1e-5 for caps up to 100
JS_DEVICE float capped(float x, float cap_log2) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return fmaf(-2.f * cap_log2, r, cap_log2);
}

JS_DEVICE void cp_async16_tc(uint32_t smem_addr, const void* gmem, bool valid) {
  const int n = valid ? 16 : 0;   // src-size 0 -> zero fill
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr), "l"(gmem), "r"(n) : "memory");
}
JS_DEVICE void cp_async_commit_tc() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
JS_DEVICE void cp_async_wait_tc() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

JS_DEVICE void tmem_st_32x32(uint32_t taddr, const uint32_t* r) {
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
// Bounded wait that backs off between polls: the waiting roles share the SM's load/store path with the
// loaders' cp.async traffic, so they must not spin on it.
JS_DEVICE bool mbar_wait_backoff(uint64_t* bar, uint32_t parity, int* status, int code) {
  for (uint32_t i = 0; i < (kSpinLimit >> 2); ++i) {
    if (mbar_test_wait(bar, parity)) return true;
    __nanosleep(20);
  }
  report(status, code);
  return false;
}
JS_DEVICE float fast_exp2(float x) {     // 2^x, flushing denormal results to zero; exp2(-inf) = 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
JS_DEVICE void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// MN-major operand tile stored as two 64-element halves of 128-byte rows (8-row groups 1024 B apart,
// halves `half_stride` bytes apart), 128-byte swizzle.
JS_DEVICE uint64_t umma_desc_sw128_mn(uint32_t smem_addr, uint32_t half_stride) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(half_stride >> 4) << 16;      // leading byte offset: next 64 elements along MN
  d |= static_cast<uint64_t>(1024 >> 4) << 32;             // stride byte offset: next 8 rows along K
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
JS_DEVICE constexpr uint32_t umma_idesc_bf16_bmn(int M, int N) {   // B operand MN-major
  return umma_idesc_bf16(M, N) | (1u << 16);
}

// Optional phase trace (nanosecond timestamps written by CTA (0,0,0)); null unless a profiling script sets it.
__device__ unsigned long long* g_attn_trace = nullptr;
JS_DEVICE void attn_trace(int slot) {
  if (g_attn_trace != nullptr && blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0) {
    unsigned long long t;
    asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
    g_attn_trace[slot] = t;
  }
}

template <int G, int MODE>
__global__ void __launch_bounds__(TTHREADS, 1) paged_tree_attn_tc_kernel(AttnTcParams p) {
  constexpr int NPT = TROWS / G;   // nodes per q tile
  constexpr int MAPS = attn_maps(MODE), TLOADERS = loader_threads(MODE), MMA_WARP = 4 * MAPS;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sKV = sQ + kSmemQ;
  uint8_t* sP = sKV + TSTAGES * kStageKV;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * MAPS * kSmemP);
  uint64_t* q_full = bars;                 // 1
  uint64_t* kv_full = bars + 1;            // TSTAGES
  uint64_t* kv_empty = kv_full + TSTAGES;  // TSTAGES
  uint64_t* s_full = kv_empty + TSTAGES;   // 2 a map
  uint64_t* p_full = s_full + 2 * MAPS;    // 2 a map
  uint64_t* pv_done = p_full + 2 * MAPS;   // 2 a map
  uint64_t* o_done = pv_done + 2 * MAPS;   // 1
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, split = blockIdx.z;

  pdl_launch_dependents();
  pdl_wait();
  if (tid == 0) attn_trace(0);

  // ---- which sequence does this q tile belong to (same numbering as the mma.sync kernel)
  int lo = 0, hi = p.B - 1;
  const int tile = blockIdx.x;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] / NPT + mid <= tile) lo = mid; else hi = mid - 1;
  }
  const int b = lo;
  const int q_begin = p.cu_q[b], n_b = p.cu_q[b + 1] - q_begin;
  const int node0 = (tile - (q_begin / NPT + b)) * NPT;
  if (node0 >= n_b) return;
  const int past = p.past_lens[b];
  const int* slots = p.slot_map + static_cast<size_t>(p.seq_rows[b]) * p.max_len;
  int L = past + n_b;
  if (p.causal) L = min(L, past + node0 + NPT);
  // first key tile any row of this CTA can see (a tree's root sits at position `past`)
  const int t_first = p.window > 0 ? max(0, past + (p.causal ? node0 : 0) - p.window + 1) / TKEYS : 0;
  // ... behind the tiles of kept first tokens: the CTA's tiles are 0 .. t_kept - 1 and t_first, t_first + 1, ...
  const int t_kept = p.window > 0 ? min(t_first, (p.keep + TKEYS - 1) / TKEYS) : 0;
  // tiles of pooled blocks come first: the blocks the CTA's last row sees (those of committed tokens, over a token tree)
  int nb_max = 0, t_pool = 0;
  if constexpr (MODE == kPooled) {
    if (p.P > 0) {
      const int behind = past + (p.causal ? min(node0 + NPT, n_b) : n_b) - p.window;      // positions behind the last row's window
      nb_max = behind > 0 ? behind / p.P : 0;
      if (!p.causal) nb_max = min(nb_max, past / p.P);
      t_pool = (nb_max + TKEYS - 1) / TKEYS;
    }
  }
  const int n_tiles = (L + TKEYS - 1) / TKEYS - t_first + t_kept + t_pool;
  const int t_begin = (n_tiles * split) / p.splits;
  const int t_end = (n_tiles * (split + 1)) / p.splits;
  const int nt = t_end - t_begin;
  auto tile_key = [&](int i) {          // first key of this split's tile i
    int t = t_begin + i;
    if constexpr (MODE == kPooled) {
      if (t < t_pool) return t * TKEYS;
      t -= t_pool;
    }
    return (t < t_kept ? t : t - t_kept + t_first) * TKEYS;
  };
  auto pooled_tile = [&](int i) { return MODE == kPooled && t_begin + i < t_pool; };      // its keys are blocks

  // softmax thread's row
  const int row = (warp & 3) * 32 + lane;
  const int node = node0 + row / G, head = h * G + row % G;
  const bool row_valid = node < n_b;
  const size_t out_row = static_cast<size_t>(q_begin + (row_valid ? node : 0)) * p.Hq + head;
  __nv_bfloat16* out_ptr = p.out + static_cast<size_t>(q_begin + (row_valid ? node : 0)) * p.ldo + head * TD;

  const bool cmerge = MODE != kDiff && p.cluster_merge != 0;
  const int map = MODE == kDiff ? warp >> 2 : 0;      // softmax threads: the map they own
  const bool softmax_warp = warp < 4 * MAPS;
  float m_run = -INFINITY, l_run = 0.f;     // softmax threads: running (integer) maximum and sum of their row
  if (p.sink && split == p.splits - 1) {    // the last split always has a tile
    const float s2 = p.sinks != nullptr && row_valid ? p.sinks[head] * 1.4426950408889634f : 0.f;
    m_run = ceilf(s2);
    l_run = exp2f(s2 - m_run);
  }
  const float gate = p.gate != nullptr && row_valid ? 1.f / (1.f + expf(-p.gate[static_cast<size_t>(q_begin + node) * p.ldg + head])) : 1.f;
  bool sm_ok = true;
  if (nt <= 0 && !cmerge) {   // more splits than key tiles: this split contributes nothing
    if (softmax_warp && row_valid && p.splits > 1) {
      float* ml = p.ws_ml + ((static_cast<size_t>(split) * p.T * p.Hq + out_row) * MAPS + map) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }

  if (tid == 0 && nt > 0) {
    mbar_init(q_full, TLOADERS);
    for (int s = 0; s < TSTAGES; ++s) { mbar_init(&kv_full[s], TLOADERS); mbar_init(&kv_empty[s], 1); }
    for (int i = 0; i < 2 * MAPS; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 128); mbar_init(&pv_done[i], 1); }
    mbar_init(o_done, 1);
    fence_barrier_init();
  }
  if (warp == MMA_WARP && nt > 0) {
    tmem_alloc(tmem_slot, 256 * MAPS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = nt > 0 ? *tmem_slot : 0u;
  if (tid == 0) attn_trace(1);      // setup done
  const uint32_t tmem_o = tmem_base + 128 * MAPS;      // map m: S buffers at columns 128 m and 128 m + 64, O behind all of them

  const uint32_t t_lane = static_cast<uint32_t>((warp & 3) * 32) << 16;
  if (nt <= 0) {
    // (cluster merge) nothing to compute: this CTA only takes part in the exchange below
  } else if (warp > MMA_WARP) {
    // ================================================================ loaders
    const int lt = tid - (MMA_WARP + 1) * 32;
    const uint32_t q_addr = smem_u32(sQ);
    for (int c = lt; c < TROWS * 16; c += TLOADERS) {
      const int r = c >> 4, ch = c & 15;
      const int nd = node0 + r / G;
      const bool valid = nd < n_b;
      const __nv_bfloat16* src = p.q + (static_cast<size_t>(q_begin + (valid ? nd : 0)) * p.Hq + h * G + r % G) * TD + ch * 8;
      cp_async16_tc(q_addr + (ch >> 3) * (TROWS * 128) + r * 128 + (((ch & 7) ^ (r & 7)) << 4), src, valid);
    }
    cp_async_commit_tc();
    constexpr int RSTEP = TLOADERS / 16;        // key rows covered by one pass of all loader threads
    const int ch = lt & 15, r0 = lt >> 4;       // this thread copies chunk `ch` of keys r0, r0+RSTEP, ...
    // slots of the first tile; the next tile's are fetched while the current tile's copies are issued
    int slot_next[TKEYS / RSTEP];
    const int* blocks = nullptr;
    if constexpr (MODE == kPooled) blocks = p.block_map + static_cast<size_t>(p.seq_rows[b]) * p.max_blocks;
    // slot of key kp of tile i, 0 past the end
    auto slot_at = [&](int i, int kp) {
      if constexpr (MODE == kPooled) {
        if (pooled_tile(i)) return kp < nb_max ? (kp < p.max_blocks ? __ldg(blocks + kp) : -1) : 0;
      }
      return kp < L ? __ldg(slots + kp) : 0;
    };
#pragma unroll
    for (int j = 0; j < TKEYS / RSTEP; ++j) slot_next[j] = slot_at(0, tile_key(0) + r0 + RSTEP * j);
    bool ok = true;
    // copies complete in issue order (Q, tile 0, tile 1, ...); `next_sig` is the next one to publish (-1 = Q)
    int next_sig = -1;
    auto publish_before = [&](int upto) {
      if (next_sig < upto) fence_proxy_async();
      for (; next_sig < upto; ++next_sig) {
        if (next_sig < 0) mbar_arrive(q_full); else mbar_arrive(&kv_full[next_sig % TSTAGES]);
        if (lt == 0 && next_sig >= 0 && next_sig < 8) attn_trace(40 + next_sig);   // tile published by loader thread 0
      }
    };
    for (int i = 0; i < nt && ok; ++i) {
      const int s = i % TSTAGES;
      if (i >= TSTAGES) {
        const uint32_t par = ((i / TSTAGES) & 1) ^ 1;
        if (!mbar_test_wait(&kv_empty[s], par)) {
          // about to block on the consumer: it may itself be waiting for tiles not yet published
          cp_async_wait_tc<0>();
          publish_before(i);
          ok = mbar_wait_backoff(&kv_empty[s], par, p.status, kTimeoutEmpty);
        }
      }
      if (!ok) break;
      const int k0 = tile_key(i), k0n = tile_key(i + 1);
      const uint32_t k_addr = smem_u32(sKV + s * kStageKV);
      int slot_cur[TKEYS / RSTEP];
#pragma unroll
      for (int j = 0; j < TKEYS / RSTEP; ++j) {
        slot_cur[j] = slot_next[j];
        slot_next[j] = i + 1 < nt ? slot_at(i + 1, k0n + r0 + RSTEP * j) : 0;
      }
      const bool is_pool = pooled_tile(i);
      const int limit = is_pool ? nb_max : L, n_slots = is_pool ? p.block_rows : p.S;
      const __nv_bfloat16 *k_src = p.k_pool, *v_src = p.v_pool;
      long long head_stride = p.kv_head, slot_stride = p.kv_slot;
      if constexpr (MODE == kPooled) {
        if (is_pool) {
          k_src = p.kb_pool;
          v_src = p.vb_pool;
          head_stride = static_cast<long long>(p.block_rows) * TD;
          slot_stride = TD;
        }
      }
#pragma unroll
      for (int j = 0; j < TKEYS / RSTEP; ++j) {
        const int r = r0 + RSTEP * j;
        const int kp = k0 + r;
        const bool valid = kp < limit;
        int slot = slot_cur[j];
        if (slot < 0 || slot >= n_slots) { report(p.status, kBadSlot); slot = 0; }
        const size_t off = static_cast<size_t>(h) * head_stride + static_cast<size_t>(slot) * slot_stride + ch * 8;
        const uint32_t dst = (ch >> 3) * (TKEYS * 128) + r * 128 + (((ch & 7) ^ (r & 7)) << 4);
        cp_async16_tc(k_addr + dst, k_src + off, valid);
        cp_async16_tc(k_addr + TKEYS * 256 + dst, v_src + off, valid);
      }
      cp_async_commit_tc();
      if (lt == 0 && i < 8) attn_trace(32 + i);    // copies of tile i issued
      cp_async_wait_tc<2>();          // everything but the two newest groups has landed
      publish_before(i - 1);
    }
    if (ok) {
      cp_async_wait_tc<0>();
      publish_before(nt);
    }
  } else if (warp == MMA_WARP) {
    // ================================================================ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = umma_idesc_bf16(TROWS, TKEYS);
      constexpr uint32_t idesc_pv = umma_idesc_bf16_bmn(TROWS, TD);
      bool ok = mbar_wait_backoff(q_full, 0, p.status, kTimeoutFull);
      attn_trace(2);                // Q landed
      // O += P V of tile j for every map, each as soon as its P is there
      auto issue_pv = [&](int j) {
        const int s = j % TSTAGES, pb = j & 1;
        const uint32_t v_addr = smem_u32(sKV + s * kStageKV + TKEYS * 256);
#pragma unroll
        for (int m = 0; m < MAPS; ++m) {
          if (!mbar_wait_backoff(&p_full[2 * m + pb], (j >> 1) & 1, p.status, kTimeoutAccum)) return false;
          tc_fence_after();
          const uint64_t a_desc = umma_desc_sw128(smem_u32(sP + (2 * m + pb) * kSmemP));
#pragma unroll
          for (int k = 0; k < TKEYS / 16; ++k)
            umma_f16(tmem_o + m * TD, a_desc + 2 * k, umma_desc_sw128_mn(v_addr + k * 2048, TKEYS * 128), idesc_pv, (j | k) != 0 ? 1u : 0u);
          if (m == MAPS - 1) umma_commit(&kv_empty[s]);
          umma_commit(&pv_done[2 * m + pb]);
        }
        return true;
      };
      for (int i = 0; i < nt && ok; ++i) {
        const int s = i % TSTAGES, sb = i & 1;
        ok = mbar_wait_backoff(&kv_full[s], (i / TSTAGES) & 1, p.status, kTimeoutFull);
        if (!ok) break;
        if (i < 8) attn_trace(8 + i);   // K/V tile i landed
        // S buffer sb was consumed when P of tile i-2 was published (waited for below, before PV(i-2))
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sKV + s * kStageKV);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint32_t hoff = (k >> 2), kk = k & 3;          // each half of the columns is a map of its own in kDiff
          umma_f16(tmem_base + (MAPS == 2 ? hoff * 2 * TKEYS : 0) + sb * TKEYS, umma_desc_sw128(smem_u32(sQ) + hoff * (TROWS * 128)) + 2 * kk,
                   umma_desc_sw128(k_addr + hoff * (TKEYS * 128)) + 2 * kk, idesc_qk, (MAPS == 2 ? kk : k) != 0 ? 1u : 0u);
          if (MAPS == 2 && k == 3) umma_commit(&s_full[sb]);
        }
        umma_commit(&s_full[2 * (MAPS - 1) + sb]);
        if (i >= 1) {
          ok = issue_pv(i - 1);
          if (!ok) break;
        }
      }
      if (ok) ok = issue_pv(nt - 1);
      umma_commit(o_done);     // also releases the epilogue on an error path
    }
  } else {
    // ================================================================ softmax + epilogue (one row per thread)
    int mw[8];
#pragma unroll
    for (int w = 0; w < 8; ++w)
      mw[w] = (!p.causal && row_valid && w < p.W) ? p.mask_bits[static_cast<size_t>(q_begin + node) * p.W + w] : 0;
    int cut = 0;                       // committed keys below it are out of the row's window
    int nb_row = 0;                    // blocks the row sees
    if (p.window > 0) {
      if (p.causal) {
        cut = past + node - p.window + 1;
        if constexpr (MODE == kPooled) nb_row = p.P > 0 && cut > 0 ? cut / p.P : 0;
      } else {                         // a node's position is its number of proper ancestors behind the committed length
        int cnt = 0;
#pragma unroll
        for (int w = 0; w < 8; ++w) cnt += __popc(static_cast<unsigned>(mw[w]));
        if constexpr (MODE == kPooled) nb_row = p.P > 0 && past + cnt > p.window ? min(past + cnt - p.window, past) / p.P : 0;
        cut = min(past, past + cnt - p.window);
        // ancestors out of the window are the lowest bits (the d-th lowest is at position past + d); kept ones stay
        int drop = cnt - p.window, spare = p.keep - past;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
          unsigned rest = static_cast<unsigned>(mw[w]);
          for (; drop > 0 && rest != 0u; --drop, --spare) {
            const unsigned low = rest & (0u - rest);
            if (spare <= 0) mw[w] &= static_cast<int>(~low);
            rest ^= low;
          }
        }
      }
    }
    bool ok = true;
    for (int i = 0; i < nt && ok; ++i) {
      const int sb = i & 1;
      ok = mbar_wait_backoff(&s_full[2 * map + sb], (i >> 1) & 1, p.status, kTimeoutAccum);
      if (!ok) break;
      tc_fence_after();
      if (tid == 0 && i < 8) attn_trace(16 + i);   // scores of tile i ready
      uint32_t sr[64];
      tmem_ld_32x32(tmem_base + t_lane + (2 * map + sb) * TKEYS, sr);
      tmem_ld_32x32(tmem_base + t_lane + (2 * map + sb) * TKEYS + 32, sr + 32);
      tmem_ld_wait();
      // visibility of the tile's 64 keys for this row, as one 64-bit word (bit c = key k0 + c)
      const int k0 = tile_key(i);
      const int jlo = k0 - past;                         // window index of the tile's first key (may be < 0)
      unsigned long long vm = 0ull;
      if (pooled_tile(i)) {
        const int seen = nb_row - k0;
        if (row_valid && seen > 0) vm = seen >= TKEYS ? ~0ull : (1ull << seen) - 1ull;
      } else if (row_valid) {
        if (jlo <= -TKEYS) {
          vm = ~0ull;                                    // the whole tile is prefix
        } else {
          if (jlo < 0) vm = (1ull << (-jlo)) - 1ull;     // prefix part of a mixed tile
          if (p.causal) {
            const int cmax = node - jlo;                 // window key j = jlo + c is visible when j <= node
            if (cmax >= 63) vm = ~0ull; else if (cmax >= 0) vm |= (1ull << (cmax + 1)) - 1ull;
          } else {
#pragma unroll
            for (int w = 0; w < 8; ++w) {
              const int sh = 32 * w - jlo;               // where bit 0 of mask word w falls in the tile
              const unsigned long long word = static_cast<unsigned int>(mw[w]);
              if (sh >= 0 && sh < 64) vm |= word << sh;
              else if (sh < 0 && sh > -32) vm |= word >> (-sh);
            }
          }
        }
        const int left = L - k0;                         // keys at or past L do not exist
        if (left < 64) vm &= (left <= 0) ? 0ull : ((1ull << left) - 1ull);
        const int hidden = cut - k0;                     // this many of the tile's keys lie before the window
        if (hidden > 0) {
          const int kept = p.keep - k0;                  // ... of which the first `kept` are visible all the same
          const unsigned long long stay = kept >= 64 ? ~0ull : kept > 0 ? (1ull << kept) - 1ull : 0ull;
          vm &= (hidden >= 64 ? 0ull : ~0ull << hidden) | stay;
        }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};   // four chains instead of one 64-deep
      float to_log2 = p.scale_log2;
      if constexpr (MODE == kPooled) {
        if (p.cap_log2 > 0.f) {
#pragma unroll
          for (int c = 0; c < 64; ++c) sr[c] = __float_as_uint(capped(__uint_as_float(sr[c]) * p.cap_in, p.cap_log2));
          to_log2 = 1.f;
        }
      }
      if (vm == ~0ull) {              // the common case: every key of the tile is visible to this row
#pragma unroll
        for (int c = 0; c < 64; ++c) {
          const float x = __uint_as_float(sr[c]) * to_log2;
          sr[c] = __float_as_uint(x);
          mx4[c & 3] = fmaxf(mx4[c & 3], x);
        }
      } else {
#pragma unroll
        for (int c = 0; c < 64; ++c) {
          const bool vis = (vm >> c) & 1ull;
          const float x = vis ? __uint_as_float(sr[c]) * to_log2 : -INFINITY;
          sr[c] = __float_as_uint(x);
          mx4[c & 3] = fmaxf(mx4[c & 3], x);
        }
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // integer running maximum in the log2 domain (probabilities are then exact powers of two apart
      // whatever the tile order or key split; see the mma.sync kernel)
      const float m_new = fmaxf(m_run, ceilf(mx));
      const float m_safe = (m_new == -INFINITY) ? 0.f : m_new;
      const float alpha = exp2f(m_run - m_safe);          // 0 when nothing was visible before
      m_run = m_new;
      // P buffer sb is free once PV of tile i-2 has completed
      if (i >= 2) ok = mbar_wait_backoff(&pv_done[2 * map + sb], ((i - 2) >> 1) & 1, p.status, kTimeoutAccum);
      if (!ok) break;
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t p_row = smem_u32(sP + (2 * map + sb) * kSmemP) + row * 128;
#pragma unroll
      for (int c8 = 0; c8 < 8; ++c8) {
        uint32_t w4[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float p0 = fast_exp2(__uint_as_float(sr[c8 * 8 + 2 * e]) - m_safe);
          const float p1 = fast_exp2(__uint_as_float(sr[c8 * 8 + 2 * e + 1]) - m_safe);
          rs4[e] += p0 + p1;
          __nv_bfloat162 v = __floats2bfloat162_rn(p0, p1);
          w4[e] = *reinterpret_cast<uint32_t*>(&v);
        }
        asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + ((c8 ^ (row & 7)) << 4)), "r"(w4[0]),
                     "r"(w4[1]), "r"(w4[2]), "r"(w4[3]) : "memory");
      }
      l_run = l_run * alpha + ((rs4[0] + rs4[1]) + (rs4[2] + rs4[3]));
      // rescale O when some row of this warp raised its maximum (tcgen05.ld/st are warp-wide)
      const bool need = i > 0 && alpha != 1.f;
      if (__any_sync(0xffffffffu, need)) {
        ok = mbar_wait_backoff(&pv_done[2 * map + ((i - 1) & 1)], ((i - 1) >> 1) & 1, p.status, kTimeoutAccum);   // every earlier PV is in O
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c0 = 0; c0 < TD; c0 += 32) {
          uint32_t orr[32];
          tmem_ld_32x32(tmem_o + map * TD + t_lane + c0, orr);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) orr[j] = __float_as_uint(__uint_as_float(orr[j]) * alpha);
          tmem_st_32x32(tmem_o + map * TD + t_lane + c0, orr);
        }
        tmem_st_wait();
      }
      fence_proxy_async();          // P (generic-proxy stores) -> visible to the MMA's async-proxy reads
      tc_fence_before();
      mbar_arrive(&p_full[2 * map + sb]);
      if (tid == 0 && i < 8) attn_trace(24 + i);   // P of tile i published
    }
    // ---- epilogue
    if (ok) ok = mbar_wait_backoff(o_done, 0, p.status, kTimeoutAccum);
    tc_fence_after();
    if (tid == 0) attn_trace(3);    // output accumulator complete
    sm_ok = ok;
    if (MODE == kDiff && p.splits == 1) {
      // both maps' threads of a row finish half of its columns each; sums and denominators pass through the dead Q tile
      float* den = reinterpret_cast<float*>(sQ);
      float* sq = den + 2 * TROWS;
      auto both_maps = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };
      den[map * TROWS + row] = l_run > 0.f ? 1.f / l_run : 0.f;
      both_maps();
      const float i1 = den[row], i2 = den[TROWS + row] * *p.lam;
      float v[64], ss = 0.f;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t a[32], c[32];
        const uint32_t at = tmem_o + t_lane + map * 64 + half * 32;
        tmem_ld_32x32(at, a);
        tmem_ld_32x32(at + TD, c);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          v[half * 32 + j] = __uint_as_float(a[j]) * i1 - __uint_as_float(c[j]) * i2;
          ss += v[half * 32 + j] * v[half * 32 + j];
        }
      }
      sq[map * TROWS + row] = ss;
      both_maps();
      const float r = p.share / sqrtf((sq[row] + sq[TROWS + row]) / p.V + p.eps);
      if (ok && row_valid) {
        uint4 pk[8];
        __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(pk);
#pragma unroll
        for (int j = 0; j < 32; ++j) o2[j] = __floats2bfloat162_rn(v[2 * j] * r, v[2 * j + 1] * r);
        uint4* dst = reinterpret_cast<uint4*>(out_ptr + map * 64);
#pragma unroll
        for (int j = 0; j < 8; ++j) dst[j] = pk[j];
      }
    } else if (ok && !cmerge) {
      const float inv = l_run > 0.f ? gate / l_run : 0.f;
#pragma unroll 1
      for (int c0 = 0; c0 < TD; c0 += 32) {
        uint32_t orr[32];
        tmem_ld_32x32(tmem_o + map * TD + t_lane + c0, orr);
        tmem_ld_wait();
        if (!row_valid) continue;
        if (p.splits == 1) {
          uint4 pk[4];
          __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(pk);
#pragma unroll
          for (int j = 0; j < 16; ++j)
            o2[j] = __floats2bfloat162_rn(__uint_as_float(orr[2 * j]) * inv, __uint_as_float(orr[2 * j + 1]) * inv);
          uint4* dst = reinterpret_cast<uint4*>(out_ptr + c0);
#pragma unroll
          for (int j = 0; j < 4; ++j) dst[j] = pk[j];
        } else {
          float4* dst = reinterpret_cast<float4*>(p.ws_o + ((static_cast<size_t>(split) * p.T * p.Hq + out_row) * MAPS + map) * TD + c0);
#pragma unroll
          for (int j = 0; j < 8; ++j)
            dst[j] = make_float4(__uint_as_float(orr[4 * j]), __uint_as_float(orr[4 * j + 1]),
                                 __uint_as_float(orr[4 * j + 2]), __uint_as_float(orr[4 * j + 3]));
        }
      }
      if (p.splits > 1 && row_valid) {
        float* ml = p.ws_ml + ((static_cast<size_t>(split) * p.T * p.Hq + out_row) * MAPS + map) * 2;
        ml[0] = m_run;
        ml[1] = l_run;
      }
    }
  }

  if (cmerge) {
    // ---------------------------------------------------------------- merge of the key splits inside the cluster
    // Column chunk c (32 of the 128 output columns) is finished by CTA c % splits.  Every CTA pushes its
    // unnormalised chunk (column-major, 16 KB) into the owner's shared memory and its rows' (max, sum) to
    // all CTAs; the receive areas reuse the K/V stages + P buffers (chunks, at most 8 x 16 KB = 128 KB) and the
    // Q tile ((max, sum) pairs, at most 8 KB), all dead once every CTA of the cluster has left its main loop.
    const int per_owner = (4 + p.splits - 1) / p.splits;
    float* recv_o = reinterpret_cast<float*>(sKV);
    float* recv_ml = reinterpret_cast<float*>(sQ);
    tc_fence_before();
    __syncthreads();
    cluster_sync();
    if (tid == 0) attn_trace(5);    // every CTA of the cluster left its main loop
    if (warp < 4) {
      const bool have = nt > 0 && sm_ok;
      const float m_pub = have ? m_run : -INFINITY;
      const uint32_t ml_addr = smem_u32(recv_ml) + static_cast<uint32_t>((split * TROWS + row) * 8);
      for (int d = 0; d < p.splits; ++d) {
        const uint32_t a = map_to_cta(ml_addr, d);
        st_dsmem_f32(a, m_pub);
        st_dsmem_f32(a + 4, have ? l_run : 0.f);
      }
      if (have) {
#pragma unroll 1
        for (int c = 0; c < 4; ++c) {
          uint32_t orr[32];
          tmem_ld_32x32(tmem_o + t_lane + c * 32, orr);
          tmem_ld_wait();
          const uint32_t dst = map_to_cta(smem_u32(recv_o), c % p.splits) +
                               static_cast<uint32_t>(((split * per_owner + c / p.splits) * 4096 + row) * 4);
#pragma unroll
          for (int j = 0; j < 32; ++j) st_dsmem_f32(dst + j * (TROWS * 4), __uint_as_float(orr[j]));
        }
      }
    }
    if (tid == 0) attn_trace(6);    // partials pushed
    tc_fence_before();
    __syncthreads();
    cluster_sync();
    if (tid == 0) attn_trace(7);    // partials of all splits landed
    if (warp < 4 && row_valid) {
      float m = -INFINITY;
      for (int s2 = 0; s2 < p.splits; ++s2) m = fmaxf(m, recv_ml[(s2 * TROWS + row) * 2]);
      float wsrc[8], lsum = 0.f;
      for (int s2 = 0; s2 < p.splits; ++s2) {
        const float ms = recv_ml[(s2 * TROWS + row) * 2];
        wsrc[s2] = (ms == -INFINITY) ? 0.f : exp2f(ms - m);
        lsum += recv_ml[(s2 * TROWS + row) * 2 + 1] * wsrc[s2];
      }
      const float inv = lsum > 0.f ? gate / lsum : 0.f;
      for (int c = split; c < 4; c += p.splits) {
        float acc[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) acc[j] = 0.f;
        for (int s2 = 0; s2 < p.splits; ++s2) {
          if (wsrc[s2] == 0.f) continue;       // that split saw no visible key (its chunk was never pushed)
          const float* src = recv_o + (s2 * per_owner + c / p.splits) * 4096 + row;
#pragma unroll
          for (int j = 0; j < 32; ++j) acc[j] += src[j * TROWS] * wsrc[s2];
        }
        uint4 pk[4];
        __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(pk);
#pragma unroll
        for (int j = 0; j < 16; ++j) o2[j] = __floats2bfloat162_rn(acc[2 * j] * inv, acc[2 * j + 1] * inv);
        uint4* dst = reinterpret_cast<uint4*>(out_ptr + c * 32);
#pragma unroll
        for (int j = 0; j < 4; ++j) dst[j] = pk[j];
      }
    }
  }

  // ------------------------------------------------------------------ teardown
  if (tid == 0) attn_trace(4);      // epilogue stores issued
  tc_fence_before();
  __syncthreads();
  if (warp == MMA_WARP && nt > 0) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256 * MAPS);
  }
}

// merge of the key splits of a differential attention: one warp per (token, head) norms the difference of the merged maps
__global__ void __launch_bounds__(256) diff_merge_kernel(AttnTcParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int rows = p.T * p.Hq;
  if (row >= rows) return;
  const float lam = *p.lam;
  float o[4] = {}, ss = 0.f;
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const size_t at = static_cast<size_t>(row) * 2 + m, stride = static_cast<size_t>(rows) * 2;
    float top = -INFINITY;
    for (int s = 0; s < p.splits; ++s) top = fmaxf(top, p.ws_ml[(s * stride + at) * 2]);
    float acc[4] = {}, l = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.ws_ml[(s * stride + at) * 2], ls = p.ws_ml[(s * stride + at) * 2 + 1];
      if (ms == -INFINITY) continue;   // this split saw no visible key (its O may be unwritten)
      const float w = exp2f(ms - top);
      l += ls * w;
      const float4 v = *reinterpret_cast<const float4*>(p.ws_o + (s * stride + at) * TD + lane * 4);
      acc[0] += v.x * w; acc[1] += v.y * w; acc[2] += v.z * w; acc[3] += v.w * w;
    }
    const float f = (l > 0.f ? 1.f / l : 0.f) * (m == 0 ? 1.f : -lam);
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] += acc[j] * f;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) ss += o[j] * o[j];
  const float r = p.share / sqrtf(warp_sum(ss) / p.V + p.eps);
  __nv_bfloat16* dst = p.out + static_cast<size_t>(row / p.Hq) * p.ldo + (row % p.Hq) * TD + lane * 4;
  *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(o[0] * r, o[1] * r);
  *reinterpret_cast<__nv_bfloat162*>(dst + 2) = __floats2bfloat162_rn(o[2] * r, o[3] * r);
}

template <int G, int MODE>
static int launch_attn_tc(const AttnTcParams& p, int q_tiles, bool pdl, cudaStream_t stream) {
  static int configured[kMaxDevicesCached] = {};
  constexpr int kAttnTcSmem = attn_tc_smem(MODE);
  auto kern = paged_tree_attn_tc_kernel<G, MODE>;
  if (ensure_dyn_smem(kern, kAttnTcSmem, configured) != 0) return -3;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(q_tiles, p.Hkv, p.splits);
  cfg.blockDim = dim3(TTHREADS);
  cfg.dynamicSmemBytes = kAttnTcSmem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (p.cluster_merge) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = 1;
    attr[na].val.clusterDim.y = 1;
    attr[na].val.clusterDim.z = p.splits;
    ++na;
  }
  if (pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  return cudaLaunchKernelEx(&cfg, kern, p) == cudaSuccess ? 0 : -4;
}

}  // namespace js

// Profiling hook: 32 timestamps of CTA (0,0,0) go to `buf` (device memory) on every launch; nullptr switches it off.
extern "C" int js_attn_tc_set_trace(unsigned long long* buf) {
  return cudaMemcpyToSymbol(js::g_attn_trace, &buf, sizeof(buf)) == cudaSuccess ? 0 : -1;
}

extern "C" int js_attn_merge(float* ws_o, float* ws_ml, const float* gate, int ldg, void* out, int ldo, int T, int Hq, int splits, int pdl,
                             cudaStream_t stream);

// How many clusters of `splits` CTAs of the kernel for GQA group size G can be resident at once on the current
// device (a cluster lives inside one GPC, so this is less than SMs / splits); 0 or negative = cannot say.  The host
// picks the number of key splits from it so that a launch is one wave.
extern "C" int js_attn_tc_max_active_clusters(int G, int splits) {
  using namespace js;
  if (splits < 1 || splits > kMaxClusterSplits) return -1;
  const void* kern = nullptr;
  constexpr int kAttnTcSmem = attn_tc_smem(kPlain);      // what kPooled takes as well
  switch (G) {
    case 1: kern = reinterpret_cast<const void*>(paged_tree_attn_tc_kernel<1, kPlain>); break;
    case 2: kern = reinterpret_cast<const void*>(paged_tree_attn_tc_kernel<2, kPlain>); break;
    case 4: kern = reinterpret_cast<const void*>(paged_tree_attn_tc_kernel<4, kPlain>); break;
    case 8: kern = reinterpret_cast<const void*>(paged_tree_attn_tc_kernel<8, kPlain>); break;
    case 16: kern = reinterpret_cast<const void*>(paged_tree_attn_tc_kernel<16, kPlain>); break;
    default: return -2;
  }
  if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kAttnTcSmem) != cudaSuccess) return -3;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(1, 1, splits);
  cfg.blockDim = dim3(TTHREADS);
  cfg.dynamicSmemBytes = kAttnTcSmem;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = splits;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  int n = 0;
  if (cudaOccupancyMaxActiveClusters(&n, kern, &cfg) != cudaSuccess) { cudaGetLastError(); return -4; }
  return n;
}

// js_paged_tree_attention with the layout of the pools and the output spelled out: head h of slot s starts at
// h * kv_head + s * kv_slot, token t of the output at t * ldo (all multiples of 8).  Needs 128 % (Hq / Hkv) == 0 and
// W <= 8 (windows of up to 256 nodes).
// window > 0 limits a row to the last `window` tokens of its own path and the positions below `keep`; sink adds a valueless
// key of score sinks[head] (null: 0); gate (T, ldg) fp32 logits multiply a head's output by their sigmoid (null: none).
// softcap > 0 caps the scores; P > 0 adds the pooled blocks of P tokens
// that end before a row's window (kb, vb (Hkv, block_rows, 128) through block_map (max_seqs, max_blocks)); over a token tree the
// window must reach past the tree.  maps 2: differential attention with lam (device), share, eps and V value columns, q and pool
// rows 64 columns a map, ws_o and ws_ml twice as many rows; without a window, sinks or gates.
extern "C" int js_window_attention_tc(const void* q, const void* k_pool, const void* v_pool, const int* slot_map,
                                      const int* seq_rows, const int* cu_q, const int* past_lens, const int* mask_bits, void* out,
                                      float* ws_o, float* ws_ml, int* status, int B, int T, int Hq, int Hkv, int S, int max_len, int W,
                                      int causal, int splits, float scale, int window, int sink, int keep, const float* sinks,
                                      const float* gate, int ldg, float softcap, int P, const void* kb, const void* vb,
                                      int block_rows, const int* block_map, int max_blocks, int maps, const float* lam, float share,
                                      float eps, int V, long long kv_head, long long kv_slot, int ldo, int pdl, cudaStream_t stream) {
  using namespace js;
  if (window < 0 || keep < 0 || softcap < 0.f || P < 0 || maps < 1 || maps > 2) return -10;
  if (P > 0 && (window < 1 || kb == nullptr || vb == nullptr || block_map == nullptr)) return -13;
  if (maps == 2 && (window || sink || gate != nullptr || P || softcap > 0.f || lam == nullptr || V < 1 || V > TD)) return -13;
  if (T <= 0 || B <= 0) return 0;
  if (Hq % Hkv) return -10;
  if ((kv_head % 8) || (kv_slot % 8) || (ldo % 8)) return -10;
  const int G = Hq / Hkv;
  if (splits < 1) return -11;
  if (splits > 1 && (ws_o == nullptr || ws_ml == nullptr)) return -12;
  if (!causal && (mask_bits == nullptr || W < 1 || W > 8)) return -13;
  // The key splits merge inside a cluster only while every cluster of the launch is resident at once (a second
  // wave would double the kernel's time); otherwise partials go through the workspace and the merge kernel.
  bool in_cluster = maps == 1 && splits >= 2 && splits <= kMaxClusterSplits;
  if (in_cluster) {
    static int room[kMaxDevicesCached][5][kMaxClusterSplits + 1] = {};     // 0 = not asked yet
    int dev = 0;
    cudaGetDevice(&dev);
    const int gi = G == 1 ? 0 : G == 2 ? 1 : G == 4 ? 2 : G == 8 ? 3 : 4;
    int r = 0;
    if (dev >= 0 && dev < kMaxDevicesCached) r = room[dev][gi][splits];
    if (r == 0) {
      r = js_attn_tc_max_active_clusters(G, splits);
      if (r <= 0) r = -1;
      if (dev >= 0 && dev < kMaxDevicesCached) room[dev][gi][splits] = r;
    }
    const int npt = 128 / G;
    in_cluster = r > 0 && ((T + npt - 1) / npt) * Hkv <= r;
  }
  AttnTcParams p{reinterpret_cast<const __nv_bfloat16*>(q), reinterpret_cast<const __nv_bfloat16*>(k_pool),
                 reinterpret_cast<const __nv_bfloat16*>(v_pool), slot_map, seq_rows, cu_q, past_lens, mask_bits,
                 reinterpret_cast<__nv_bfloat16*>(out), ws_o, ws_ml, status, B, T, Hq, Hkv, S, max_len, W, causal,
                 splits, scale * 1.4426950408889634f, kv_head, kv_slot, ldo, window, sink, keep, sinks, gate, ldg,
                 in_cluster ? 1 : 0, softcap * 1.4426950408889634f, softcap > 0.f ? 2.8853900817779268f * scale / softcap : 0.f, P,
                 reinterpret_cast<const __nv_bfloat16*>(kb), reinterpret_cast<const __nv_bfloat16*>(vb), block_map, block_rows, max_blocks,
                 lam, share, eps, V};
  auto launch = [&](auto mode) {
    constexpr int M = decltype(mode)::value;
    switch (G) {
      case 1: return launch_attn_tc<1, M>(p, (T + 127) / 128 + B, pdl != 0, stream);
      case 2: return launch_attn_tc<2, M>(p, (T + 63) / 64 + B, pdl != 0, stream);
      case 4: return launch_attn_tc<4, M>(p, (T + 31) / 32 + B, pdl != 0, stream);
      case 8: return launch_attn_tc<8, M>(p, (T + 15) / 16 + B, pdl != 0, stream);
      case 16: return launch_attn_tc<16, M>(p, (T + 7) / 8 + B, pdl != 0, stream);
      default: return -14;
    }
  };
  const int rc = maps == 2 ? launch(std::integral_constant<int, kDiff>{})
               : P > 0 || softcap > 0.f ? launch(std::integral_constant<int, kPooled>{}) : launch(std::integral_constant<int, kPlain>{});
  if (rc != 0 || splits == 1 || p.cluster_merge) return rc;
  if (maps == 1) return js_attn_merge(ws_o, ws_ml, gate, ldg, out, ldo, T, Hq, splits, pdl, stream);
  cudaLaunchConfig_t c2 = {};
  c2.gridDim = dim3((T * Hq + 7) / 8);
  c2.blockDim = dim3(256);
  c2.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  c2.attrs = attr;
  c2.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&c2, diff_merge_kernel, p) == cudaSuccess ? 0 : -5;
}

// The same without a window; sinks and gate may be null.
extern "C" int js_paged_attention_tc_strided(const void* q, const void* k_pool, const void* v_pool, const int* slot_map,
                                          const int* seq_rows, const int* cu_q, const int* past_lens,
                                          const int* mask_bits, void* out, float* ws_o, float* ws_ml, int* status, int B,
                                          int T, int Hq, int Hkv, int S, int max_len, int W, int causal, int splits,
                                          float scale, const float* sinks, const float* gate, int ldg, long long kv_head,
                                          long long kv_slot, int ldo, int pdl, cudaStream_t stream) {
  return js_window_attention_tc(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, out, ws_o, ws_ml, status, B, T, Hq,
                                Hkv, S, max_len, W, causal, splits, scale, 0, sinks != nullptr, 0, sinks, gate, ldg, 0.f, 0, nullptr, nullptr, 0,
                                nullptr, 0, 1, nullptr, 0.f, 0.f, js::TD, kv_head, kv_slot, ldo, pdl, stream);
}

// Same arguments as js_paged_tree_attention.
extern "C" int js_paged_tree_attention_tc(const void* q, const void* k_pool, const void* v_pool, const int* slot_map,
                                          const int* seq_rows, const int* cu_q, const int* past_lens,
                                          const int* mask_bits, void* out, float* ws_o, float* ws_ml, int* status, int B,
                                          int T, int Hq, int Hkv, int S, int max_len, int W, int causal, int splits,
                                          float scale, int pdl, cudaStream_t stream) {
  return js_paged_attention_tc_strided(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, out, ws_o, ws_ml, status,
                                       B, T, Hq, Hkv, S, max_len, W, causal, splits, scale, nullptr, nullptr, 0,
                                       static_cast<long long>(S) * js::TD, js::TD, Hq * js::TD, pdl, stream);
}
