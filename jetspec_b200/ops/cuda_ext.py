"""Loader and thin tensor-level wrappers for the sm_100a kernel library.

The kernels live in ``csrc/*.cu`` and are compiled by ``nvcc`` for
``compute_100a/sm_100a`` into one shared library inside the package
(``jetspec_b200/_C/libjetspec_sm100.so``).  They export plain C entry points that
take raw device pointers and a stream, so there is no framework ABI to match and
the library builds in seconds; this module binds them with ``ctypes`` and passes
``tensor.data_ptr()`` and the current CUDA stream (launches are therefore
graph-capturable).

On a machine with a GPU a missing or unloadable library is an error, never a
silent fallback.

What these kernels stand in for in the reference: the fused verify stack's cuBLAS GEMMs and ATen glue
(``jetspec/inference_engine/compiled_verify_stack.py:170-272``), the Triton paged tree-attention kernel
(``jetspec/inference_engine/paged_tree_attn.py:55-367``, op wrapper ``paged_tree_attn_op.py:29-79``), the dense
tree-attention kernel of the HF path (``jetspec/core/tree_attention_kernel.py:63-216``), the graphed accept
(``jetspec/inference_engine/graph_capture.py:240-323``) and the grouped-GEMM MoE (``jetspec/models/moe_fused.py:16-116``).
"""
from __future__ import annotations

import ctypes
import glob
import os
import subprocess
import sys
from typing import Optional

import torch

_PKG = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_ROOT = os.path.dirname(_PKG)
# kernel sources: inside the installed package (wheel), else beside it (source checkout)
_CSRC = os.path.join(_PKG, "csrc") if os.path.isdir(os.path.join(_PKG, "csrc")) else os.path.join(_ROOT, "csrc")
_OUT_DIR = os.path.join(_PKG, "_C")
LIB_PATH = os.path.join(_OUT_DIR, "libjetspec_sm100.so")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-shared"]

_lib = None


def sources() -> list:
    return sorted(glob.glob(os.path.join(_CSRC, "*.cu")))


def _stale() -> bool:
    if not os.path.exists(LIB_PATH):
        return True
    t = os.path.getmtime(LIB_PATH)
    deps = sources() + glob.glob(os.path.join(_CSRC, "*.cuh")) + glob.glob(os.path.join(_CSRC, "*.h"))
    return any(os.path.getmtime(f) > t for f in deps)


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile every ``csrc/*.cu`` for sm_100a into the in-tree shared library."""
    if not force and not _stale():
        return LIB_PATH
    if not os.path.isdir(_CSRC):
        raise RuntimeError(f"kernel sources not found at {_CSRC}")
    os.makedirs(_OUT_DIR, exist_ok=True)
    # Several ranks may find the library stale at the same moment: one builds under a file lock, into a
    # temporary name that replaces the library atomically; the others wait and then find it fresh.
    import fcntl
    with open(os.path.join(_OUT_DIR, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        try:
            if not force and not _stale():
                return LIB_PATH
            nvcc = os.environ.get("NVCC", "nvcc")
            tmp = f"{LIB_PATH}.{os.getpid()}.tmp"
            # one object per source, compiled concurrently and kept beside the library, so a change to one
            # kernel file recompiles that file only; headers invalidate everything
            obj_dir = os.path.join(_OUT_DIR, "obj")
            os.makedirs(obj_dir, exist_ok=True)
            hdr_time = max([os.path.getmtime(f) for f in glob.glob(os.path.join(_CSRC, "*.cuh")) +
                            glob.glob(os.path.join(_CSRC, "*.h"))] or [0.0])
            compile_flags = [f for f in NVCC_FLAGS if f != "-shared"] + (["-Xptxas=-v"] if verbose else [])
            jobs = []
            for src in sources():
                obj = os.path.join(obj_dir, os.path.basename(src)[:-3] + ".o")
                fresh = (not force and os.path.exists(obj)
                         and os.path.getmtime(obj) >= max(os.path.getmtime(src), hdr_time))
                jobs.append((src, obj, fresh))
            procs = [(src, subprocess.Popen([nvcc] + compile_flags + ["-I", _CSRC, "-c", src, "-o", obj],
                                            stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True))
                     for src, obj, fresh in jobs if not fresh]
            log = []
            for src, pr in procs:
                out, err = pr.communicate()
                log.append(err)
                if pr.returncode != 0:
                    for _, other in procs:
                        if other.poll() is None:
                            other.kill()
                    raise RuntimeError(f"nvcc failed on {os.path.basename(src)}:\n{out}\n{err}")
            r = subprocess.run([nvcc] + NVCC_FLAGS + [obj for _, obj, _ in jobs] + ["-o", tmp],
                               capture_output=True, text=True)
            if r.returncode != 0:
                if os.path.exists(tmp):
                    os.remove(tmp)
                raise RuntimeError(f"nvcc link failed:\n{r.stdout}\n{r.stderr}")
            os.replace(tmp, LIB_PATH)
            if verbose:
                print("".join(log), file=sys.stderr)
        finally:
            fcntl.flock(lock, fcntl.LOCK_UN)
    return LIB_PATH


def available() -> bool:
    return os.path.exists(LIB_PATH)


def load():
    """``ctypes`` handle of the kernel library (built on first use when a compiler is present)."""
    global _lib
    if _lib is not None:
        return _lib
    if _stale():
        try:
            build()
        except Exception as e:  # no compiler on this machine: use an existing library if there is one
            if not os.path.exists(LIB_PATH):
                raise RuntimeError(f"sm_100a kernel library is missing and could not be built: {e}") from e
    lib = ctypes.CDLL(LIB_PATH)
    for name in ("js_gemm_bf16", "js_paged_tree_attention", "js_embed", "js_rmsnorm", "js_qkv_post", "js_silu_mul",
                 "js_gather_rows", "js_argmax_merge", "js_topk_merge", "js_tree_build", "js_tree_accept_commit",
                 "js_draft_prep"):
        getattr(lib, name).restype = ctypes.c_int
    _lib = lib
    return lib


# ------------------------------------------------------------------ helpers
_vp = ctypes.c_void_p


def _p(t: Optional[torch.Tensor]):
    return _vp(t.data_ptr()) if t is not None else _vp(0)


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_cur_device = getattr(torch._C, "_cuda_getDevice", None)


def _stream():
    """The current stream of the current device as a raw handle.  ``torch.cuda.current_stream()`` builds a Python
    ``Stream`` object and resolves the device index on every call (~10 us, paid per kernel launch on the eager
    path); the raw accessor is a plain C call."""
    if _raw_stream is not None and _cur_device is not None:
        return _vp(_raw_stream(_cur_device()))
    return _vp(torch.cuda.current_stream().cuda_stream)


def _check(rc: int, what: str):
    if rc != 0:
        raise RuntimeError(f"{what} failed with code {rc}")


_status: dict = {}


def status_word(device) -> torch.Tensor:
    """Per-device int32 the kernels write an error code to (0 = ok)."""
    dev = torch.device(device)
    key = dev.index if dev.index is not None else (torch.cuda.current_device() if dev.type == "cuda" else -1)
    if key not in _status:
        with torch.inference_mode(False):       # a normal tensor: it is cleared in place from any calling context
            _status[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status[key]


STATUS_NAMES = {0: "ok", 1: "timeout waiting for a TMA stage", 2: "timeout waiting for a free stage",
                3: "timeout waiting for the accumulator", 4: "timeout waiting for a peer flag",
                5: "KV slot out of range", 6: "tree node index out of range",
                7: "expert-parallel dispatch: a rank's expert counts never arrived",
                8: "expert-parallel dispatch: a source rank's rows never arrived",
                9: "all-reduce tail / expert combine: partial cells never arrived",
                10: "all-reduce tail: a slice owner's result cells never arrived",
                11: "vocabulary-parallel top-k: a rank's record never arrived",
                12: "expert-parallel dispatch: more rows for one expert than the grouped launch covers"}


def check_status(device) -> None:
    """Raise if any kernel recorded an error since the last check (one host sync)."""
    w = status_word(device)
    code = int(w.item())
    if code != 0:
        w.zero_()
        raise RuntimeError(f"kernel status {code}: {STATUS_NAMES.get(code, 'unknown')}")


_inv_freq: dict = {}


def inv_freq(head_dim: int, theta: float, device) -> torch.Tensor:
    key = (head_dim, float(theta), str(device))
    if key not in _inv_freq:
        from .reference import rope_inv_freq
        _inv_freq[key] = rope_inv_freq(head_dim, theta, device).contiguous()
    return _inv_freq[key]


# ------------------------------------------------------------------ GEMM
EPI_STORE, EPI_SWIGLU, EPI_ARGMAX, EPI_TOPK, EPI_STORE_F32 = 0, 1, 2, 3, 4
EPI_RELU2 = 8
ACT_GELU_GLU, ACT_RELU2, ACT_NONE, ACT_GELU_ERF, ACT_XIELU = 0, 1, 2, 3, 4
SM_COUNT = 148
_DEEP = os.environ.get("JETSPEC_GEMM_DEEP", "0") == "1"
_SPLIT_DEEP = os.environ.get("JETSPEC_SPLIT_DEEP")      # force the split-K pipeline: 1 = 192 KB, 2 = 128 KB, 0 = 96 KB
_SPLIT_DEEP = int(_SPLIT_DEEP) if _SPLIT_DEEP is not None else None


# measured best (bn, split, deep) per (M, N, K, epilogue); filled from the tuning sweep
GEMM_TUNING: dict = {}


def gemm_supported(M: int, N: int, K: int) -> bool:
    return K % 8 == 0 and N % 8 == 0 and K >= 64


def gu_tile(intermediate: int) -> int:
    """Tile width of the fused gate/up GEMM (the weight is interleaved at this granularity): 128, or the value of
    ``JETSPEC_GU_TILE`` (128, 192 or 256).  192 columns turn Qwen3-8B's 192 tiles of 128 columns (two CTAs on 44 of
    the 148 SMs) into one even wave of 128 CTAs, but measured slower in the decode round (5.77 against 5.61 ms):
    with one CTA per SM nothing streams while a tile's SwiGLU epilogue runs, whereas two shallow CTAs per SM
    overlap one's epilogue with the other's loads."""
    env = os.environ.get("JETSPEC_GU_TILE")
    return int(env) if env else 128


def pick_gemm_config(M: int, N: int, K: int, epi: int, bn: Optional[int] = None):
    """``(bn, split, deep)``: tile width, K-split cluster size, pipeline variant.

    Decode shapes are weight-streaming bound, so the goal is enough CTAs to cover the
    SMs (two CTAs fit per SM with the shallow pipeline) without re-reading the
    activations more than necessary.
    """
    key = (M, N, K, epi)
    if key in GEMM_TUNING:
        return GEMM_TUNING[key]
    m_tiles = (M + 127) // 128
    if bn is None and epi == EPI_STORE and m_tiles >= 4 and N % 256 == 0 and m_tiles * (N // 256) >= 64:
        # prefill / batched verify (>= 512 rows): compute bound, and a 128x128 tile asks more of the L2-to-SM path
        # than it gives; 128x256 tiles with the deep pipeline measured 5-12 % faster at 2048 rows
        # (qkv 97 -> 91 us, o 62 -> 56, down 182 -> 165) and equal or better at 512.  From 1024 rows on, two row tiles
        # per CTA (deep = 3: 256 x 256 outputs per CTA, every weight stage feeds two accumulators) when that does not
        # cost a wave: at 2048 rows o 53.9 -> 48.7 us, down 155.4 -> 146.3 (128 CTAs, one wave), but qkv
        # 88.1 -> 96.2 (192 CTAs: two waves of big tiles against three of small ones), gate/up equal.
        if m_tiles >= 8:
            t1, t2 = m_tiles * (N // 256), ((m_tiles + 1) // 2) * (N // 256)
            if 2 * ((t2 + SM_COUNT - 1) // SM_COUNT) <= (t1 + SM_COUNT - 1) // SM_COUNT:
                return 256, 1, 3
        return 256, 1, 1
    bn = bn or 128
    tiles = m_tiles * ((N + bn - 1) // bn)
    kb = (K + 63) // 64
    split = 1
    if epi in (EPI_STORE, EPI_STORE_F32, EPI_SWIGLU):
        # SwiGLU tiles hold two (gate, up) chunk pairs, so a split of 4 leaves two CTAs of each cluster without
        # output columns; it still pays when the projection is narrow (tensor-parallel shards: 24 tiles -> 96 CTAs)
        max_split = 4
        # Measured on chains of L2-cold GEMMs (M = 128): a K split helps while the whole grid is one
        # wave of one CTA per SM AND the clusters can be placed (a cluster lives inside one GPC, so only
        # ~32 clusters of 4, ~40 of 3 or ~72 of 2 fit at once; 48 clusters of 3 ran as two waves).
        room = {2: 72, 3: 40, 4: 32}
        for c in (4, 3, 2):
            if c <= max_split and tiles <= room[c] and tiles * c <= SM_COUNT and kb // c >= 4:
                split = c
                break
    if split > 1:
        # deep pipeline (192 KB, one CTA per SM; the receive area aliases the stages), except for the narrow shards of
        # a tensor-parallel rank (at most 96 CTAs with at most 16 k-blocks each): 128 KB serves those as well and
        # leaves room for the next kernel's CTA and its first weight stages on the same SM (compute-only round of a
        # 1/8 shard: 2.96 -> 2.92 ms).  The full-size o_proj (128 CTAs) measured slower that way inside the round
        # (5.45 -> 5.50 ms) although faster in a chain of its own.  JETSPEC_SPLIT_DEEP forces 1 (192 KB), 2 (128 KB)
        # or 0 (96 KB) for every split launch.
        if _SPLIT_DEEP is not None:
            return bn, split, _SPLIT_DEEP
        return bn, split, (2 if (kb + split - 1) // split <= 16 and tiles * split <= 96 else 1)
    # no split: a deep pipeline when the tiles fit one CTA per SM, else two shallow CTAs per SM
    return bn, 1, (1 if tiles <= SM_COUNT or _DEEP else 0)


def gemm(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None,
         residual: Optional[torch.Tensor] = None, epi: int = EPI_STORE, bn: Optional[int] = None,
         split: Optional[int] = None, deep: Optional[bool] = None, pdl: bool = False,
         part_val=None, part_idx=None, part_lse=None, trace: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out = x @ w.T`` (+ ``residual``) on the tcgen05 kernel.  ``x (M, K)``, ``w (N, K)`` bf16."""
    lib = load()
    M, K = x.shape
    N = w.shape[0]
    assert w.shape[1] == K and x.stride(1) == 1 and w.stride(1) == 1
    cb, cs, cd = pick_gemm_config(M, N, K, epi, bn)
    bn = bn or cb
    split = split or cs
    deep = cd if deep is None else deep
    if out is None:
        if epi == EPI_SWIGLU:
            out = torch.empty(M, N // 2, dtype=torch.bfloat16, device=x.device)
        elif epi == EPI_STORE_F32:
            out = torch.empty(M, N, dtype=torch.float32, device=x.device)
        elif epi in (EPI_STORE,):
            out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    ldc = out.stride(0) if out is not None else 0
    rc = lib.js_gemm_bf16(_p(x), _p(w), _p(out), _p(residual), M, N, K, x.stride(0), w.stride(0), ldc, epi, bn,
                          split, int(deep), _p(part_val), _p(part_idx), _p(part_lse),
                          _p(status_word(x.device)), _p(trace), int(pdl), _stream())
    _check(rc, f"js_gemm_bf16(M={M},N={N},K={K},epi={epi},bn={bn},split={split})")
    return out


def interleave_gate_up(gate_w: torch.Tensor, up_w: torch.Tensor, bn: int = 128) -> torch.Tensor:
    """Weight layout for the SwiGLU epilogue: every ``bn``-row tile holds ``bn/2`` gate rows
    followed by the ``bn/2`` up rows of the same outputs."""
    I, H = gate_w.shape
    h = bn // 2
    assert I % h == 0
    if not isinstance(gate_w, torch.Tensor):      # NVFP4: stack, then permute rows (exact: rows are independent)
        t = torch.arange(I, device=gate_w.packed.device).view(I // h, h)
        order = torch.cat((t, t + I), dim=1).reshape(-1)
        return type(gate_w).cat_rows([gate_w, up_w]).index_rows(order)
    g = gate_w.view(I // h, h, H)
    u = up_w.view(I // h, h, H)
    return torch.cat((g, u), dim=1).reshape(2 * I, H).contiguous()


def n_tiles(N: int, bn: int = 128) -> int:
    return (N + bn - 1) // bn


# ------------------------------------------------------------------ NVFP4
def nvfp4_act_buffers(M: int, K: int, device) -> dict:
    """Device buffers one quantised activation matrix needs (allocate once, reuse across graph replays)."""
    tiles = (M + 127) // 128
    return {"packed": torch.zeros(M, K // 2, dtype=torch.uint8, device=device),
            "sf": torch.zeros(tiles * (K // 64) * 512, dtype=torch.uint8, device=device),
            "outer": torch.zeros(M, dtype=torch.float32, device=device), "M": M, "K": K}


def quant_nvfp4(x: torch.Tensor, buf: Optional[dict] = None, norm_w: Optional[torch.Tensor] = None, eps: float = 1e-6,
                norm_out: Optional[torch.Tensor] = None, pdl: bool = False) -> dict:
    """Quantise ``x (M, K)`` bf16 to NVFP4 with one outer scale per row; with ``norm_w`` the RMSNorm of ``x`` is
    quantised instead (and also written to ``norm_out`` as bf16 when given)."""
    lib = load()
    M, K = x.shape
    assert x.dtype == torch.bfloat16 and x.stride(1) == 1
    if buf is None:
        buf = nvfp4_act_buffers(M, K, x.device)
    assert buf["K"] == K and buf["M"] >= M
    lib.js_quant_nvfp4.restype = ctypes.c_int
    rc = lib.js_quant_nvfp4(_p(x), x.stride(0), _p(norm_w), ctypes.c_float(eps), M, K, _p(buf["packed"]), _p(buf["sf"]),
                            _p(buf["outer"]), _p(norm_out), norm_out.stride(0) if norm_out is not None else 0,
                            int(pdl), _stream())
    _check(rc, f"js_quant_nvfp4(M={M},K={K})")
    return buf


def pick_nvfp4_split(M: int, N: int, K: int, epi: int) -> int:
    """K split for the NVFP4 GEMM: same placement rule as the bf16 kernel (clusters of 4 / 2 that fit one wave)."""
    tiles = ((M + 127) // 128) * ((N + 127) // 128)
    kb = K // 256
    max_split = 2 if epi == EPI_SWIGLU else 4
    room = {2: 72, 4: 32}
    for c in (4, 2):
        if c <= max_split and tiles <= room[c] and tiles * c <= SM_COUNT and kb // c >= 2:
            return c
    return 1


def gemm_nvfp4(x, qw, out: Optional[torch.Tensor] = None, residual: Optional[torch.Tensor] = None,
               epi: int = EPI_STORE, split: Optional[int] = None, pdl: bool = False, act_buf: Optional[dict] = None):
    """``out = q(x) @ dequant(qw).T`` on the block-scaled tcgen05 kernel.

    ``x`` is either a bf16 ``(M, K)`` matrix (quantised here, per row) or the dict ``quant_nvfp4`` returned;
    ``qw`` is an ``NVFP4Tensor`` with per-tensor outer scale and swizzled block scales.
    """
    lib = load()
    act = x if isinstance(x, dict) else quant_nvfp4(x, act_buf, pdl=pdl)
    M = x.shape[0] if not isinstance(x, dict) else act.get("rows", act["M"])
    N, K = qw.shape
    assert act["K"] == K
    qw.swizzled()
    split = split or pick_nvfp4_split(M, N, K, epi)
    dev = qw.packed.device
    if out is None:
        out = torch.empty(M, N // 2 if epi == EPI_SWIGLU else N,
                          dtype=torch.float32 if epi == EPI_STORE_F32 else torch.bfloat16, device=dev)
    if not hasattr(qw, "_w_scale"):
        qw._w_scale = float(qw.outer)           # one host read per weight, outside any graph capture
    lib.js_gemm_nvfp4.restype = ctypes.c_int
    rc = lib.js_gemm_nvfp4(_p(act["packed"]), _p(act["sf"]), _p(act["outer"]), _p(qw.packed), _p(qw.scales_swizzled),
                           ctypes.c_float(qw._w_scale), _p(out), _p(residual), M, N, K, act["packed"].stride(0),
                           qw.packed.stride(0), out.stride(0), epi, split, _p(status_word(dev)), int(pdl), _stream())
    _check(rc, f"js_gemm_nvfp4(M={M},N={N},K={K},epi={epi},split={split})")
    return out


def lm_head_argmax(h: torch.Tensor, w: torch.Tensor, ws: Optional[dict] = None, pdl: bool = False,
                   out_idx: Optional[torch.Tensor] = None, out_val: Optional[torch.Tensor] = None):
    """Greedy token per row: vocabulary GEMM with a per-tile argmax epilogue, then a merge.
    The ``(M, V)`` logits are never written."""
    lib = load()
    M, N = h.shape[0], w.shape[0]
    nt = n_tiles(N)
    if ws is None:
        ws = {"val": torch.empty(M, nt, dtype=torch.float32, device=h.device),
              "idx": torch.empty(M, nt, dtype=torch.int32, device=h.device)}
    gemm(h, w, out=None, epi=EPI_ARGMAX, bn=128, split=1, pdl=pdl, part_val=ws["val"], part_idx=ws["idx"])
    if out_idx is None:
        out_idx = torch.empty(M, dtype=torch.int32, device=h.device)
    if out_val is None:
        out_val = torch.empty(M, dtype=torch.float32, device=h.device)
    _check(lib.js_argmax_merge(_p(ws["val"]), _p(ws["idx"]), nt, M, _p(out_idx), _p(out_val), int(pdl), _stream()),
           "js_argmax_merge")
    return out_idx, out_val


# Few-row top-k over the vocabulary in two passes over materialised logits (JETSPEC_TOPK_TWO_PASS=0: inside the GEMM
# epilogue, as for many rows).  The partial lists reuse the epilogue's workspace: (rows, slices, 8) fits (rows, tiles, 8).
TOPK_TWO_PASS = os.environ.get("JETSPEC_TOPK_TWO_PASS", "1") != "0"
TOPK_TWO_PASS_ROWS = 32
TOPK_SLICES = 64


def lm_head_topk_logprobs(h: torch.Tensor, w: torch.Tensor, k: int, ws: Optional[dict] = None, pdl: bool = False,
                          out_tok: Optional[torch.Tensor] = None, out_lp: Optional[torch.Tensor] = None):
    """Per-row top-``k`` tokens with full-vocabulary log-probabilities, without materialising logits."""
    lib = load()
    assert 1 <= k <= 8
    M, N = h.shape[0], w.shape[0]
    nt = n_tiles(N)
    if ws is None:
        ws = {"val": torch.empty(M, nt, 8, dtype=torch.float32, device=h.device),
              "idx": torch.empty(M, nt, 8, dtype=torch.int32, device=h.device),
              "lse": torch.empty(M, nt, 2, dtype=torch.float32, device=h.device)}
    if out_tok is None:
        out_tok = torch.empty(M, k, dtype=torch.int32, device=h.device)
    if out_lp is None:
        out_lp = torch.empty(M, k, dtype=torch.float32, device=h.device)
    if TOPK_TWO_PASS and M <= TOPK_TWO_PASS_ROWS and N % 4 == 0 and nt >= TOPK_SLICES:
        # A draft block has a few rows, so one warp per CTA would carry the in-epilogue sorted insertion and the
        # weight stream stalls behind it.  Store the (few) logits with the plain fp32 epilogue instead, which streams
        # at the argmax epilogue's rate, and take the top-k from them in two small passes (they stay in L2).
        if "logits" not in ws or ws["logits"].shape[0] < M or ws["logits"].shape[1] != N:
            ws["logits"] = torch.empty(max(M, TOPK_TWO_PASS_ROWS), N, dtype=torch.float32, device=h.device)
        logits = ws["logits"][:M]
        gemm(h, w, out=logits, epi=EPI_STORE_F32, bn=128, split=1, pdl=pdl)
        lib.js_logits_topk_slices.restype = ctypes.c_int
        _check(lib.js_logits_topk_slices(_p(logits), ctypes.c_longlong(logits.stride(0)), M, N, TOPK_SLICES,
                                         _p(ws["val"]), _p(ws["idx"]), _p(ws["lse"]), int(pdl), _stream()),
               "js_logits_topk_slices")
        _check(lib.js_topk_merge(_p(ws["val"]), _p(ws["idx"]), _p(ws["lse"]), TOPK_SLICES, M, k, _p(out_tok),
                                 _p(out_lp), int(pdl), _stream()), "js_topk_merge")
        return out_tok, out_lp
    gemm(h, w, out=None, epi=EPI_TOPK, bn=128, split=1, pdl=pdl, part_val=ws["val"], part_idx=ws["idx"],
         part_lse=ws["lse"])
    _check(lib.js_topk_merge(_p(ws["val"]), _p(ws["idx"]), _p(ws["lse"]), nt, M, k, _p(out_tok), _p(out_lp),
                             int(pdl), _stream()), "js_topk_merge")
    return out_tok, out_lp


# ------------------------------------------------------------------ elementwise
def embed(ids: torch.Tensor, table: torch.Tensor, out: Optional[torch.Tensor] = None, pdl: bool = False):
    lib = load()
    T, (V, H) = ids.numel(), table.shape
    if out is None:
        out = torch.empty(T, H, dtype=table.dtype, device=table.device)
    _check(lib.js_embed(_p(ids), _p(table), _p(out), T, H, V, int(pdl), _stream()), "js_embed")
    return out


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, out: Optional[torch.Tensor] = None, pdl: bool = False):
    lib = load()
    shp = x.shape
    x2 = x.reshape(-1, shp[-1])
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    if out is None:
        out = torch.empty(x2.shape, dtype=x.dtype, device=x.device)
    o2 = out.reshape(-1, shp[-1])
    _check(lib.js_rmsnorm(_p(x2), _p(w), _p(o2), x2.shape[0], shp[-1], x2.stride(0), o2.stride(0),
                          ctypes.c_float(eps), int(pdl), _stream()), "js_rmsnorm")
    return out.reshape(shp)


def silu_mul(gate_up: torch.Tensor, out: Optional[torch.Tensor] = None, pdl: bool = False):
    lib = load()
    T, I2 = gate_up.shape
    gate_up = gate_up.contiguous()
    if out is None:
        out = torch.empty(T, I2 // 2, dtype=gate_up.dtype, device=gate_up.device)
    _check(lib.js_silu_mul(_p(gate_up), _p(out), T, I2 // 2, int(pdl), _stream()), "js_silu_mul")
    return out


def qkv_post(qkv: torch.Tensor, q_norm_w, k_norm_w, positions: torch.Tensor, slots: torch.Tensor,
             freq: torch.Tensor, q_out: Optional[torch.Tensor], k_pool: torch.Tensor, v_pool: torch.Tensor,
             Hq: int, Hkv: int, eps: float, n_valid: Optional[torch.Tensor] = None, pdl: bool = False):
    """Per-head RMSNorm + RoPE on the fused QKV rows; q → ``q_out``, k/v → pools at ``slots``."""
    lib = load()
    T = qkv.shape[0]
    S = k_pool.shape[1]
    _check(lib.js_qkv_post(_p(qkv), qkv.stride(0), _p(q_norm_w), _p(k_norm_w), _p(positions), _p(slots), _p(freq),
                           _p(q_out), _p(k_pool), _p(v_pool), T, Hq, Hkv, S, ctypes.c_float(eps), _p(n_valid),
                           _p(status_word(qkv.device)), int(pdl), _stream()), "js_qkv_post")
    return q_out


def gather_rows(src: torch.Tensor, idx: Optional[torch.Tensor], dst: torch.Tensor, dst_col0: int = 0,
                n_valid: Optional[torch.Tensor] = None, rows: Optional[int] = None, pdl: bool = False):
    lib = load()
    rows = rows if rows is not None else (idx.numel() if idx is not None else src.shape[0])
    H = src.shape[1]
    _check(lib.js_gather_rows(_p(src), src.stride(0), _p(idx), _p(n_valid), _p(dst), dst.stride(0), dst_col0, rows, H,
                              src.shape[0], int(pdl), _stream()), "js_gather_rows")
    return dst


# ------------------------------------------------------------------ attention
def attn_splits(q_tiles: int, Hkv: int, max_keys: int) -> int:
    # the launcher adds one q tile per sequence for raggedness; keep the whole grid in ONE wave
    # (two CTAs fit per SM) and give every split at least a couple of key tiles
    ctas = max(1, (q_tiles + 1) * Hkv)
    want = max(1, (2 * SM_COUNT) // ctas)
    return max(1, min(want, (max_keys + 127) // 128, 16))


ATTN_CLUSTER_SPLITS = 8       # key splits the tcgen05 kernel merges inside one cluster (kMaxClusterSplits)
ATTN_IMPL = os.environ.get("JETSPEC_ATTN", "tc")     # "tc": tcgen05 kernel where it applies; "mma": mma.sync kernel


def attn_impl(Hq: int, Hkv: int, W: int = 0) -> str:
    G = Hq // Hkv
    return "tc" if ATTN_IMPL == "tc" and 128 % G == 0 and W <= 8 else "mma"


_ATTN_ROOM: dict = {}


def _attn_cluster_room(G: int, splits: int) -> int:
    """Clusters of ``splits`` CTAs of the tcgen05 attention kernel the current device holds at once."""
    dev = torch.cuda.current_device() if torch.cuda.is_available() else -1
    key = (dev, G, splits)
    if key not in _ATTN_ROOM:
        n = 0
        if dev >= 0:
            lib = load()
            lib.js_attn_tc_max_active_clusters.restype = ctypes.c_int
            n = int(lib.js_attn_tc_max_active_clusters(int(G), int(splits)))
        if n <= 0:       # no device / no answer: what was measured on a 148-SM part, else a conservative guess
            n = {2: 72, 3: 40, 4: 32}.get(splits, SM_COUNT // (splits + 2))
        _ATTN_ROOM[key] = n
    return _ATTN_ROOM[key]


def attn_merges_in_cluster(T: int, Hq: int, Hkv: int, splits: int) -> bool:
    """Whether the tcgen05 kernel merges ``splits`` key splits itself (they form one cluster and exchange partial
    outputs through distributed shared memory): up to ATTN_CLUSTER_SPLITS, and only while all clusters of the
    launch are resident at once (a cluster lives inside one GPC: 148 SMs hold 33 clusters of 4 but only 15 of 8)."""
    G = Hq // Hkv
    if attn_impl(Hq, Hkv) != "tc" or not 2 <= splits <= ATTN_CLUSTER_SPLITS:
        return False
    npt = 128 // G
    return ((T + npt - 1) // npt) * Hkv <= _attn_cluster_room(G, splits)


def attn_splits_for(T: int, Hq: int, Hkv: int, max_keys: int, seqs: int = 1) -> int:
    """Key splits for ``T`` query tokens of ``seqs`` sequences: fill the SMs with ONE wave of CTAs, a couple of key tiles per
    split."""
    G = Hq // Hkv
    if attn_impl(Hq, Hkv) == "tc":                      # 128 rows per CTA, one CTA per SM
        # one wave of CTAs, a couple of key tiles per split.  Measured on the decode round (prefix ~2.5 k keys): more,
        # shorter splits win even when they need the separate merge launch (TP=2: 9 splits + merge 4.60 ms per round,
        # 6 splits merged inside a cluster 4.71 ms), because the kernel's time is the chain of key tiles of one CTA.
        npt = 128 // G
        ctas = max(1, max((T + npt - 1) // npt, seqs) * Hkv)             # a tile's rows are one sequence's
        return max(1, min(SM_COUNT // ctas, (max_keys + 127) // 128, 16))
    npt = max(1, 64 // G)
    return attn_splits((T + npt - 1) // npt, Hkv, max_keys)


def paged_tree_attention(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale: float,
                         causal: bool, max_q: int, out: Optional[torch.Tensor] = None, splits: Optional[int] = None,
                         ws: Optional[dict] = None, max_keys: Optional[int] = None, pdl: bool = False,
                         impl: Optional[str] = None):
    """Ragged paged attention with tree (packed-bit) or causal masking.  See
    :func:`jetspec_b200.ops.reference.paged_tree_attention` for the contract."""
    lib = load()
    T, Hq, D = q.shape
    assert D == 128
    Hkv, S = k_pool.shape[0], k_pool.shape[1]
    B = seq_rows.numel()
    G = Hq // Hkv
    if out is None:
        out = torch.empty(T, Hq * D, dtype=q.dtype, device=q.device)
    if splits is None:
        mk = max_keys if max_keys is not None else slot_map.shape[1]
        splits = attn_splits_for(T, Hq, Hkv, mk)
    ws_o = ws_ml = None
    if splits > 1:
        if ws is None:
            ws = {"o": torch.empty(splits, T, Hq, D, dtype=torch.float32, device=q.device),
                  "ml": torch.empty(splits, T, Hq, 2, dtype=torch.float32, device=q.device)}
        ws_o, ws_ml = ws["o"], ws["ml"]
    W = mask_bits.shape[1] if mask_bits is not None else 0
    impl = impl or attn_impl(Hq, Hkv, W)
    fn = lib.js_paged_tree_attention_tc if impl == "tc" else lib.js_paged_tree_attention
    fn.restype = ctypes.c_int
    _check(fn(_p(q), _p(k_pool), _p(v_pool), _p(slot_map), _p(seq_rows), _p(cu_q),
              _p(past_lens), _p(mask_bits), _p(out), _p(ws_o), _p(ws_ml),
              _p(status_word(q.device)), B, T, Hq, Hkv, S, slot_map.shape[1], W,
              int(bool(causal)), int(splits), ctypes.c_float(scale), int(pdl), _stream()),
           f"js_paged_tree_attention[{impl}]")
    return out


def _head_gate(gate: Optional[torch.Tensor]) -> tuple:
    """Pointer and leading dimension of the fp32 gate logits ``(T, >= heads)`` of an attention kernel."""
    assert gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1)
    return _p(gate), gate.stride(0) if gate is not None else 0


def _sinks(sinks: Optional[torch.Tensor], heads: int):
    """Pointer to the fp32 sink scores of an attention kernel's heads."""
    assert sinks is None or (sinks.dtype == torch.float32 and sinks.is_contiguous() and sinks.numel() == heads)
    return _p(sinks)


def paged_attention_rows(q, k_rows, v_rows, slot_map, seq_rows, cu_q, past_lens, scale: float, max_q: int, out, max_keys: int,
                         pdl: bool = False, sinks: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention over keys and values stored row-major, ``k_rows, v_rows (keys, Hkv*128)`` (views of one wider
    matrix are fine), on the tcgen05 kernel; ``out (T, >= Hq*128)`` may be a column block of a wider matrix.  ``sinks (Hq,)``:
    score of a valueless key per head; ``gate (T, >= Hq)``: logits whose sigmoid multiplies a head's output."""
    lib = load()
    T, Hq, D = q.shape
    Hkv = k_rows.shape[1] // 128
    assert D == 128 and q.is_contiguous() and k_rows.stride(1) == 1 and v_rows.stride() == k_rows.stride()
    splits = attn_splits_for(T, Hq, Hkv, max_keys)
    ws_o = ws_ml = None
    if splits > 1:
        ws_o = torch.empty(splits, T, Hq, D, dtype=torch.float32, device=q.device)
        ws_ml = torch.empty(splits, T, Hq, 2, dtype=torch.float32, device=q.device)
    _check(lib.js_paged_attention_tc_strided(
        _p(q), _p(k_rows), _p(v_rows), _p(slot_map), _p(seq_rows), _p(cu_q), _p(past_lens), None, _p(out), _p(ws_o), _p(ws_ml),
        _p(status_word(q.device)), seq_rows.numel(), T, Hq, Hkv, k_rows.shape[0], slot_map.shape[1], 0, 1, splits,
        ctypes.c_float(scale), _sinks(sinks, Hq), *_head_gate(gate), ctypes.c_longlong(128), ctypes.c_longlong(k_rows.stride(0)),
        out.stride(0), int(pdl), _stream()), "js_paged_attention_tc_strided")
    return out


def l2_prefetch(t: torch.Tensor, max_bytes: Optional[int] = None, ctas: int = 8) -> None:
    """Ask the memory system to pull the first ``max_bytes`` of ``t`` into L2 (launch on the CURRENT stream;
    the kernel only issues ``cp.async.bulk.prefetch.L2`` requests and exits)."""
    lib = load()
    n = t.numel() * t.element_size()
    if max_bytes is not None:
        n = min(n, int(max_bytes))
    lib.js_l2_prefetch.restype = ctypes.c_int
    _check(lib.js_l2_prefetch(_p(t), ctypes.c_size_t(n), int(ctas), _stream()), "js_l2_prefetch")


# ------------------------------------------------------------------ routing, sampling, compaction
def moe_route(router_logits: torch.Tensor, top_k: int, renorm: bool, pdl: bool = False):
    """``(weights (T, k) fp32, experts (T, k) int32)``: softmax over the experts, top-k, optional renormalisation."""
    lib = load()
    lg = router_logits.float().contiguous()
    T, E = lg.shape
    wts = torch.empty(T, top_k, dtype=torch.float32, device=lg.device)
    idx = torch.empty(T, top_k, dtype=torch.int32, device=lg.device)
    lib.js_moe_route.restype = ctypes.c_int
    _check(lib.js_moe_route(_p(lg), T, E, top_k, int(bool(renorm)), _p(wts), _p(idx), int(pdl), _stream()), "js_moe_route")
    return wts, idx


def moe_route_sort(router_logits: torch.Tensor, top_k: int, renorm: bool, first_expert: int, n_local: int,
                   pdl: bool = False, with_tokens: bool = False):
    """Routing plus the stable permutation of the (token, choice) pairs by local expert, all on the device.
    Returns ``(order int32 (T*k), row_weight fp32 (T*k), group_off int32 (n_local+1), counts_all int32 (E))``."""
    lib = load()
    wts, idx = moe_route(router_logits, top_k, renorm, pdl)
    T, E = router_logits.shape
    P = T * top_k
    dev = wts.device
    order = torch.empty(P, dtype=torch.int32, device=dev)
    row_w = torch.empty(P, dtype=torch.float32, device=dev)
    group_off = torch.empty(n_local + 1, dtype=torch.int32, device=dev)
    counts_all = torch.empty(E, dtype=torch.int32, device=dev)
    tok = torch.empty(P, dtype=torch.int32, device=dev) if with_tokens else None
    lib.js_moe_sort.restype = ctypes.c_int
    _check(lib.js_moe_sort(_p(idx), _p(wts), P, E, int(first_expert), int(n_local), _p(order), _p(row_w), _p(group_off),
                           _p(counts_all), int(top_k), _p(tok), int(pdl), _stream()), "js_moe_sort")
    if with_tokens:
        return order, row_w, group_off, counts_all, tok
    return order, row_w, group_off, counts_all


def sample_temperature(logits: torch.Tensor, temperature: float, generator=None) -> torch.Tensor:
    """Draw one token per row from ``softmax(logits / temperature)`` (inverse CDF with one uniform per row)."""
    lib = load()
    shp = logits.shape[:-1]
    flat = logits.reshape(-1, logits.shape[-1])
    if flat.dtype not in (torch.float32, torch.bfloat16):
        flat = flat.float()
    flat = flat.contiguous()
    N, V = flat.shape
    u = torch.rand(N, dtype=torch.float32, device=flat.device, generator=generator)
    out = torch.empty(N, dtype=torch.int64, device=flat.device)
    lib.js_sample_temperature.restype = ctypes.c_int
    _check(lib.js_sample_temperature(_p(flat), int(flat.dtype == torch.bfloat16), N, V, flat.stride(0),
                                     ctypes.c_float(temperature), _p(u), _p(out), _stream()), "js_sample_temperature")
    return out.view(shp)


def kv_compact(k: torch.Tensor, v: torch.Tensor, past_len: int, keep: torch.Tensor) -> None:
    """In place: positions ``past_len + i`` of ``k, v (Hkv, capacity, 128)`` take the rows ``past_len + keep[i]``."""
    lib = load()
    assert k.dtype == torch.bfloat16 and k.shape[-1] == 128 and k.is_contiguous() and v.is_contiguous()
    keep = keep.to(device=k.device, dtype=torch.int32).contiguous()
    lib.js_kv_compact.restype = ctypes.c_int
    _check(lib.js_kv_compact(_p(k), _p(v), k.shape[0], k.shape[1], int(past_len), _p(keep), keep.numel(), _stream()),
           "js_kv_compact")


# ------------------------------------------------------------------ latent attention, Dynamic Tanh, sigmoid routing
def _is_bf16(t: torch.Tensor) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32), t.dtype
    return int(t.dtype == torch.bfloat16)


def dynamic_tanh(x: torch.Tensor, alpha, weight, bias, out_dtype) -> torch.Tensor:
    """``tanh(alpha x) * weight + bias`` of fp32 rows ``x (T, W)``, result in ``out_dtype``."""
    lib = load()
    T, W = x.shape
    assert x.dtype == torch.float32 and x.stride(1) == 1
    out = torch.empty(T, W, dtype=out_dtype, device=x.device)
    _check(lib.js_dynamic_tanh(_p(x), x.stride(0), _p(alpha), _p(weight), _p(bias), _is_bf16(weight), _p(out), W,
                               _is_bf16(out), T, W, _stream()), "js_dynamic_tanh")
    return out


def gelu_tanh_mul(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    lib = load()
    gate, up = gate.contiguous(), up.contiguous()
    out = torch.empty_like(gate)
    _check(lib.js_gelu_tanh_mul(_p(gate), _p(up), _p(out), ctypes.c_longlong(gate.numel()), _is_bf16(gate), _stream()),
           "js_gelu_tanh_mul")
    return out


def relu_squared(x: torch.Tensor) -> torch.Tensor:
    lib = load()
    x = x.contiguous()
    out = torch.empty_like(x)
    _check(lib.js_relu_squared(_p(x), _p(out), ctypes.c_longlong(x.numel()), _is_bf16(x), _stream()), "js_relu_squared")
    return out


def latent_scatter(c: torch.Tensor, pool: torch.Tensor, slots: torch.Tensor) -> None:
    """Rows ``c (T, R)`` into ``pool (S, Rp)`` at ``slots``; columns past ``R`` are zeroed."""
    lib = load()
    assert c.dtype == pool.dtype and c.stride(1) == 1 and pool.is_contiguous() and slots.dtype == torch.int32
    _check(lib.js_latent_scatter(_p(c), c.stride(0), c.shape[1], _p(pool), pool.shape[1], pool.shape[0], _p(slots), c.shape[0],
                                 _is_bf16(c), _p(status_word(c.device)), _stream()), "js_latent_scatter")


LATENT_TC_MAX = 512        # most value columns of the tensor-core kernel
LATENT_TC_ROW = 768        # widest cached row of the tensor-core kernel


def latent_tc_ok(Rp: int, out_cols: Optional[int] = None) -> bool:
    """Whether the tensor-core kernel takes rows of ``Rp`` columns whose first ``out_cols`` are values."""
    return Rp <= LATENT_TC_ROW and (Rp if out_cols is None else out_cols) <= LATENT_TC_MAX


def latent_attn_splits(T: int, heads: int, seqs: int, max_q: int, Rp: int, max_keys: int, out_cols: Optional[int] = None) -> int:
    """Key splits of the tensor-core latent attention: one wave of CTAs (128 query rows of one sequence each, 64 for rows
    wider than 512; two column groups for more than 256 value columns), at least a couple of key tiles each."""
    per = 64 if Rp > 512 else 128
    tiles = min(T * heads // per + seqs, seqs * ((max_q * heads + per - 1) // per))
    ctas = max(1, tiles * (2 if (Rp if out_cols is None else out_cols) > 256 else 1))
    return max(1, min(SM_COUNT // ctas, (max_keys + 127) // 128, 16))


def latent_attention_rows(qa: torch.Tensor, pool: torch.Tensor, heads: int, slot_map, seq_rows, cu_q, past_lens, mask_bits,
                          scale: float, causal: bool, max_q: int, out: Optional[torch.Tensor] = None,
                          splits: Optional[int] = None, ws: Optional[dict] = None, max_keys: Optional[int] = None,
                          pdl: bool = False, impl: Optional[str] = None, tile: int = 0, out_cols: Optional[int] = None,
                          sinks: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of absorbed query rows ``qa (T*heads, Rp)`` over the latent rows of ``pool (S, Rp)``; ``out`` has the
    shape of ``qa``, of which the first ``out_cols`` columns are wanted.  ``impl``: ``"tc"`` (bf16, see :func:`latent_tc_ok`,
    masks up to 256 nodes) or ``"simt"``.  ``sinks (heads,)``: score of a valueless key per head; ``gate (T, >= heads)``: logits
    whose sigmoid multiplies a head's output."""
    lib = load()
    rows, Rp = qa.shape
    T, B = rows // heads, seq_rows.numel()
    assert qa.is_contiguous() and pool.is_contiguous() and pool.shape[1] == Rp and qa.dtype == pool.dtype
    if out is None:
        out = torch.empty_like(qa)
    W = mask_bits.shape[1] if mask_bits is not None else 0
    if impl is None:
        impl = "tc" if qa.dtype == torch.bfloat16 and latent_tc_ok(Rp, out_cols) and W <= 8 else "simt"
    st = _p(status_word(qa.device))
    if impl == "simt":
        _check(lib.js_latent_attention_simt(_p(qa), _p(pool), _p(slot_map), _p(seq_rows), _p(cu_q), _p(past_lens),
                                            _p(mask_bits), _p(out), B, T, heads, Rp, pool.shape[0], slot_map.shape[1], W,
                                            int(causal), ctypes.c_float(scale), _sinks(sinks, heads), *_head_gate(gate),
                                            _is_bf16(qa), st, _stream()),
               "js_latent_attention_simt")
        return out
    if splits is None:
        splits = latent_attn_splits(T, heads, B, max_q, Rp, max_keys if max_keys is not None else slot_map.shape[1], out_cols)
    if splits > 1 and ws is None:
        ws = {"o": torch.empty(splits, rows, Rp, dtype=torch.float32, device=qa.device),
              "ml": torch.empty(splits, rows, 2, dtype=torch.float32, device=qa.device)}
    _check(lib.js_latent_attention_tc(_p(qa), _p(pool), _p(slot_map), _p(seq_rows), _p(cu_q), _p(past_lens), _p(mask_bits),
                                      _p(out), _p(ws["o"] if splits > 1 else None), _p(ws["ml"] if splits > 1 else None), st,
                                      B, T, heads, Rp, Rp if out_cols is None else int(out_cols), pool.shape[0], slot_map.shape[1], W,
                                      int(causal), int(splits), int(max_q), ctypes.c_float(scale), _sinks(sinks, heads), *_head_gate(gate),
                                      int(tile), int(pdl), _stream()), "js_latent_attention_tc")
    return out


def latent_attention(q: torch.Tensor, w_uk, w_uv, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale: float,
                     causal: bool, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Unfused form (see :func:`jetspec_b200.ops.reference.latent_attention`): the key expansion is moved onto the
    query, the value expansion behind the attention, with library products around the attention kernel."""
    T, H, _ = q.shape
    R, D, Rp = w_uk.shape[1], w_uk.shape[0] // H, pool.shape[1]
    V, E = w_uv.shape[0] // H, q.shape[2] - D
    qa = torch.zeros(T, H, Rp, dtype=q.dtype, device=q.device)
    qa[:, :, :R] = torch.bmm(q[..., :D].transpose(0, 1), w_uk.view(H, D, R)).transpose(0, 1)
    qa[:, :, R:R + E] = q[..., D:]
    sinks = sink.detach().float().contiguous() if sink is not None else None
    o = latent_attention_rows(qa.view(T * H, Rp), pool, H, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale, causal, T, sinks=sinks,
                              out_cols=R)
    o = o.view(T, H, Rp)[:, :, :R].transpose(0, 1)
    return torch.bmm(o, w_uv.view(H, V, R).transpose(1, 2)).transpose(0, 1).reshape(T, H * V)


def sigmoid_route(logits: torch.Tensor, correction: torch.Tensor, top: int, scale: float, gate_col: int = -1,
                  act: Optional[torch.Tensor] = None, wts: Optional[torch.Tensor] = None, idx: Optional[torch.Tensor] = None,
                  pdl: bool = False):
    """``(weights (T, k) fp32, experts (T, k) int32)`` from fp32 router logits (a strided view may be wider than the
    experts: the first ``correction.numel()`` columns count); with ``act`` its rows are scaled in place by
    ``sigmoid(logits[:, gate_col])``."""
    lib = load()
    T, E = logits.shape[0], correction.numel()
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    correction = correction.float().contiguous()
    if wts is None:
        wts = torch.empty(T, top, dtype=torch.float32, device=logits.device)
        idx = torch.empty(T, top, dtype=torch.int32, device=logits.device)
    _check(lib.js_sigmoid_route(_p(logits), logits.stride(0), _p(correction), T, E, int(top), ctypes.c_float(scale), _p(wts),
                                _p(idx), int(gate_col), _p(act), act.stride(0) if act is not None else 0,
                                act.shape[1] if act is not None else 0, int(pdl), _stream()), "js_sigmoid_route")
    return wts, idx


def gemm_inproj(x, w, raw: Optional[torch.Tensor], n_raw: int, act_out: Optional[torch.Tensor], gelu: bool, pdl: bool = False,
                bn: Optional[int] = None, split: Optional[int] = None, deep: Optional[int] = None,
                act: Optional[int] = None, act_args: tuple = (0.0, 0.0)) -> None:
    """Fused input projections: ``x @ w.T`` whose first ``n_raw`` columns go to ``raw`` as fp32 and the rest through the
    activation (``gelu``: tanh-GELU gate * up on 64-row interleaved weights, else relu^2; ``act`` names any ``ACT_*``
    instead, with its constants ``act_args``) to ``act_out`` as bf16."""
    act = act if act is not None else ACT_GELU_GLU if gelu else ACT_RELU2
    lib = load()
    M, K = x.shape
    N = w.shape[0]
    if bn is None:
        tiles2 = ((M + 127) // 128) * (N // 256)
        if M >= 512 and N % 256 == 0 and tiles2 >= 64:
            bn, split, deep = 256, 1, 0
        else:
            bn, split, deep = pick_gemm_config(M, N, K, EPI_SWIGLU, 128)
    _check(lib.js_gemm_inproj(_p(x), _p(w), _p(raw), _p(act_out), M, N, K, x.stride(0), w.stride(0),
                              raw.stride(0) if raw is not None else 0, act_out.stride(0) if act_out is not None else 0,
                              int(n_raw), int(act), *map(ctypes.c_float, act_args), bn, split, int(deep), _p(status_word(x.device)), int(pdl),
                              _stream()), f"js_gemm_inproj(M={M},N={N},K={K},bn={bn},split={split})")


def gemm_resid32(a, w, x: torch.Tensor, norm=None, h: Optional[torch.Tensor] = None, emb: Optional[torch.Tensor] = None,
                 pdl: bool = False, bn: Optional[int] = None, split: Optional[int] = None, deep: Optional[int] = None) -> None:
    """``x += a @ w.T (+ emb)`` on the fp32 residual stream; ``norm = (weight fp32, bias fp32, alpha)`` also writes the
    Dynamic Tanh of the new ``x`` to ``h``."""
    lib = load()
    M, K = a.shape
    N = w.shape[0]
    if bn is None:
        bn, split, deep = pick_gemm_config(M, N, K, EPI_STORE)
        if bn == 256 and deep != 3:
            deep = 1
    nw, nb, alpha = norm if norm is not None else (None, None, 0.0)
    _check(lib.js_gemm_resid32(_p(a), _p(w), _p(x), _p(x), M, N, K, a.stride(0), w.stride(0), x.stride(0), _p(emb),
                               emb.stride(0) if emb is not None else 0, _p(h), h.stride(0) if h is not None else 0, _p(nw),
                               _p(nb), ctypes.c_float(alpha), bn, split, int(deep), _p(status_word(a.device)), int(pdl),
                               _stream()), f"js_gemm_resid32(M={M},N={N},K={K},bn={bn},split={split})")


def gemm_batched(a, w, out, batch: int, N: int, K: int, a_batch_k: int, c_batch_stride: int, ldc: int, pdl: bool = False) -> None:
    """``batch`` products in one launch: columns ``[z * a_batch_k, + K)`` of ``a`` times rows ``[z * N, + N)`` of ``w``
    (transposed), to ``out + z * c_batch_stride`` with leading dimension ``ldc``."""
    lib = load()
    _check(lib.js_gemm_bf16_batched(_p(a), _p(w), _p(out), a.shape[0], N, K, batch, a_batch_k, ctypes.c_longlong(c_batch_stride),
                                    a.stride(0), w.stride(0), ldc, _p(status_word(a.device)), int(pdl), _stream()),
           f"js_gemm_bf16_batched(M={a.shape[0]},N={N},K={K},batch={batch})")


def gemm_grouped(a, w, out, total_rows: int, N: int, groups: int, group_off, cover: int, epi: int) -> None:
    """Grouped GEMM over experts (rows of ``a`` sorted by expert, weights stacked)."""
    lib = load()
    _check(lib.js_gemm_bf16_grouped(_p(a), _p(w), _p(out), total_rows, N, a.shape[1], a.stride(0), w.stride(0), out.stride(0), epi,
                                    groups, _p(group_off), cover, None, None, None, None, 1, _p(status_word(a.device)), 0,
                                    _stream()), f"js_gemm_bf16_grouped(rows={total_rows},N={N},groups={groups},epi={epi})")


# ------------------------------------------------------------------ window attention, delta rules, post-norm steps
_pair_freq: dict = {}


def pair_freq(dims: int, base: float, device) -> torch.Tensor:
    key = (dims, float(base), str(device))
    if key not in _pair_freq:
        from .reference import pair_freq as table
        _pair_freq[key] = table(dims, base, device)
    return _pair_freq[key]


def rmsnorm_f32(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    lib = load()
    assert x.dim() == 2 and x.dtype == torch.float32 and x.stride(1) == 1
    out = torch.empty_like(x, memory_format=torch.contiguous_format)
    assert w.is_contiguous()
    _check(lib.js_rmsnorm_f32(_p(x), x.stride(0), _p(w), _is_bf16(w), _p(out), x.shape[0], x.shape[1], ctypes.c_float(eps),
                              _stream()), "js_rmsnorm_f32")
    return out


def rotate_norm(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, eps: Optional[float]) -> torch.Tensor:
    lib = load()
    T, heads, D = x.shape
    x = x.contiguous()
    out = torch.empty_like(x)
    # named: a temporary would be freed, and its memory possibly handed out again, before the launch
    pos, freq = positions.to(torch.int32), pair_freq(dims, base, x.device)
    _check(lib.js_rotate_norm(_p(x), _p(out), _p(pos), T, heads, D, dims, _p(freq),
                              int(eps is not None), ctypes.c_float(eps or 0.0), _is_bf16(x), _stream()), "js_rotate_norm")
    return out


def window_attention(q, k_pool, v_pool, vdim: int, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale: float, window: int,
                     sink, causal: bool, out: Optional[torch.Tensor] = None, pdl: bool = False, keep_first: int = 0,
                     gate: Optional[torch.Tensor] = None, softcap: float = 0.0, blocks=None, diff=None,
                     norm_dim: Optional[int] = None) -> torch.Tensor:
    """Window attention on the plain cores (bf16 or fp32, heads of up to 512); see the reference op for the arguments.  ``gate``:
    logits whose sigmoid multiplies a head's output (one map a head).  ``norm_dim``: columns of ``vdim`` that are not padding."""
    sinks = sink.detach().float().contiguous() if isinstance(sink, torch.Tensor) else None
    lib = load()
    T, H, D = q.shape
    assert q.stride(2) == 1 and q.stride(1) == D
    maps, (lam, share, eps) = (1, (None, 0.0, 0.0)) if diff is None else (2, diff)
    H //= maps
    lam = lam.detach().float().contiguous() if lam is not None else None
    kb, vb, block_map, P = blocks if blocks is not None else (None, None, None, 0)
    G, S, Dp = k_pool.shape
    if out is None:
        out = torch.empty(T, H * vdim, dtype=q.dtype, device=q.device)
    _check(lib.js_window_attention_simt(
        _p(q), ctypes.c_longlong(q.stride(0)), _p(k_pool), _p(v_pool), Dp, v_pool.shape[2], _p(slot_map), _p(seq_rows), _p(cu_q),
        _p(past_lens), _p(mask_bits), _p(out), out.stride(0), seq_rows.numel(), T, H, G, D, vdim, S, slot_map.shape[1],
        mask_bits.shape[1] if mask_bits is not None else 0, int(causal), ctypes.c_float(scale), int(window),
        int(sinks is not None or bool(sink)), int(keep_first), _sinks(sinks, H), *_head_gate(gate), ctypes.c_float(softcap), int(P), _p(kb),
        _p(vb), kb.shape[1] if P else 0, _p(block_map), block_map.shape[1] if P else 0, maps, _p(lam), ctypes.c_float(share), ctypes.c_float(eps),
        int(norm_dim or vdim), _is_bf16(q), _p(status_word(q.device)), int(pdl), _stream()), "js_window_attention_simt")
    return out


def pool_blocks(k_pool, v_pool, kb_pool, vb_pool, block_map, P: int, slot_map, seq_rows, cu_q, past_lens, rows: Optional[int] = None,
                counts=None, most: int = 0, pdl: bool = False) -> None:
    """Pool the blocks whose last token is among the sequences' new rows (see the reference op).  ``rows`` bounds the new rows
    where ``cu_q`` must not be read.  With ``counts`` (device) instead of ``cu_q`` the new tokens of a sequence are the last
    ``counts`` ones ahead of ``past_lens``, at most ``most``."""
    lib = load()
    G, S, Kw = k_pool.shape
    rows = int(cu_q[-1]) if rows is None and counts is None else rows or 0
    _check(lib.js_pool_blocks(_p(k_pool), _p(v_pool), _p(kb_pool), _p(vb_pool), G, S, kb_pool.shape[1], Kw, v_pool.shape[2], _p(block_map),
                              block_map.shape[1], P, _p(slot_map), slot_map.shape[1], _p(seq_rows), _p(cu_q), _p(past_lens), _p(counts),
                              most // P + 1, seq_rows.numel(), rows, _is_bf16(k_pool), _p(status_word(k_pool.device)), int(pdl), _stream()),
           "js_pool_blocks")


def xielu(x: torch.Tensor, up: float, down: float) -> torch.Tensor:
    lib = load()
    x = x.contiguous()
    out = torch.empty_like(x)
    _check(lib.js_xielu(_p(x), _p(out), ctypes.c_longlong(x.numel()), ctypes.c_float(up), ctypes.c_float(down), _is_bf16(x), _stream()), "js_xielu")
    return out


def depth_average(history: list, weights: torch.Tensor) -> torch.Tensor:
    lib = load()
    history, w = [x.contiguous() for x in history], weights.detach().float().contiguous()
    out = torch.empty_like(history[0])
    addr = (ctypes.c_ulonglong * len(history))(*[x.data_ptr() for x in history])
    _check(lib.js_depth_average(addr, len(history), _p(w), _p(out), ctypes.c_longlong(out.numel()), _stream()), "js_depth_average")
    return out


def sandwich(y, src, w, x, next_norm, eps: float, h, width: int, hist: Optional[torch.Tensor] = None, d: Optional[torch.Tensor] = None,
             tap: Optional[torch.Tensor] = None, pdl: bool = False) -> None:
    """Residual step of a sublayer whose output is normed: ``x = src + rms(y) w`` and ``h`` its norm with ``next_norm``.  At the
    end of a layer, ``hist (layers + 1, T, ld)`` and ``d`` (the layer's depth weights): the sum is the layer's result, kept as
    the next entry of ``hist``, and ``x`` the weighted sum over the entries so far."""
    lib = load()
    T, ld = x.shape
    assert src.stride(0) == ld and h.stride(0) == ld
    terms = d.numel() - 1 if d is not None else 0
    assert d is None or (hist.shape[1:] == x.shape and hist.shape[0] > terms)
    _check(lib.js_sandwich(_p(y), y.stride(0), _p(src), _p(w), _p(d), terms, _p(hist if d is not None else None), ctypes.c_longlong(T * ld),
                           _p(x), _p(next_norm), ctypes.c_float(eps), _p(h), ld, _p(tap), tap.stride(0) if tap is not None else 0, T, width,
                           int(pdl), _stream()), "js_sandwich")


def window_tc_ok(maps: int, pool: int, softcap: float) -> bool:
    """Whether the tensor-core kernel has a form for these options."""
    return maps == 1 or (maps == 2 and pool == 0 and softcap == 0.0)


def window_attn_splits(T: int, Hq: int, Hkv: int, max_keys: int, window: int, keep_first: int = 0, pool: int = 0,
                       seqs: int = 1) -> int:
    """Key splits of the tensor-core kernel: a CTA's rows span at most the window, their own tokens, the kept first ones and the
    pooled blocks."""
    keys = min(max_keys, window + 128 // (Hq // Hkv) + keep_first) if window else max_keys
    return attn_splits_for(T, Hq, Hkv, keys + (max_keys // pool if pool else 0), seqs)


def window_attention_tc(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale: float, window: int, sink,
                        causal: bool, out: torch.Tensor, splits: int = 1, ws: Optional[dict] = None, pdl: bool = False,
                        keep_first: int = 0, gate: Optional[torch.Tensor] = None, softcap: float = 0.0,
                        blocks=None, diff=None, vdim: int = 128) -> torch.Tensor:
    """Window attention on the tcgen05 kernel: bf16, heads padded to 128, groups of 1, 2, 4, 8 or 16 query heads.  ``sink``:
    whether a valueless key of score 0 takes part, or its score per head, fp32 ``(Hq,)``; ``gate (T, >= Hq)``: logits whose
    sigmoid multiplies a head's output.  ``softcap``, ``blocks``: see the reference op (trees must not be deeper than the window).
    ``diff = (lam, share, eps)``: ``q (T, Hq, 128)`` and the
    pools' keys hold 64 columns for each of two maps, ``vdim`` is the true width of the values."""
    lib = load()
    maps, (lam, share, eps) = (1, (None, 0.0, 0.0)) if diff is None else (2, diff)
    kb, vb, block_map, P = blocks if blocks is not None else (None, None, None, 0)
    T, Hq, D = q.shape
    sinks = sink if isinstance(sink, torch.Tensor) else None
    G, S, _ = k_pool.shape
    assert D == 128 and q.is_contiguous() and k_pool.shape[2] == 128 and v_pool.shape[2] == 128
    _check(lib.js_window_attention_tc(
        _p(q), _p(k_pool), _p(v_pool), _p(slot_map), _p(seq_rows), _p(cu_q), _p(past_lens), _p(mask_bits), _p(out),
        _p(ws["o"] if splits > 1 else None), _p(ws["ml"] if splits > 1 else None), _p(status_word(q.device)), seq_rows.numel(), T, Hq,
        G, S, slot_map.shape[1], mask_bits.shape[1] if mask_bits is not None else 0, int(causal), int(splits), ctypes.c_float(scale),
        int(window), int(sinks is not None or bool(sink)), int(keep_first), _sinks(sinks, Hq), *_head_gate(gate), ctypes.c_float(softcap),
        int(P), _p(kb), _p(vb), kb.shape[1] if P else 0, _p(block_map), block_map.shape[1] if P else 0, maps, _p(lam),
        ctypes.c_float(share), ctypes.c_float(eps), int(vdim), ctypes.c_longlong(S * 128), ctypes.c_longlong(128), out.stride(0), int(pdl), _stream()), "js_window_attention_tc")
    return out


def delta_buffers(T: int, cfg, device) -> dict:
    """Prepared inputs of a delta rule for ``T`` rows and its read-outs, all fp32."""
    f = lambda *n: torch.empty(T, *n, dtype=torch.float32, device=device)
    return {"q": f(cfg.kv_heads * cfg.dim), "k": f(cfg.kv_heads * cfg.dim), "v": f(cfg.heads * cfg.vdim), "gl": f(cfg.decays),
            "beta": f(cfg.heads), "o": f(cfg.heads, cfg.vdim)}


def _check_delta_pool(cfg, pre, z, b, conv, state=None) -> None:
    """Shapes the kernels index by: the state pool's slots and the width of the rows."""
    assert pre.shape[1] == cfg.channels and z.shape[1] >= cfg.decays and b.shape[1] >= cfg.heads and z.shape[0] == b.shape[0] == pre.shape[0]
    assert conv.is_contiguous() and conv.shape[1:] == (cfg.taps, cfg.channels), conv.shape
    if state is not None:
        assert state.is_contiguous() and state.shape == (conv.shape[0], cfg.heads, cfg.dim, cfg.vdim), state.shape


def delta_prep(buf: dict, cfg, pre, z, b, taps, A_log, dt_bias, conv, rows, cu_q, past_lens, mask_bits, pdl: bool = False) -> None:
    """Short convolutions, unit norms, decays and step sizes of every row into ``buf``."""
    lib = load()
    T = pre.shape[0]
    assert pre.stride(1) == 1 and z.stride(1) == 1 and b.stride(1) == 1 and z.dtype == b.dtype == torch.float32
    assert taps.dtype == pre.dtype == A_log.dtype == dt_bias.dtype == conv.dtype and taps.is_contiguous()
    _check_delta_pool(cfg, pre, z, b, conv)
    _check(lib.js_delta_prep(
        cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim, cfg.taps, int(cfg.decay == "channel"), _p(pre), pre.stride(0), _p(z), z.stride(0),
        _p(b), b.stride(0), _p(taps), _p(A_log), _p(dt_bias), _p(conv), _p(rows), _p(cu_q), _p(past_lens), _p(mask_bits),
        mask_bits.shape[1] if mask_bits is not None else 0, rows.numel(), T, _p(buf["q"]), _p(buf["k"]), _p(buf["v"]), _p(buf["gl"]),
        _p(buf["beta"]), _is_bf16(pre), int(pdl), _stream()), "js_delta_prep")


def delta_seq(buf: dict, cfg, state, conv, pre, rows, cu_q, past_lens, mask_bits=None, path=None, path_len=None, pdl: bool = False) -> None:
    """The recurrence over prepared rows: causal (states advance), over token trees (``mask_bits``: nothing is stored), or
    along the rows ``path[:path_len]`` of one sequence (states advance, nothing is read out)."""
    lib = load()
    assert conv.shape[1:] == (cfg.taps, cfg.channels) and state.shape == (conv.shape[0], cfg.heads, cfg.dim, cfg.vdim)
    assert conv.is_contiguous() and state.is_contiguous() and state.dtype == torch.float32 and conv.dtype == pre.dtype
    mode = 1 if mask_bits is not None else 2 if path is not None else 0
    B = rows.numel()
    W = mask_bits.shape[1] if mask_bits is not None else 0
    # paths of a tree are walked by several CTAs: enough of them to fill the device, at most one per 4 nodes
    groups = max(1, min(32 * W // 4, 4 * SM_COUNT // max(1, B * cfg.heads * ((cfg.vdim + 31) // 32)))) if W else 1
    _check(lib.js_delta_seq(
        mode, cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim, cfg.taps, int(cfg.decay == "channel"), _p(buf["q"]), _p(buf["k"]), _p(buf["v"]),
        _p(buf["gl"]), _p(buf["beta"]), _p(state), _p(rows), _p(cu_q), _p(past_lens), B, _p(mask_bits), W, groups, _p(path), _p(path_len),
        _p(buf["o"] if mode != 2 else None), _p(pre), pre.stride(0), _p(conv), _is_bf16(pre), int(pdl), _stream()), "js_delta_seq")


def delta_mix(pre, z, b, taps, A_log, dt_bias, cfg, state, conv, rows, cu_q, past_lens, mask_bits, causal: bool) -> torch.Tensor:
    """Unfused form of a delta rule; see the reference op for the contract."""
    if not causal and mask_bits.shape[1] > 8:
        from . import reference as ref
        return ref.delta_mix(pre, z, b, taps, A_log, dt_bias, cfg, state, conv, rows, cu_q, past_lens, mask_bits, causal)
    buf = delta_buffers(pre.shape[0], cfg, pre.device)
    mask = None if causal else mask_bits
    delta_prep(buf, cfg, pre, z, b, taps, A_log, dt_bias, conv, rows, cu_q, past_lens, mask)
    delta_seq(buf, cfg, state, conv, pre, rows, cu_q, past_lens, mask)
    return buf["o"]


def delta_step_ok(cfg) -> bool:
    """Whether the one-kernel decode step takes this shape (a head's state fits one CTA's registers)."""
    groups = 1
    while 4 * groups < cfg.vdim:
        groups *= 2
    return cfg.vdim % 4 == 0 and cfg.vdim <= 256 and cfg.dim <= 256 and cfg.dim * groups <= 4096


def delta_blocks_ok(cfg) -> bool:
    return cfg.vdim % 4 == 0 and cfg.dim <= 128


def delta_block_buffers(T: int, B: int, cfg, device) -> dict:
    """Rows of the block form for ``T`` rows of ``B`` sequences, all fp32."""
    R, DP, H = 8 * (T // 8 + B), 64 if cfg.dim <= 64 else 128, cfg.heads
    f = lambda *n: torch.empty(H, *n, dtype=torch.float32, device=device)
    return {"kt": f(R, DP), "qt": f(R, DP), "kh": f(R, DP), "bv": f(R, cfg.vdim), "pt": f(R, 8), "ge": f(R // 8, DP),
            "o": torch.empty(T, H, cfg.vdim, dtype=torch.float32, device=device)}


def delta_forward(cfg, pre, z, b, taps, A_log, dt_bias, state, conv, rows, cu_q, past_lens, gate, o_norm, kind: str, eps: float, out,
                  max_rows: int, buffers=None, pdl: bool = False) -> int:
    """Everything between a delta layer's projections, bf16, causal: one kernel for decode steps (one row a sequence), blocks
    of 8 rows for portions, the row-by-row kernels for shapes neither takes.  ``buffers(kind)`` hands out the workspace of
    ``"blocks"`` or ``"rows"``.  Returns the number of kernels launched."""
    lib = load()
    T, B = pre.shape[0], rows.numel()
    get = buffers or (lambda k: delta_block_buffers(T, B, cfg, pre.device) if k == "blocks" else delta_buffers(T, cfg, pre.device))
    assert pre.dtype == torch.bfloat16 and pre.stride(1) == 1 and z.stride(1) == 1 and b.stride(1) == 1 and gate.stride(1) == 1
    assert conv.dtype == torch.bfloat16 and state.dtype == torch.float32
    _check_delta_pool(cfg, pre, z, b, conv, state)
    head = (cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim, cfg.taps, int(cfg.decay == "channel"), _p(pre), pre.stride(0), _p(z), z.stride(0),
            _p(b), b.stride(0), _p(taps), _p(A_log), _p(dt_bias), _p(conv), _p(state), _p(rows), _p(cu_q), _p(past_lens), B)
    if max_rows == 1 and T == B and delta_step_ok(cfg):
        _check(lib.js_delta_step(*head, _p(gate), gate.stride(0), _p(o_norm), int(kind == "silu"), ctypes.c_float(eps), _p(out),
                                 out.stride(0), int(pdl), _stream()), "js_delta_step")
        return 1
    if delta_blocks_ok(cfg):
        w = get("blocks")
        # 32 value columns a CTA share the loads, 16 fill the device: a lone sequence of few heads wants the latter
        wide = B * cfg.heads * ((cfg.vdim + 31) // 32) >= SM_COUNT * 3 // 4
        _check(lib.js_delta_blocks(*head, T, *(_p(w[n]) for n in ("kt", "qt", "kh", "bv", "pt", "ge", "o")), int(wide), int(pdl), _stream()),
               "js_delta_blocks")
    else:
        w = get("rows")
        delta_prep(w, cfg, pre, z, b, taps, A_log, dt_bias, conv, rows, cu_q, past_lens, None, pdl=pdl)
        delta_seq(w, cfg, state, conv, pre, rows, cu_q, past_lens, None, pdl=pdl)
    gated_head_norm(w["o"], o_norm, gate, kind, eps, out=out, pdl=pdl)
    return 3


def gated_head_norm(o: torch.Tensor, w: torch.Tensor, gate: torch.Tensor, kind: str, eps: float, out: Optional[torch.Tensor] = None,
                    vp: Optional[int] = None, pdl: bool = False) -> torch.Tensor:
    """``o (T, H, V)`` fp32 -> ``out (T, H * vp)`` in the gate's dtype; columns of a head past ``V`` are zero."""
    lib = load()
    T, H, V = o.shape
    vp = vp or V
    if out is None:
        out = torch.empty(T, H * vp, dtype=gate.dtype, device=gate.device)
    assert (w is None or w.dtype == gate.dtype) and gate.dtype == out.dtype and gate.stride(1) == 1
    _check(lib.js_gated_head_norm(_p(o), _p(w), _p(gate), gate.stride(0), _p(out), out.stride(0), T, H, V, vp, int(kind == "silu"),
                                  ctypes.c_float(eps), _is_bf16(gate), int(pdl), _stream()), "js_gated_head_norm")
    return out


# ------------------------------------------------------------------ pre-norm steps, general rotations, retention
_rot_freq: dict = {}


def rot_freq(rot, device) -> torch.Tensor:
    """fp32 frequencies of a ``RotaryConfig`` on the device."""
    key = (rot, str(device))
    if key not in _rot_freq:
        _rot_freq[key] = torch.tensor(rot.frequencies(), dtype=torch.float32, device=device)
    return _rot_freq[key]


def gelu_erf(x: torch.Tensor) -> torch.Tensor:
    lib = load()
    x = x.contiguous()
    out = torch.empty_like(x)
    _check(lib.js_gelu_erf(_p(x), _p(out), ctypes.c_longlong(x.numel()), _is_bf16(x), _stream()), "js_gelu_erf")
    return out


def rotate(x: torch.Tensor, positions: torch.Tensor, rot, out_dtype) -> torch.Tensor:
    lib = load()
    T, heads, D = x.shape
    x = x.contiguous()
    out = torch.empty(T, heads, D, dtype=out_dtype, device=x.device)
    pos, freq = positions.to(torch.int32), rot_freq(rot, x.device)      # named: they outlive the launch
    _check(lib.js_rotate(_p(x), _is_bf16(x), _p(out), _is_bf16(out), _p(pos), T, heads, D, rot.dims, int(rot.pairing == "next"), _p(freq),
                         ctypes.c_float(rot.amplitude()), _stream()), "js_rotate")
    return out


def head_gate(y: torch.Tensor, logits: torch.Tensor) -> torch.Tensor:
    lib = load()
    T, H = logits.shape
    y, logits = y.contiguous(), logits.float()
    assert logits.stride(1) == 1 and y.shape[0] == T and y.shape[1] % H == 0
    out = torch.empty_like(y)
    _check(lib.js_head_gate(_p(y), _p(logits), logits.stride(0), _p(out), T, H, y.shape[1] // H, _is_bf16(y), _stream()), "js_head_gate")
    return out


_decays: dict = {}


def retention_decays(cfg, device) -> torch.Tensor:
    """The heads' decays, fp32 on the device."""
    key = (tuple(cfg.decay), str(device))
    if key not in _decays:
        _decays[key] = torch.tensor(cfg.decay, dtype=torch.float32, device=device)
    return _decays[key]


def retention_seq(q, k, v, cfg, state, rows, cu_q, past_lens, mask_bits=None, path=None, path_len=None, out=None, pdl: bool = False):
    """Retention row by row over fp32 rows ``q, k (T, H*D)``, ``v (T, H*V)``: causal (states advance), over token trees
    (``mask_bits``: nothing is stored), or along the rows ``path[:path_len]`` of one sequence (nothing is read out)."""
    lib = load()
    assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (k, v, state))
    assert k.shape[1] == cfg.heads * cfg.dim and v.shape[1] == cfg.heads * cfg.vdim and state.shape[1:] == (cfg.heads, cfg.dim, cfg.vdim)
    mode = 1 if mask_bits is not None else 2 if path is not None else 0
    assert mode == 2 or (q.dtype == torch.float32 and q.is_contiguous() and q.shape == k.shape)
    B, W = rows.numel(), mask_bits.shape[1] if mask_bits is not None else 0
    groups = max(1, min(32 * W // 4, 4 * SM_COUNT // max(1, B * cfg.heads * ((cfg.vdim + 31) // 32)))) if W else 1
    if out is None and mode != 2:
        out = torch.empty(k.shape[0], cfg.heads, cfg.vdim, dtype=torch.float32, device=k.device)
    _check(lib.js_retention_seq(mode, cfg.heads, cfg.dim, cfg.vdim, _p(q), _p(k), _p(v), _p(retention_decays(cfg, k.device)), _p(state), _p(rows),
                                _p(cu_q), _p(past_lens), B, _p(mask_bits), W, groups, _p(path), _p(path_len), _p(out), int(pdl), _stream()),
           "js_retention_seq")
    return out


def retention(q, k, v, cfg, state, rows, cu_q, past_lens, mask_bits, causal: bool) -> torch.Tensor:
    """Unfused form; see the reference op for the contract."""
    q, k, v = (x.float().contiguous() for x in (q, k, v))
    return retention_seq(q, k, v, cfg, state, rows, cu_q, past_lens, None if causal else mask_bits)


RETENTION_CHUNK = 128


def retention_powers(cfg, device) -> torch.Tensor:
    """Powers 0 .. 256 of the heads' decays ``(H, 257)``, evaluated in double and rounded to fp32 once."""
    key = ("powers", tuple(cfg.decay), str(device))
    if key not in _decays:
        _decays[key] = torch.tensor([[d ** j for j in range(257)] for d in cfg.decay], dtype=torch.float64).float().to(device)
    return _decays[key]


def retention_fused_ok(cfg) -> bool:
    """Whether the chunk and tree kernels take this shape (the step kernel and the row walk take dims up to 256)."""
    return cfg.dim <= 128 and cfg.vdim <= 256


def _retention_args(cfg, act, cols, rot, powers, state=None) -> tuple:
    """The arguments all retention kernels start with.  ``cols``: where k, v and the gate start in ``act``; ``rot``: the layer's
    columns ``(T, >= dims / 2, 2)`` of the rotary table."""
    assert act.dtype == torch.bfloat16 and act.stride(1) == 1 and rot.dtype == torch.float32 and rot.stride(2) == 1 and rot.stride(1) == 2
    assert act.shape[1] >= cols[2] + cfg.heads * cfg.vdim and rot.shape[0] >= act.shape[0] and rot.shape[1] >= cfg.rot.dims // 2
    assert state is None or (state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (cfg.heads, cfg.dim, cfg.vdim))
    return (cfg.heads, cfg.dim, cfg.vdim, cfg.rot.dims, _p(act), act.stride(0), *cols, _p(rot), rot.stride(0) // 2, _p(powers))


def retention_rows_buffers(T: int, cfg, device) -> dict:
    """Rotated fp32 rows and read-outs of the row-by-row walk."""
    f = lambda n: torch.empty(T, cfg.heads * n, dtype=torch.float32, device=device)
    return {"q": f(cfg.dim), "k": f(cfg.dim), "v": f(cfg.vdim), "o": torch.empty(T, cfg.heads, cfg.vdim, dtype=torch.float32, device=device)}


def retention_chunk_buffer(T: int, B: int, cfg, device) -> torch.Tensor:
    """States before every chunk of a portion's rows."""
    return torch.empty(T // RETENTION_CHUNK + B, cfg.heads, cfg.dim, cfg.vdim, dtype=torch.float32, device=device)


def retention_forward(cfg, act, cols, rot, state, rows, cu_q, past_lens, mask_bits, eps: float, out, max_rows: int, buffers=None,
                      pdl: bool = False) -> int:
    """Everything between a retention layer's projections ``act`` (bf16, q | k | v | gate) and its output product: rotations,
    the recurrence, per-head norm and silu gate to ``out``.  One kernel for decode steps (one row a sequence) and for token
    trees (``mask_bits``; nothing is stored), three for portions; row by row for shapes these do not take.
    ``buffers(kind)`` hands out the workspace of ``"chunks"`` or ``"rows"``.  Returns the number of kernels launched."""
    lib = load()
    T, B = act.shape[0], rows.numel()
    get = buffers or (lambda k: (retention_chunk_buffer if k == "chunks" else lambda t, b, c, d: retention_rows_buffers(t, c, d))(T, B, cfg, act.device))
    assert out.dtype == torch.bfloat16 and out.stride(1) == 1 and out.shape[1] >= cfg.heads * cfg.vdim
    args = _retention_args(cfg, act, cols, rot, retention_powers(cfg, act.device), state)
    seqs = (_p(rows), _p(cu_q), _p(past_lens), B)
    if mask_bits is None and max_rows == 1 and T == B and cfg.vdim <= 1024:
        cl = 1               # CTAs a head's value columns are dealt to: enough to fill the device, at least 32 columns each
        while cl < 8 and (cfg.vdim > 256 * cl or (cfg.vdim >= 64 * cl and B * cfg.heads * cl < 2 * SM_COUNT)):
            cl *= 2
        _check(lib.js_retention_step(*args, *seqs, _p(state), ctypes.c_float(eps), _p(out), out.stride(0), cl, int(pdl), _stream()),
               "js_retention_step")
        return 1
    if retention_fused_ok(cfg) and mask_bits is None:
        U = get("chunks")
        assert U.shape[0] >= T // RETENTION_CHUNK + B
        _check(lib.js_retention_chunks(*args, *seqs, T, _p(state), _p(U), ctypes.c_float(eps), _p(out), out.stride(0), int(pdl), _stream()),
               "js_retention_chunks")
        return 3
    if retention_fused_ok(cfg) and mask_bits.shape[1] <= 8:
        _check(lib.js_retention_tree(*args, *seqs, T, _p(state), _p(mask_bits), mask_bits.shape[1], ctypes.c_float(eps), _p(out), out.stride(0),
                                     int(pdl), _stream()), "js_retention_tree")
        return 1
    w = get("rows")
    _check(lib.js_retention_prep(*args[:-1], T, _p(w["q"]), _p(w["k"]), _p(w["v"]), int(pdl), _stream()), "js_retention_prep")
    retention_seq(w["q"], w["k"], w["v"], cfg, state, rows, cu_q, past_lens, mask_bits, out=w["o"], pdl=pdl)
    gated_head_norm(w["o"], None, act[:, cols[2]:cols[2] + cfg.heads * cfg.vdim], "silu", eps, out=out, pdl=pdl)
    return 3


def retention_path(cfg, act, cols, rot, state, rows, cu_q, past_lens, path, path_len, pdl: bool = False) -> None:
    """Advance one sequence's state along the rows ``path[:path_len]`` of a tree forward; ``past_lens`` is the committed length
    behind the path."""
    _check(load().js_retention_path(*_retention_args(cfg, act, cols, rot, retention_powers(cfg, act.device), state), _p(rows), _p(cu_q),
                                    _p(past_lens), _p(state), _p(path), _p(path_len), int(pdl), _stream()), "js_retention_path")


# ------------------------------------------------------------------ MoE (grouped through the dense GEMM)
_moe_cache: dict = {}


def moe_forward(x, gate_w, w_gate_up, w_down, top_k: int, renorm: bool, router_logits=None, residual=None):
    """Sparse MoE on one GPU: route, sort the (token, choice) pairs by expert, run all experts'
    SwiGLU MLPs with two grouped tcgen05 GEMMs (one launch each), combine with the routing weights.
    With ``residual`` (T, H) the combine kernel adds the layer output onto it in place and returns it."""
    from . import reference as ref
    from ..parallel.ep import interleave_experts, route_and_sort
    lib = load()
    T, H = x.shape
    E, I2, _ = w_gate_up.shape
    I = I2 // 2
    if I % 64 or H % 128:
        y = ref.moe_forward(x, gate_w, w_gate_up, w_down, top_k, renorm, router_logits)
        return y if residual is None else residual.add_(y)
    key = (w_gate_up.data_ptr(), w_down.data_ptr())
    if key not in _moe_cache:
        _moe_cache[key] = (interleave_experts(w_gate_up), w_down.reshape(E * H, I).contiguous())
    gu, dn = _moe_cache[key]
    if router_logits is None:
        router_logits = gemm(x, gate_w, epi=EPI_STORE_F32) if gemm_supported(T, E, H) else torch.nn.functional.linear(x, gate_w)
    on_device = E <= 256 and T * top_k <= 16384
    if on_device:    # router + permutation kernels: int32 order, no host synchronisation, static shapes
        order, row_w, group_off, _, tok = moe_route_sort(router_logits.float(), top_k, renorm, 0, E, with_tokens=True)
    else:
        order, row_w, group_off, _ = route_and_sort(router_logits, top_k, renorm, 0, E)
        tok = torch.div(order, top_k, rounding_mode="floor")
    if on_device and x.dtype == torch.bfloat16 and x.stride(1) == 1:
        xs = torch.empty(T * top_k, H, dtype=x.dtype, device=x.device)
        gather_rows(x, tok, xs)                   # expert-sorted copy of the token rows
    else:
        xs = x.index_select(0, tok)
    h = torch.empty(T * top_k, I, dtype=x.dtype, device=x.device)
    ys = torch.empty(T * top_k, H, dtype=x.dtype, device=x.device)
    st = _p(status_word(x.device))
    # launch for a few times the balanced rows per expert (an expert can hold at most T rows); hotter experts are
    # finished by their CTAs walking on through the remaining row tiles, empty tiles are never launched in bulk
    cover = min(T, ((4 * T * top_k // E + 128 + 127) // 128) * 128)
    _check(lib.js_gemm_bf16_grouped(_p(xs), _p(gu), _p(h), T * top_k, 2 * I, H, xs.stride(0), gu.stride(0), h.stride(0),
                                    EPI_SWIGLU, E, _p(group_off), cover, None, None, None, None, 1, st, 0, _stream()),
           "grouped gate/up")
    _check(lib.js_gemm_bf16_grouped(_p(h), _p(dn), _p(ys), T * top_k, H, I, h.stride(0), dn.stride(0), ys.stride(0),
                                    EPI_STORE, E, _p(group_off), cover, None, None, None, None, 1, st, 0, _stream()),
           "grouped down")
    if on_device and x.dtype == torch.bfloat16:
        # weighted sum of each token's expert outputs in choice order (fixed order, no atomics)
        fused = residual is not None and residual.dtype == x.dtype and residual.stride(1) == 1
        out = residual if fused else torch.empty(T, H, dtype=x.dtype, device=x.device)
        inv = torch.empty(T * top_k, dtype=torch.int32, device=x.device)
        lib.js_moe_combine.restype = ctypes.c_int
        _check(lib.js_moe_combine(_p(ys), ys.stride(0), _p(order), _p(row_w), T, top_k, H, _p(inv),
                                  _p(residual) if fused else None, _p(out), out.stride(0), 0, _stream()),
               "js_moe_combine")
        return out if fused or residual is None else residual.add_(out)
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    out.index_add_(0, tok.long(), ys.float() * row_w[:, None])
    out = out.to(x.dtype)
    return out if residual is None else residual.add_(out)
