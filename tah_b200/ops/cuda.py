"""ctypes bindings for the hand-written sm_100a kernels in ``csrc/`` (``libtahb200.so``).

Every wrapper takes torch CUDA tensors, launches on the current torch stream and
returns torch tensors.  The library is built in-tree by :mod:`tah_b200.ops.build`; if it
is missing on a machine with a CUDA device, loading raises (no silent fallback).

Kernels that wait on hardware barriers give up after a bounded time and set a status
word; :func:`check_status` reads it (a host sync) and raises :class:`KernelTimeout`.
"""
from __future__ import annotations

import ctypes
import os
from typing import List, Optional, Sequence

import torch

_LIB = None
# TAH_B200_LIB: load another build of the library (A/B timing of kernel changes)
_LIB_PATH = os.environ.get("TAH_B200_LIB") or os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))),
                                                           "lib", "libtahb200.so")

c_void_p, c_int, c_ll, c_float = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float


class KernelTimeout(RuntimeError):
    pass


STATUS_NAMES = {1: "timeout waiting for a TMA load", 2: "timeout waiting for a free pipeline stage",
                3: "timeout waiting for the accumulator", 4: "timeout waiting for a peer flag",
                5: "index out of range / KV pages exhausted"}


def lib():
    global _LIB
    if _LIB is None:
        if not os.path.exists(_LIB_PATH):
            from tah_b200.ops.build import build
            build()
        _LIB = ctypes.CDLL(_LIB_PATH)
        if hasattr(_LIB, "tahb_decode_attn_ws_floats"):      # absent from the group builds
            _LIB.tahb_decode_attn_ws_floats.restype = c_ll
    return _LIB


def use_group_build(group: str) -> None:
    """Load the library of a source group (:data:`tah_b200.ops.build.GROUPS`), compiling only its sources when the full
    library is not there (a process that replays a trace of one model; nothing may have been loaded yet)."""
    global _LIB_PATH
    if _LIB is None and not os.path.exists(_LIB_PATH):
        from tah_b200.ops.build import build
        _LIB_PATH = build(group=group)


def available() -> bool:
    return torch.cuda.is_available()


def _stream() -> c_void_p:
    return c_void_p(torch.cuda.current_stream().cuda_stream)


def _p(t: Optional[torch.Tensor]) -> c_void_p:
    return c_void_p(0 if t is None else t.data_ptr())


_status = {}


def status_word(device=None) -> torch.Tensor:
    dev = torch.device(device if device is not None else torch.cuda.current_device())
    if dev.type != "cuda":
        dev = torch.device("cuda", torch.cuda.current_device())
    key = dev.index if dev.index is not None else torch.cuda.current_device()
    if key not in _status:
        _status[key] = torch.zeros(1, dtype=torch.int32, device=torch.device("cuda", key))
    return _status[key]


def check_status(device=None) -> None:
    """Read the status word (synchronises) and raise if a kernel reported a failure."""
    w = status_word(device)
    code = int(w.item())
    if code != 0:
        w.zero_()
        raise KernelTimeout(f"tah_b200 kernel status {code}: {STATUS_NAMES.get(code, 'unknown')}")


launch_count = 0      # number of library entry points called (each launches at least one kernel)


def _rc(rc: int, what: str) -> None:
    global launch_count
    launch_count += 1
    if rc != 0:
        raise RuntimeError(f"{what} failed on the host side (code {rc})")


def _check_bf16_2d(t: torch.Tensor, name: str):
    if t.dtype != torch.bfloat16 or t.dim() != 2 or t.stride(1) != 1 or not t.is_cuda:
        raise ValueError(f"{name}: need a 2-D bf16 CUDA tensor with unit inner stride, got {t.dtype} {tuple(t.shape)} {t.stride()}")


# -------------------------------------------------------------------------------------------
# GEMM
# -------------------------------------------------------------------------------------------
SM_COUNT = 148


def _fits(bn: int, s: int, nacc: int) -> bool:
    stage = 16384 * nacc + bn * 128
    ns = min(8, (196 * 1024) // stage)
    if s == 1:
        return True
    per = bn // s
    if bn % s or per % 16:
        return False
    red = ((s - 1) * 128 * nacc * per * 4 + 1023) // 1024 * 1024
    return red + per * 256 <= ns * stage


def plan_gemm(M: int, F: int, K: int, R: int = 0, dual: bool = False):
    """Pick the token-tile width and the split-K cluster size with a small cost model.

    Measured on B200: a k-block (64 of K) costs about 0.3 us of load latency per CTA unless the
    tensor-core time of the tile is larger, the epilogue about 0.5 us + 8 ns per token column,
    and clusters larger than 4 CTAs (one ~200 KB CTA per SM) no longer fit in one wave.
    """
    nacc = 2 if dual else 1
    kb = K // 64 + R // 64
    base = 16 if M <= 16 else 32 if M <= 32 else 64 if M <= 64 else 128 if M <= 128 else 256
    cands = [base] + ([128, 64] if base == 256 else [64] if base == 128 else [])
    best = None
    for bn in cands:
        for s in (1, 2, 4):
            if s > 1 and (kb // s < 2 or not _fits(bn, s, nacc)):
                continue
            ctas = ((F + 127) // 128) * ((M + bn - 1) // bn) * s
            waves = (ctas + SM_COUNT - 1) // SM_COUNT
            t_kb = max(0.30, 128 * bn * 64 * 2 * nacc / 8192 / 1900.0)
            per = bn // s
            t_cta = (kb / s) * t_kb + 0.5 + 0.009 * per
            if s > 1:
                pushed_kb = (s - 1) * per * nacc * 0.5            # KiB sent to the peers through DSMEM
                t_cta += 1.0 + pushed_kb / 19.0 + (0.07 * per if dual else 0.0)
            t = waves * t_cta
            if best is None or t < best[0] - 1e-9:
                best = (t, bn, s)
    return best[1], best[2]


# token count from which the two-tile ("pair") GEMM is the default; TAH_B200_GEMM_PAIR=0 turns it off
PAIR_AUTO = os.environ.get("TAH_B200_GEMM_PAIR", "1") != "0"
PAIR_MIN_TOKENS = 1024


def interleave_gate_up(w: torch.Tensor) -> torch.Tensor:
    """``[2I, K]`` gate rows then up rows -> ``[2I, K]`` with rows ``gate_0, up_0, gate_1, up_1, ...`` (the layout
    :func:`gemm` wants for ``swiglu_interleaved``; apply it to the LoRA-B extension of the projection as well)."""
    half = w.shape[0] // 2
    return torch.stack((w[:half], w[half:]), dim=1).reshape(w.shape).contiguous()


def pick_splits(M: int, F: int, K: int, R: int = 0, dual: bool = False) -> int:
    return plan_gemm(M, F, K, R, dual)[1]


_pending_gemm_wait = None


def set_pending_gemm_wait(desc) -> None:
    """The next :func:`gemm` / :func:`gemm_qkv` call without a ``tp_wait`` of its own takes ``desc = (flags,
    targets)``: its TMA producer waits for those landing flags before the first load.  Used by parameter-sharded
    training, where the first GEMM of a layer consumes the all-gather of the layer's weights."""
    global _pending_gemm_wait
    _pending_gemm_wait = desc


def clear_pending_gemm_wait() -> bool:
    """Drop a pending wait; returns True if one was still pending (nobody consumed it)."""
    global _pending_gemm_wait
    had = _pending_gemm_wait is not None
    _pending_gemm_wait = None
    return had


def _take_pending_wait(tp_wait):
    global _pending_gemm_wait
    if tp_wait is None and _pending_gemm_wait is not None:
        tp_wait, _pending_gemm_wait = _pending_gemm_wait, None
    return tp_wait


def wait_flags(flags: torch.Tensor, targets: torch.Tensor) -> None:
    """Stream-ordered bounded wait (one tiny kernel) until ``flags[q] >= targets[q]`` for every q: gates kernels
    that cannot wait themselves, e.g. library GEMMs reading a gather buffer that peers fill."""
    _rc(lib().tahb_wait_flags(_p(flags), _p(targets), c_int(flags.numel()), _p(status_word(flags.device)), _stream()),
        "tahb_wait_flags")


def gemm(x: torch.Tensor, w: torch.Tensor, *, out: Optional[torch.Tensor] = None,
         residual: Optional[torch.Tensor] = None, x2: Optional[torch.Tensor] = None,
         w2: Optional[torch.Tensor] = None, swiglu: bool = False, splits: Optional[int] = None,
         bn: int = 0, tp_push=None, tp_wait=None, gelu: bool = False, swiglu_interleaved: bool = False,
         pair: Optional[bool] = None) -> torch.Tensor:
    """``out[M,F] = x[M,K] @ w[F,K]^T (+ x2[M,R] @ w2[F,R]^T) (+ residual)``; with ``swiglu`` the
    weight is ``[2F, K]`` (gate rows then up rows) and ``out = silu(gate) * up``.

    ``gelu``: the epilogue applies the erf GELU to the bf16-rounded output (not together with ``residual``).

    ``pair``: every CTA computes two 128-feature output tiles (features ``f`` and ``F/2 + f``) from one 256-token
    activation tile, unsplit.  It halves the activation bytes a CTA pulls per unit of work, which is what bounds
    the kernel at large token counts (1350-1400 vs 915-1100 TFLOP/s at 8192+ tokens); default: on from
    ``PAIR_MIN_TOKENS`` tokens when the shape allows it (also with ``swiglu_interleaved``).

    ``swiglu_interleaved``: the rows of ``w`` (and ``w2``) alternate ``gate_i, up_i`` (see :func:`interleave_gate_up`)
    and ``out[M, F/2] = silu(gate) * up``: one accumulator and one wide MMA per k step, the faster SwiGLU form.

    Tensor parallel (see :class:`tah_b200.parallel.tp.TensorParallel`): ``tp_push =
    (slot_ptrs, cnt_ptrs, rank, rows_per_rank)`` replaces the output by peer stores of the tile
    rows into their owners' slot buffers (reduce-scatter by push, ``out`` is not written);
    ``tp_wait = (flags, targets)`` makes the kernel wait for the broadcast rows of ``x``."""
    _check_bf16_2d(x, "x")
    _check_bf16_2d(w, "w")
    tp_wait = _take_pending_wait(tp_wait)
    M, K = x.shape
    F = w.shape[0] // 2 if swiglu else w.shape[0]
    F_out = F // 2 if swiglu_interleaved else F
    if swiglu_interleaved and (swiglu or gelu or residual is not None or tp_push is not None or F % 2):
        raise ValueError("swiglu_interleaved excludes swiglu / gelu / residual / tp_push")
    if w.shape[1] != K:
        raise ValueError(f"K mismatch: x {tuple(x.shape)} w {tuple(w.shape)}")
    R = 0
    if x2 is not None:
        _check_bf16_2d(x2, "x2")
        _check_bf16_2d(w2, "w2")
        R = x2.shape[1]
        if w2.shape[1] != R or w2.shape[0] != w.shape[0] or x2.shape[0] != M:
            raise ValueError("K-extension operands do not match")
    if tp_push is not None:
        out = x.new_empty(0, F) if out is None else out
    elif out is None:
        out = torch.empty(M, F_out, dtype=torch.bfloat16, device=x.device)
    else:
        _check_bf16_2d(out, "out")
    if residual is not None:
        _check_bf16_2d(residual, "residual")
    if pair is None:
        pair = (PAIR_AUTO and M >= PAIR_MIN_TOKENS and bn == 0 and splits is None and not swiglu and not gelu
                and w.shape[0] % 256 == 0)
    pair = bool(pair) and not swiglu and not gelu and w.shape[0] % 256 == 0
    if pair:
        bn, splits = 256, 1
    elif swiglu_interleaved:
        splits = 1                       # the interleaved epilogue exists for unsplit tiles
        if bn == 0:
            bn = 16 if M <= 16 else 32 if M <= 32 else 64 if M <= 64 else 128 if M <= 128 else 256
    elif splits is None and bn == 0:
        bn, splits = plan_gemm(M, F, K, R, swiglu)
    elif splits is None:
        splits = 1
    args = (_p(w), _p(x), _p(out), _p(residual), _p(w2), _p(x2), c_int(M), c_int(F), c_int(K), c_int(R),
            c_ll(w.stride(0)), c_ll(x.stride(0)), c_ll(out.stride(0)),
            c_ll(residual.stride(0) if residual is not None else 0),
            c_ll(w2.stride(0) if w2 is not None else 0), c_ll(x2.stride(0) if x2 is not None else 0),
            c_int(1 if swiglu else 3 if gelu else (6 if pair else 4) if swiglu_interleaved else 2 if pair else 0), c_int(F if swiglu else 0), c_int(splits), c_int(bn),
            _p(status_word(x.device)), _stream())
    if tp_push is None and tp_wait is None:
        rc = lib().tahb_gemm(*args)
    else:
        if tp_push is not None:
            slot_ptrs, cnt_ptrs, rank, rpr = tp_push
            n = len(slot_ptrs)
            push = ((c_void_p * n)(*slot_ptrs), (c_void_p * n)(*cnt_ptrs), c_int(n), c_int(rank), c_int(rpr))
        else:
            push = (None, None, c_int(0), c_int(0), c_int(0))
        if tp_wait is not None:
            flags, targets = tp_wait
            wait = (_p(flags), _p(targets), c_int(flags.numel()))
        else:
            wait = (None, None, c_int(0))
        rc = lib().tahb_gemm_tp(*args, *push, *wait)
    _rc(rc, "tahb_gemm")
    return out


def gemm_t(x: torch.Tensor, w: torch.Tensor, *, x_t: bool = False, w_t: bool = False, out: Optional[torch.Tensor] = None,
           residual: Optional[torch.Tensor] = None, splits: Optional[int] = None, bn: int = 0,
           pair: Optional[bool] = None) -> torch.Tensor:
    """GEMM with operands read transposed straight from their row-major storage (the backward GEMMs):

    * ``w_t``: ``w`` is ``[K, F]`` (instead of ``[F, K]``); * ``x_t``: ``x`` is ``[K, M]`` (instead of ``[M, K]``);

    ``out[M, F] = op(x) @ op(w)^T (+ residual)``.  Data gradient of ``y = x W^T``: ``gemm_t(dy, W, w_t=True)``; weight
    gradient: ``gemm_t(dy, x, x_t=True, w_t=True, residual=grad, out=grad)`` (reduction over the tokens, any count).
    Same tcgen05 kernel as :func:`gemm`; the transposed tiles are described to the tensor core as MN-major."""
    _check_bf16_2d(x, "x")
    _check_bf16_2d(w, "w")
    if x_t:
        Kx, M = x.shape
    else:
        M, Kx = x.shape
    if w_t:
        Kw, F = w.shape
    else:
        F, Kw = w.shape
    if Kx != Kw:
        raise ValueError(f"reduction mismatch: x {tuple(x.shape)} (x_t={x_t}) w {tuple(w.shape)} (w_t={w_t})")
    if not (x_t or w_t):
        return gemm(x, w, out=out, residual=residual, splits=splits, bn=bn, pair=pair)
    if out is None:
        out = torch.empty(M, F, dtype=torch.bfloat16, device=x.device)
    if residual is not None:
        _check_bf16_2d(residual, "residual")
    if pair is None:
        pair = PAIR_AUTO and M >= PAIR_MIN_TOKENS and bn == 0 and splits is None
    pair = bool(pair) and F % 256 == 0 and (not x_t or M % 64 == 0)
    if pair:
        bn, splits = 256, 1
    elif splits is None and bn == 0:
        bn, splits = plan_gemm(M, F, (Kx + 63) // 64 * 64, 0, False)
        if x_t:
            bn = max(bn, 64)
    elif splits is None:
        splits = 1
    _rc(lib().tahb_gemm_t(_p(w), _p(x), _p(out), _p(residual), c_int(M), c_int(F), c_int(Kx), c_ll(w.stride(0)),
                          c_ll(x.stride(0)), c_ll(out.stride(0)), c_ll(residual.stride(0) if residual is not None else 0),
                          c_int(1 if w_t else 0), c_int(1 if x_t else 0), c_int(splits), c_int(bn),
                          _p(status_word(x.device)), _stream(), c_int(1 if pair else 0)), "tahb_gemm_t")
    return out


# -------------------------------------------------------------------------------------------
# elementwise / norm / rope
# -------------------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    _check_bf16_2d(x, "x")
    if out is None:
        out = torch.empty_like(x)
    _rc(lib().tahb_rmsnorm(_p(x), _p(w), _p(out), c_int(x.shape[0]), c_int(x.shape[1]), c_ll(x.stride(0)),
                           c_ll(out.stride(0)), c_float(eps), _stream()), "tahb_rmsnorm")
    return out


def rms_norm_lora(x: torch.Tensor, w: torch.Tensor, eps: float, gate: torch.Tensor, A: torch.Tensor,
                  out: Optional[torch.Tensor] = None, t_out: Optional[torch.Tensor] = None):
    """RMSNorm of every row and, in the same launch, ``t[r] = gate[r] ? y[r] @ A^T : 0`` (the LoRA-A product of the
    rows at depth >= 1 of a decode tick).  Returns ``(y, t)``."""
    _check_bf16_2d(x, "x")
    M, H = x.shape
    R = A.shape[0]
    if out is None:
        out = torch.empty_like(x)
    if t_out is None:
        t_out = torch.empty(M, R, dtype=torch.bfloat16, device=x.device)
    if A.shape[1] != H or not A.is_contiguous():
        raise ValueError("rms_norm_lora: A must be a contiguous [R, H] matrix")
    _rc(lib().tahb_rmsnorm_lora(_p(x), _p(w), _p(out), c_int(M), c_int(H), c_ll(x.stride(0)), c_ll(out.stride(0)),
                                c_float(eps), _p(gate), _p(A), _p(t_out), c_int(R), c_ll(t_out.stride(0)), _stream()),
        "tahb_rmsnorm_lora")
    return out, t_out


def layer_norm(x, w, b, eps: float = 1e-5, out=None):
    """LayerNorm over the last dimension of bf16 ``x [M, D]`` (fp32 statistics)."""
    _check_bf16_2d(x, "x")
    M, D = x.shape
    if out is None:
        out = torch.empty(M, D, dtype=torch.bfloat16, device=x.device)
    _rc(lib().tahb_layernorm(_p(x), _p(w), _p(b), _p(out), None, None, None, c_int(M), c_int(D), c_ll(x.stride(0)),
                             c_ll(out.stride(0)), c_float(eps), _stream()), "tahb_layernorm")
    return out


def layer_norm_dot(x, w, b, dot_w, dot_b, eps: float = 1e-5, out=None):
    """``z[r] = bf16(LayerNorm(x[r]) . dot_w + dot_b)`` as fp32: LayerNorm followed by ``Linear(D, 1)``."""
    _check_bf16_2d(x, "x")
    M, D = x.shape
    if out is None:
        out = torch.empty(M, dtype=torch.float32, device=x.device)
    _rc(lib().tahb_layernorm(_p(x), _p(w), _p(b), None, _p(dot_w), _p(dot_b), _p(out), c_int(M), c_int(D),
                             c_ll(x.stride(0)), c_ll(0), c_float(eps), _stream()), "tahb_layernorm")
    return out


def rope_table(pos: torch.Tensor, hd: int, theta: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``[M, hd]`` bf16 RoPE table of a pass: ``cos`` of the ``hd/2`` frequencies at ``pos[t]``, then ``sin``."""
    M = pos.shape[0]
    if out is None:
        out = torch.empty(M, hd, dtype=torch.bfloat16, device=pos.device)
    _rc(lib().tahb_rope_table(_p(pos), _p(out), c_int(M), c_int(hd), c_float(theta), _stream()), "tahb_rope_table")
    return out


def set_peer_wait_limit_ns(ns: int) -> int:
    """How long kernels wait for a flag that a peer GPU advances before they give up (status 4); 0 = default
    (2 s).  Returns the previous limit."""
    fn = lib().tahb_set_peer_wait_limit_ns
    fn.restype = ctypes.c_ulonglong
    return int(fn(ctypes.c_ulonglong(int(ns))))


class _QkvEpilogue(ctypes.Structure):
    _fields_ = [("q_norm_w", c_void_p), ("k_norm_w", c_void_p), ("q_out", c_void_p), ("k_dense", c_void_p),
                ("v_dense", c_void_p), ("kv_cache", c_void_p * 4), ("cache_sel", c_void_p), ("slot", c_void_p),
                ("pos", c_void_p), ("rope_cs", c_void_p), ("n_caches", c_int), ("nq", c_int), ("nkv", c_int), ("page_size", c_int),
                ("eps", c_float), ("theta", c_float)]


def gemm_qkv(x: torch.Tensor, w: torch.Tensor, q_w, k_w, pos, nq: int, nkv: int, eps: float, theta: float, *,
             x2: Optional[torch.Tensor] = None, w2: Optional[torch.Tensor] = None, q_out=None, k_dense=None,
             v_dense=None, caches: Sequence[torch.Tensor] = (), cache_sel=None, slot=None, page_size: int = 16,
             tp_wait=None, splits: Optional[int] = None, bn: int = 0, rope_cs: Optional[torch.Tensor] = None):
    """QKV projection (``x @ w^T`` + LoRA K-extension) whose epilogue applies the per-head QK RMSNorm and RoPE and
    writes q to ``q_out`` and K / V into the paged cache slots (and / or ``k_dense`` / ``v_dense``): the fused form
    of :func:`gemm` followed by :func:`qk_norm_rope_kv`, for head_dim 128 (one 128-feature tile = one head)."""
    _check_bf16_2d(x, "x")
    _check_bf16_2d(w, "w")
    M, K = x.shape
    F = w.shape[0]
    if F != (nq + 2 * nkv) * 128:
        raise ValueError("gemm_qkv needs head_dim 128 and w of (nq + 2 nkv) * 128 rows")
    R = 0
    if x2 is not None:
        _check_bf16_2d(x2, "x2")
        _check_bf16_2d(w2, "w2")
        R = x2.shape[1]
    if q_out is None:
        q_out = torch.empty(M, nq * 128, dtype=torch.bfloat16, device=x.device)
    if splits is None and bn == 0:
        bn, splits = plan_gemm(M, F, K, R, False)
    elif splits is None:
        splits = 1
    e = _QkvEpilogue()
    e.q_norm_w, e.k_norm_w, e.q_out = q_w.data_ptr(), k_w.data_ptr(), q_out.data_ptr()
    e.k_dense = 0 if k_dense is None else k_dense.data_ptr()
    e.v_dense = 0 if v_dense is None else v_dense.data_ptr()
    for i in range(4):
        e.kv_cache[i] = caches[i].data_ptr() if i < len(caches) else 0
    e.cache_sel = 0 if cache_sel is None else cache_sel.data_ptr()
    e.slot = 0 if slot is None else slot.data_ptr()
    e.pos = pos.data_ptr()
    e.rope_cs = 0 if rope_cs is None else rope_cs.data_ptr()     # [M, 128] table from rope_table(), else computed in place
    e.n_caches, e.nq, e.nkv, e.page_size, e.eps, e.theta = len(caches), nq, nkv, page_size, eps, theta
    if tp_wait is not None:
        flags, targets = tp_wait
        wait = (_p(flags), _p(targets), c_int(flags.numel()))
    else:
        wait = (None, None, c_int(0))
    _rc(lib().tahb_gemm_qkv(_p(w), _p(x), _p(w2), _p(x2), c_int(M), c_int(F), c_int(K), c_int(R), c_ll(w.stride(0)),
                            c_ll(x.stride(0)), c_ll(w2.stride(0) if w2 is not None else 0),
                            c_ll(x2.stride(0) if x2 is not None else 0), c_int(splits), c_int(bn),
                            _p(status_word(x.device)), _stream(), *wait, ctypes.byref(e)), "tahb_gemm_qkv")
    return q_out


def _ptr_array(tensors: Sequence[Optional[torch.Tensor]]):
    arr = (c_void_p * len(tensors))()
    for i, t in enumerate(tensors):
        arr[i] = 0 if t is None else t.data_ptr()
    return arr


def qk_norm_rope_kv(qkv, q_w, k_w, pos, nq: int, nkv: int, hd: int, eps: float, theta: float, *,
                    q_out=None, k_dense=None, v_dense=None, caches: Sequence[torch.Tensor] = (),
                    cache_sel=None, slot=None, page_size: int = 16):
    """Per-head QK RMSNorm + RoPE on a fused ``[M, (nq+2nkv)*hd]`` projection; writes normed/rotated
    q to ``q_out``, K/V to ``k_dense``/``v_dense`` and/or into the paged cache(s) at ``slot``."""
    _check_bf16_2d(qkv, "qkv")
    M = qkv.shape[0]
    if q_out is None:
        q_out = torch.empty(M, nq * hd, dtype=torch.bfloat16, device=qkv.device)
    arr = _ptr_array(list(caches)) if caches else (c_void_p * 1)()
    _rc(lib().tahb_qk_norm_rope_kv(_p(qkv), _p(q_w), _p(k_w), _p(q_out), _p(k_dense), _p(v_dense), arr,
                                   c_int(len(caches)), _p(cache_sel), _p(slot), _p(pos), c_int(M), c_int(nq),
                                   c_int(nkv), c_int(hd), c_int(page_size), c_ll(qkv.stride(0)), c_float(eps),
                                   c_float(theta), _stream()), "tahb_qk_norm_rope_kv")
    return q_out


def rms_norm_bwd(x: torch.Tensor, w: torch.Tensor, gy: torch.Tensor, eps: float, want_gw: bool = True):
    """Backward of :func:`rms_norm` on contiguous ``[M, H]`` bf16 tensors: returns ``(gx, gw_fp32 or None)``."""
    M, H = x.shape
    gx = torch.empty_like(x)
    gw = torch.zeros(H, dtype=torch.float32, device=x.device) if want_gw else None
    _rc(lib().tahb_rmsnorm_bwd(_p(x), _p(w), _p(gy), _p(gx), _p(gw), c_int(M), c_int(H), c_float(eps), _stream()),
        "tahb_rmsnorm_bwd")
    return gx, gw


def swiglu_bwd(gate_up: torch.Tensor, gy: torch.Tensor) -> torch.Tensor:
    """Backward of :func:`swiglu`: ``gate_up`` ``[M, 2I]``, ``gy`` ``[M, I]`` (contiguous bf16) -> ``[M, 2I]``."""
    M, I2 = gate_up.shape
    out = torch.empty_like(gate_up)
    _rc(lib().tahb_swiglu_bwd(_p(gate_up), _p(gy), _p(out), c_ll(M), c_int(I2 // 2), _stream()), "tahb_swiglu_bwd")
    return out


def qk_norm_rope_bwd(qkv, q_w, k_w, gq, gk, gv, pos, nq: int, nkv: int, hd: int, eps: float, theta: float):
    """Backward of :func:`qk_norm_rope_kv` (dense outputs): returns ``(gqkv, gq_w_fp32, gk_w_fp32)``."""
    M = qkv.shape[0]
    gqkv = torch.empty_like(qkv)
    gqw = torch.zeros(hd, dtype=torch.float32, device=qkv.device)
    gkw = torch.zeros(hd, dtype=torch.float32, device=qkv.device)
    _rc(lib().tahb_qk_norm_rope_bwd(_p(qkv), _p(q_w), _p(k_w), _p(gq), _p(gk), _p(gv), _p(gqkv), _p(gqw), _p(gkw),
                                    _p(pos), c_int(M), c_int(nq), c_int(nkv), c_int(hd), c_float(eps), c_float(theta),
                                    _stream()), "tahb_qk_norm_rope_bwd")
    return gqkv, gqw, gkw


def embed_gather(E, tok, out=None):
    M, H = tok.shape[0], E.shape[1]
    if out is None:
        out = torch.empty(M, H, dtype=E.dtype, device=E.device)
    _rc(lib().tahb_embed_gather(_p(E), _p(tok), _p(out), c_int(M), c_int(H), c_ll(out.stride(0)), _stream()),
        "tahb_embed_gather")
    return out


def lora_a_rows(x, A, gate=None, out=None, tp_wait=None):
    """``out[r] = gate[r] ? x[r] @ A^T : 0`` for the few gated rows of a decode tick.  ``tp_wait =
    (flags, targets)``: gated rows first wait for the tensor-parallel broadcast of ``x``."""
    _check_bf16_2d(x, "x")
    M, K = x.shape
    R = A.shape[0]
    if out is None:
        out = torch.empty(M, R, dtype=torch.bfloat16, device=x.device)
    if tp_wait is None:
        _rc(lib().tahb_lora_a_rows(_p(x), _p(A), _p(out), _p(gate), c_int(M), c_int(K), c_int(R), c_ll(x.stride(0)),
                                   c_ll(out.stride(0)), _stream()), "tahb_lora_a_rows")
    else:
        flags, targets = tp_wait
        _rc(lib().tahb_lora_a_rows_tp(_p(x), _p(A), _p(out), _p(gate), c_int(M), c_int(K), c_int(R),
                                      c_ll(x.stride(0)), c_ll(out.stride(0)), _p(flags), _p(targets),
                                      c_int(flags.numel()), _p(status_word(x.device)), _stream()), "tahb_lora_a_rows_tp")
    return out


def swiglu(gate_up, out=None):
    _check_bf16_2d(gate_up, "gate_up")
    M, I2 = gate_up.shape
    if out is None:
        out = torch.empty(M, I2 // 2, dtype=torch.bfloat16, device=gate_up.device)
    _rc(lib().tahb_swiglu(_p(gate_up), _p(out), c_int(M), c_int(I2 // 2), c_ll(gate_up.stride(0)),
                          c_ll(out.stride(0)), _stream()), "tahb_swiglu")
    return out


def logits_post(logits, cum, depth, best, best_val=None):
    fn = lib().tahb_logits_post_f32 if logits.dtype == torch.float32 else lib().tahb_logits_post
    _rc(fn(_p(logits), _p(cum), _p(depth), _p(best), _p(best_val), c_int(logits.shape[0]), c_int(logits.shape[1]),
           c_ll(logits.stride(0)), c_ll(cum.stride(0)), _stream()), "tahb_logits_post")
    return best


# -------------------------------------------------------------------------------------------
# decoders with an fp32 residual stream (activations bf16, or fp32 in the 32-bit mode)
# -------------------------------------------------------------------------------------------
def _act_f32(*ts: torch.Tensor) -> int:
    """1 when the activation operands are fp32, 0 when they are bf16 (they must agree)."""
    dt = ts[0].dtype
    if dt not in (torch.float32, torch.bfloat16) or any(t.dtype != dt for t in ts):
        raise ValueError(f"activations must be all bf16 or all fp32, got {[t.dtype for t in ts]}")
    return 1 if dt == torch.float32 else 0


def linear(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[M, F] = x[M, K] @ w[F, K]^T``: the tensor-core GEMM for bf16, the fp32 FMA kernel for fp32 operands."""
    if not _act_f32(x, w):
        return gemm(x, w, out=out)
    if x.dim() != 2 or w.dim() != 2 or x.shape[1] != w.shape[1] or x.stride(1) != 1 or w.stride(1) != 1:
        raise ValueError(f"linear: x {tuple(x.shape)} w {tuple(w.shape)}")
    M, Kd = x.shape
    if out is None:
        out = torch.empty(M, w.shape[0], dtype=torch.float32, device=x.device)
    _rc(lib().tahb_gemm_f32(_p(x), c_ll(x.stride(0)), _p(w), c_ll(w.stride(0)), _p(out), c_ll(out.stride(0)), c_int(M),
                            c_int(w.shape[0]), c_int(Kd), _stream()), "tahb_gemm_f32")
    return out


def swiglu_linear(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``silu(gate) * up`` of ``x @ w^T``: bf16 weights have interleaved gate / up rows (:func:`interleave_gate_up`, the
    fused GEMM epilogue), fp32 weights the stacked ``[gate; up]`` rows (product, then an activation kernel)."""
    if not _act_f32(x, w):
        return gemm(x, w, out=out, swiglu_interleaved=True)
    gu = linear(x, w)
    M, inter = gu.shape[0], gu.shape[1] // 2
    if out is None:
        out = torch.empty(M, inter, dtype=torch.float32, device=x.device)
    _rc(lib().tahb_swiglu_f32(_p(gu), _p(out), c_int(M), c_int(inter), c_ll(gu.stride(0)), c_ll(out.stride(0)),
                              _stream()), "tahb_swiglu_f32")
    return out


def xielu_linear(x: torch.Tensor, w: torch.Tensor, up: float, low: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """xIELU of ``x @ w^T``: ``up z^2 + z / 2`` for ``z > 0`` and ``low (exp(z) - 1 - z) + z / 2`` otherwise; in the epilogue of
    the product for bf16 (on ``z`` rounded to bf16), a kernel behind it for fp32."""
    M, Kd = x.shape
    F = w.shape[0]
    if w.shape[1] != Kd:
        raise ValueError(f"xielu_linear: x {tuple(x.shape)} w {tuple(w.shape)}")
    if _act_f32(x, w):
        out = linear(x, w, out=out)
        _rc(lib().tahb_xielu_f32(_p(out), c_float(up), c_float(low), c_int(M), c_int(F), c_ll(out.stride(0)), _stream()), "tahb_xielu_f32")
        return out
    if out is None:
        out = torch.empty(M, F, dtype=torch.bfloat16, device=x.device)
    for n, t in (("x", x), ("w", w), ("out", out)):
        _check_bf16_2d(t, n)
    pair = PAIR_AUTO and M >= PAIR_MIN_TOKENS and F % 256 == 0
    bn, splits = (256, 1) if pair else plan_gemm(M, F, Kd)
    _rc(lib().tahb_gemm_xielu(_p(w), _p(x), _p(out), c_int(M), c_int(F), c_int(Kd), c_ll(w.stride(0)), c_ll(x.stride(0)), c_ll(out.stride(0)),
                              c_float(up), c_float(low), c_int(int(pair)), c_int(splits), c_int(bn), _p(status_word(x.device)), _stream()),
        "tahb_gemm_xielu")
    return out


def embed_norm(E, tok, scale: float, w, width: int, eps: float, x, h, groups: int = 1, pos=None, freq=None, streams: int = 1,
               w_in=None, add=None, centered: bool = False):
    """``x = scale * E[tok]`` (fp32 residual stream) and ``h = rms(x) * w`` in the activation type of ``E``.  Rows are
    padded to ``E.shape[1]`` columns, ``width`` of them real.  ``groups``: parts of the row with a root mean square of
    their own; ``pos`` / ``freq``: token positions and :func:`sinusoid_frequencies`, adds sinusoidal positions to ``x``;
    ``streams`` / ``w_in``: that many copies in ``x [M, streams, ld]``, and the fp32 weights of their sum (what ``h`` sees);
    ``add``: fp32 vector added to ``x``; ``centered``: a layer norm in the place of the RMS norm."""
    f32 = _act_f32(E, h)
    if x.numel() != tok.shape[0] * streams * E.shape[1]:
        raise ValueError(f"embed_norm: residual {tuple(x.shape)} for {streams} streams of {E.shape[1]} columns")
    _rc(lib().tahb_embed_norm(_p(E), _p(tok), c_float(scale), _p(pos if freq is not None else None), _p(freq), c_int(streams),
                              _p(w_in), _p(add), _p(x), _p(w), _p(h), c_int(tok.shape[0]), c_int(E.shape[0]), c_int(width),
                              c_int(groups), c_int(E.shape[1]), c_float(eps), c_int(int(centered)), c_int(f32), _stream()),
        "tahb_embed_norm")


def sinusoid_frequencies(width: int, base: float = 10000.0, device=None) -> torch.Tensor:
    """``[2, (width + 1) // 2]`` fp32: the frequency ``base ** (-2 i / width)`` of the entry pair ``(2 i, 2 i + 1)`` as a
    high and a low part, so that the kernel can form angles beyond fp32 rounding."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / width)
    hi = f.float()
    return torch.stack([hi, (f - hi.double()).float()]).contiguous().to(device)


def rotary_table(pos, freq, mscale: float, out):
    """``out [n, half, 2]``: ``mscale * (cos, sin)`` of ``pos * f``; ``freq [2, half]``: frequencies as high and low parts."""
    _rc(lib().tahb_rotary_table(_p(pos), _p(freq), c_float(mscale), _p(out), c_int(pos.shape[0]), c_int(freq.shape[1]), _stream()),
        "tahb_rotary_table")
    return out


class _Streams(ctypes.Structure):
    _fields_ = [("y", c_void_p), ("ldy", c_ll), ("y_bias", c_void_p), ("y_ex", c_void_p), ("slot", c_void_p), ("y_weight", c_void_p),
                ("top", c_int), ("x", c_void_p), ("hc", c_void_p), ("w_next", c_void_p), ("h", c_void_p), ("width", c_int),
                ("groups", c_int), ("ld", c_int), ("eps", c_float)]


def streams_norm(y, x, hc, w_next, width: int, groups: int, eps: float, h, y_bias=None, y_ex=None, slot=None, y_weight=None):
    """The seam of hyper-connections: with ``x [M, S, ld]`` (fp32, in place) and ``hc`` = mix ``[S, S]`` (from, to), out
    ``[S]``, in ``[S]`` back to back, ``x_t <- sum_s mix[s, t] x_s + out[t] * y`` and ``h = rms(sum_t in[t] x_t) * w_next``.
    ``y`` may be None; ``y_bias [ld]`` is added to it; ``y_ex [list rows, ld]`` / ``slot [M, top]`` / ``y_weight [M, top]``:
    expert outputs that are gathered and added with their weights."""
    M, S, ld = x.shape
    a = _Streams()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    if hc.numel() != S * S + 2 * S or hc.dtype != torch.float32:
        raise ValueError(f"streams_norm: {hc.numel()} weights for {S} streams")
    a.y, a.ldy, a.y_bias, a.y_ex, a.slot, a.y_weight = ptr(y), 0 if y is None else y.stride(0), ptr(y_bias), ptr(y_ex), ptr(slot), ptr(y_weight)
    a.top, a.x, a.hc, a.w_next, a.h = 0 if slot is None else slot.shape[1], ptr(x), ptr(hc), ptr(w_next), ptr(h)
    a.width, a.groups, a.ld, a.eps = width, groups, ld, eps
    f32 = _act_f32(h, *[t for t in (y, y_ex) if t is not None])
    _rc(lib().tahb_streams_norm(ctypes.byref(a), c_int(M), c_int(S), c_int(f32), _stream()), "tahb_streams_norm")


def residual_add_norm(y, x, mult: float, w_next, width: int, groups: int, eps: float, h, y_ex=None, slot=None):
    """``x += mult * y`` (fp32, in place) and ``h = rms(x) * w_next`` with ``groups`` parts per row: the seam behind a
    layer whose mixer and feed-forward run in parallel.  ``y_ex [list rows, ld]`` / ``slot [M, top]``: expert outputs that
    are gathered and added to ``y``."""
    f32 = _act_f32(y, h)
    _rc(lib().tahb_residual_add_norm(_p(y), c_ll(y.stride(0)), _p(y_ex), _p(slot), c_int(0 if slot is None else slot.shape[1]),
                                     c_float(mult), _p(x), _p(w_next), _p(h), c_int(y.shape[0]), c_int(width), c_int(groups),
                                     c_int(x.shape[1]), c_float(eps), c_int(f32), _stream()), "tahb_residual_add_norm")


class _ResidualNorm(ctypes.Structure):
    _fields_ = [("y", c_void_p), ("ldy", c_ll), ("x", c_void_p), ("w_out", c_void_p), ("w_next", c_void_p), ("h", c_void_p), ("width", c_int),
                ("ld", c_int), ("eps", c_float), ("add", c_void_p), ("E", c_void_p), ("tok", c_void_p), ("vocab", c_int), ("scale", c_float),
                ("before", c_void_p)]


def residual_norm(y, x, w_out, w_next, width: int, eps: float, h, centered: bool = False, add=None, embedding=None, before=None):
    """``x += norm(y) * w_out`` (fp32, in place) and ``h = norm(x) * w_next``: output norm, layer scale, residual sum and
    the next sublayer's input norm in one launch.  ``w_out`` / ``w_next``: fp32 rows padded with zeros.  The norms are RMS norms,
    or layer norms when ``centered``.  ``add`` (fp32 vector) and ``embedding = (E, tok, scale)``: what the residual gets in
    addition behind the sublayer's sum; ``before`` receives it without."""
    a = _ResidualNorm()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    E, tok, scale = (None, None, 0.0) if embedding is None else embedding
    f32 = _act_f32(y, h) if E is None else _act_f32(y, h, E)
    if E is not None and E.shape[1] != x.shape[1] or before is not None and before.shape != x.shape:
        raise ValueError(f"residual_norm: rows of {x.shape[1]} columns")
    a.y, a.ldy, a.x, a.w_out, a.w_next, a.h = ptr(y), y.stride(0), ptr(x), ptr(w_out), ptr(w_next), ptr(h)
    a.width, a.ld, a.eps, a.add, a.E, a.tok, a.before = width, x.shape[1], eps, ptr(add), ptr(E), ptr(tok), ptr(before)
    a.vocab, a.scale = 0 if E is None else E.shape[0], scale
    _rc(lib().tahb_residual_norm(ctypes.byref(a), c_int(y.shape[0]), c_int(int(centered)), c_int(f32), _stream()), "tahb_residual_norm")


def few_linear(x, w, b, out=None):
    """``x @ w^T + b`` with an fp32 result for a handful of output features (gates of a recurrence)."""
    M, F = x.shape[0], w.shape[0]
    if out is None:
        out = torch.empty(M, F, dtype=torch.float32, device=x.device)
    _rc(lib().tahb_few_linear(_p(x), c_ll(x.stride(0)), _p(w), _p(b), _p(out), c_int(M), c_int(w.shape[1]), c_int(F),
                              c_int(_act_f32(x, w)), _stream()), "tahb_few_linear")
    return out


APPEND_MAX_ENTRIES = 1024


def kv_append(rows, counts, starts, cache, depth: int, pos, row_of, slot):
    """Append ``counts[e]`` tokens to row ``rows[e]`` of the paged cache for every entry of a step (pages from the device
    free stack); fills position, row and slot of every packed token (entry ``e`` starts at ``starts[e]``)."""
    pt = cache.page_table[depth]
    _rc(lib().tahb_kv_append(_p(rows), _p(counts), _p(starts), c_int(rows.numel()), _p(cache.len[depth]), _p(pt),
                             _p(cache.free_stack[depth]), _p(cache.free_count[depth]), c_int(cache.rows), c_int(pt.shape[1]),
                             c_int(cache.page_size), _p(pos), _p(row_of), _p(slot), _p(status_word(pt.device)), _stream()),
        "tahb_kv_append")


class _QkvPost(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("qkv", "bias", "q_w", "k_w", "q_out", "cache", "slot")] + \
               [(n, c_int) for n in ("M", "nq", "nkv", "dk", "dv", "dim", "page_size")] + [("ld", c_ll), ("eps", c_float),
                ("rope", c_void_p), ("rot", c_int), ("interleaved", c_int), ("v_first", c_void_p), ("lam", c_void_p),
                ("v_keep", c_void_p)]


def qkv_post(qkv, bias, q_w, k_w, q_out, cache, slot, nq: int, nkv: int, dk: int, dv: int, dim: int, page_size: int,
             eps: float, rope=None, rot: int = 0, interleaved: bool = False, v_first=None, lam=None, v_keep=None):
    """Projection bias, per-head RMS norm of q / k, rotation of their first ``rot`` dims (``rope [n, rot / 2, 2]``, see
    :func:`rotary_table`; pairs ``(2 i, 2 i + 1)`` when ``interleaved``, else ``(i, i + rot / 2)``), q to ``q_out``, k / v into
    the paged cache.  ``nkv = 0``: queries only (a layer that reads another layer's keys); ``nq = 0``: keys and values only
    (``qkv`` starts at the keys).  ``v_first [n, nkv * dv]`` / ``lam [1]``: values become ``(1 - lam) v + lam v_first``;
    ``v_keep [n, nkv * dv]`` receives the values instead."""
    a = _QkvPost()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    for n, t in (("qkv", qkv), ("bias", bias), ("q_w", q_w), ("k_w", k_w), ("q_out", q_out), ("cache", cache), ("slot", slot),
                 ("rope", rope), ("v_first", v_first), ("lam", lam), ("v_keep", v_keep)):
        setattr(a, n, ptr(t))
    a.M, a.nq, a.nkv, a.dk, a.dv, a.dim, a.page_size = qkv.shape[0], nq, nkv, dk, dv, dim, page_size
    a.ld, a.eps, a.rot, a.interleaved = qkv.stride(0), eps, rot, int(interleaved)
    _rc(lib().tahb_qkv_post(ctypes.byref(a), c_int(_act_f32(qkv, qkv if q_out is None else q_out)), _stream()), "tahb_qkv_post")


class _WindowAttn(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("out", c_void_p), ("cache", c_void_p), ("page_table", c_void_p), ("pos", c_void_p),
                ("row", c_void_p), ("bias", c_void_p), ("sink", c_void_p), ("gate", c_void_p), ("wide_gate", c_void_p)] + \
               [(n, c_int) for n in ("n", "nq", "nkv", "dk", "dv", "page_size", "max_pages", "window", "keep_first", "far")] + \
               [("ld_q", c_ll), ("ld_out", c_ll), ("ld_gate", c_ll), ("scale", c_float), ("softcap", c_float),
                ("temp_coef", c_float), ("temp_every", ctypes.c_double), ("ws", c_void_p), ("n_split", c_int),
                ("status", c_void_p), ("slope", c_void_p), ("factor", c_void_p), ("pooled", c_void_p), ("tied", c_int), ("n_pages", c_int), ("pool", c_int),
                ("pool_rows", c_int), ("out_scale", c_float)]


def window_attn_args(q, out, pool, page_table, pos, row, *, nq: int, nkv: int, dk: int, dv: int, page_size: int,
                     scale: float, window: int, keep_first: int, bias=None, sink=None, gate=None, softcap=None, q_temp=None,
                     n_split: int = 1, ws=None, wide_gate=None, slope=None, tied: bool = False, factor=None, pooled=None,
                     block: int = 0, pool_rows: int = 0, out_scale: float = 1.0):
    """Arguments of one windowed attention launch: queries ``q [n, nq * dk]`` (any row pitch) at positions ``pos`` of cache
    rows ``row`` over the paged ``pool`` of the layer that owns the keys; ``softcap``: score cap, ``q_temp = (coef,
    every)``: query temperature, ``slope [nq]``: taken off the scores per token of distance; ``tied``: the pool holds keys only,
    which are the values, with an optional ``factor [pages, page_size]`` of every key's scores, and optional block means
    ``pooled`` of ``block`` keys each, ``pool_rows`` of them a page; ``out_scale``: factor of the output; see
    ``csrc/attn_window.cu`` for the rule."""
    a = _WindowAttn()
    a.tied, a.n_pages, a.pool, a.pool_rows, a.out_scale = int(tied), pool.shape[0], block, pool_rows, out_scale
    ptr = lambda t: 0 if t is None else t.data_ptr()
    a.q, a.out, a.cache, a.page_table, a.pos, a.row = (ptr(t) for t in (q, out, pool, page_table, pos, row))
    a.bias, a.sink, a.gate, a.wide_gate = ptr(bias), ptr(sink), ptr(gate), ptr(wide_gate)
    a.slope, a.factor, a.pooled = ptr(slope), ptr(factor), ptr(pooled)
    gate = wide_gate if gate is None else gate
    a.n, a.nq, a.nkv, a.dk, a.dv, a.page_size, a.max_pages = q.shape[0], nq, nkv, dk, dv, page_size, page_table.shape[1]
    a.window, a.keep_first, a.far = window, keep_first, 0 if bias is None else bias.shape[1] - 1
    a.softcap = 0.0 if softcap is None else softcap
    a.temp_coef, a.temp_every = (0.0, 1.0) if q_temp is None else q_temp
    a.ld_q, a.ld_out, a.ld_gate = q.stride(0), out.stride(0), 0 if gate is None else gate.stride(0)
    a.scale, a.ws, a.n_split, a.status = scale, ptr(ws), n_split, status_word(q.device).data_ptr()
    return a


def window_attn_plain(q, out, pool, page_table, pos, row, **kw):
    """Windowed attention, one warp per (query, head): any head size up to 256, bf16 or fp32."""
    a = window_attn_args(q, out, pool, page_table, pos, row, **kw)
    _rc(lib().tahb_window_attn_plain(ctypes.byref(a), c_int(_act_f32(q, out)), _stream()), "tahb_window_attn_plain")
    return out


def window_attn_decode(q, out, pool, page_table, pos, row, **kw):
    """Windowed attention of single tokens (bf16, pages of 16): pipelined page copies, optional key splits (``n_split``,
    ``ws`` of ``n * nq * n_split * (dv + 2)`` floats).  ``bias``, ``sink`` and ``slope`` in log2 units."""
    a = window_attn_args(q, out, pool, page_table, pos, row, **kw)
    _rc(lib().tahb_window_attn_decode(ctypes.byref(a), _stream()), "tahb_window_attn_decode")
    return out


def window_attn_tiles(q, out, pool, page_table, pos, row, tile_q0, tile_qn, n_pages: int, kv_ld: int = 0, pool_base=None, **kw):
    """Windowed attention of prompt portions on the tensor cores (bf16, pages of 16): tiles of up to 128 consecutive
    tokens of one row.  ``bias``, ``sink`` and ``slope`` in log2 units.  ``kv_ld``: ``pool`` is not a paged cache but a matrix of that
    pitch whose rows ``[keys of all heads | values of all heads]`` are a token each, 16 of them a page.  ``wide_gate``: gate
    pre-activations of every output element (``gate``: of every head).  ``pooled`` is then the matrix of :func:`pool_gather`, and
    ``pool_base`` the first of its pages of 16 rows that belongs to a tile's row."""
    a = window_attn_args(q, out, pool, page_table, pos, row, **kw)
    pooled = kw.get("pooled")
    _rc(lib().tahb_window_attn_tiles(ctypes.byref(a), _p(tile_q0), _p(tile_qn), c_int(tile_q0.numel()), c_int(n_pages),
                                     c_ll(kv_ld), _p(pool_base), c_int(0 if pooled is None else pooled.shape[0] // 16), _stream()),
        "tahb_window_attn_tiles")
    return out


class _TiedKeys(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("k", "cache", "pooled", "slot", "pos", "row", "page_table")] + \
               [(n, c_int) for n in ("M", "nkv", "dk", "page_size", "max_pages", "pool", "pool_rows")] + [("ld", c_ll)]


def tied_keys(k, cache, slot, pos, row, page_table, nkv: int, dk: int, page_size: int, pooled=None, block: int = 0, pool_rows: int = 0):
    """Keys ``k [n, nkv * dk]`` (any row pitch) of a tied layer to the paged cache, and the mean of every block of ``block`` keys
    that a token completes to its ``pooled`` row."""
    a = _TiedKeys()
    for n, t in (("k", k), ("cache", cache), ("pooled", pooled), ("slot", slot), ("pos", pos), ("row", row), ("page_table", page_table)):
        setattr(a, n, 0 if t is None else t.data_ptr())
    a.M, a.nkv, a.dk, a.page_size, a.max_pages = k.shape[0], nkv, dk, page_size, page_table.shape[1]
    a.pool, a.pool_rows, a.ld = block, pool_rows, k.stride(0)
    _rc(lib().tahb_tied_keys(ctypes.byref(a), c_int(_act_f32(k, cache)), _stream()), "tahb_tied_keys")


def pool_gather(pooled, src, nkv: int, dk: int, pool_rows: int, out):
    """Pooled rows ``src`` (page * pool_rows + row; negative: zeros) one after another: ``out [n, nkv * dk]``."""
    if out.shape[0] < src.numel() or out.shape[1] != nkv * dk or not out.is_contiguous():
        raise ValueError(f"pool_gather: {tuple(out.shape)} for {src.numel()} rows of {nkv} x {dk}")
    _act_f32(pooled, out)
    _rc(lib().tahb_pool_gather(_p(pooled), _p(src), c_int(src.numel()), c_int(nkv), c_int(dk * pooled.element_size()), c_int(pool_rows),
                               c_int(pooled.shape[0]), _p(out), _stream()), "tahb_pool_gather")
    return out


class _NormAll(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("q", "k", "w", "q_out", "cache", "factor", "slot")] + \
               [(n, c_int) for n in ("M", "nq", "nkv", "dk", "dim", "page_size")] + [("ld", c_ll), ("eps", c_float)]


def norm_all(q, k, w, q_out, cache, factor, slot, *, nq: int, nkv: int, dk: int, dim: int, page_size: int, eps: float):
    """RMS norms of q and k over all heads of a token, in a tied layer: ``q_out`` = ``q`` with its norm's factor and the weights
    ``w [nq * dk]`` of both norms; ``k`` as it is to the paged cache, its norm's factor to ``factor [pages, page_size]``."""
    a = _NormAll()
    for n, t in (("q", q), ("k", k), ("w", w), ("q_out", q_out), ("cache", cache), ("factor", factor), ("slot", slot)):
        setattr(a, n, t.data_ptr())
    if q.stride(0) != k.stride(0) or not q_out.is_contiguous() or w.numel() != nq * dk:
        raise ValueError("norm_all: queries and keys of one projection, packed output")
    a.M, a.nq, a.nkv, a.dk, a.dim, a.page_size, a.ld, a.eps = q.shape[0], nq, nkv, dk, dim, page_size, q.stride(0), eps
    _rc(lib().tahb_norm_all(ctypes.byref(a), c_int(_act_f32(q, k, q_out, cache)), _stream()), "tahb_norm_all")


# -------------------------------------------------------------------------------------------
# elementwise recurrence (csrc/min_gru.cu)
# -------------------------------------------------------------------------------------------
class _MinGru(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("proj", "zb", "xb", "out", "S", "seq_start", "seq_len", "pos", "row", "slot", "ws")] + \
               [(n, c_int) for n in ("n", "d", "n_split")] + [("ld", c_ll), ("ld_out", c_ll), ("out_scale", c_float)]


def _min_gru_args(proj, zb, xb, out, state, pos, row, out_scale, seq_start=None, seq_len=None, slot=None, n_split=1, ws=None):
    a = _MinGru()
    for n, t in (("proj", proj), ("zb", zb), ("xb", xb), ("out", out), ("S", state[0]), ("seq_start", seq_start), ("seq_len", seq_len),
                 ("pos", pos), ("row", row), ("slot", slot), ("ws", ws)):
        setattr(a, n, 0 if t is None else t.data_ptr())
    d = zb.numel()
    if proj.shape[1] < 3 * d or out.shape[1] < d or state[0].shape[1] != d:
        raise ValueError(f"min_gru: {d} channels in a projection of {proj.shape[1]}")
    a.n, a.d, a.n_split, a.ld, a.ld_out, a.out_scale = proj.shape[0], d, n_split, proj.stride(0), out.stride(0), out_scale
    return a


def min_gru_step(proj, zb, xb, out, state, pos, row, out_scale: float, slot=None):
    """One token per row of ``S <- (1 - z) S + z c(u)``, ``out = out_scale * S * silu(g)``, from columns ``[z | u | g]`` of ``proj``
    (biases ``zb``, ``xb``); updates ``state = (S [rows, d],)`` in place.  Rows with a negative ``slot`` are left alone."""
    a = _min_gru_args(proj, zb, xb, out, state, pos, row, out_scale, slot=slot)
    _rc(lib().tahb_min_gru_step(ctypes.byref(a), c_int(_act_f32(proj, out)), _stream()), "tahb_min_gru_step")
    return out


def min_gru_scan(proj, zb, xb, out, state, pos, row, out_scale: float, *, seq_start, seq_len, n_split: int = 1, ws=None):
    """The same for portions ``seq_start`` / ``seq_len``, each cut into ``n_split`` segments that run side by side (``ws``: portions
    * n_split * 2 * d floats)."""
    a = _min_gru_args(proj, zb, xb, out, state, pos, row, out_scale, seq_start, seq_len, None, n_split, ws)
    n_seq = seq_start.numel()
    if n_split > 1 and ws.numel() < n_seq * n_split * 2 * a.d:
        raise ValueError("min_gru_scan: workspace too small")
    _rc(lib().tahb_min_gru_scan(ctypes.byref(a), c_int(n_seq), c_int(_act_f32(proj, out)), _stream()), "tahb_min_gru_scan")
    return out


# -------------------------------------------------------------------------------------------
# latent attention (csrc/attn_latent.cu)
# -------------------------------------------------------------------------------------------
class _LatentPost(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("proj", "q_w", "c_w", "rope", "cq", "cache", "slot")] + \
               [(n, c_int) for n in ("M", "q_rank", "Qp", "q_col", "kv_rank", "Rp", "c_col", "rot", "rw", "r_col")] + \
               [("ld", c_ll), ("eps", c_float)]


def latent_post(proj, q_w, c_w, rope, cq, cache, slot, *, q_rank: int, q_col: int, kv_rank: int, Rp: int, c_col: int, rot: int,
                rw: int, r_col: int, eps: float):
    """After the projection ``[query latent | c | r | ...]``: ``cq`` = RMS norm of the query latent, and the cached row
    ``[norm of c (Rp columns) | rotated r (rw columns)]`` of every token."""
    a = _LatentPost()
    for n, t in (("proj", proj), ("q_w", q_w), ("c_w", c_w), ("rope", rope), ("cq", cq), ("cache", cache), ("slot", slot)):
        setattr(a, n, t.data_ptr())
    a.M, a.q_rank, a.Qp, a.q_col, a.kv_rank, a.Rp, a.c_col = proj.shape[0], q_rank, cq.shape[1], q_col, kv_rank, Rp, c_col
    a.rot, a.rw, a.r_col, a.ld, a.eps = rot, rw, r_col, proj.stride(0), eps
    _rc(lib().tahb_latent_post(ctypes.byref(a), c_int(_act_f32(proj, cq, cache)), _stream()), "tahb_latent_post")


class _LatentQuery(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("q", "rope", "list")] + \
               [(n, c_int) for n in ("n", "n_list", "npad", "heads", "dk", "dq", "dim", "rot")] + [("ld", c_ll)]


class HeadLists:
    """Block table of head lists (``heads`` runs of ``npad`` rows), in the form the grouped products take."""

    def __init__(self, n: int, heads: int, dtype: torch.dtype, device):
        self.bn = 64 if dtype == torch.float32 else 16 if n <= 16 else 32 if n <= 32 else 64 if n <= 64 else 128
        self.n, self.heads, self.npad = n, heads, (n + self.bn - 1) // self.bn * self.bn
        self.rows = heads * self.npad
        self.blk_expert = torch.arange(heads, dtype=torch.int32, device=device).repeat_interleave(self.npad // self.bn)
        self.n_blocks = torch.full((1,), self.rows // self.bn, dtype=torch.int32, device=device)


def latent_query(q, rope, lists: Optional[HeadLists], list_out, *, heads: int, dk: int, dim: int, rot: int):
    """Rotate the last ``rot`` dims of every head of ``q [n, heads * dk]``: the first ``lists.n`` tokens go to the head lists
    ``list_out [lists.rows, dq]``, the others are rotated in place."""
    a = _LatentQuery()
    a.q, a.rope, a.list = q.data_ptr(), rope.data_ptr(), 0 if lists is None else list_out.data_ptr()
    a.n, a.n_list, a.npad = q.shape[0], 0 if lists is None else lists.n, 0 if lists is None else lists.npad
    a.heads, a.dk, a.dq, a.dim, a.rot, a.ld = heads, dk, dk if lists is None else list_out.shape[1], dim, rot, q.stride(0)
    _rc(lib().tahb_latent_query(ctypes.byref(a), c_int(_act_f32(q)), _stream()), "tahb_latent_query")


def latent_gather(pool, src_pages, page_size: int, row: int, out):
    """Pages ``src_pages`` of a latent cache (rows of ``row`` elements) one after another as rows of ``out [pages * page_size,
    lp]``, zeros behind the cached row."""
    es = pool.element_size()
    if out.shape[0] < src_pages.numel() * page_size or not out.is_contiguous():
        raise ValueError(f"latent_gather: {tuple(out.shape)} for {src_pages.numel()} pages")
    _rc(lib().tahb_latent_gather(_p(pool), _p(src_pages), c_int(src_pages.numel()), c_int(pool.shape[0]), c_int(page_size),
                                 c_int(row * es), c_int(out.shape[1] * es), _p(out), _stream()), "tahb_latent_gather")
    return out


def latent_gate(list_v, lists: HeadLists, gate, out, dv: int):
    """``out[t, h * dv + d] = list_v[h * npad + t, d] * sigmoid(gate[t, h * dv + d])`` (``gate`` None: no factor): back from head
    lists to token rows."""
    _rc(lib().tahb_latent_gate(_p(list_v), c_int(lists.npad), c_int(list_v.shape[1]), _p(gate), c_ll(0 if gate is None else gate.stride(0)),
                               _p(out), c_ll(out.stride(0)), c_int(lists.n), c_int(lists.heads), c_int(dv), c_int(_act_f32(list_v, out)),
                               _stream()), "tahb_latent_gate")
    return out


class _LatentAttn(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("q", "out", "cache", "page_table", "pos", "row", "sink")] + \
               [(n, c_int) for n in ("n", "npad", "heads", "Rp", "rw", "lq", "page_size", "max_pages")] + \
               [("scale", c_float), ("ws", c_void_p), ("n_split", c_int), ("n_pages", c_int), ("status", c_void_p), ("window", c_int)]


def _latent_attn_args(q, out, pool, page_table, pos, row, lists: HeadLists, *, Rp: int, rw: int, page_size: int, scale: float,
                      sink=None, n_split: int = 1, ws=None, window: int = 2 ** 31 - 1):
    a = _LatentAttn()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    a.q, a.out, a.cache, a.page_table, a.pos, a.row, a.sink = (ptr(t) for t in (q, out, pool, page_table, pos, row, sink))
    a.n, a.npad, a.heads, a.Rp, a.rw, a.lq = lists.n, lists.npad, lists.heads, Rp, rw, q.shape[1]
    a.page_size, a.max_pages, a.scale, a.ws, a.n_split = page_size, page_table.shape[1], scale, ptr(ws), n_split
    a.n_pages, a.status, a.window = pool.shape[0], status_word(q.device).data_ptr(), window
    if n_split > 1 and ws.numel() < lists.n * lists.heads * n_split * (Rp + 2):
        raise ValueError("latent attention: workspace too small")
    return a


def latent_attn_plain(q, out, pool, page_table, pos, row, lists: HeadLists, **kw):
    """Absorbed latent attention of the tokens of ``lists`` over the cached rows: ``q [lists.rows, lq]`` -> ``out [lists.rows,
    Rp]``, any sizes, bf16 or fp32.  ``sink`` in natural units."""
    a = _latent_attn_args(q, out, pool, page_table, pos, row, lists, **kw)
    _rc(lib().tahb_latent_attn_plain(ctypes.byref(a), c_int(_act_f32(q, out, pool)), _stream()), "tahb_latent_attn_plain")
    return out


def latent_attn_decode(q, out, pool, page_table, pos, row, lists: HeadLists, **kw):
    """The same on the tensor cores (bf16, pages of 16), with optional key splits.  ``sink`` in log2 units."""
    a = _latent_attn_args(q, out, pool, page_table, pos, row, lists, **kw)
    _rc(lib().tahb_latent_attn_decode(ctypes.byref(a), _stream()), "tahb_latent_attn_decode")
    return out


def latent_decode_fits(heads: int, Rp: int, rw: int) -> bool:
    return bool(lib().tahb_latent_decode_fits(c_int(heads), c_int(Rp), c_int(rw)))


# -------------------------------------------------------------------------------------------
# feed-forward mechanisms (csrc/feed_forward.cu)
# -------------------------------------------------------------------------------------------
def poly_norm(z, act, n: int, eps: float, out):
    """``a N(z) + b N(z^2) + c N(z^3) + e`` of every row, ``act = (a, b, c, e)`` fp32 on the device, ``N`` the division by
    the root mean square over the first ``n`` columns (the rest is padding)."""
    _rc(lib().tahb_poly_norm(_p(z), c_ll(z.stride(0)), _p(act), _p(out), c_ll(out.stride(0)), c_int(z.shape[0]), c_int(n),
                             c_int(z.shape[1]), c_float(eps), c_int(_act_f32(z, out)), _stream()), "tahb_poly_norm")
    return out


def clamped_glu(gu, limit: float, out, in_scale=None, gate=None, lists=None, slope: float = 1.702, offset: float = 1.0):
    """``g sigmoid(slope g) (u + offset)`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)`` of interleaved columns
    ``gate_0, up_0, gate_1, ...``.  ``in_scale``: factor of both per row; ``gate``: fp32 column whose sigmoid multiplies
    the row's result; ``lists``: :class:`ExpertLists` that the rows are those of."""
    _rc(lib().tahb_clamped_glu(_p(gu), c_ll(gu.stride(0)), _p(out), c_ll(out.stride(0)), c_int(gu.shape[0]), c_int(out.shape[1]),
                               c_float(limit), c_float(slope), c_float(offset), _p(in_scale), _p(gate),
                               c_ll(0 if gate is None else gate.stride(0)), _p(None if lists is None else lists.n_blocks),
                               c_int(0 if lists is None else lists.bn), c_int(_act_f32(gu, out)), _stream()), "tahb_clamped_glu")
    return out


def expert_block(pairs: int, experts: int, dtype: torch.dtype) -> int:
    """Rows of a block of the expert lists for ``pairs`` (token, expert) pairs: the token tile of the grouped product."""
    if dtype == torch.float32:
        return 64
    avg = pairs / experts
    return 16 if avg <= 10 else 32 if avg <= 21 else 64 if avg <= 42 else 128 if avg <= 192 else 256


class ExpertLists:
    """Buffers of a routed pass over ``M`` tokens: the tokens' experts and weights, and the experts' token lists in blocks
    of ``bn`` rows (``rows`` of them at most, however the router decides)."""

    def __init__(self, M: int, experts: int, top: int, dtype: torch.dtype, device, bn: Optional[int] = None):
        i32 = lambda *s: torch.empty(*s, dtype=torch.int32, device=device)
        self.M, self.experts, self.top = M, experts, top
        self.bn = bn or expert_block(M * top, experts, dtype)
        self.max_blocks = M * top // self.bn + min(experts, M * top)
        self.rows = self.max_blocks * self.bn
        self.expert, self.rank, self.slot = i32(M, top), i32(M, top), i32(M, top)
        self.weight = torch.empty(M, top, dtype=torch.float32, device=device)
        self.count = torch.zeros(experts + 1, dtype=torch.int32, device=device)
        self.seg, self.blk_expert, self.n_blocks = i32(experts), i32(self.max_blocks), i32(1)
        self.row_weight = torch.empty(self.rows, dtype=torch.float32, device=device)


def moe_route(z, lists: ExpertLists, softmax: bool = False):
    """Choose ``lists.top`` experts per row of router logits ``z [M, >= experts]`` (fp32) and build the experts' lists; the
    weights are the chosen experts' sigmoid scores, or their softmax scores over all experts."""
    L = lists
    if z.dtype != torch.float32 or z.shape[0] != L.M or z.shape[1] < L.experts:
        raise ValueError(f"moe_route: logits {z.dtype} {tuple(z.shape)} for {L.M} tokens and {L.experts} experts")
    _rc(lib().tahb_moe_route(_p(z), c_ll(z.stride(0)), c_int(L.M), c_int(L.experts), c_int(L.top), c_int(L.bn), c_int(int(softmax)), _p(L.expert),
                             _p(L.rank), _p(L.weight), _p(L.count), _p(L.seg), _p(L.blk_expert), _p(L.n_blocks),
                             c_int(L.max_blocks), _p(status_word(z.device)), _stream()), "tahb_moe_route")


def moe_gather(h, lists: ExpertLists, out):
    """Copy the rows of ``h`` into the experts' lists ``out [lists.rows, width]``."""
    L, es = lists, h.element_size()
    if out.shape != (L.rows, h.shape[1]) or not out.is_contiguous():
        raise ValueError(f"moe_gather: list buffer {tuple(out.shape)}, need {(L.rows, h.shape[1])}")
    _rc(lib().tahb_moe_gather(_p(h), c_int(h.shape[1] * es), c_ll(h.stride(0) * es), c_int(L.M), c_int(L.top), _p(L.expert),
                              _p(L.rank), _p(L.weight), _p(L.seg), _p(out), _p(L.row_weight), _p(L.slot), c_int(L.rows),
                              _p(status_word(h.device)), _stream()), "tahb_moe_gather")
    return out


def moe_linear(x, w, lists: ExpertLists, out):
    """``out[r] = x[r] @ w[expert of r]^T`` for the rows of the experts' lists; ``w [experts, F, K]``."""
    E, F, Kd = w.shape
    if not (x.is_contiguous() and w.is_contiguous() and out.is_contiguous()) or x.shape != (lists.rows, Kd) or out.shape != (lists.rows, F):
        raise ValueError(f"moe_linear: x {tuple(x.shape)} w {tuple(w.shape)} out {tuple(out.shape)}")
    if _act_f32(x, w, out):
        _rc(lib().tahb_moe_gemm_f32(_p(w), _p(x), _p(out), c_int(F), c_int(Kd), c_int(lists.rows), _p(lists.blk_expert),
                                    _p(lists.n_blocks), _stream()), "tahb_moe_gemm_f32")
    else:
        _rc(lib().tahb_moe_gemm(_p(w), _p(x), _p(out), c_int(E), c_int(F), c_int(Kd), c_int(lists.rows), c_int(lists.bn),
                                _p(lists.blk_expert), _p(lists.n_blocks), c_int(0), _p(None), c_float(0.0), c_float(0.0), c_float(0.0),
                                _p(status_word(x.device)), _stream()), "tahb_moe_gemm")
    return out


def moe_glu_linear(x, w, limit: float, lists: ExpertLists, out, slope: float = 1.702, offset: float = 1.0, weighted: bool = True):
    """:func:`clamped_glu` of :func:`moe_linear` with interleaved gate / up rows in ``w [experts, 2 F, K]``; ``weighted``: every
    list row's weight multiplies gate and up (the projection of the weighted input).  bf16: one kernel."""
    E, F2, Kd = w.shape
    if not (x.is_contiguous() and w.is_contiguous() and out.is_contiguous()) or x.shape != (lists.rows, Kd) or out.shape != (lists.rows, F2 // 2):
        raise ValueError(f"moe_glu_linear: x {tuple(x.shape)} w {tuple(w.shape)} out {tuple(out.shape)}")
    row_weight = lists.row_weight if weighted else None
    if _act_f32(x, w, out):
        gu = moe_linear(x, w, lists, torch.empty(lists.rows, F2, dtype=torch.float32, device=x.device))
        return clamped_glu(gu, limit, out, in_scale=row_weight, lists=lists, slope=slope, offset=offset)
    _rc(lib().tahb_moe_gemm(_p(w), _p(x), _p(out), c_int(E), c_int(F2), c_int(Kd), c_int(lists.rows), c_int(lists.bn),
                            _p(lists.blk_expert), _p(lists.n_blocks), c_int(1), _p(row_weight), c_float(limit), c_float(slope),
                            c_float(offset), _p(status_word(x.device)), _stream()), "tahb_moe_gemm")
    return out


class _Mlstm(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("qkvg", "gates", "norm_w", "out", "S", "nvec", "mval", "seq_start", "seq_len", "pos",
                                        "row", "slot")] + \
               [(n, c_int) for n in ("n_seq", "heads", "dk", "dv", "dim", "vdim")] + [("ld", c_ll), ("ld_out", c_ll)] + \
               [(n, c_float) for n in ("cap", "eps", "q_scale")]


def mlstm_args(qkvg, gates, norm_w, out, state, pos, row, *, heads: int, dk: int, dv: int, dim: int, vdim: int, cap: float,
               eps: float, seq_start=None, seq_len=None, slot=None):
    a = _Mlstm()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    S, nvec, mval = state
    a.qkvg, a.gates, a.norm_w, a.out = ptr(qkvg), ptr(gates), ptr(norm_w), ptr(out)
    a.S, a.nvec, a.mval = ptr(S), ptr(nvec), ptr(mval)
    a.seq_start, a.seq_len, a.pos, a.row, a.slot = ptr(seq_start), ptr(seq_len), ptr(pos), ptr(row), ptr(slot)
    a.n_seq = qkvg.shape[0] if seq_start is None else seq_start.shape[0]
    a.heads, a.dk, a.dv, a.dim, a.vdim = heads, dk, dv, dim, vdim
    a.ld, a.ld_out, a.cap, a.eps, a.q_scale = qkvg.stride(0), out.stride(0), cap, eps, dim ** -0.5
    return a


class _MlstmChunks(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("c_start", "c_len", "seq_chunk0", "seq_chunks", "dS", "dn", "cg", "s0", "n0", "m0")] + \
               [("n_chunks", c_int), ("status", c_void_p)]


def mlstm_chunk_ws_floats(n_chunks: int, heads: int, dk: int, dv: int) -> int:
    """fp32 workspace of :func:`mlstm_chunks`: dS, the incoming state as a bf16 pair, dn, n0, chunk scalars."""
    return n_chunks * heads * (2 * dk * dv + 2 * dk + 4)


def mlstm_chunks(qkvg, gates, norm_w, out, state, pos, row, *, chunk_start, chunk_len, seq_chunk0, seq_chunks, ws, **kw):
    """mLSTM of prompt portions in chunks of up to 128 tokens on the tensor cores (bf16, dk <= 128, dv <= 256); updates
    ``state`` in place.  Chunk ``c`` = tokens ``chunk_start[c] .. + chunk_len[c]``; portion ``s`` = chunks ``seq_chunk0[s]
    .. + seq_chunks[s]``."""
    a = mlstm_args(qkvg, gates, norm_w, out, state, pos, row, **kw)
    a.n_seq = seq_chunk0.shape[0]
    heads, dk, dv, n = kw["heads"], kw["dk"], kw["dv"], chunk_start.shape[0]
    c = _MlstmChunks()
    c.c_start, c.c_len, c.seq_chunk0, c.seq_chunks = (t.data_ptr() for t in (chunk_start, chunk_len, seq_chunk0, seq_chunks))
    at = ws.data_ptr()
    if ws.numel() < mlstm_chunk_ws_floats(n, heads, dk, dv):
        raise ValueError("mlstm_chunks: workspace too small")
    for name, floats in (("dS", dk * dv), ("s0", dk * dv), ("dn", dk), ("n0", dk), ("cg", 2), ("m0", 1)):
        setattr(c, name, at)
        at += 4 * n * heads * floats
    c.n_chunks, c.status = n, status_word(qkvg.device).data_ptr()
    _rc(lib().tahb_mlstm_chunks(ctypes.byref(a), ctypes.byref(c), c_int(qkvg.shape[0]), _stream()), "tahb_mlstm_chunks")
    return out


def mlstm_recurrent(qkvg, gates, norm_w, out, state, pos, row, **kw):
    """mLSTM token by token (the decode step; also any portion): updates ``state = (S, n, m)`` in place."""
    a = mlstm_args(qkvg, gates, norm_w, out, state, pos, row, **kw)
    _rc(lib().tahb_mlstm_recurrent(ctypes.byref(a), c_int(_act_f32(qkvg, out)), _stream()), "tahb_mlstm_recurrent")
    return out


class _Gla(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("qkvg", "low", "w2", "b2", "norm_w", "out", "S", "seq_start", "seq_len", "pos", "row",
                                        "slot")] + \
               [(n, c_int) for n in ("n_seq", "heads", "dk", "dv", "vdim", "rank")] + [("ld", c_ll), ("ld_out", c_ll)] + \
               [(n, c_float) for n in ("inv_tau", "eps", "q_scale")]


def _gla_args(qkvg, low, w2, b2, norm_w, out, state, pos, row, *, heads: int, dk: int, dv: int, dim: int, vdim: int, tau: float,
              eps: float, seq_start=None, seq_len=None, slot=None):
    a = _Gla()
    ptr = lambda t: 0 if t is None else t.data_ptr()
    for n, t in (("qkvg", qkvg), ("low", low), ("w2", w2), ("b2", b2), ("norm_w", norm_w), ("out", out), ("S", state[0]),
                 ("seq_start", seq_start), ("seq_len", seq_len), ("pos", pos), ("row", row), ("slot", slot)):
        setattr(a, n, ptr(t))
    if not low.is_contiguous() or low.shape[1] != w2.shape[1] or low.dtype != torch.float32:
        raise ValueError(f"gla: decay features {low.dtype} {tuple(low.shape)} for weights {tuple(w2.shape)}")
    a.n_seq = qkvg.shape[0] if seq_start is None else seq_start.shape[0]
    a.heads, a.dk, a.dv, a.vdim, a.rank, a.ld, a.ld_out = heads, dk, dv, vdim, w2.shape[1], qkvg.stride(0), out.stride(0)
    a.inv_tau, a.eps, a.q_scale = 1.0 / tau, eps, dim ** -0.5
    return a


class _GlaChunks(ctypes.Structure):
    _fields_ = [(n, c_void_p) for n in ("c_start", "c_len", "seq_chunk0", "seq_chunks", "G", "dS", "s0")] + \
               [("n_chunks", c_int), ("status", c_void_p)]


def gla_chunk_ws_floats(n_tokens: int, n_chunks: int, heads: int, dk: int, dv: int) -> int:
    """fp32 workspace of :func:`gla_chunks`: running log decays of the tokens, state sums, incoming states as bf16 pairs."""
    return n_tokens * heads * dk + n_chunks * heads * 2 * dk * dv


def gla_chunks(qkvg, low, w2, b2, norm_w, out, state, pos, row, *, chunk_start, chunk_len, seq_chunk0, seq_chunks, ws, **kw):
    """Gated linear attention of prompt portions in chunks of up to 128 tokens on the tensor cores (bf16, dk <= 128, dv <=
    256); updates ``state`` in place.  Chunks and portions as in :func:`mlstm_chunks`."""
    a = _gla_args(qkvg, low, w2, b2, norm_w, out, state, pos, row, **kw)
    a.n_seq = seq_chunk0.shape[0]
    heads, dk, dv, n, T = kw["heads"], kw["dk"], kw["dv"], chunk_start.shape[0], qkvg.shape[0]
    c = _GlaChunks()
    c.c_start, c.c_len, c.seq_chunk0, c.seq_chunks = (t.data_ptr() for t in (chunk_start, chunk_len, seq_chunk0, seq_chunks))
    if ws.numel() < gla_chunk_ws_floats(T, n, heads, dk, dv):
        raise ValueError("gla_chunks: workspace too small")
    at = ws.data_ptr()
    for name, floats in (("dS", n * heads * dk * dv), ("s0", n * heads * dk * dv), ("G", T * heads * dk)):
        setattr(c, name, at)
        at += 4 * floats
    c.n_chunks, c.status = n, status_word(qkvg.device).data_ptr()
    _rc(lib().tahb_gla_chunks(ctypes.byref(a), ctypes.byref(c), c_int(T), _stream()), "tahb_gla_chunks")
    return out


def gla_recurrent(qkvg, low, w2, b2, norm_w, out, state, pos, row, **kw):
    """Gated linear attention token by token (the decode step; also any portion): updates ``state = (S,)`` in place.
    ``low [n, rank]`` fp32 features, decay ``exp(logsigmoid(w2 low + b2) / tau)`` per key channel."""
    a = _gla_args(qkvg, low, w2, b2, norm_w, out, state, pos, row, **kw)
    _rc(lib().tahb_gla_recurrent(ctypes.byref(a), c_int(_act_f32(qkvg, w2, out)), _stream()), "tahb_gla_recurrent")
    return out


# -------------------------------------------------------------------------------------------
# attention
# -------------------------------------------------------------------------------------------
def decode_attn(q, caches: Sequence[torch.Tensor], page_tables: Sequence[torch.Tensor], lens: Sequence[torch.Tensor],
                depth, nq: int, nkv: int, hd: int, page_size: int, scale: float, out=None, n_split: int = 1,
                ws: Optional[torch.Tensor] = None):
    rows = q.shape[0]
    if out is None:
        out = torch.empty_like(q)
    n = len(caches)
    mp = (c_int * n)(*[pt.shape[1] for pt in page_tables])
    if n_split > 1 and ws is None:
        ws = torch.empty(int(lib().tahb_decode_attn_ws_floats(rows, nq, hd, n_split)), dtype=torch.float32, device=q.device)
    _rc(lib().tahb_decode_attn(_p(q), _p(out), _ptr_array(caches), _ptr_array(page_tables), _ptr_array(lens), mp,
                               c_int(n), _p(depth), c_int(rows), c_int(nq), c_int(nkv), c_int(hd), c_int(page_size),
                               c_float(scale), c_int(n_split), _p(ws), _p(status_word(q.device)), _stream()), "tahb_decode_attn")
    return out


def varlen_attn_naive(q, ks, vs, bases, counts, nq, nkv, hd, scale, out=None):
    """Packed duo-causal attention: query i attends rows ``bases[s][i] + j, j < counts[s][i]`` of the
    packed ``ks[s]``/``vs[s]`` for each of up to three segments ``s``."""
    if out is None:
        out = torch.empty_like(q)
    n = len(ks)
    _rc(lib().tahb_varlen_attn_naive(_p(q), _p(out), _ptr_array(ks), _ptr_array(vs), _ptr_array(bases),
                                     _ptr_array(counts), c_int(n), c_int(q.shape[0]), c_int(nq), c_int(nkv),
                                     c_int(hd), c_float(scale), _stream()), "tahb_varlen_attn_naive")
    return out


def attn_tiles(seq_counts: torch.Tensor, tile: int = 128):
    """Query tiles for :func:`prefill_attn`: every sequence's packed tokens (``seq_counts[b]`` of
    them, sequences laid out back to back) are cut into runs of at most ``tile`` tokens.  Returns
    int32 ``(tile_q0, tile_qn)``."""
    cnt = seq_counts.to(torch.int64)
    per = (cnt + tile - 1) // tile
    n_tiles = int(per.sum())
    dev = cnt.device
    seq_of = torch.repeat_interleave(torch.arange(cnt.numel(), device=dev), per, output_size=n_tiles)
    rank = torch.arange(n_tiles, device=dev) - (torch.cumsum(per, 0) - per)[seq_of]
    q0 = (torch.cumsum(cnt, 0) - cnt)[seq_of] + tile * rank
    qn = torch.clamp(cnt[seq_of] - tile * rank, max=tile)
    return q0.to(torch.int32).contiguous(), qn.to(torch.int32).contiguous()


def prefill_attn(q, ks, vs, bases, counts, tile_q0, tile_qn, nq, nkv, hd, scale, out=None, lse=None, bounds=None):
    """Packed duo-causal attention on the tensor cores (``csrc/attn_prefill.cu``).  The reference builds a
    dense additive mask ``(kv_pos <= q_pos) & (kv_iter <= q_iter) & kv_valid`` per pass (reference
    ``tah/model/tah_model.py:744-791``) and hands it to SDPA; here the same rule is the per-query prefix
    ``bases[s] .. bases[s] + counts[s]`` of every depth's K/V and no mask tensor exists.  Same contract as
    :func:`varlen_attn_naive` plus the query tiling of :func:`attn_tiles`: the tokens of a tile belong
    to one sequence and share ``bases[s]``.  ``counts[s]`` must be non-decreasing along a sequence's rows, or
    ``bounds[s]`` must give such a non-decreasing upper bound (rows whose count was zeroed, e.g. padding).  ``lse`` (optional fp32
    ``[n_q, nq]``) receives the base-2 log-sum-exp of the scaled scores, which the backward kernels take."""
    if out is None:
        out = torch.empty_like(q)
    n = len(ks)
    for t in (q, out, *ks, *vs):
        if t.dtype != torch.bfloat16 or not t.is_contiguous():
            raise ValueError("prefill_attn wants contiguous bf16 tensors")
    n_kv = (c_ll * n)(*[k.shape[0] for k in ks])
    _rc(lib().tahb_prefill_attn(_p(q), _p(out), _ptr_array(ks), _ptr_array(vs), n_kv, _ptr_array(bases),
                                _ptr_array(counts), _ptr_array(bounds if bounds is not None else counts), c_int(n), _p(tile_q0), _p(tile_qn), c_int(tile_q0.numel()),
                                c_ll(q.shape[0]), c_int(nq), c_int(nkv), c_int(hd), c_float(scale), _p(lse),
                                _p(status_word(q.device)), _stream()), "tahb_prefill_attn")
    return out


def attn_kv_items(seq_kv_counts: torch.Tensor, seq_kv_base: torch.Tensor, seq_q_counts: torch.Tensor, block: int = 128):
    """Work items of :func:`attn_bwd_dkv` for one KV segment: every sequence's ``seq_kv_counts[b]`` keys
    (stored from row ``seq_kv_base[b]`` of the segment's K/V matrices) are cut into blocks of ``block``.
    Returns int32 ``(row0, nkeys, kidx0, qa, qb)``; ``qa:qb`` are the sequence's packed query rows
    (sequences laid out back to back, ``seq_q_counts[b]`` rows each)."""
    cnt = seq_kv_counts.to(torch.int64)
    per = (cnt + block - 1) // block
    n = int(per.sum())
    dev = cnt.device
    seq_of = torch.repeat_interleave(torch.arange(cnt.numel(), device=dev), per, output_size=n)
    rank = torch.arange(n, device=dev) - (torch.cumsum(per, 0) - per)[seq_of]
    kidx0 = block * rank
    row0 = seq_kv_base.to(torch.int64)[seq_of] + kidx0
    nkeys = torch.clamp(cnt[seq_of] - kidx0, max=block)
    qc = seq_q_counts.to(torch.int64)
    qstart = torch.cumsum(qc, 0) - qc
    qa = qstart[seq_of]
    qb = qa + qc[seq_of]
    i32 = lambda t: t.to(torch.int32).contiguous()
    return i32(row0), i32(nkeys), i32(kidx0), i32(qa), i32(qb)


def attn_bwd_dq(q, dout, ks, vs, bases, counts, tile_q0, tile_qn, nq, nkv, hd, scale, lse, dsum, out=None,
                bounds=None):
    """dQ of :func:`prefill_attn` (``csrc/attn_prefill_bwd.cu``); ``dsum = rowsum(dO * O)`` per (query, head)."""
    if out is None:
        out = torch.empty_like(q)
    n = len(ks)
    n_kv = (c_ll * n)(*[k.shape[0] for k in ks])
    _rc(lib().tahb_attn_bwd_dq(_p(q), _p(dout), _p(out), _ptr_array(ks), _ptr_array(vs), n_kv, _ptr_array(bases),
                               _ptr_array(counts), _ptr_array(bounds if bounds is not None else counts), c_int(n), _p(tile_q0), _p(tile_qn), c_int(tile_q0.numel()),
                               c_ll(q.shape[0]), c_int(nq), c_int(nkv), c_int(hd), c_float(scale), _p(lse), _p(dsum),
                               _p(status_word(q.device)), _stream()), "tahb_attn_bwd_dq")
    return out


def attn_bwd_dkv(q, dout, k, v, count, items, nq, nkv, hd, scale, lse, dsum, dk=None, dv=None, bound=None):
    """dK, dV of one KV segment of :func:`prefill_attn`; ``items`` from :func:`attn_kv_items`, ``count`` the
    segment's visible-key counts per packed query.  Keys outside every item keep a zero gradient."""
    if dk is None:
        dk = torch.zeros_like(k)
    if dv is None:
        dv = torch.zeros_like(v)
    row0, nkeys, kidx0, qa, qb = items
    _rc(lib().tahb_attn_bwd_dkv(_p(q), _p(dout), _p(k), _p(v), _p(dk), _p(dv), c_ll(k.shape[0]), _p(count),
                                _p(bound if bound is not None else count), _p(row0),
                                _p(nkeys), _p(kidx0), _p(qa), _p(qb), c_int(row0.numel()), c_ll(q.shape[0]),
                                c_int(nq), c_int(nkv), c_int(hd), c_float(scale), _p(lse), _p(dsum),
                                _p(status_word(q.device)), _stream()), "tahb_attn_bwd_dkv")
    return dk, dv


# -------------------------------------------------------------------------------------------
# losses
# -------------------------------------------------------------------------------------------
def ce_fwd(logits: torch.Tensor, labels: torch.Tensor, ignore_index: int = -100):
    """Per-row cross entropy of bf16 ``logits [rows, V]`` in fp32 without an fp32 copy: returns ``(loss, lse)``."""
    _check_bf16_2d(logits, "logits")
    rows, V = logits.shape
    loss = torch.empty(rows, dtype=torch.float32, device=logits.device)
    lse = torch.empty(rows, dtype=torch.float32, device=logits.device)
    _rc(lib().tahb_ce_fwd(_p(logits), _p(labels), _p(loss), _p(lse), c_int(rows), c_int(V), c_ll(logits.stride(0)),
                          c_int(ignore_index), _stream()), "tahb_ce_fwd")
    return loss, lse


def ce_bwd(logits: torch.Tensor, labels: torch.Tensor, lse: torch.Tensor, gscale: torch.Tensor, ignore_index: int = -100):
    """``dlogits = (softmax(logits) - onehot(labels)) * gscale[0]`` in bf16 (zero rows where the label is ignored)."""
    rows, V = logits.shape
    d = torch.empty(rows, V, dtype=torch.bfloat16, device=logits.device)
    _rc(lib().tahb_ce_bwd(_p(logits), _p(labels), _p(lse), _p(gscale), _p(d), c_int(rows), c_int(V),
                          c_ll(logits.stride(0)), c_ll(d.stride(0)), c_int(ignore_index), _stream()), "tahb_ce_bwd")
    return d


def soft_embed_bwd(dout: torch.Tensor, val: torch.Tensor, idx: torch.Tensor, E: torch.Tensor, dE: torch.Tensor):
    """Backward of :func:`soft_embed_rows`: returns ``dval [rows, K]`` (fp32) and adds ``p_k * dout`` into the fp32
    accumulator ``dE [V, H]`` at the rows ``idx``."""
    rows, Kk = val.shape
    dval = torch.empty(rows, Kk, dtype=torch.float32, device=val.device)
    _rc(lib().tahb_soft_embed_bwd(_p(dout), _p(val), _p(idx), _p(E), _p(dval), _p(dE), c_int(rows), c_int(Kk),
                                  c_int(E.shape[1]), c_ll(dout.stride(0)), _stream()), "tahb_soft_embed_bwd")
    return dval


def bce_logits(z: torch.Tensor, labels: torch.Tensor, depth: int, pos_weight: float, thr: float, g=None):
    """Forward (``g`` None): fp32 ``[3]`` = (sum of BCE terms over labelled tokens, their count, correct threshold
    decisions).  Backward (``g`` = upstream gradient scalar tensor): ``dz``."""
    n = z.shape[0]
    if g is None:
        out = torch.zeros(3, dtype=torch.float32, device=z.device)
        _rc(lib().tahb_bce_logits(_p(z), _p(labels), c_int(depth), c_float(pos_weight), c_float(thr), c_int(n), _p(out),
                                  None, None, _stream()), "tahb_bce_logits")
        return out
    dz = torch.empty(n, dtype=torch.float32, device=z.device)
    _rc(lib().tahb_bce_logits(_p(z), _p(labels), c_int(depth), c_float(pos_weight), c_float(thr), c_int(n), None, _p(g),
                              _p(dz), _stream()), "tahb_bce_logits")
    return dz


# -------------------------------------------------------------------------------------------
# sampling / control
# -------------------------------------------------------------------------------------------
def topk_rows(x, k: int, flag=None, out_val=None, out_idx=None, ordered: bool = False):
    """Sorted top-``k`` (value desc, index asc) of every flagged bf16 row.  ``ordered=True`` forces
    the kernel's slower index-ordered path (its fallback for rows with > 1024 near-threshold ties)."""
    rows, V = x.shape
    if out_val is None:
        out_val = torch.zeros(rows, k, dtype=torch.float32, device=x.device)
    if out_idx is None:
        out_idx = torch.zeros(rows, k, dtype=torch.int32, device=x.device)
    fn = lib().tahb_topk_rows_ordered if ordered else lib().tahb_topk_rows
    _rc(fn(_p(x), _p(flag), _p(out_val), _p(out_idx), c_int(rows), c_int(V), c_int(k), c_ll(x.stride(0)), _stream()),
        "tahb_topk_rows")
    return out_val, out_idx


def soft_embed_rows(val, idx, E, flag=None, out=None):
    rows, K = val.shape
    H = E.shape[1]
    if out is None:
        out = torch.zeros(rows, H, dtype=E.dtype, device=E.device)
    _rc(lib().tahb_soft_embed_rows(_p(val), _p(idx), _p(flag), _p(E), _p(out), c_int(rows), c_int(K), c_int(H),
                                   c_ll(out.stride(0)), _stream()), "tahb_soft_embed_rows")
    return out


def sample_topk(val, idx, temperature: float, top_p: float, min_p: float, seed: int, step=None, out=None,
                seed_dev: Optional[torch.Tensor] = None):
    """Draw one token per row from a sorted top-k set.  ``seed_dev`` (optional int64 device scalar) is mixed
    into the seed on the device, so a captured launch can be replayed with a fresh seed."""
    rows, K = val.shape
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=val.device)
    _rc(lib().tahb_sample_topk(_p(val), _p(idx), _p(out), c_int(rows), c_int(K), c_float(temperature), c_float(top_p),
                               c_float(min_p), ctypes.c_ulonglong(seed & (2 ** 64 - 1)), _p(seed_dev), _p(step),
                               _stream()),
        "tahb_sample_topk")
    return out


def sample_full(x, temperature: float, top_k: int, top_p: float, min_p: float, seed: int, step=None, out=None,
                seed_dev: Optional[torch.Tensor] = None):
    """Draw one token per row of bf16 logits ``x [rows, V]`` over the whole vocabulary (temperature ->
    softmax -> min_p -> top_k -> top_p -> draw, reference ``tah/model/utils.py:84-125``); ``top_k <= 0``
    means no top-k filter.  Used where the sorted top-k route (``top_k <= 128``) does not apply."""
    _check_bf16_2d(x, "x")
    rows, V = x.shape
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=x.device)
    _rc(lib().tahb_sample_full(_p(x), _p(out), c_int(rows), c_int(V), c_ll(x.stride(0)), c_float(temperature),
                               c_int(top_k), c_float(top_p), c_float(min_p), ctypes.c_ulonglong(seed & (2 ** 64 - 1)),
                               _p(seed_dev), _p(step), _stream()), "tahb_sample_full")
    return out


def decider_head(h, w2, b2, out=None):
    """``z[r] = bf16(sum_j bf16(silu(h[r, j])) * w2[j] + b2)`` as fp32: the output layer of the two-layer
    decider MLP on the first layer's bf16 activations ``h`` (``[rows, inner]``)."""
    rows, inner = h.shape
    if out is None:
        out = torch.empty(rows, dtype=torch.float32, device=h.device)
    _rc(lib().tahb_decider_head(_p(h), _p(w2), _p(b2), _p(out), c_int(rows), c_int(inner), c_ll(h.stride(0)),
                                _stream()), "tahb_decider_head")
    return out


def decide(z, threshold: float, override, pos, depth, max_iter: int, need_soft):
    rows = need_soft.shape[0]
    _rc(lib().tahb_decide(_p(z), c_float(threshold), _p(override), c_int(override.shape[1] if override is not None else 0),
                          _p(pos), _p(depth), c_int(max_iter), _p(need_soft), c_int(rows), _stream()), "tahb_decide")
    return need_soft


def fused_reduce_residual_norm(partial_ptrs, xout_ptrs, mc_partial: int, mc_xout: int, h, ln_w, flag_ptrs, epoch,
                               M: int, H: int, rank: int, world: int, eps: float, add_residual: bool, grid: int):
    """Row-parallel epilogue over NVLink: all-reduce of the ranks' partial [M, H] results + residual
    add + RMSNorm + broadcast of the normalised rows, one launch per rank (see csrc/comm.cu)."""
    n = len(partial_ptrs)
    arr = lambda ptrs: (c_void_p * n)(*ptrs)
    _rc(lib().tahb_fused_reduce_residual_norm(arr(partial_ptrs), arr(xout_ptrs), c_void_p(mc_partial),
                                              c_void_p(mc_xout), _p(h), _p(ln_w), arr(flag_ptrs), _p(epoch),
                                              _p(status_word(h.device)), c_int(M), c_int(H), c_int(rank),
                                              c_int(world), c_float(eps), c_int(1 if add_residual else 0),
                                              c_int(grid), _stream()), "tahb_fused_reduce_residual_norm")


def push_reduce_norm_bcast(slot, cnt, cnt_target, xout_ptrs, mc_xout: int, xflag_ptrs, xtarget, arrive, h, ln_w,
                           M: int, H: int, rank: int, world: int, rpr: int, eps: float, add_residual: bool,
                           final_wait: bool, grid: int, tap_ptrs=None, mc_tap: int = 0, tap_ld: int = 0):
    """Owner side of the push-based row-parallel epilogue: sum the slots that the peers' GEMMs
    filled, residual add, RMSNorm, broadcast, flag (see ``push_reduce_norm_bcast_kernel``).  ``tap_ptrs``:
    every rank's address of the tap column that also receives the updated residual rows (row pitch ``tap_ld``)."""
    n = len(xout_ptrs)
    arr = lambda ptrs: (c_void_p * n)(*ptrs)
    _rc(lib().tahb_push_reduce_norm_bcast(_p(slot), _p(cnt), _p(cnt_target), arr(xout_ptrs), c_void_p(mc_xout),
                                          arr(xflag_ptrs), _p(xtarget), _p(arrive), _p(h), _p(ln_w),
                                          _p(status_word(h.device)), c_int(M), c_int(H), c_int(rank), c_int(world),
                                          c_int(rpr), c_float(eps), c_int(1 if add_residual else 0),
                                          c_int(1 if final_wait else 0), c_int(grid), _stream(),
                                          arr(tap_ptrs) if tap_ptrs else None, c_void_p(mc_tap if tap_ptrs else 0),
                                          c_ll(tap_ld if tap_ptrs else 0)),
        "tahb_push_reduce_norm_bcast")


def tp_topk_merge(xval_ptrs, xidx_ptrs, arrive_ptrs, epoch, vals, idx, out_val, out_idx, buf_rows: int, k: int, rank: int,
                  world: int, vocab_lo: int):
    """Exchange sorted per-shard top-``k`` candidates with the peers of a tensor-parallel group through
    symmetric memory and merge them (``tp_topk_merge_kernel``).  ``buf_rows``: the row capacity the exchange
    buffers were laid out for."""
    n = len(xval_ptrs)
    arr = lambda ptrs: (c_void_p * n)(*ptrs)
    rows = vals.shape[0]
    if rows != buf_rows:
        raise ValueError("tp_topk_merge: the exchange buffers are laid out for a fixed number of rows")
    _rc(lib().tahb_tp_topk_merge(arr(xval_ptrs), arr(xidx_ptrs), arr(arrive_ptrs), _p(epoch), _p(vals), _p(idx),
                                 _p(out_val), _p(out_idx), _p(status_word(vals.device)), c_int(rows), c_int(k),
                                 c_int(vals.stride(0)), c_int(out_idx.stride(0)), c_int(rank), c_int(world),
                                 c_int(vocab_lo), _stream()), "tahb_tp_topk_merge")


def shard_gather_push(shard, dst_ptrs, mc_dst: int, landed_ptrs, ready_ptrs, target, state, rank: int, world: int,
                      grid: int):
    """Store this rank's parameter shard into every rank's gather buffer and advance the landing flags
    (``shard_gather_push_kernel`` in ``csrc/comm.cu``); the consumer is :func:`gemm` with ``tp_wait``."""
    n = len(dst_ptrs)
    arr = lambda ptrs: (c_void_p * n)(*ptrs)
    _rc(lib().tahb_shard_gather_push(_p(shard), arr(dst_ptrs), c_void_p(mc_dst), arr(landed_ptrs), arr(ready_ptrs),
                                     _p(target), _p(state), c_ll(shard.numel() * shard.element_size()), c_int(rank),
                                     c_int(world), c_int(grid), _p(status_word(shard.device)), _stream()),
        "tahb_shard_gather_push")


class TickStateBinding:
    """Packs the scheduler state tensors into the pointer/int arrays the tick kernels take."""

    def __init__(self, tensors: List[Optional[torch.Tensor]], ints: List[int]):
        assert len(tensors) == 28 and len(ints) == 10
        self._keep = tensors
        self.ptrs = _ptr_array(tensors)
        self.ints = (c_int * len(ints))(*ints)

    def tick_begin(self, E, soft, x_in, rope_cs=None, hd: int = 0, theta: float = 0.0):
        """``rope_cs`` (optional ``[rows, hd]`` bf16): also write the RoPE cos | sin row of every row's position.
        ``E = None``: only the scheduler part (KV slots); the caller gathers the embeddings itself."""
        _rc(lib().tahb_tick_begin(self.ptrs, self.ints, _p(E), _p(soft), _p(x_in), c_int(0 if E is None else E.shape[1]), _p(rope_cs),
                                  c_int(hd), c_float(theta), _stream()), "tahb_tick_begin")

    def tick_end(self, need_soft, next_tok):
        _rc(lib().tahb_tick_end(self.ptrs, self.ints, _p(need_soft), _p(next_tok), _stream()), "tahb_tick_end")
