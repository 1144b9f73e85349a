"""Kernels of hybrid decoders (latent attention, gated linear recurrence, dropless experts, fp32 residual stream):
allocation-explicit wrappers over ``csrc/{gemm_grouped,latent_attention,recurrent,moe_local,stream_norm}.cu``.

Everything here runs on a CUDA device in bfloat16 or float32 (true fp32 multiply-adds); there is no CPU form.
"""
from __future__ import annotations

import ctypes
from typing import Optional, Sequence

import torch

from .. import _native as N

P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float


class GroupedSegArgs(ctypes.Structure):
    _fields_ = [("x", P), ("w", P), ("out", P), ("offsets", P), ("ldx", L), ("ldw", L), ("ldc", L), ("groups", I),
                ("N", I), ("K", I), ("M", I), ("x_cols", I), ("x_col_stride", I), ("out_col_stride", I), ("f32", I),
                ("act", I), ("out_f32", I), ("rows_hint", I)]


class LatentArgs(ctypes.Structure):
    _fields_ = [("d", P), ("gq", P), ("gc", P), ("cq", P), ("c_new", P), ("q", P), ("o", P), ("ws", P), ("cache", P), ("pos_ptr", P), ("ldd", L), ("ws_floats", L), ("B", I), ("S", I), ("H", I), ("Rq", I),
                ("R", I), ("cap", I), ("pos", I), ("splits", I), ("f32", I), ("force_simt", I),
                ("eps", F), ("scale", F)]


class RecurrentArgs(ctypes.Structure):
    _fields_ = [("x", P), ("taps", P), ("conv_bias", P), ("conv_state", P), ("u", P), ("z", P), ("br", P), ("bi", P),
                ("lam", P), ("y", P), ("state", P), ("out", P), ("agg", P), ("ldx", L), ("ldy", L), ("agg_floats", L),
                ("B", I), ("S", I), ("C", I), ("K", I), ("blocks", I), ("chunk", I), ("f32", I), ("c", F)]


class MoeArgs(ctypes.Structure):
    _fields_ = [("x", P), ("router", P), ("logits", P), ("idx", P), ("w", P), ("count", P), ("cursor", P),
                ("offsets", P), ("slot", P), ("xs", P), ("ldx", L), ("ld_logits", L), ("T", I), ("D", I), ("E", I),
                ("top", I), ("f32", I)]


class StreamArgs(ctypes.Structure):
    _fields_ = [("x", P), ("mix", P), ("shared", P), ("y", P), ("slot", P), ("w", P), ("embed", P), ("tokens", P),
                ("pick", P), ("g1", P), ("g2", P), ("shift", P), ("shift_state", P), ("x_out", P), ("h1", P), ("h2", P),
                ("rows", I), ("S", I), ("D", I), ("top", I), ("vocab", I), ("f32", I), ("eps", F)]


_declared = False


def _lib():
    global _declared
    lib = N.load()
    if not _declared:
        lib.dptb_gemm_grouped.argtypes = [ctypes.POINTER(GroupedSegArgs), I, I, P]
        lib.dptb_latent_norm_append.argtypes = [ctypes.POINTER(LatentArgs), P]
        lib.dptb_latent_attn.argtypes = [ctypes.POINTER(LatentArgs), P]
        lib.dptb_latent_attn_splits.argtypes = [I] * 5
        lib.dptb_latent_attn_ws_floats.argtypes = [I] * 4
        lib.dptb_latent_attn_ws_floats.restype = L
        lib.dptb_conv_state.argtypes = [ctypes.POINTER(RecurrentArgs), P]
        lib.dptb_lru_scan.argtypes = [ctypes.POINTER(RecurrentArgs), P]
        lib.dptb_moe_router.argtypes = [ctypes.POINTER(MoeArgs), P]
        lib.dptb_moe_place.argtypes = [ctypes.POINTER(MoeArgs), P]
        lib.dptb_stream_norm.argtypes = [ctypes.POINTER(StreamArgs), P]
        _declared = True
    return lib


def _f32(t: torch.Tensor) -> int:
    if not t.is_cuda:
        raise RuntimeError("these kernels run on a CUDA device only")
    return int(N.dtype_code(t) == 0)


def _same(t: Optional[torch.Tensor], dtype: torch.dtype, shape: Sequence[int], what: str) -> Optional[int]:
    """Pointer of a contiguous tensor after checking dtype and shape (None passes through)."""
    if t is None:
        return None
    if t.dtype != dtype or list(t.shape) != list(shape) or not t.is_contiguous():
        raise ValueError(f"{what}: expected a contiguous {dtype} tensor {list(shape)}, got {t.dtype} {list(t.shape)}")
    return t.data_ptr()


# --------------------------------------------------------------------------- grouped GEMM
def grouped_segment(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, groups: int, N_: int, K: int,
                    offsets: Optional[torch.Tensor] = None, x_col_stride: int = 0, out_col_stride: int = 0, act=None,
                    rows_hint: Optional[int] = None) -> GroupedSegArgs:
    """``out_g = act(x_g @ w_g^T)``; ``w [groups * N, K]``.  With ``offsets`` (int32, device, ``groups + 1``) group ``g``
    owns rows ``offsets[g] : offsets[g+1]`` of ``x``; without, all rows and its own column range of ``x`` and ``out``."""
    a = GroupedSegArgs()
    if x.dtype != w.dtype or x.stride(-1) != 1 or out.stride(-1) != 1 or not w.is_contiguous():
        raise ValueError("grouped_gemm: unsupported layout or mixed dtypes")
    if w.numel() != groups * N_ * K:
        raise ValueError("grouped_gemm: weight size does not match groups * N * K")
    M = x.shape[0]
    cols = N_ if offsets is not None else (groups - 1) * out_col_stride + N_
    if out.shape[0] < M or out.shape[1] < cols:
        raise ValueError("grouped_gemm: output too small")
    if offsets is not None and (offsets.dtype != torch.int32 or offsets.numel() != groups + 1):
        raise ValueError("grouped_gemm: offsets must be int32 [groups + 1]")
    if out.dtype not in (x.dtype, torch.float32):
        raise TypeError("grouped_gemm: output must have the input's dtype or be float32")
    a.x, a.w, a.out, a.offsets = x.data_ptr(), w.data_ptr(), out.data_ptr(), N.ptr(offsets)
    a.ldx, a.ldw, a.ldc = x.stride(0) if M > 1 else max(x.shape[1], x.stride(0)), K, out.stride(0)
    a.groups, a.N, a.K, a.M, a.x_cols = groups, N_, K, M, x.shape[1]
    a.x_col_stride, a.out_col_stride = x_col_stride, out_col_stride
    a.f32, a.act, a.out_f32 = _f32(x), {None: 0, "relu2": 1}[act], int(out.dtype == torch.float32)
    a.rows_hint = M if rows_hint is None else max(1, rows_hint)
    return a


def grouped_gemm(*segs: GroupedSegArgs, force_simt: bool = False) -> None:
    arr = (GroupedSegArgs * len(segs))(*segs)
    N.check(_lib().dptb_gemm_grouped(arr, len(segs), int(force_simt), N.stream_ptr()), "gemm_grouped")


# --------------------------------------------------------------------------- latent attention
def _latent_args(cache: torch.Tensor, B: int, S: int, pos: int, pos_ptr: Optional[torch.Tensor]) -> LatentArgs:
    a = LatentArgs()
    if cache.dim() != 3 or not cache.is_contiguous() or cache.shape[0] < B:
        raise ValueError("latent cache must be contiguous [B, capacity, R]")
    a.cache, a.B, a.S, a.R, a.cap = cache.data_ptr(), B, S, cache.shape[2], cache.shape[1]
    a.pos, a.pos_ptr, a.f32 = pos, N.ptr(pos_ptr), _f32(cache)
    return a


def latent_norm_append(d: torch.Tensor, gq, gc, cache, B: int, S: int, pos: int, eps: float,
                       pos_ptr: Optional[torch.Tensor] = None, dense: bool = False):
    """``d [B*S, Rq + R]``: RMS-normalise both parts; the query latent is returned ``[B*S, Rq]``, the key/value latent goes
    into ``cache[:, pos : pos + S]`` (and, with ``dense``, is returned as ``[B*S, R]`` as well)."""
    a = _latent_args(cache, B, S, pos, pos_ptr)
    a.Rq = gq.numel()
    if d.shape[0] != B * S or d.shape[1] != a.Rq + a.R or d.dtype != cache.dtype or d.stride(1) != 1:
        raise ValueError("latent_norm_append: projections do not match the norms and the cache")
    cq = torch.empty(B * S, a.Rq, dtype=d.dtype, device=d.device)
    c_new = torch.empty(B * S, a.R, dtype=d.dtype, device=d.device) if dense else None
    a.d, a.ldd, a.eps, a.cq, a.c_new = d.data_ptr(), d.stride(0), eps, cq.data_ptr(), N.ptr(c_new)
    a.gq, a.gc = _same(gq, d.dtype, [a.Rq], "gq"), _same(gc, d.dtype, [a.R], "gc")
    N.check(_lib().dptb_latent_norm_append(ctypes.byref(a), N.stream_ptr()), "latent_norm_append")
    return cq, c_new


def latent_attn_plan(rows: int, H: int, R: int, max_keys: int, f32: bool):
    """(key slices, workspace floats) for ``rows`` queries over up to ``max_keys`` cached tokens."""
    lib = _lib()
    s = lib.dptb_latent_attn_splits(rows, H, R, max_keys, int(f32))
    return s, int(lib.dptb_latent_attn_ws_floats(rows, H, R, s))


def latent_attn(q: torch.Tensor, cache: torch.Tensor, B: int, S: int, H: int, pos: int, scale: float,
                pos_ptr: Optional[torch.Tensor] = None, splits: int = 1, ws: Optional[torch.Tensor] = None,
                force_simt: bool = False) -> torch.Tensor:
    """Causal attention in latent space: ``q [B*S, H*R]`` against ``cache [B, cap, R]``, query ``s`` seeing the rows up to
    ``pos + s``; returns ``[B*S, H*R]``."""
    a = _latent_args(cache, B, S, pos, pos_ptr)
    out = torch.empty_like(q)
    a.q, a.o, a.H, a.scale = _same(q, cache.dtype, [B * S, H * a.R], "q"), out.data_ptr(), H, scale
    a.splits, a.ws, a.ws_floats = splits, N.ptr(ws), 0 if ws is None else ws.numel()
    a.force_simt = int(force_simt)
    N.check(_lib().dptb_latent_attn(ctypes.byref(a), N.stream_ptr()), "latent_attn")
    return out


# --------------------------------------------------------------------------- convolution + recurrence
def lru_chunk(S: int) -> int:
    """Tokens per chunk of the two-pass recurrence: about 0.7 sqrt(S), where the steps inside a chunk and the chunks to fold
    balance (measured between 512 and 8192 tokens)."""
    return 16 if S <= 1024 else 32 if S <= 4096 else 64 if S <= 32768 else 128


def conv_state(x: torch.Tensor, taps, bias, state: torch.Tensor, B: int, S: int, blocks: int) -> torch.Tensor:
    """Causal depthwise convolution over ``x [B*S, >= C]`` with ``state [B, K-1, C]`` (fp32, updated).  Returns
    ``[B*S, blocks, 2, C/blocks]`` (high and low bf16 parts) for bf16, ``[B*S, C]`` for fp32."""
    a = RecurrentArgs()
    C, K = taps.shape
    f32 = _f32(x)
    u = torch.empty((B * S, C) if f32 else (B * S, 2 * C), dtype=x.dtype, device=x.device)
    if x.shape[0] != B * S or x.shape[1] < C or x.stride(1) != 1:
        raise ValueError("conv_state: input does not match the taps")
    a.x, a.ldx, a.u = x.data_ptr(), x.stride(0) if B * S > 1 else max(x.stride(0), C), u.data_ptr()
    a.taps, a.conv_bias = _same(taps, x.dtype, [C, K], "taps"), _same(bias, x.dtype, [C], "bias")
    a.conv_state = _same(state, torch.float32, [B, K - 1, C], "conv state")
    a.B, a.S, a.C, a.K, a.blocks, a.f32 = B, S, C, K, blocks, f32
    N.check(_lib().dptb_conv_state(ctypes.byref(a), N.stream_ptr()), "conv_state")
    return u


def lru_scan(u, z, br, bi, lam, y, state, B: int, S: int, blocks: int, c: float,
             chunk: Optional[int] = None) -> torch.Tensor:
    """Gated linear recurrence from ``state [B, C]`` (fp32, updated) and its product with ``gelu_tanh(y)``; ``z`` holds the
    fp32 gate products ``[B*S, blocks, 2, C/blocks]`` and is used as scratch.  Returns ``[B*S, C]``."""
    a = RecurrentArgs()
    C = lam.numel()
    out = torch.empty(B * S, C, dtype=y.dtype, device=y.device)
    chunk = lru_chunk(S) if chunk is None else chunk
    chunks = (S + chunk - 1) // chunk
    agg = torch.empty(B * (chunks + 1) * 2 * C, dtype=torch.float32, device=y.device) if chunks > 1 else None
    f32 = _f32(y)
    if y.shape[0] != B * S or y.shape[1] < C or y.stride(1) != 1:
        raise ValueError("lru_scan: gate branch does not match")
    a.u = _same(u, y.dtype, [B * S, C if f32 else 2 * C], "u")
    a.z = _same(z, torch.float32, [B * S, 2 * C], "z")
    a.br, a.bi, a.lam = _same(br, y.dtype, [C], "br"), _same(bi, y.dtype, [C], "bi"), _same(lam, y.dtype, [C], "lam")
    a.y, a.ldy = y.data_ptr(), y.stride(0) if B * S > 1 else max(y.stride(0), C)
    a.state, a.out, a.agg = _same(state, torch.float32, [B, C], "state"), out.data_ptr(), N.ptr(agg)
    a.agg_floats = 0 if agg is None else agg.numel()
    a.B, a.S, a.C, a.K, a.blocks, a.chunk, a.f32, a.c = B, S, C, 1, blocks, chunk, f32, c
    N.check(_lib().dptb_lru_scan(ctypes.byref(a), N.stream_ptr()), "lru_scan")
    return out


# --------------------------------------------------------------------------- routing
ROUTER_KERNEL_ROWS = 64


def moe_route(x: torch.Tensor, router: torch.Tensor, top: int, counters: torch.Tensor):
    """Experts ``idx [T, top]`` with the largest ``router @ x`` and their softmax weights; counts go to ``counters[:E]``
    (zeroed by the caller)."""
    from . import kernels as K
    T, D = x.shape
    E = router.shape[0]
    a = MoeArgs()
    a.f32 = _f32(x)
    idx = torch.empty(T, top, dtype=torch.int32, device=x.device)
    w = torch.empty(T, top, dtype=torch.float32, device=x.device)
    a.x, a.ldx, a.router = _same(x, router.dtype, [T, D], "x"), D, _same(router, x.dtype, [E, D], "router")
    if (T > ROUTER_KERNEL_ROWS and not a.f32) or 4 * (D + E) > 48 * 1024:
        logits = torch.empty(T, E, dtype=torch.float32, device=x.device)
        if a.f32:
            K.gemm(x, router, logits, trans_b=True)
        else:       # few output features: narrow token tiles put the product on all SMs
            grouped_gemm(grouped_segment(x, router, logits, groups=1, N_=E, K=D, rows_hint=64))
        a.logits, a.ld_logits = logits.data_ptr(), E
    a.idx, a.w, a.count = idx.data_ptr(), w.data_ptr(), counters.data_ptr()
    a.T, a.D, a.E, a.top = T, D, E, top
    N.check(_lib().dptb_moe_router(ctypes.byref(a), N.stream_ptr()), "moe_router")
    return idx, w


def moe_place(x: torch.Tensor, idx: torch.Tensor, counters: torch.Tensor, E: int):
    """Rows of ``x`` in expert order ``[T*top, D]``, row offsets ``[E+1]`` and the slot of every choice ``[T, top]``.
    ``counters`` is the ``[2 * E]`` buffer whose first half ``moe_route`` filled (the second half must be zero)."""
    T, D = x.shape
    top = idx.shape[1]
    a = MoeArgs()
    xs = torch.empty(T * top, D, dtype=x.dtype, device=x.device)
    slot = torch.empty_like(idx)
    offsets = torch.empty(E + 1, dtype=torch.int32, device=x.device)
    a.x, a.ldx, a.f32 = _same(x, x.dtype, [T, D], "x"), D, _f32(x)
    a.idx, a.count, a.cursor = idx.data_ptr(), counters.data_ptr(), counters.data_ptr() + 4 * E
    a.offsets, a.slot, a.xs = offsets.data_ptr(), slot.data_ptr(), xs.data_ptr()
    a.T, a.D, a.E, a.top = T, D, E, top
    if counters.dtype != torch.int32 or counters.numel() < 2 * E:
        raise ValueError("moe_place: counters must be int32 [2 * experts]")
    N.check(_lib().dptb_moe_place(ctypes.byref(a), N.stream_ptr()), "moe_place")
    return xs, offsets, slot


# --------------------------------------------------------------------------- residual stream
class LayerTerms:
    """What a layer adds to the stream: its mixer's output, the shared expert's, and the routed experts' rows with the
    slot and weight of every (token, choice)."""

    __slots__ = ("mix", "shared", "y", "slot", "w")

    def __init__(self, mix=None, shared=None, y=None, slot=None, w=None):
        self.mix, self.shared, self.y, self.slot, self.w = mix, shared, y, slot, w


def stream_norm(x: Optional[torch.Tensor], terms: Optional[LayerTerms], rows: int, S: int, g1: torch.Tensor, eps: float, *,
                g2: Optional[torch.Tensor] = None, shift: Optional[torch.Tensor] = None,
                shift_state: Optional[torch.Tensor] = None, embed: Optional[torch.Tensor] = None,
                tokens: Optional[torch.Tensor] = None, pick: Optional[torch.Tensor] = None,
                keep: bool = True):
    """``(x', h1, h2)``: the stream after adding ``terms`` (and embedding rows), its norm with scale ``g1`` mixed with the
    previous token's by ``shift``, and its norm with scale ``g2``.  ``pick`` selects the output rows."""
    a = StreamArgs()
    dt = g1.dtype
    D = x.shape[1] if x is not None else embed.shape[1]
    dev = g1.device
    src = rows if pick is None else (x.shape[0] if x is not None else tokens.numel())
    a.f32 = _f32(g1)
    a.x = _same(x, torch.float32, [src, D], "x")
    if terms is not None:
        a.mix, a.shared = _same(terms.mix, dt, [src, D], "mix"), _same(terms.shared, dt, [src, D], "shared")
        if terms.y is not None:
            a.top = terms.slot.shape[1]
            a.y = terms.y.data_ptr()
            a.slot = _same(terms.slot, torch.int32, [src, a.top], "slot")
            a.w = _same(terms.w, torch.float32, [src, a.top], "w")
    if embed is not None:
        a.embed, a.vocab = _same(embed, dt, [embed.shape[0], D], "embed"), embed.shape[0]
        a.tokens = _same(tokens, torch.int64, [src], "tokens")
    a.pick = _same(pick, torch.int32, [rows], "pick")
    x_out = torch.empty(rows, D, dtype=torch.float32, device=dev) if keep else None
    h1 = torch.empty(rows, D, dtype=dt, device=dev)
    h2 = torch.empty(rows, D, dtype=dt, device=dev) if g2 is not None else None
    a.g1, a.g2 = g1.data_ptr(), N.ptr(g2)
    a.shift = _same(shift, dt, [D], "shift")
    if shift is not None:
        a.shift_state = _same(shift_state, torch.float32, [rows // S, D], "shift state")
    a.x_out, a.h1, a.h2 = N.ptr(x_out), h1.data_ptr(), N.ptr(h2)
    a.rows, a.S, a.D, a.eps = rows, S, D, eps
    N.check(_lib().dptb_stream_norm(ctypes.byref(a), N.stream_ptr()), "stream_norm")
    return x_out, h1, h2
