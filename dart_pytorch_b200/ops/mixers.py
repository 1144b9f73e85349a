"""Kernels of decoders with windowed attention, linear attention and a depth-averaged stream: allocation-explicit wrappers over
``csrc/{linear_attention,window_attention,branch_norm,attention_fwd,attention_decode}.cu``.

Everything here runs on a CUDA device in bfloat16 or float32 (true fp32 multiply-adds); there is no CPU form.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .. import _native as N
from .hybrid import _f32, _same

P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float


def _fields(*groups):
    return [(name, kind) for kind, names in groups for name in names.split()]


class LinearArgs(ctypes.Structure):
    _fields_ = _fields((P, "p w2 b2 decay log_a state o ws"), (L, "ld ws_floats"), (I, "oq ok ov orank"),
                       (I, "B S H dk dv rank silu f32 chunked segments"), (F, "q_scale inv_tau"))


class HeadNormArgs(ctypes.Structure):
    _fields_ = _fields((P, "o w g out"), (L, "ldg"), (I, "rows groups n sigmoid f32"), (F, "eps"))


class PrepArgs(ctypes.Structure):
    _fields_ = _fields((P, "p gq gk rot rot_v q k_ring v_ring k_lin v_lin k_pool v_pool pos_ptr"), (L, "ld"),
                       (I, "oq ok ov B S H G dk dv whole rot_dims ring lin_rows hist pos rot_rows pool pool_rows f32"),
                       (F, "eps"))


class PoolArgs(ctypes.Structure):
    _fields_ = _fields((P, "k v k_pool v_pool"), (L, "k_batch v_batch"), (I, "B nk nv ring lin0 pool pool_rows first count f32"))


class WindowArgs(ctypes.Structure):
    _fields_ = _fields((P, "q k v k_pool v_pool sink rot_v o pos_ptr"), (L, "k_batch v_batch"),
                       (I, "B S H G dk dv ring lin0 window pool pool_rows pos f32"), (F, "scale"))


class WindowFwdArgs(ctypes.Structure):
    _fields_ = _fields((P, "q k v k_pool v_pool sink rot o"), (I, "B S H G dk dv rows hist window pool pool_rows pos"),
                       (F, "scale"))


class WindowDecodeArgs(ctypes.Structure):
    _fields_ = _fields((P, "q k v k_pool v_pool sink rot o ws pos_ptr"), (L, "ws_floats"),
                       (I, "B S H G dk dv ring window pool pool_rows pos splits"), (F, "scale"))


class BranchArgs(ctypes.Structure):
    _fields_ = _fields((P, "x embed tokens m1 m2 w stack avg pick wf result x_out h"), (L, "stack_stride"),
                       (I, "rows D n vocab f32"), (F, "c1 c2 eps"))


_declared = False


def _lib():
    global _declared
    lib = N.load()
    if not _declared:
        for name, args in (("dptb_linear_attn", LinearArgs), ("dptb_head_norm_gate", HeadNormArgs), ("dptb_qkv_prep", PrepArgs),
                           ("dptb_pool_blocks", PoolArgs), ("dptb_window_attn", WindowArgs),
                           ("dptb_window_attn_fwd", WindowFwdArgs), ("dptb_window_attn_decode", WindowDecodeArgs),
                           ("dptb_branch_norm", BranchArgs)):
            getattr(lib, name).argtypes = [ctypes.POINTER(args), P]
        lib.dptb_linear_chunkable.argtypes = [I] * 3
        lib.dptb_linear_segments.argtypes = [I] * 5
        lib.dptb_linear_ws_floats.argtypes = [I] * 5
        lib.dptb_linear_ws_floats.restype = L
        lib.dptb_attn_decode_splits_hd.argtypes = [I] * 5
        lib.dptb_attn_decode_ws_floats.argtypes = [I] * 5
        lib.dptb_attn_decode_ws_floats.restype = L
        _declared = True
    return lib


def _call(name: str, args) -> None:
    N.check(getattr(_lib(), "dptb_" + name)(ctypes.byref(args), N.stream_ptr()), name)


def _rows(p: torch.Tensor, rows: int, cols: int, what: str) -> int:
    """Row stride of a projection's output ``[rows, >= cols]``."""
    if p.dim() != 2 or p.shape[0] != rows or p.shape[1] < cols or p.stride(1) != 1:
        raise ValueError(f"{what}: expected rows [{rows}, >= {cols}], got {list(p.shape)}")
    return p.stride(0) if rows > 1 else max(p.stride(0), p.shape[1])


# --------------------------------------------------------------------------- linear attention
CHUNK_ROWS = 16       # tokens per sequence from which the tensor-core form runs
MAX_CHUNK_RANK = 192  # of the low-rank decay in that form (shared memory of the kernel that sums the decays)


def linear_chunkable(dk: int, dv: int, f32: bool) -> bool:
    return bool(_lib().dptb_linear_chunkable(dk, dv, int(f32)))


def linear_attn(p: torch.Tensor, cols: dict, state: torch.Tensor, B: int, S: int, H: int, dk: int, dv: int, *,
                w2: Optional[torch.Tensor] = None, b2: Optional[torch.Tensor] = None, tau: float = 1.0,
                decay: Optional[torch.Tensor] = None, silu: bool = False, q_scale: float = 1.0,
                chunked: Optional[bool] = None, segments: Optional[int] = None) -> torch.Tensor:
    """``S_t = diag(a_t) S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t`` from ``state [B, H, dk, dv]`` (fp32, updated); returns
    ``[B*S, H*dv]``.  ``cols`` are the columns of ``q``, ``k``, ``v`` (and ``r``, the low-rank decay input) in ``p``.
    ``a = sigmoid(w2 r + b2)^(1/tau)`` per key channel, or ``decay [H, 2]`` (log a, a - 1) per head."""
    a = LinearArgs()
    f32 = _f32(p)
    ends = [cols["q"] + H * dk, cols["k"] + H * dk, cols["v"] + H * dv]
    if decay is None:
        a.rank = w2.shape[1]
        ends.append(cols["r"] + a.rank)
        a.w2, a.b2 = _same(w2, p.dtype, [H * dk, a.rank], "w2"), _same(b2, p.dtype, [H * dk], "b2")
        a.orank, a.inv_tau = cols["r"], 1.0 / tau
    else:
        a.decay = _same(decay, torch.float32, [H, 2], "decay")
    a.p, a.ld = p.data_ptr(), _rows(p, B * S, max(ends), "linear_attn")
    a.oq, a.ok, a.ov = cols["q"], cols["k"], cols["v"]
    a.state = _same(state, torch.float32, [B, H, dk, dv], "state")
    o = torch.empty(B * S, H * dv, dtype=p.dtype, device=p.device)
    a.o = o.data_ptr()
    a.B, a.S, a.H, a.dk, a.dv, a.silu, a.f32, a.q_scale = B, S, H, dk, dv, int(silu), f32, q_scale
    if chunked is None:
        chunked = S >= CHUNK_ROWS and linear_chunkable(dk, dv, bool(f32)) and a.ld % 8 == 0 and p.data_ptr() % 16 == 0 and \
            a.rank <= MAX_CHUNK_RANK and q_scale > 0.0
    a.chunked = int(chunked)
    if chunked:
        a.segments = _lib().dptb_linear_segments(B, S, H, dk, dv) if segments is None else segments
        a.ws_floats = _lib().dptb_linear_ws_floats(B, H, dk, dv, a.segments)
        keep = (torch.empty(a.ws_floats, dtype=torch.float32, device=p.device) if a.ws_floats else None,
                torch.empty(B * S, H * dk, dtype=torch.float32, device=p.device) if decay is None else None)
        a.ws, a.log_a = N.ptr(keep[0]), N.ptr(keep[1])
    _call("linear_attn", a)
    return o


def head_norm_gate(o: torch.Tensor, w: torch.Tensor, g: torch.Tensor, eps: float, gate: str) -> torch.Tensor:
    """``rms(o) * w * act(g)``: ``o [rows, groups * n]`` normalised over every group of ``n = len(w)`` features; ``act`` is
    ``silu`` or ``sigmoid``."""
    a = HeadNormArgs()
    rows, cols = o.shape
    a.n = w.numel()
    if cols % a.n:
        raise ValueError("head_norm_gate: the norm's size must divide the features")
    out = torch.empty_like(o)
    a.o, a.w, a.out = _same(o, w.dtype, [rows, cols], "o"), _same(w, w.dtype, [a.n], "w"), out.data_ptr()
    a.g, a.ldg = g.data_ptr(), _rows(g, rows, cols, "head_norm_gate")
    a.rows, a.groups, a.sigmoid, a.f32, a.eps = rows, cols // a.n, {"silu": 0, "sigmoid": 1}[gate], _f32(o), eps
    _call("head_norm_gate", a)
    return out


# --------------------------------------------------------------------------- windowed attention
def qkv_prep(p: torch.Tensor, cols: dict, B: int, S: int, H: int, G: int, dk: int, dv: int, *, eps: float, gq=None, gk=None,
             whole: bool, rot: Optional[torch.Tensor], rot_v: Optional[torch.Tensor], k_ring: torch.Tensor,
             v_ring: torch.Tensor, pos: int, pos_ptr: Optional[torch.Tensor] = None, k_lin=None, v_lin=None, hist: int = 0,
             k_pool=None, v_pool=None, pool: int = 0) -> torch.Tensor:
    """Norm and rotation of the projected queries, keys and values; returns ``q [B*S, H*dk]`` and writes the keys and values to
    the ring (and to row ``hist + s`` of the linear buffers).  With ``k_pool`` (one-token steps) the block that ended just
    before this token is pooled from the ring."""
    a = PrepArgs()
    dt = p.dtype
    a.p, a.ld = p.data_ptr(), _rows(p, B * S, max(cols["q"] + H * dk, cols["k"] + G * dk, cols["v"] + G * dv), "qkv_prep")
    a.oq, a.ok, a.ov = cols["q"], cols["k"], cols["v"]
    if gq is not None:
        a.gq = _same(gq, dt, [H * dk if whole else dk], "q norm")
        a.gk = _same(gk, dt, [G * dk if whole else dk], "k norm")
    n_rot = k_ring.shape[0]
    a.rot_rows = 1 << 30
    if rot is not None:
        a.rot_dims, a.rot_rows = 2 * rot.shape[1], rot.shape[0]
        a.rot = _same(rot, torch.float32, [a.rot_rows, a.rot_dims // 2, 2], "rot")
    if rot_v is not None:
        a.rot_rows = min(a.rot_rows, rot_v.shape[0])
        a.rot_v = _same(rot_v, torch.float32, [rot_v.shape[0], dv // 2, 2], "rot_v")
    if n_rot < B:
        raise ValueError("qkv_prep: the ring holds fewer sequences than the step")
    a.ring = k_ring.shape[1]
    a.k_ring = _same(k_ring, dt, [n_rot, a.ring, G * dk], "k ring")
    a.v_ring = _same(v_ring, dt, [n_rot, a.ring, G * dv], "v ring")
    if k_lin is not None:
        a.lin_rows, a.hist = k_lin.shape[1], hist
        a.k_lin = _same(k_lin, dt, [B, a.lin_rows, G * dk], "k_lin")
        a.v_lin = _same(v_lin, dt, [B, a.lin_rows, G * dv], "v_lin")
    if k_pool is not None:
        if S != 1:
            raise ValueError("qkv_prep: pools in one-token steps only")
        a.pool, a.pool_rows = pool, k_pool.shape[1]
        a.k_pool = _same(k_pool, dt, [n_rot, a.pool_rows, G * dk], "k_pool")
        a.v_pool = _same(v_pool, dt, [n_rot, a.pool_rows, G * dv], "v_pool")
    q = torch.empty(B * S, H * dk, dtype=dt, device=p.device)
    a.q, a.pos, a.pos_ptr = q.data_ptr(), pos, N.ptr(pos_ptr)
    a.B, a.S, a.H, a.G, a.dk, a.dv, a.whole, a.f32, a.eps = B, S, H, G, dk, dv, int(whole), _f32(p), eps
    _call("qkv_prep", a)
    return q


def pool_blocks(k: torch.Tensor, v: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, B: int, *, pool: int, first: int,
                count: int, ring: int = 0, lin0: int = 0) -> None:
    """Means of the blocks ``first .. first + count`` into ``k_pool`` / ``v_pool [B, rows, n]``; ``k``, ``v [B, rows, n]`` are a
    ring (``ring`` rows) or start at position ``lin0``."""
    if count <= 0:
        return
    a = PoolArgs()
    a.nk, a.nv, a.pool_rows = k.shape[2], v.shape[2], k_pool.shape[1]
    if (first + count) * pool - lin0 > k.shape[1] and not ring:
        raise ValueError("pool_blocks: blocks beyond the rows")
    a.k, a.v = _same(k, k.dtype, list(k.shape), "k"), _same(v, k.dtype, [k.shape[0], k.shape[1], a.nv], "v")
    a.k_pool = _same(k_pool, k.dtype, [k_pool.shape[0], a.pool_rows, a.nk], "k_pool")
    a.v_pool = _same(v_pool, k.dtype, [k_pool.shape[0], a.pool_rows, a.nv], "v_pool")
    if min(k.shape[0], k_pool.shape[0]) < B:
        raise ValueError("pool_blocks: fewer sequences than the step")
    a.k_batch, a.v_batch = k.stride(0), v.stride(0)
    a.B, a.ring, a.lin0, a.pool, a.first, a.count, a.f32 = B, ring, lin0, pool, first, count, _f32(k)
    _call("pool_blocks", a)


class WindowKeys:
    """What the queries of a windowed attention see: token rows ``[B, rows, n]`` (a ring when ``ring`` is set, otherwise
    starting at position ``lin0``), the window's size and the pooled rows before it."""

    __slots__ = ("k", "v", "window", "ring", "lin0", "pool", "k_pool", "v_pool")

    def __init__(self, k, v, window: int, ring: bool = False, lin0: int = 0, pool: int = 0, k_pool=None, v_pool=None):
        self.k, self.v, self.window, self.ring, self.lin0 = k, v, window, k.shape[1] if ring else 0, lin0
        self.pool, self.k_pool, self.v_pool = pool, k_pool, v_pool


def _window_args(a, q, keys: WindowKeys, B, S, H, G, dk, dv, pos, scale, sink, rot):
    dt, n = q.dtype, keys.k.shape[0]
    if n < B:
        raise ValueError("windowed attention: fewer cached sequences than the step brings")
    a.q = _same(q, dt, [B * S, H * dk], "q")
    a.k = _same(keys.k, dt, [n, keys.k.shape[1], G * dk], "k")
    a.v = _same(keys.v, dt, [n, keys.k.shape[1], G * dv], "v")
    if keys.pool:
        a.pool, a.pool_rows = keys.pool, keys.k_pool.shape[1]
        a.k_pool = _same(keys.k_pool, dt, [n, a.pool_rows, G * dk], "k_pool")
        a.v_pool = _same(keys.v_pool, dt, [n, a.pool_rows, G * dv], "v_pool")
    a.sink = _same(sink, dt, [H], "sink")
    if rot is not None:
        if rot.dtype != torch.float32 or rot.shape[1] != dv // 2 or not rot.is_contiguous() or rot.shape[0] < pos + S:
            raise ValueError("windowed attention: rotation table does not match")
    o = torch.empty(B * S, H * dv, dtype=dt, device=q.device)
    a.o, a.window, a.pos, a.scale = o.data_ptr(), keys.window, pos, scale
    a.B, a.S, a.H, a.G, a.dk, a.dv = B, S, H, G, dk, dv
    return o


def window_attn(q, keys: WindowKeys, B: int, S: int, H: int, G: int, dk: int, dv: int, pos: int, scale: float, *, sink=None,
                rot=None, pos_ptr: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Windowed attention, any dtype and size; ``q [B*S, H*dk]`` at positions ``pos ...``; returns ``[B*S, H*dv]``."""
    a = WindowArgs()
    o = _window_args(a, q, keys, B, S, H, G, dk, dv, pos, scale, sink, rot)
    if not keys.ring and (pos - keys.lin0 < min(pos, keys.window - 1) or pos + S - keys.lin0 > keys.k.shape[1]):
        raise ValueError("window_attn: the rows do not cover the window")
    a.k_batch, a.v_batch = keys.k.stride(0), keys.v.stride(0)
    a.ring, a.lin0, a.rot_v, a.pos_ptr, a.f32 = keys.ring, keys.lin0, N.ptr(rot), N.ptr(pos_ptr), _f32(q)
    _call("window_attn", a)
    return o


def window_flash_ok(dtype, dk: int, dv: int, scale: float) -> bool:
    return dtype == torch.bfloat16 and dk % 8 == 0 and dv % 8 == 0 and max(dk, dv) <= 128 and scale > 0


def window_attn_fwd(q, keys: WindowKeys, B: int, S: int, H: int, G: int, dk: int, dv: int, pos: int, scale: float, *, sink=None,
                    rot=None) -> torch.Tensor:
    """The same for long bf16 steps over linear rows (``[history | step]``) on the tensor cores."""
    a = WindowFwdArgs()
    o = _window_args(a, q, keys, B, S, H, G, dk, dv, pos, scale, sink, rot)
    if keys.ring or keys.k.shape[0] != B:
        raise ValueError("window_attn_fwd: takes linear rows")
    a.rows, a.hist, a.rot = keys.k.shape[1], pos - keys.lin0, N.ptr(rot)
    if a.hist < min(pos, keys.window - 1):
        raise ValueError("window_attn_fwd: the rows do not cover the window")
    _call("window_attn_fwd", a)
    return o


def window_decode_ok(dtype, H: int, G: int, dk: int, dv: int) -> bool:
    return dtype == torch.bfloat16 and dk % 8 == 0 and dv % 8 == 0 and max(dk, dv) <= 128 and H // G <= 8


def window_decode_plan(rows: int, H: int, G: int, dk: int, dv: int, max_keys: int):
    """(key slices, workspace floats) for ``rows`` queries over up to ``max_keys`` keys."""
    lib, hd = _lib(), 64 if max(dk, dv) <= 64 else 128
    s = lib.dptb_attn_decode_splits_hd(1, rows, G, max_keys, hd)
    return s, int(lib.dptb_attn_decode_ws_floats(1, rows, H, hd, s))


def window_attn_decode(q, keys: WindowKeys, B: int, S: int, H: int, G: int, dk: int, dv: int, pos: int, scale: float, *,
                       sink=None, rot=None, pos_ptr: Optional[torch.Tensor] = None, splits: int = 1,
                       ws: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The same for short bf16 steps straight from the ring."""
    a = WindowDecodeArgs()
    o = _window_args(a, q, keys, B, S, H, G, dk, dv, pos, scale, sink, rot)
    if not keys.ring:
        raise ValueError("window_attn_decode: takes a ring")
    a.ring, a.rot, a.pos_ptr = keys.ring, N.ptr(rot), N.ptr(pos_ptr)
    a.splits, a.ws, a.ws_floats = splits, N.ptr(ws), 0 if ws is None else ws.numel()
    _call("window_attn_decode", a)
    return o


# --------------------------------------------------------------------------- residual stream
def branch_norm(x: Optional[torch.Tensor], rows: int, D: int, dtype, eps: float, *, m1=None, m2=None, c1: float = 1.0,
                c2: float = 1.0, w=None, embed=None, tokens=None, stack: Optional[torch.Tensor] = None, n: int = 0, avg=None,
                pick: Optional[torch.Tensor] = None, wf=None, result: Optional[torch.Tensor] = None, x_out=None,
                h: bool = True) -> Optional[torch.Tensor]:
    """``x' = x + rms(c1 m1 + c2 m2) * w`` (``x`` fp32 or embedding rows), optionally averaged with the first ``n`` streams of
    ``stack [>= n, rows, D]`` by the weights ``avg [n + 1]``.  ``result`` receives ``x'``, ``x_out`` the average; returns it in
    ``dtype``, normed by ``wf`` if given (None with ``h=False``).  ``pick`` selects the output rows."""
    a = BranchArgs()
    src = x.shape[0] if x is not None else tokens.numel()
    if pick is None and src != rows:
        raise ValueError("branch_norm: wrong number of rows")
    dev = x.device if x is not None else tokens.device
    a.x = _same(x, torch.float32, [src, D], "x")
    if x is None:
        a.embed, a.vocab = _same(embed, dtype, [embed.shape[0], D], "embed"), embed.shape[0]
        a.tokens = _same(tokens, torch.int64, [src], "tokens")
    a.m1, a.m2 = _same(m1, dtype, [src, D], "m1"), _same(m2, dtype, [src, D], "m2")
    a.w, a.wf = _same(w, dtype, [D], "w"), _same(wf, dtype, [D], "wf")
    if avg is not None:
        if stack.shape[0] < n or list(stack.shape[1:]) != [src, D] or stack.dtype != torch.float32 or not stack.is_contiguous():
            raise ValueError("branch_norm: stack does not match")
        a.stack, a.avg, a.n, a.stack_stride = stack.data_ptr(), _same(avg, dtype, [n + 1], "avg"), n, src * D
    a.pick = _same(pick, torch.int32, [rows], "pick")
    a.result, a.x_out = _same(result, torch.float32, [rows, D], "result"), _same(x_out, torch.float32, [rows, D], "x_out")
    out = torch.empty(rows, D, dtype=dtype, device=dev) if h else None
    a.h = N.ptr(out)
    a.rows, a.D, a.c1, a.c2, a.eps, a.f32 = rows, D, c1, c2, eps, int(dtype == torch.float32)
    if not dev.type == "cuda":
        raise RuntimeError("these kernels run on a CUDA device only")
    _call("branch_norm", a)
    return out
