"""Mixers and a feed-forward of hybrid decoders on CUDA devices: windowed attention (sinks, pooled blocks before the window,
rotated values), linear attention with a decay (gated or constant), two mixers side by side, and the gated MLP.

Like the blocks of ``hybrid`` they take the rows of a whole step (``[B*S, D]``) and a ``StepContext``, and their ``new_state``
makes the part of a ``HybridCache`` that belongs to them: a ring of the window's keys and values with the pooled rows behind
it, or a matrix per head.  Inference only: the kernels have no backward.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Sequence, Tuple

import torch

from .. import ops as F
from .hybrid import StepContext, _full, _weight
from .layers import Linear
from .module import Module

SHORT_STEP = 32       # steps of up to this many tokens per sequence attend straight to the ring


def row_layout(**rows: int) -> Tuple[Dict[str, int], int]:
    """First row of every part of a fused projection, each at a multiple of 8 (16-byte aligned columns), and the total."""
    at, out = 0, {}
    for name, n in rows.items():
        out[name] = at
        at += (n + 7) // 8 * 8
    return out, at


class _Projected(Module):
    """A mixer that reads column ranges (``cols``) of one fused projection of its input.  ``own_input=False``: the projection
    belongs to a parent, which hands over this mixer's columns."""

    def _make_input(self, width: int, device, seed: int, dtype, init_std, bias: bool, own_input: bool) -> None:
        self.w_in = self.b_in = None
        if own_input:
            self.w_in = _weight(self.in_rows, width, seed, device, dtype, init_std)
            self.b_in = _full((self.in_rows,), 0.0, device, dtype) if bias else None

    def _input_parameters(self):
        return [t for t in (self.w_in, self.b_in) if t is not None]

    def forward(self, h: torch.Tensor, ctx: StepContext, state) -> torch.Tensor:
        return self.mix(F.linear(h, self.w_in, self.b_in), ctx, state)


# --------------------------------------------------------------------------------------------- rotary angles --
class RotaryTable:
    """Cosines and sines of ``position * f_i``, ``f_i = base^(-2i/dims)``, as ``[positions, dims/2, 2]`` (fp32, angles computed
    in fp64).  ``scaling`` divides low frequencies by ``factor``: those with a wavelength above ``original / low``, none below
    ``original / high``, a linear blend between the two."""

    _tables: Dict[tuple, torch.Tensor] = {}

    def __init__(self, base: float, dims: int, scaling: Optional[dict] = None):
        if dims % 2 or dims < 0:
            raise ValueError("RotaryTable: an even number of dimensions")
        self.base, self.dims = float(base), int(dims)
        self.scaling = None if not scaling else tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))

    def frequencies(self) -> torch.Tensor:
        f = self.base ** (-2.0 * torch.arange(self.dims // 2, dtype=torch.float64) / max(self.dims, 1))
        if self.scaling is None:
            return f
        factor, low, high, original = self.scaling
        turns = original * f / (2.0 * math.pi)            # over the original context
        keep = ((turns - low) / (high - low)).clamp(0.0, 1.0) if high != low else (turns > low).double()
        return (1.0 - keep) * f / factor + keep * f

    def rows(self, positions: int, device) -> torch.Tensor:
        """A table of at least ``positions`` rows; tables of one specification are shared."""
        key = (self.base, self.dims, self.scaling, str(torch.device(device)))
        got = self._tables.get(key)
        if got is None or got.shape[0] < positions:
            n = max(positions, 2 * (0 if got is None else got.shape[0]))
            a = torch.arange(n, dtype=torch.float64)[:, None] * self.frequencies()[None]
            got = self._tables[key] = torch.stack([a.cos(), a.sin()], -1).float().to(device).contiguous()
        return got


# --------------------------------------------------------------------------------------- windowed attention --
class WindowState:
    """Keys and values of one layer: rings ``[B, ring, n]`` (position ``p`` in row ``p % ring``) and, with pooling, one row for
    every block of ``pool`` tokens.  A ring outlasts the window by the longest step that reads it in place."""

    def __init__(self, nk: int, nv: int, window: int, pool: int, rotary: Optional[RotaryTable], rotary_v: Optional[RotaryTable]):
        self.nk, self.nv, self.window, self.pool = nk, nv, window, pool
        self.rotary, self.rotary_v = rotary, rotary_v
        self.ring = (max(window, pool) + SHORT_STEP + 7) // 8 * 8
        self.k = self.v = self.k_pool = self.v_pool = self.rot = self.rot_v = None

    def floats(self, batch: int) -> int:
        return 0

    def bind(self, flat: torch.Tensor, batch: int) -> None:
        pass

    def grow(self, batch: int, capacity: int, valid: int, dtype, device) -> None:
        if self.k is None:
            self.k = torch.zeros(batch, self.ring, self.nk, dtype=dtype, device=device)
            self.v = torch.zeros(batch, self.ring, self.nv, dtype=dtype, device=device)
        if self.pool:
            rows, old = max(1, capacity // self.pool), self.k_pool
            # zeros: rows that are not visible yet meet weights of zero
            new = [torch.zeros(batch, rows, n, dtype=dtype, device=device) for n in (self.nk, self.nv)]
            if old is not None and valid:
                new[0][:, :old.shape[1]] = old
                new[1][:, :old.shape[1]] = self.v_pool
            self.k_pool, self.v_pool = new
        if self.rotary is not None:
            self.rot = self.rotary.rows(capacity, device)
        if self.rotary_v is not None:
            self.rot_v = self.rotary_v.rows(capacity, device)

    def history(self, ring: torch.Tensor, B: int, pos: int, hist: int, S: int) -> torch.Tensor:
        """``[B, hist + S, n]`` whose first rows are the last ``hist`` positions before ``pos``."""
        out = torch.empty(B, hist + S, ring.shape[2], dtype=ring.dtype, device=ring.device)
        at, done = (pos - hist) % self.ring, 0
        while done < hist:
            n = min(hist - done, self.ring - at)
            out[:, done:done + n] = ring[:B, at:at + n]
            at, done = 0, done + n
        return out


class WindowAttention(_Projected):
    """Grouped-query attention over the last ``window`` tokens.

    * ``qk_norm``: RMS norm of queries and keys before the rotation, per ``"head"`` (one weight of ``dim``), over all heads
      ``"together"`` (a weight for every feature), or None.
    * ``rotary``: rotation of the first dimensions of queries and keys, pairs ``(2i, 2i + 1)``; ``rotary_v``: values are turned by
      their position over ``vdim`` and outputs back by the query's.
    * ``pool``: in front of the window one key and value per block of ``pool`` tokens, the mean of the cached ones, visible
      once the whole block has left the window.
    * ``sink``: ``exp(sink_h)`` joins the softmax's denominator."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int, scale: float, eps: float, *,
                 qk_norm: Optional[str] = None, rotary: Optional[RotaryTable] = None, rotary_v: Optional[RotaryTable] = None,
                 pool: int = 0, sink: bool = False, bias: bool = False, out_bias: bool = False, own_input: bool = True,
                 device=None, seed: int = 0, dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("WindowAttention: the query heads must share the key/value heads equally")
        if window < 1 or pool < 0:
            raise ValueError("WindowAttention: a window of at least one token")
        if rotary is not None and rotary.dims > dim:
            raise ValueError("WindowAttention: more rotated dimensions than a head has")
        if qk_norm not in (None, "head", "together"):
            raise ValueError(f"WindowAttention: unknown norm {qk_norm!r}")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.window, self.scale, self.eps, self.pool, self.qk_norm = window, float(scale), eps, pool, qk_norm
        self.rotary, self.rotary_v = rotary, rotary_v
        self.cols, self.in_rows = row_layout(q=heads * dim, k=kv_heads * dim, v=kv_heads * vdim)
        self._make_input(width, device, seed, dtype, init_std, bias, own_input)
        whole = qk_norm == "together"
        self.q_norm = _full((heads * dim if whole else dim,), 1.0, device, dtype) if qk_norm else None
        self.k_norm = _full((kv_heads * dim if whole else dim,), 1.0, device, dtype) if qk_norm else None
        self.sink = _full((heads,), 0.0, device, dtype) if sink else None
        self.wo = Linear(heads * vdim, width, bias=out_bias, device=device, seed=seed + 4, dtype=dtype, init_std=init_std)

    def own_parameters(self):
        return self._input_parameters() + [t for t in (self.q_norm, self.k_norm, self.sink) if t is not None]

    def submodules(self):
        return [self.wo]

    def new_state(self):
        return WindowState(self.kv_heads * self.dim, self.kv_heads * self.vdim, self.window, self.pool, self.rotary,
                           self.rotary_v)

    def mix(self, p: torch.Tensor, ctx: StepContext, state: WindowState) -> torch.Tensor:
        from ..ops import mixers as X
        B, S, P, pos = ctx.B, ctx.S, self.pool, ctx.pos
        sizes = (self.heads, self.kv_heads, self.dim, self.vdim)
        prep = dict(eps=self.eps, gq=self.q_norm, gk=self.k_norm, whole=self.qk_norm == "together", rot=state.rot,
                    rot_v=state.rot_v, k_ring=state.k, v_ring=state.v, pos=pos, pos_ptr=ctx.pos_ptr)
        attn = dict(sink=self.sink, rot=state.rot_v)
        # blocks this step completes, and the one that a one-token step before it may have left
        first = pos // P - (1 if pos and pos % P == 0 else 0) if P else 0
        count = (pos + S) // P - first if P else 0
        keys = dict(window=self.window, pool=P, k_pool=state.k_pool, v_pool=state.v_pool)
        if S <= SHORT_STEP:
            if S == 1 and P:
                prep.update(k_pool=state.k_pool, v_pool=state.v_pool, pool=P)
            q = X.qkv_prep(p, self.cols, B, S, *sizes, **prep)
            if S > 1 and P:
                X.pool_blocks(state.k, state.v, state.k_pool, state.v_pool, B, pool=P, first=first, count=count, ring=state.ring)
            keys = X.WindowKeys(state.k, state.v, ring=True, **keys)
            if X.window_decode_ok(p.dtype, *sizes):
                most = min(self.window, ctx.max_keys) + (ctx.max_keys // P if P else 0)
                splits, floats = X.window_decode_plan(B * S, *sizes, most)
                ws = ctx.cache.workspace(B * S, floats) if splits > 1 else None
                o = X.window_attn_decode(q, keys, B, S, *sizes, pos, self.scale, pos_ptr=ctx.pos_ptr, splits=splits, ws=ws,
                                         **attn)
            else:
                o = X.window_attn(q, keys, B, S, *sizes, pos, self.scale, pos_ptr=ctx.pos_ptr, **attn)
        else:
            hist = min(pos, max(self.window - 1, P))
            k, v = state.history(state.k, B, pos, hist, S), state.history(state.v, B, pos, hist, S)
            q = X.qkv_prep(p, self.cols, B, S, *sizes, k_lin=k, v_lin=v, hist=hist, **prep)
            if P:
                X.pool_blocks(k, v, state.k_pool, state.v_pool, B, pool=P, first=first, count=count, lin0=pos - hist)
            keys = X.WindowKeys(k, v, lin0=pos - hist, **keys)
            run = X.window_attn_fwd if X.window_flash_ok(p.dtype, self.dim, self.vdim, self.scale) else X.window_attn
            o = run(q, keys, B, S, *sizes, pos, self.scale, **attn)
        return F.linear(o, self.wo.weight, self.wo.bias)


# ------------------------------------------------------------------------------------------ linear attention --
class MatrixState:
    """One fp32 matrix ``[dk, dv]`` per sequence and head."""

    def __init__(self, heads: int, dk: int, dv: int):
        self.shape = (heads, dk, dv)
        self.s: Optional[torch.Tensor] = None

    def floats(self, batch: int) -> int:
        return batch * math.prod(self.shape)

    def bind(self, flat: torch.Tensor, batch: int) -> None:
        self.s = flat[:self.floats(batch)].view(batch, *self.shape)

    def grow(self, batch: int, capacity: int, valid: int, dtype, device) -> None:
        pass


class LinearAttention(_Projected):
    """Per head ``S_t = diag(a_t) S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t``; then ``Wo (rms(o) * w * act(Wg h))``.

    The decay is either one constant per head (``decay``) or, with ``rank``, one number per key channel and token:
    ``a = sigmoid(W2 W1 h + b)^(1/tau)``.  ``silu``: queries, keys and values pass through it.  The output norm covers every head
    by itself (one weight of ``vdim``) or, ``joint_norm``, all heads together; ``gate`` is ``"silu"`` or ``"sigmoid"``."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, eps: float, *, rank: int = 0, tau: float = 1.0,
                 decay: Optional[Sequence[float]] = None, q_scale: float = 1.0, silu: bool = False, joint_norm: bool = False,
                 gate: str = "silu", own_input: bool = True, device=None, seed: int = 0, dtype=torch.float32,
                 init_std: Optional[float] = None):
        super().__init__()
        if (decay is None) == (rank <= 0):
            raise ValueError("LinearAttention: either a rank for its decay or constant decays")
        if decay is not None and (len(decay) != heads or min(decay) <= 0.0 or max(decay) > 1.0):
            raise ValueError("LinearAttention: one decay in (0, 1] per head")
        self.width, self.heads, self.dim, self.vdim, self.eps = width, heads, dim, vdim, eps
        self.rank, self.tau, self.q_scale, self.silu, self.gate = rank, float(tau), float(q_scale), silu, gate
        parts = dict(q=heads * dim, k=heads * dim, v=heads * vdim, g=heads * vdim)
        if rank:
            parts["r"] = rank
        self.cols, self.in_rows = row_layout(**parts)
        self._make_input(width, device, seed, dtype, init_std, False, own_input)
        self.w2 = _weight(heads * dim, rank, seed + 1, device, dtype, init_std) if rank else None
        self.b2 = _full((heads * dim,), 4.0, device, dtype) if rank else None
        self._decay = None
        if decay is not None:
            d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
            self._decay = torch.stack([d.log(), d - 1.0], 1).float().to(device)
        self.norm = _full((heads * vdim if joint_norm else vdim,), 1.0, device, dtype)
        self.wo = Linear(heads * vdim, width, bias=False, device=device, seed=seed + 4, dtype=dtype, init_std=init_std)

    def own_parameters(self):
        return self._input_parameters() + [t for t in (self.w2, self.b2) if t is not None] + [self.norm]

    def submodules(self):
        return [self.wo]

    def _moved(self, device, dtype) -> None:
        if self._decay is not None and device is not None:
            self._decay = self._decay.to(device)

    def new_state(self):
        return MatrixState(self.heads, self.dim, self.vdim)

    def mix(self, p: torch.Tensor, ctx: StepContext, state: MatrixState) -> torch.Tensor:
        from ..ops import mixers as X
        o = X.linear_attn(p, self.cols, state.s, ctx.B, ctx.S, self.heads, self.dim, self.vdim, w2=self.w2, b2=self.b2,
                          tau=self.tau, decay=self._decay, silu=self.silu, q_scale=self.q_scale)
        g = p[:, self.cols["g"]:self.cols["g"] + self.heads * self.vdim]
        return F.linear(X.head_norm_gate(o, self.norm, g, self.eps, self.gate), self.wo.weight)


# ------------------------------------------------------------------------------------------- side by side --
class PairState:
    """The states of two mixers of one layer."""

    def __init__(self, left, right):
        self.left, self.right = left, right

    def floats(self, batch: int) -> int:
        return (self.left.floats(batch) + 3) // 4 * 4 + self.right.floats(batch)      # 16-byte aligned parts

    def bind(self, flat: torch.Tensor, batch: int) -> None:
        self.left.bind(flat, batch)
        self.right.bind(flat[(self.left.floats(batch) + 3) // 4 * 4:], batch)

    def grow(self, batch: int, capacity: int, valid: int, dtype, device) -> None:
        self.left.grow(batch, capacity, valid, dtype, device)
        self.right.grow(batch, capacity, valid, dtype, device)


class SideBySide(_Projected):
    """Two mixers (built with ``own_input=False``) that read the same input through one projection; returns both results, to be
    added with ``scales`` by whoever normalises the sum."""

    def __init__(self, width: int, left, right, scales: Tuple[float, float], bias: bool = False, device=None, seed: int = 0,
                 dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        self.left, self.right, self.scales = left, right, (float(scales[0]), float(scales[1]))
        self.in_rows = left.in_rows + right.in_rows
        self._make_input(width, device, seed, dtype, init_std, bias, True)

    def own_parameters(self):
        return self._input_parameters()

    def submodules(self):
        return [self.left, self.right]

    def new_state(self):
        return PairState(self.left.new_state(), self.right.new_state())

    def mix(self, p: torch.Tensor, ctx: StepContext, state: PairState):
        n = self.left.in_rows
        return self.left.mix(p[:, :n], ctx, state.left), self.right.mix(p[:, n:], ctx, state.right)


# ------------------------------------------------------------------------------------------- feed-forward --
class GatedMLP(Module):
    """``Wdown (gelu_tanh(Wgate h) * Wup h)``; gate and up are one product."""

    def __init__(self, width: int, ff: int, device=None, seed: int = 0, dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        self.width, self.ff = width, ff
        self.cols, rows = row_layout(gate=ff, up=ff)
        self.w_in = _weight(rows, width, seed, device, dtype, init_std)
        self.down = Linear(ff, width, bias=False, device=device, seed=seed + 1, dtype=dtype, init_std=init_std)

    def own_parameters(self):
        return [self.w_in]

    def submodules(self):
        return [self.down]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        from ..ops import kernels as K
        gu, up = F.linear(h, self.w_in), self.cols["up"]
        return F.linear(K.geglu_fwd(gu[:, :self.ff], gu[:, up:up + self.ff]), self.down.weight)
