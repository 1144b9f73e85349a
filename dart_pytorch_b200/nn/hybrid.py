"""Building blocks of hybrid decoders on CUDA devices: one-number RMS norm, token shift, latent attention, gated linear
recurrence, dropless top-k experts, and the state cache they share.

The mixers take the normalised rows of a whole step (``[B*S, D]``) and a ``StepContext``; every sequence of the batch
brings the same number of tokens and stands at the same position.  A mixer's part of a sequence's state is created by its
``new_state`` and lives in a ``HybridCache``: latent rows (appended) or convolution inputs and recurrent state (replaced,
fp32), so a step never recomputes earlier tokens.  Inference only: the kernels have no backward.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from .. import ops as F
from .layers import Linear
from .module import Module, make_param, normal_, uniform_


def _weight(rows: int, cols: int, seed: int, device, dtype, init_std):
    t = uniform_((rows, cols), 1.0 / math.sqrt(cols), seed, device, dtype) if init_std is None else \
        normal_((rows, cols), init_std, seed, device, dtype)
    return make_param(t)


def _full(shape, value: float, device, dtype):
    return make_param(torch.full(shape, value, dtype=torch.float32).to(device=device, dtype=dtype))


# ------------------------------------------------------------------------------------------------- state --
class LatentState:
    """Latent rows ``[B, capacity, R]`` of one layer run."""

    def __init__(self, rank: int):
        self.rank = rank
        self.buf: Optional[torch.Tensor] = None

    def floats(self, batch: int) -> int:
        return 0

    def bind(self, flat: torch.Tensor, batch: int) -> None:
        pass

    def grow(self, batch: int, capacity: int, valid: int, dtype, device) -> None:
        new = torch.zeros(batch, capacity, self.rank, dtype=dtype, device=device)
        if self.buf is not None and valid:
            new[:, :valid] = self.buf[:, :valid]
        self.buf = new


class RecurrentState:
    """Convolution inputs ``[B, K-1, C]`` and recurrent state ``[B, C]`` of one layer run, fp32."""

    def __init__(self, channels: int, taps: int):
        self.channels, self.taps = channels, taps
        self.conv: Optional[torch.Tensor] = None
        self.s: Optional[torch.Tensor] = None

    def floats(self, batch: int) -> int:
        return batch * self.channels * self.taps          # (taps - 1) inputs and the state

    def bind(self, flat: torch.Tensor, batch: int) -> None:
        n = batch * (self.taps - 1) * self.channels
        self.conv = flat[:n].view(batch, self.taps - 1, self.channels)
        self.s = flat[n:n + batch * self.channels].view(batch, self.channels)

    def grow(self, batch: int, capacity: int, valid: int, dtype, device) -> None:
        pass


class HybridCache:
    """State of ``batch`` sequences over all layer runs of a model (a layer that runs several times has one state per run).

    ``seq_len`` tokens have been processed; ``pos`` is the same number on the device, where the kernels of a captured decode
    step read it.  ``width`` is the size of the row every layer run keeps for a token shift (0: none).  Fixed-size state sits
    in one flat fp32 buffer, so that a reset is one fill.  What grows with the sequence (latents, pooled blocks, rotary tables)
    doubles when a step needs more than the capacity."""

    def __init__(self, states: List[object], width: int, batch: int, max_len: int, dtype, device, counters: int = 0):
        self.states, self.batch, self.dtype, self.device = states, batch, dtype, torch.device(device)
        self.seq_len = 0
        self.pos = torch.zeros(1, dtype=torch.int32, device=device)
        sizes = [batch * width + s.floats(batch) for s in states]
        sizes = [(n + 3) // 4 * 4 for n in sizes]         # 16-byte aligned parts
        self.flat = torch.zeros(max(1, sum(sizes)), dtype=torch.float32, device=device)
        self.shift: List[torch.Tensor] = []
        off = 0
        for s, n in zip(states, sizes):
            # the shift state comes first: it is read in 16-byte vectors
            self.shift.append(self.flat[off:off + batch * width].view(batch, width))
            s.bind(self.flat[off + batch * width:off + n], batch)
            off += n
        # per layer run: rows per expert and places handed out, zeroed at the start of a step
        self.counters = torch.zeros(max(1, len(states)), max(1, counters), dtype=torch.int32, device=device)
        self.capacity = 0
        self.plan: Dict[int, torch.Tensor] = {}           # attention workspace by rows of a step
        self.graph = None
        self.ensure(max(1, max_len))

    def ensure(self, need: int) -> None:
        """Room for ``need`` tokens.  New buffers invalidate a captured decode step."""
        if need <= self.capacity:
            return
        cap = (max(need, 2 * self.capacity) + 127) // 128 * 128
        for s in self.states:
            s.grow(self.batch, cap, self.seq_len, self.dtype, self.device)
        self.capacity = cap
        self.plan.clear()
        self.graph = None

    def attn_workspace(self, rows: int, H: int, R: int, max_keys: int):
        """(slices, workspace) of the latent attention kernel; all layers share one workspace."""
        from ..ops import hybrid as Y
        splits, floats = Y.latent_attn_plan(rows, H, R, max_keys, self.dtype == torch.float32)
        return (1, None) if splits <= 1 else (splits, self.workspace(rows, floats))

    def workspace(self, rows: int, floats: int) -> torch.Tensor:
        """fp32 scratch of an attention kernel for steps of ``rows`` rows, shared by all layers."""
        got = self.plan.get(rows)
        if got is None or got.numel() < floats:
            got = self.plan[rows] = torch.empty(floats, dtype=torch.float32, device=self.device)
        return got

    def advance(self, n: int) -> None:
        self.seq_len += n
        self.pos.fill_(self.seq_len)

    def reset(self) -> None:
        """Forget the sequences.  Latent rows need no clearing: positions at or beyond ``seq_len`` are never read."""
        self.flat.zero_()
        self.seq_len = 0
        self.pos.zero_()


class CachePool:
    """Caches of finished requests, handed out again (with their captured decode step) to new ones of the same batch."""

    def __init__(self, make, keep: int = 8):
        self._make, self._keep = make, keep
        self._free: List[HybridCache] = []

    def acquire(self, batch: int, max_len: int) -> HybridCache:
        fits = [c for c in self._free if c.batch == batch and c.capacity >= max_len]
        if fits:
            cache = min(fits, key=lambda c: c.capacity)
            self._free.remove(cache)
            cache.reset()
            return cache
        return self._make(batch, max_len)

    def release(self, cache: HybridCache) -> None:
        if cache not in self._free:
            self._free.append(cache)
        if len(self._free) > self._keep:
            self._free.pop(0)

    def clear(self) -> None:
        self._free.clear()


@dataclass
class StepContext:
    """One step: ``S`` new tokens for each of ``B`` sequences whose first stands at position ``pos``.  ``pos_ptr`` is set
    where the position has to come from the device (a decode step that is captured once and replayed)."""
    cache: HybridCache
    B: int
    S: int
    pos: int
    pos_ptr: Optional[torch.Tensor] = None

    @property
    def max_keys(self) -> int:
        return self.cache.capacity if self.pos_ptr is not None else self.pos + self.S


# ---------------------------------------------------------------------------------------------- small parts --
class ScalarRMSNorm(Module):
    """``x / sqrt(mean(x^2) + eps) * g`` with one number ``g`` for all features."""

    def __init__(self, eps: float, device=None, dtype=torch.float32):
        super().__init__()
        self.eps = eps
        self.gamma = _full((1,), 1.0, device, dtype)

    def own_parameters(self):
        return [self.gamma]


class TokenShift(Module):
    """``n_t + (n_{t-1} - n_t) * mu``, feature by feature; ``n_{-1} = 0``."""

    def __init__(self, dim: int, device=None, dtype=torch.float32, init: float = 0.5):
        super().__init__()
        self.mu = _full((dim,), init, device, dtype)

    def own_parameters(self):
        return [self.mu]


class _Packed(Module):
    """Modules that keep rearranged copies of their weights for the kernels, rebuilt when the weights change."""

    def __init__(self):
        super().__init__()
        self._pack = None

    def packed(self):
        key = tuple((p.data_ptr(), p._version, p.dtype) for p in self.parameters())
        if self._pack is None or self._pack[0] != key:
            with torch.no_grad():
                self._pack = (key, self._build_pack())
        return self._pack[1]

    def _build_pack(self):
        raise NotImplementedError

    def _moved(self, device, dtype):
        self._pack = None


# ------------------------------------------------------------------------------------------ latent attention --
EXPAND_ROWS = 32      # tokens per sequence from which keys and values are expanded for the flash kernel


class LatentAttention(_Packed):
    """Attention whose keys and values are linear maps of one cached latent per token, without positions.

    Queries: ``q = Wuq rms(Wdq h)``.  Latent: ``c = rms(Wdkv h)``; per head ``k = Wuk c`` and ``v = Wuv c``, scores
    ``scale * q . k``, causal softmax, ``Wo`` over the concatenated heads.  Storage: ``w_down = [Wdq; Wdkv]`` is one product.

    Short steps and fp32 run in latent space (``Wuk`` is applied to the queries, ``Wuv`` to the weighted latent).  Prompts in
    bf16 expand the cached latents to keys and values and run the flash kernel, heads zero-padded to its sizes."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, eps: float,
                 device=None, seed: int = 0, dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        self.width, self.heads, self.dim, self.vdim = width, heads, dim, vdim
        self.q_rank, self.kv_rank, self.scale, self.eps = q_rank, kv_rank, float(scale), eps
        mk = lambda r, c, s: _weight(r, c, seed + s, device, dtype, init_std)  # noqa: E731
        self.w_down = mk(q_rank + kv_rank, width, 0)
        self.q_norm, self.kv_norm = _full((q_rank,), 1.0, device, dtype), _full((kv_rank,), 1.0, device, dtype)
        self.w_uq = mk(heads * dim, q_rank, 1)
        self.w_uk = mk(heads * dim, kv_rank, 2)
        self.w_uv = mk(heads * vdim, kv_rank, 3)
        self.wo = Linear(heads * vdim, width, bias=False, device=device, seed=seed + 4, dtype=dtype, init_std=init_std)

    def own_parameters(self):
        return [self.w_down, self.q_norm, self.kv_norm, self.w_uq, self.w_uk, self.w_uv]

    def submodules(self):
        return [self.wo]

    def new_state(self):
        return LatentState(self.kv_rank)

    def _build_pack(self):
        from ..ops import flash
        H, dk, dv, R = self.heads, self.dim, self.vdim, self.kv_rank
        uk = self.w_uk.detach()
        pack = {"uk_t": uk.view(H, dk, R).transpose(1, 2).contiguous().view(H * R, dk)}
        pd = flash.kernel_head_dim((max(dk, dv) + 7) // 8 * 8) if uk.dtype == torch.bfloat16 else None
        pack["pd"] = pd
        if pd is not None:
            def heads_to(w, d):       # rows of every head zero-padded to pd
                return w if d == pd else torch.nn.functional.pad(w.view(H, d, -1), (0, 0, 0, pd - d)).reshape(H * pd, -1)
            pack["uq"] = heads_to(self.w_uq.detach(), dk).contiguous()
            pack["ukv"] = torch.cat([heads_to(uk, dk), heads_to(self.w_uv.detach(), dv)], 0).contiguous()
            wo = self.wo.weight.detach()
            pack["wo"] = wo if dv == pd else \
                torch.nn.functional.pad(wo.view(-1, H, dv), (0, pd - dv)).reshape(-1, H * pd).contiguous()
        return pack

    def forward(self, h: torch.Tensor, ctx: StepContext, state: LatentState) -> torch.Tensor:
        from ..ops import hybrid as Y
        B, S = ctx.B, ctx.S
        pack = self.packed()
        expand = pack["pd"] is not None and S >= EXPAND_ROWS
        cq, dense = Y.latent_norm_append(F.linear(h, self.w_down), self.q_norm, self.kv_norm, state.buf, B, S, ctx.pos,
                                         self.eps, pos_ptr=ctx.pos_ptr, dense=expand and ctx.pos == 0 and B > 1)
        return self._expanded(cq, dense, ctx, state, pack) if expand else self._in_latent_space(cq, ctx, state, pack)

    def _in_latent_space(self, cq, ctx: StepContext, state: LatentState, pack) -> torch.Tensor:
        from ..ops import hybrid as Y
        H, dk, dv, R = self.heads, self.dim, self.vdim, self.kv_rank
        M = ctx.B * ctx.S
        q = F.linear(cq, self.w_uq)
        ql = torch.empty(M, H * R, dtype=q.dtype, device=q.device)
        Y.grouped_gemm(Y.grouped_segment(q, pack["uk_t"], ql, groups=H, N_=R, K=dk, x_col_stride=dk, out_col_stride=R))
        splits, ws = ctx.cache.attn_workspace(M, H, R, ctx.max_keys)
        ol = Y.latent_attn(ql, state.buf, ctx.B, ctx.S, H, ctx.pos, self.scale, pos_ptr=ctx.pos_ptr, splits=splits, ws=ws)
        o = torch.empty(M, H * dv, dtype=q.dtype, device=q.device)
        Y.grouped_gemm(Y.grouped_segment(ol, self.w_uv.detach(), o, groups=H, N_=dv, K=R, x_col_stride=R,
                                         out_col_stride=dv))
        return F.linear(o, self.wo.weight)

    def _expanded(self, cq, dense, ctx: StepContext, state: LatentState, pack) -> torch.Tensor:
        from ..ops import flash
        H, pd, B, S = self.heads, pack["pd"], ctx.B, ctx.S
        n = ctx.pos + S
        q = F.linear(cq, pack["uq"])
        if dense is not None:                       # a batch of whole prompts: the step's latents are all there is
            kv = F.linear(dense, pack["ukv"])
        elif B == 1:
            kv = F.linear(state.buf[0, :n], pack["ukv"])
        else:
            kv = torch.cat([F.linear(state.buf[b, :n], pack["ukv"]) for b in range(B)], 0)
        o, _ = flash.attn_fwd(q, kv[:, :H * pd], kv[:, H * pd:], B, S, n, H, H, pd, True, q_offset=ctx.pos,
                              scale=self.scale, need_lse=False, precise=True)
        return F.linear(o, pack["wo"])


# ---------------------------------------------------------------------------------- gated linear recurrence --
class GatedLinearRecurrence(_Packed):
    """Recurrent block: ``y = gelu_tanh(Wy h + by)``, ``u = conv(Wx h + bx)`` (causal, per channel, no activation), gates
    ``r, i = sigmoid(block-diagonal products of u + bias)``, ``log a = -decay * r * softplus(lam)``,
    ``S_t = a S_{t-1} + sqrt(1 - a^2) i u``, output ``Wo (S * y)``.  ``w_yx = [Wy; Wx]`` is one product."""

    def __init__(self, width: int, channels: int, blocks: int, taps: int, decay: float = 8.0, device=None, seed: int = 0,
                 dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        if channels % blocks:
            raise ValueError("GatedLinearRecurrence: channels must divide into equal blocks")
        if not 1 <= taps <= 16:
            raise ValueError("GatedLinearRecurrence: between 1 and 16 convolution taps")
        self.width, self.channels, self.blocks, self.taps, self.decay = width, channels, blocks, taps, float(decay)
        n = channels // blocks
        mk = lambda r, c, s: _weight(r, c, seed + s, device, dtype, init_std)  # noqa: E731
        zeros = lambda *shape: _full(shape, 0.0, device, dtype)  # noqa: E731
        self.w_yx, self.b_yx = mk(2 * channels, width, 0), zeros(2 * channels)
        self.conv_w, self.conv_b = mk(channels, taps, 1), zeros(channels)
        self.w_r, self.b_r = mk(channels, n, 2), zeros(channels)        # [blocks * n, n]: block g owns rows g*n .. g*n+n
        self.w_i, self.b_i = mk(channels, n, 3), zeros(channels)
        # decay rates spread over (0.9, 0.999) at r = 1
        a = torch.linspace(0.9, 0.999, channels) if channels > 1 else torch.tensor([0.95])
        self.lam = make_param(torch.log(torch.expm1(-torch.log(a) / self.decay)).to(device=device, dtype=dtype))
        self.wo = Linear(channels, width, bias=False, device=device, seed=seed + 4, dtype=dtype, init_std=init_std)

    def own_parameters(self):
        return [self.w_yx, self.b_yx, self.conv_w, self.conv_b, self.w_r, self.b_r, self.w_i, self.b_i, self.lam]

    def submodules(self):
        return [self.wo]

    def new_state(self):
        return RecurrentState(self.channels, self.taps)

    def _build_pack(self):
        G, n = self.blocks, self.channels // self.blocks
        w = torch.cat([self.w_r.detach().view(G, n, n), self.w_i.detach().view(G, n, n)], 1)     # [G, 2n, n]
        if w.dtype == torch.bfloat16:
            w = torch.cat([w, w], 2)       # against [high | low] parts of the input
        return w.contiguous().view(G * 2 * n, -1)

    def forward(self, h: torch.Tensor, ctx: StepContext, state: RecurrentState) -> torch.Tensor:
        from ..ops import hybrid as Y
        C, G, B, S = self.channels, self.blocks, ctx.B, ctx.S
        n = C // G
        yx = F.linear(h, self.w_yx, self.b_yx)
        u = Y.conv_state(yx[:, C:], self.conv_w, self.conv_b, state.conv, B, S, G)
        w = self.packed()
        z = torch.empty(B * S, 2 * C, dtype=torch.float32, device=h.device)
        Y.grouped_gemm(Y.grouped_segment(u, w, z, groups=G, N_=2 * n, K=w.shape[1], x_col_stride=w.shape[1],
                                         out_col_stride=2 * n))
        s = Y.lru_scan(u, z, self.b_r, self.b_i, self.lam, yx[:, :C], state.s, B, S, G, self.decay)
        return F.linear(s, self.wo.weight)


# ------------------------------------------------------------------------------------------ dropless experts --
class DroplessMoE(Module):
    """Experts ``Wdown relu(Wup h)^2``; every token uses the ``top`` with the largest router logits, weighted by the softmax
    over those logits alone; a shared expert (``shared_ff`` > 0) of the same form runs for every token.  No token is dropped.
    All experts' weights are one ``[E, ff, D]`` and one ``[E, D, ff]`` tensor for the grouped GEMM."""

    def __init__(self, width: int, experts: int, top: int, ff: int, shared_ff: int = 0, device=None, seed: int = 0,
                 dtype=torch.float32, init_std: Optional[float] = None):
        super().__init__()
        if not 1 <= top <= experts:
            raise ValueError(f"DroplessMoE: top ({top}) must be in [1, experts ({experts})]")
        if top > 32 or experts > 1000:
            raise ValueError("DroplessMoE: at most 1000 experts and 32 per token")
        self.width, self.experts, self.top, self.ff, self.shared_ff = width, experts, top, ff, shared_ff
        mk = lambda r, c, s: _weight(r, c, seed + s, device, dtype, init_std)  # noqa: E731
        self.router = mk(experts, width, 0)
        self.w_up = mk(experts * ff, width, 1)
        self.w_down = mk(experts * width, ff, 2)
        self.s_up = mk(shared_ff, width, 3) if shared_ff else None
        self.s_down = mk(width, shared_ff, 4) if shared_ff else None

    def own_parameters(self):
        return [self.router, self.w_up, self.w_down] + ([self.s_up, self.s_down] if self.shared_ff else [])

    def forward(self, h: torch.Tensor, counters: torch.Tensor):
        """``counters``: zeroed int32 ``[>= 2 * experts]``.  Returns the shared expert's output (or None), the routed
        experts' rows, and the slot and weight of every (token, choice); the caller adds them up."""
        from ..ops import hybrid as Y
        E, D, ff, top, M = self.experts, self.width, self.ff, self.top, h.shape[0]
        idx, w = Y.moe_route(h, self.router.detach(), top, counters)
        xs, offsets, slot = Y.moe_place(h, idx, counters, E)
        hint = (M * top + E - 1) // E
        new = lambda rows, cols: torch.empty(rows, cols, dtype=h.dtype, device=h.device)  # noqa: E731
        up, y = new(M * top, ff), new(M * top, D)
        segs_up = [Y.grouped_segment(xs, self.w_up.detach(), up, groups=E, N_=ff, K=D, offsets=offsets, act="relu2",
                                     rows_hint=hint)]
        segs_down = [Y.grouped_segment(up, self.w_down.detach(), y, groups=E, N_=D, K=ff, offsets=offsets, rows_hint=hint)]
        shared = None
        if self.shared_ff:
            s_up, shared = new(M, self.shared_ff), new(M, D)
            segs_up.append(Y.grouped_segment(h, self.s_up.detach(), s_up, groups=1, N_=self.shared_ff, K=D, act="relu2"))
            segs_down.append(Y.grouped_segment(s_up, self.s_down.detach(), shared, groups=1, N_=D, K=self.shared_ff))
        Y.grouped_gemm(*segs_up)
        Y.grouped_gemm(*segs_down)
        return shared, y, slot, w
