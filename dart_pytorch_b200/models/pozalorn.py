"""Pozalorn: a decoder of gated linear attention, windowed attention with pooled blocks, and layers that run windowed attention
and lightning attention side by side.

Norms stand behind the sublayers only: ``x <- x + norm1(mixer(x))``, ``x <- x + norm2(mlp(x))`` on an fp32 stream.  After every
layer the stream becomes a weighted sum of all results so far, the embedding first (``average``).

Layers, sizes and constants come from ``config.json``, the rank of the decay projections from the checkpoint.  State, ``step``
and decoding are those of ``HybridDecoder``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..nn.hybrid import HybridCache, StepContext, _full
from ..nn.layers import Embedding, Linear, RMSNorm
from ..nn.mixers import GatedMLP, LinearAttention, RotaryTable, SideBySide, WindowAttention
from ..nn.module import Module
from .hybrid import HybridDecoder

DEFAULT_RANK = 16     # of the decay projections, when there is no checkpoint to tell
_ATTENTION = ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot")
_NEEDS = {"gla": ("heads", "dim", "vdim", "tau"), "attention": _ATTENTION,
          "parallel": ("left", "right", "left_scale", "right_scale")}


def _check(kind: str, what: dict, keys) -> None:
    missing = [k for k in keys if k not in what]
    if missing:
        raise ValueError(f"PozalornConfig: {kind} lacks {missing}")


@dataclass
class PozalornLayerConfig:
    type: str
    mixer: dict
    mlp: Optional[dict] = None
    rank: int = DEFAULT_RANK

    def __post_init__(self):
        if self.type not in _NEEDS:
            raise ValueError(f"PozalornConfig: unknown mixer {self.type!r}")
        _check(f"mixer {self.type}", self.mixer, _NEEDS[self.type])
        if self.type == "parallel":
            _check("the left mixer", self.mixer["left"], _ATTENTION)
            _check("the right mixer", self.mixer["right"], ("heads", "dim", "vdim", "decay"))
        if self.mlp is not None:
            if self.mlp.get("kind", "dense") != "dense":
                raise ValueError(f"PozalornConfig: unknown feed-forward {self.mlp['kind']!r}")
            _check("the feed-forward", self.mlp, ("ff",))


@dataclass
class PozalornConfig:
    vocab_size: int
    width: int
    layers: List[PozalornLayerConfig]
    norm_eps: float
    max_ctx: int = 1 << 20                             # only bounds the cache and the rotary tables
    device: object = None
    seed: int = 0
    dtype: torch.dtype = torch.float32
    init_std: Optional[float] = None

    def __post_init__(self):
        self.layers = [s if isinstance(s, PozalornLayerConfig) else
                       PozalornLayerConfig(s["type"], s["mixer"], s.get("mlp"), s.get("rank", DEFAULT_RANK))
                       for s in self.layers]
        if not self.layers:
            raise ValueError("PozalornConfig: no layers")

    @staticmethod
    def from_json(config: dict, state: Optional[Dict[str, torch.Tensor]] = None, **kw) -> "PozalornConfig":
        """``state``: the checkpoint, for the sizes that only its shapes give."""
        layers = []
        for i, spec in enumerate(config["layers"]):
            down = (state or {}).get(f"l{i}.mix.a1")
            layers.append(PozalornLayerConfig(spec["type"], spec["mixer"], spec.get("mlp"),
                                              DEFAULT_RANK if down is None else int(down.shape[0])))
        return PozalornConfig(vocab_size=config["vocab"], width=config["width"], layers=layers,
                              norm_eps=config["norm"]["eps"], **kw)

    # names the runners and servers read
    @property
    def embed_dim(self) -> int:
        return self.width

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_heads(self) -> int:
        return max((s.mixer["left"] if s.type == "parallel" else s.mixer)["heads"] for s in self.layers)


def _attention(c: PozalornConfig, m: dict, seed: int, together: bool, **kw) -> WindowAttention:
    rot = m["rot"]
    return WindowAttention(c.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"], c.norm_eps,
                           qk_norm="together" if together else "head",
                           rotary=RotaryTable(rot["base"], rot["dims"], rot.get("scaling")), seed=seed, bias=True,
                           init_std=c.init_std, device=c.device, dtype=c.dtype, **kw)


def make_mixer(c: PozalornConfig, spec: PozalornLayerConfig, seed: int):
    m, kw = spec.mixer, dict(device=c.device, dtype=c.dtype, init_std=c.init_std)
    if spec.type == "gla":
        return LinearAttention(c.width, m["heads"], m["dim"], m["vdim"], c.norm_eps, rank=spec.rank, tau=m["tau"],
                               q_scale=m["dim"] ** -0.5, gate="silu", seed=seed, **kw)
    if spec.type == "attention":
        return _attention(c, m, seed, True, pool=m["mask"].get("pool") or 0, rotary_v=RotaryTable(m["rot"]["base"], m["vdim"]))
    left = _attention(c, m["left"], seed, False, sink=True, out_bias=True, own_input=False)
    r = m["right"]
    right = LinearAttention(c.width, r["heads"], r["dim"], r["vdim"], c.norm_eps, decay=r["decay"], silu=True, joint_norm=True,
                            gate="sigmoid", own_input=False, seed=seed + 10, **kw)
    return SideBySide(c.width, left, right, (m["left_scale"], m["right_scale"]), bias=True, seed=seed + 20, **kw)


class PozalornLayer(Module):
    def __init__(self, c: PozalornConfig, index: int, seed: int):
        super().__init__()
        spec = c.layers[index]
        kw = dict(device=c.device, dtype=c.dtype)
        self.mixer = make_mixer(c, spec, seed)
        self.norm1 = RMSNorm(c.width, c.norm_eps, **kw)
        self.norm2 = self.mlp = None
        if spec.mlp is not None:
            self.norm2 = RMSNorm(c.width, c.norm_eps, **kw)
            self.mlp = GatedMLP(c.width, spec.mlp["ff"], seed=seed + 1000, init_std=c.init_std, **kw)
        # weights of the embedding, every earlier layer's result and this one's
        self.average = _full((index + 2,), 0.0, c.device, c.dtype)
        self.average.data[-1] = 1.0

    def own_parameters(self):
        return [self.average]

    def submodules(self):
        return [self.mixer, self.norm1] + ([self.norm2, self.mlp] if self.mlp is not None else [])


class Pozalorn(HybridDecoder):
    _name = "Pozalorn"

    def __init__(self, config: PozalornConfig):
        super().__init__()
        c = config
        self.config = c
        self.embed = Embedding(c.vocab_size, c.width, device=c.device, seed=c.seed, dtype=c.dtype, init_std=c.init_std)
        self.layers = [PozalornLayer(c, i, c.seed + 100000 + i * 10000) for i in range(len(c.layers))]
        self.final_norm = RMSNorm(c.width, c.norm_eps, device=c.device, dtype=c.dtype)
        self.head = Linear(c.width, c.vocab_size, bias=False, device=c.device, seed=c.seed + 900000, dtype=c.dtype,
                           init_std=c.init_std)
        self._init_serving()

    def submodules(self):
        return [self.embed] + list(self.layers) + [self.final_norm, self.head]

    def _make_cache(self, batch: int, max_len: int) -> HybridCache:
        return HybridCache([layer.mixer.new_state() for layer in self.layers], 0, batch, max_len, self.dtype, self.device)

    def _run(self, tokens: torch.Tensor, ctx: StepContext, pick: Optional[torch.Tensor]) -> torch.Tensor:
        """All layers over ``tokens [B*S]``; final-norm rows (those in ``pick``)."""
        from ..ops import mixers as X
        M, D, eps, dt = ctx.B * ctx.S, self.config.width, self.config.norm_eps, self.dtype
        new = lambda: torch.empty(M, D, dtype=torch.float32, device=tokens.device)  # noqa: E731
        half = dt != torch.float32          # the sublayers read a rounded copy of the stream, in fp32 the stream itself
        # results so far: the embedding, then the layers' (all but the last one's are read again)
        stack = torch.empty(len(self.layers), M, D, dtype=torch.float32, device=tokens.device)
        x = stack[0]
        h = X.branch_norm(None, M, D, dt, eps, embed=self.embed.weight, tokens=tokens, result=x, h=half)
        for i, layer in enumerate(self.layers):
            m = layer.mixer(x if h is None else h, ctx, ctx.cache.states[i])
            m1, m2 = m if isinstance(m, tuple) else (m, None)
            c1, c2 = layer.mixer.scales if m2 is not None else (1.0, 1.0)
            term = dict(m1=m1, m2=m2, c1=c1, c2=c2, w=layer.norm1.gamma)
            if layer.mlp is not None:
                y = new()
                h = X.branch_norm(x, M, D, dt, eps, x_out=y, h=half, **term)
                x = y
                term = dict(m1=layer.mlp(x if h is None else h), w=layer.norm2.gamma)
            term.update(stack=stack, n=i + 1, avg=layer.average)
            if i + 1 == len(self.layers):
                rows = M if pick is None else pick.numel()
                return X.branch_norm(x, rows, D, dt, eps, pick=pick, wf=self.final_norm.gamma, **term)
            y = new()
            h = X.branch_norm(x, M, D, dt, eps, result=stack[i + 1], x_out=y, h=half, **term)
            x = y
