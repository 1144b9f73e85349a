"""Famudra: a hybrid decoder of latent-attention and gated-linear-recurrence layers with dropless experts.

A layer reads the fp32 residual stream through two one-number RMS norms and adds both branches at once,
``x + (mixer(shift(norm1(x))) + experts(norm2(x)))``; the mixer's input is mixed with the previous token's.  A range of
layers may run several times with the same weights (each run with a state of its own); before every run of the range but
the first the token embedding is added to the stream again.

Layers, sizes and constants come from ``config.json``.  The state of a batch of sequences is a ``HybridCache``; ``step`` is
the one function that processes tokens: prompts, portions of prompts and decode steps.  A step of one token per sequence is
captured in a CUDA graph, once per cache, and replayed.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from ..nn.hybrid import (DroplessMoE, GatedLinearRecurrence, HybridCache, LatentAttention, ScalarRMSNorm,
                         StepContext, TokenShift)
from ..nn.layers import Embedding, Linear
from ..nn.module import Module
from .hybrid import HybridDecoder

MIXERS = ("latent_attention", "rglru")


@dataclass
class FamudraLayerConfig:
    type: str
    mixer: dict
    mlp: Optional[dict] = None

    def __post_init__(self):
        if self.type not in MIXERS:
            raise ValueError(f"FamudraConfig: unknown mixer {self.type!r}")
        need = ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale") if self.type == "latent_attention" else \
            ("width", "blocks", "conv")
        missing = [k for k in need if k not in self.mixer]
        if missing:
            raise ValueError(f"FamudraConfig: mixer {self.type} lacks {missing}")
        if self.mlp is not None and self.mlp.get("kind", "moe") != "moe":
            raise ValueError(f"FamudraConfig: unknown feed-forward {self.mlp['kind']!r}")


@dataclass
class FamudraConfig:
    vocab_size: int
    width: int
    layers: List[FamudraLayerConfig]
    norm_eps: float
    loop: Optional[Tuple[int, int, int]] = None        # layers [start, stop) run `times` times
    max_ctx: int = 1 << 20                             # the design has no positions; this only bounds the cache
    device: object = None
    seed: int = 0
    dtype: torch.dtype = torch.float32
    init_std: Optional[float] = None

    def __post_init__(self):
        self.layers = [s if isinstance(s, FamudraLayerConfig) else
                       FamudraLayerConfig(s["type"], s["mixer"], s.get("mlp")) for s in self.layers]
        if not self.layers:
            raise ValueError("FamudraConfig: no layers")
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a <= b <= len(self.layers)) or times < 1:
                raise ValueError(f"FamudraConfig: bad loop {self.loop}")

    @staticmethod
    def from_json(config: dict, **kw) -> "FamudraConfig":
        loop = config.get("loop")
        return FamudraConfig(vocab_size=config["vocab"], width=config["width"], layers=config["layers"],
                             norm_eps=config["norm"]["eps"],
                             loop=None if not loop else (loop["start"], loop["stop"], loop["times"]), **kw)

    @property
    def schedule(self) -> List[Tuple[int, bool]]:
        """(layer, embedding is added before it) for every layer run, in order."""
        a, b, times = self.loop or (0, 0, 1)
        runs = [(i, False) for i in range(a)]
        for t in range(times):
            runs += [(i, t > 0 and i == a) for i in range(a, b)]
        return runs + [(i, False) for i in range(b, len(self.layers))]

    # names the runners and servers read
    @property
    def embed_dim(self) -> int:
        return self.width

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_heads(self) -> int:
        return max([s.mixer.get("heads", 0) for s in self.layers])


class FamudraLayer(Module):
    def __init__(self, c: FamudraConfig, spec: FamudraLayerConfig, seed: int):
        super().__init__()
        kw = dict(device=c.device, dtype=c.dtype)
        m = spec.mixer
        self.norm1 = ScalarRMSNorm(c.norm_eps, **kw)
        self.shift = TokenShift(c.width, **kw)
        if spec.type == "latent_attention":
            self.mixer = LatentAttention(c.width, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"],
                                         c.norm_eps, seed=seed, init_std=c.init_std, **kw)
        else:
            self.mixer = GatedLinearRecurrence(c.width, m["width"], m["blocks"], m["conv"], seed=seed,
                                               init_std=c.init_std, **kw)
        self.norm2 = self.mlp = None
        if spec.mlp is not None:
            self.norm2 = ScalarRMSNorm(c.norm_eps, **kw)
            self.mlp = DroplessMoE(c.width, spec.mlp["router"]["experts"], spec.mlp["router"]["top"],
                                   spec.mlp["expert"]["ff"], (spec.mlp.get("shared") or {}).get("ff", 0), seed=seed + 1000,
                                   init_std=c.init_std, **kw)

    def submodules(self):
        return [self.norm1, self.shift, self.mixer] + ([self.norm2, self.mlp] if self.mlp is not None else [])


class Famudra(HybridDecoder):
    _name = "Famudra"

    def __init__(self, config: FamudraConfig):
        super().__init__()
        c = config
        self.config = c
        self.embed = Embedding(c.vocab_size, c.width, device=c.device, seed=c.seed, dtype=c.dtype, init_std=c.init_std)
        self.layers = [FamudraLayer(c, s, c.seed + 100000 + i * 10000) for i, s in enumerate(c.layers)]
        self.final_norm = ScalarRMSNorm(c.norm_eps, device=c.device, dtype=c.dtype)
        self.head = Linear(c.width, c.vocab_size, bias=False, device=c.device, seed=c.seed + 900000, dtype=c.dtype,
                           init_std=c.init_std)
        self.schedule = c.schedule
        self._init_serving()

    def submodules(self):
        return [self.embed] + list(self.layers) + [self.final_norm, self.head]

    # ---- state -----------------------------------------------------------------------------------
    def _make_cache(self, batch: int, max_len: int) -> HybridCache:
        experts = [layer.mlp.experts for layer in self.layers if layer.mlp is not None]
        return HybridCache([self.layers[i].mixer.new_state() for i, _ in self.schedule], self.config.width, batch, max_len,
                           self.dtype, self.device, counters=2 * max(experts, default=0))

    # ---- one step --------------------------------------------------------------------------------
    def _run(self, tokens: torch.Tensor, ctx: StepContext, pick: Optional[torch.Tensor]) -> torch.Tensor:
        """All layers over ``tokens [B*S]``; final-norm rows (those in ``pick``)."""
        from ..ops import hybrid as Y
        cache, M, eps = ctx.cache, ctx.B * ctx.S, self.config.norm_eps
        table = self.embed.weight
        cache.counters.zero_()
        x = terms = None
        for run, (i, add_embedding) in enumerate(self.schedule):
            layer = self.layers[i]
            x, h1, h2 = Y.stream_norm(x, terms, M, ctx.S, layer.norm1.gamma, eps,
                                      g2=None if layer.mlp is None else layer.norm2.gamma, shift=layer.shift.mu,
                                      shift_state=cache.shift[run],
                                      embed=table if run == 0 or add_embedding else None, tokens=tokens)
            mix = layer.mixer(h1, ctx, cache.states[run])
            terms = Y.LayerTerms(mix) if layer.mlp is None else \
                Y.LayerTerms(mix, *layer.mlp(h2, cache.counters[run]))
        rows = M if pick is None else pick.numel()
        return Y.stream_norm(x, terms, rows, 1, self.final_norm.gamma, eps, pick=pick, keep=False)[1]
