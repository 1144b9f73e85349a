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

import gc
import os
from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch

from .. import _native as N
from ..nn.hybrid import (CachePool, DroplessMoE, GatedLinearRecurrence, HybridCache, LatentAttention, ScalarRMSNorm,
                         StepContext, TokenShift)
from ..nn.layers import Embedding, Linear
from ..nn.module import Module
from .gpt import _as_token_tensor
from .neox import CausalLMMixin

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


class Famudra(CausalLMMixin, Module):
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
        self.caches = CachePool(self._make_cache)
        self._capture_stream = None

    def submodules(self):
        return [self.embed] + list(self.layers) + [self.final_norm, self.head]

    def _moved(self, device, dtype):
        self.caches.clear()

    # ---- state -----------------------------------------------------------------------------------
    def _make_cache(self, batch: int, max_len: int) -> HybridCache:
        experts = [layer.mlp.experts for layer in self.layers if layer.mlp is not None]
        return HybridCache([self.layers[i].mixer.new_state() for i, _ in self.schedule], self.config.width, batch, max_len,
                           self.dtype, self.device, counters=2 * max(experts, default=0))

    def new_cache(self, max_len: Optional[int] = None, batch: int = 1) -> HybridCache:
        """State for ``batch`` new sequences; give it back with ``free_cache`` when they are finished."""
        return self.caches.acquire(batch, max_len or 256)

    def cache_for(self, tokens: int) -> HybridCache:
        return self.new_cache(tokens)

    def free_cache(self, cache: HybridCache) -> None:
        self.caches.release(cache)

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

    def _head(self, h: torch.Tensor) -> torch.Tensor:
        """fp32 logits."""
        from ..ops import hybrid as Y
        from ..ops import kernels as K
        w = self.head.weight.detach()
        out = torch.empty(h.shape[0], w.shape[0], dtype=torch.float32, device=h.device)
        if h.shape[0] <= K.SKINNY_MAX_ROWS and h.dtype == torch.bfloat16:
            Y.grouped_gemm(Y.grouped_segment(h, w, out, groups=1, N_=w.shape[0], K=w.shape[1]))
        else:
            K.gemm(h, w, out, trans_b=True)
        return out

    def _capture(self, cache: HybridCache):
        """Record a decode step of this cache: token buffer in, logits out, position advanced on the device."""
        tokens = torch.zeros(cache.batch, dtype=torch.long, device=cache.device)
        ctx = StepContext(cache, cache.batch, 1, 0, pos_ptr=cache.pos)
        lib = N.load()

        def body():
            lib.dptb_gemm_skinny_set_pdl(1)
            try:
                out = self._head(self._run(tokens, ctx, None))
            finally:
                lib.dptb_gemm_skinny_set_pdl(0)
            cache.pos.add_(1)
            return out
        if self._capture_stream is None:
            self._capture_stream = torch.cuda.Stream(device=cache.device)
        s = self._capture_stream
        saved = (cache.flat.clone(), cache.pos.clone())
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s):
            body()                                    # warm-up: workspaces, packed weights, kernel attributes
            cache.flat.copy_(saved[0])
            cache.pos.copy_(saved[1])
            torch.cuda.synchronize()
            launches = lib.dptb_launch_count()
            graph = torch.cuda.CUDAGraph()
            # an unreachable older graph must not be destroyed while this one is being recorded
            gc.collect()
            collecting = gc.isenabled()
            gc.disable()
            try:
                with torch.cuda.graph(graph, stream=s):
                    logits = body()
            finally:
                if collecting:
                    gc.enable()
        torch.cuda.current_stream().wait_stream(s)
        cache.graph = (graph, tokens, logits, int(lib.dptb_launch_count() - launches))

    def step(self, cache: HybridCache, tokens: torch.Tensor, rows: Optional[Sequence[int]] = None) -> torch.Tensor:
        """Process ``tokens [B, S]`` after what ``cache`` already holds; fp32 logits ``[len(rows), vocab]`` at the flat
        places ``rows`` of ``tokens`` (None: all).  The result may be overwritten by the next step of this cache."""
        if not tokens.is_cuda:
            raise RuntimeError("Famudra runs on a CUDA device (bfloat16 or float32); there is no CPU path")
        B, S = tokens.shape
        if B != cache.batch:
            raise ValueError(f"Famudra.step: the cache holds {cache.batch} sequences, got {B}")
        if S == 0:
            raise ValueError("Famudra.step: no tokens")
        if cache.seq_len + S > self.config.max_ctx:
            raise ValueError(f"Famudra: {cache.seq_len + S} tokens exceed maxCtx {self.config.max_ctx}")
        cache.ensure(cache.seq_len + S)
        tokens = tokens.reshape(-1).contiguous()
        with torch.no_grad():
            if S == 1 and os.environ.get("DPTB200_DECODE_GRAPH", "1") != "0":
                if cache.graph is None:
                    self._capture(cache)
                graph, buf, logits, _ = cache.graph
                buf.copy_(tokens)
                graph.replay()
                cache.seq_len += 1
                return logits if rows is None or list(rows) == list(range(B)) else logits[list(rows)]
            pick = None
            if rows is not None and len(rows) < B * S:
                pick = torch.tensor(list(rows), dtype=torch.int32, device=tokens.device)
            ctx = StepContext(cache, B, S, cache.seq_len)
            if pick is not None and pick.numel() == 0:      # nothing asked for: the state still moves on
                self._run(tokens, ctx, torch.zeros(1, dtype=torch.int32, device=tokens.device))
                cache.advance(S)
                return torch.empty(0, self.config.vocab_size, dtype=torch.float32, device=tokens.device)
            out = self._head(self._run(tokens, ctx, pick))
            cache.advance(S)
            return out

    # ---- the interface the generation loops and services use -----------------------------------------
    def _as_batch(self, tokens) -> torch.Tensor:
        t = _as_token_tensor(tokens, self.device)
        if t.dim() not in (1, 2):
            raise ValueError("Famudra: tokens must be [N] or [B, N]")
        return t if t.dim() == 2 else t.unsqueeze(0)

    def _check_start(self, start_pos: int, cache: HybridCache) -> None:
        if start_pos != cache.seq_len:
            raise ValueError(f"Famudra: start_pos {start_pos} but the cache holds {cache.seq_len} tokens")

    def logits(self, tokens, start_pos: int = 0, cache: Optional[HybridCache] = None) -> torch.Tensor:
        """fp32 logits of every token, ``[N, V]`` or ``[B, N, V]``."""
        t = self._as_batch(tokens)
        own = cache is None
        cache = self.new_cache(t.shape[1], t.shape[0]) if own else cache
        self._check_start(start_pos, cache)
        out = self.step(cache, t).clone()
        if own:
            self.free_cache(cache)
        return out if getattr(tokens, "ndim", 1) == 1 else out.view(*t.shape, -1)

    def last_logits(self, tokens, start_pos: int = 0, cache: Optional[HybridCache] = None) -> torch.Tensor:
        t = self._as_batch(tokens)
        if cache is None:
            return super().last_logits(tokens, start_pos, cache)
        self._check_start(start_pos, cache)
        B, S = t.shape
        return self.step(cache, t, [b * S + S - 1 for b in range(B)])

    def hidden(self, tokens, start_pos: int = 0, cache: Optional[HybridCache] = None) -> torch.Tensor:
        """Final-norm hidden states ``[N, D]`` or ``[B, N, D]``."""
        t = self._as_batch(tokens)
        own = cache is None
        cache = self.new_cache(t.shape[1], t.shape[0]) if own else cache
        self._check_start(start_pos, cache)
        cache.ensure(cache.seq_len + t.shape[1])
        with torch.no_grad():
            h = self._run(t.reshape(-1).contiguous(), StepContext(cache, *t.shape, cache.seq_len), None)
        cache.advance(t.shape[1])
        if own:
            self.free_cache(cache)
        return h if getattr(tokens, "ndim", 1) == 1 else h.view(*t.shape, -1)

    def forward(self, tokens):
        return self.logits(tokens)
