"""What the hybrid decoder families share: the cache pool, the step function, its captured form for decoding, and the interface
of the generation loops and services.

A family derives from ``HybridDecoder``, calls ``_init_serving`` and provides ``config`` (``max_ctx``, ``vocab_size``), ``head``
(a Linear), ``_make_cache(batch, max_len)`` and ``_run(tokens, ctx, pick)``, which puts the tokens of one step through all layers.
"""
from __future__ import annotations

import gc
import os
from typing import Optional, Sequence

import torch

from .. import _native as N
from ..nn.hybrid import CachePool, HybridCache, StepContext
from ..nn.module import Module
from .gpt import _as_token_tensor
from .neox import CausalLMMixin


class HybridDecoder(CausalLMMixin, Module):
    def _init_serving(self) -> None:
        self.caches = CachePool(self._make_cache)
        self._capture_stream = None

    def _moved(self, device, dtype):
        self.caches.clear()

    # ---- what a family provides ------------------------------------------------------------------
    def _make_cache(self, batch: int, max_len: int) -> HybridCache:
        raise NotImplementedError

    def _run(self, tokens: torch.Tensor, ctx: StepContext, pick: Optional[torch.Tensor]) -> torch.Tensor:
        """All layers over ``tokens [B*S]``; final-norm rows (those in ``pick``)."""
        raise NotImplementedError

    # ---- state -----------------------------------------------------------------------------------
    def new_cache(self, max_len: Optional[int] = None, batch: int = 1) -> HybridCache:
        """State for ``batch`` new sequences; give it back with ``free_cache`` when they are finished."""
        return self.caches.acquire(batch, max_len or 256)

    def cache_for(self, tokens: int) -> HybridCache:
        return self.new_cache(tokens)

    def free_cache(self, cache: HybridCache) -> None:
        self.caches.release(cache)

    # ---- one step --------------------------------------------------------------------------------
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
            raise RuntimeError(f"{self._name} runs on a CUDA device (bfloat16 or float32); there is no CPU path")
        B, S = tokens.shape
        if B != cache.batch:
            raise ValueError(f"{self._name}.step: the cache holds {cache.batch} sequences, got {B}")
        if S == 0:
            raise ValueError(f"{self._name}.step: no tokens")
        if cache.seq_len + S > self.config.max_ctx:
            raise ValueError(f"{self._name}: {cache.seq_len + S} tokens exceed maxCtx {self.config.max_ctx}")
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
            raise ValueError(f"{self._name}: tokens must be [N] or [B, N]")
        return t if t.dim() == 2 else t.unsqueeze(0)

    def _check_start(self, start_pos: int, cache: HybridCache) -> None:
        if start_pos != cache.seq_len:
            raise ValueError(f"{self._name}: start_pos {start_pos} but the cache holds {cache.seq_len} tokens")

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
