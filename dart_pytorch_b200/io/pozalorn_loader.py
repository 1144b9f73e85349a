"""Pozalorn checkpoints: ``{name: tensor}`` maps with the layer prefix ``l<i>.`` (``embed``, ``l0.norm1``, ``l0.mix.*``,
``l0.mlp.*``, ``l0.dwa``, ..., ``final.norm``, ``head``), Linear weights stored ``[out, in]``."""
from __future__ import annotations

from typing import Dict, Iterator, Tuple

import torch

from ..models.pozalorn import Pozalorn
from ..nn.mixers import LinearAttention, SideBySide, WindowAttention
from .hf_loaders import LoadReport, _copy, _Taker
from .safetensors import SafeTensors

Entry = Tuple[str, torch.Tensor]


def _window(p: str, m: WindowAttention, w_in: torch.Tensor, b_in: torch.Tensor) -> Iterator[Entry]:
    for name, heads, d in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim), ("v", m.kv_heads, m.vdim)):
        at = m.cols[name]
        yield p + name, w_in[at:at + heads * d]
        yield p + name + ".b", b_in[at:at + heads * d]
    yield p + "q.norm", m.q_norm.data
    yield p + "k.norm", m.k_norm.data
    if m.sink is not None:
        yield p + "sink", m.sink.data
    yield p + "o", m.wo.weight.data
    if m.wo.bias is not None:
        yield p + "o.b", m.wo.bias.data.view(-1)


def _linear(p: str, m: LinearAttention, w_in: torch.Tensor) -> Iterator[Entry]:
    for name, d in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim)):
        yield p + name, w_in[m.cols[name]:m.cols[name] + m.heads * d]
    if m.rank:
        yield p + "a1", w_in[m.cols["r"]:m.cols["r"] + m.rank]
        yield p + "a2", m.w2.data
        yield p + "a2.b", m.b2.data
    yield p + "norm", m.norm.data
    yield p + "o", m.wo.weight.data


def _entries(model: Pozalorn) -> Iterator[Entry]:
    """(name, view of the model's storage) of every tensor; fused weights appear as row ranges."""
    yield "embed", model.embed.weight.data
    for i, layer in enumerate(model.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, SideBySide):
            n = m.left.in_rows
            yield from _window(p + "mix.left.", m.left, m.w_in.data[:n], m.b_in.data[:n])
            yield from _linear(p + "mix.right.", m.right, m.w_in.data[n:])
        elif isinstance(m, WindowAttention):
            yield from _window(p + "mix.", m, m.w_in.data, m.b_in.data)
        else:
            yield from _linear(p + "mix.", m, m.w_in.data)
        yield p + "norm1", layer.norm1.gamma.data
        if layer.mlp is not None:
            f = layer.mlp
            yield p + "norm2", layer.norm2.gamma.data
            yield p + "mlp.gate", f.w_in.data[:f.ff]
            yield p + "mlp.up", f.w_in.data[f.cols["up"]:f.cols["up"] + f.ff]
            yield p + "mlp.down", f.down.weight.data
        yield p + "dwa", layer.average.data
    yield "final.norm", model.final_norm.gamma.data
    yield "head", model.head.weight.data


class PozalornLoader:
    @staticmethod
    def load_map(model: Pozalorn, state: Dict[str, torch.Tensor]) -> LoadReport:
        taker = _Taker(state, "pozalorn")
        for name, view in _entries(model):
            _copy(view, taker.take(name, list(view.shape)))
        model.caches.clear()
        return taker.report()

    @staticmethod
    def load_file(model: Pozalorn, path: str) -> LoadReport:
        return PozalornLoader.load_map(model, SafeTensors.load_file(path))

    @staticmethod
    def dump(model: Pozalorn) -> Dict[str, torch.Tensor]:
        return {name: view.detach().float().cpu().clone() for name, view in _entries(model)}

    loadMap, loadFile = load_map, load_file
