"""Famudra checkpoints: ``{name: tensor}`` maps with the layer prefix ``l<i>.`` (``embed``, ``l0.norm1``, ``l0.shift``,
``l0.mix.*``, ``l0.mlp.*``, ..., ``final.norm``, ``head``), Linear weights stored ``[out, in]``."""
from __future__ import annotations

from typing import Dict, Iterator, Tuple

import torch

from ..models.famudra import Famudra
from ..nn.hybrid import LatentAttention
from .hf_loaders import LoadReport, _copy, _Taker
from .safetensors import SafeTensors


def _entries(model: Famudra) -> Iterator[Tuple[str, torch.Tensor, list]]:
    """(name, view of the model's storage, shape in the file) of every tensor; fused weights appear as row ranges."""
    c = model.config

    def t(name, view, shape=None):
        return name, view, list(view.shape) if shape is None else shape
    yield t("embed", model.embed.weight.data)
    for i, layer in enumerate(model.layers):
        p = f"l{i}."
        yield t(p + "norm1", layer.norm1.gamma.data, [])
        yield t(p + "shift", layer.shift.mu.data)
        m = layer.mixer
        if isinstance(m, LatentAttention):
            yield t(p + "mix.dq", m.w_down.data[:m.q_rank])
            yield t(p + "mix.dkv", m.w_down.data[m.q_rank:])
            yield t(p + "mix.dq.norm", m.q_norm.data)
            yield t(p + "mix.dkv.norm", m.kv_norm.data)
            yield t(p + "mix.uq", m.w_uq.data)
            yield t(p + "mix.uk", m.w_uk.data)
            yield t(p + "mix.uv", m.w_uv.data)
        else:
            C, G = m.channels, m.blocks
            n = C // G
            yield t(p + "mix.y", m.w_yx.data[:C])
            yield t(p + "mix.x", m.w_yx.data[C:])
            yield t(p + "mix.y.b", m.b_yx.data[:C])
            yield t(p + "mix.x.b", m.b_yx.data[C:])
            yield t(p + "mix.conv", m.conv_w.data)
            yield t(p + "mix.conv.b", m.conv_b.data)
            for gate, w, b in (("ra", m.w_r, m.b_r), ("ri", m.w_i, m.b_i)):
                yield t(p + f"mix.{gate}", w.data.view(G, n, n))
                yield t(p + f"mix.{gate}.b", b.data.view(G, n))
            yield t(p + "mix.lam", m.lam.data)
        yield t(p + "mix.o", m.wo.weight.data)
        if layer.mlp is not None:
            e = layer.mlp
            yield t(p + "norm2", layer.norm2.gamma.data, [])
            yield t(p + "mlp.router", e.router.data)
            for k in range(e.experts):
                yield t(p + f"mlp.e{k}.up", e.w_up.data[k * e.ff:(k + 1) * e.ff])
                yield t(p + f"mlp.e{k}.down", e.w_down.data[k * c.width:(k + 1) * c.width])
            if e.shared_ff:
                yield t(p + "mlp.shared.up", e.s_up.data)
                yield t(p + "mlp.shared.down", e.s_down.data)
    yield t("final.norm", model.final_norm.gamma.data, [])
    yield t("head", model.head.weight.data)


class FamudraLoader:
    @staticmethod
    def load_map(model: Famudra, state: Dict[str, torch.Tensor]) -> LoadReport:
        taker = _Taker({k: (v.reshape(()) if v.numel() == 1 and v.dim() == 1 else v) for k, v in state.items()}, "famudra")
        for name, view, shape in _entries(model):
            src = taker.take(name, shape if taker.has(name) and taker.state[name].dim() else [])
            if src.numel() != view.numel():
                raise ValueError(f'famudra loader: "{name}" has {src.numel()} values, expected {view.numel()}')
            _copy(view, src.reshape(view.shape))
        for m in model.modules():
            if hasattr(m, "_pack"):
                m._pack = None
        model.caches.clear()
        return taker.report()

    @staticmethod
    def load_file(model: Famudra, path: str) -> LoadReport:
        return FamudraLoader.load_map(model, SafeTensors.load_file(path))

    @staticmethod
    def dump(model: Famudra) -> Dict[str, torch.Tensor]:
        return {name: view.detach().float().cpu().reshape(shape).clone() for name, view, shape in _entries(model)}

    loadMap, loadFile = load_map, load_file
