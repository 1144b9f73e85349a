"""Pozalorn without a GPU: configuration, registry, checkpoint loading, rotary tables, state bookkeeping, and the plain
implementation the GPU tests compare against (checked against itself and for the mistakes it should expose)."""
import copy
import json
import math

import pytest
import torch

import pozalorn_oracle as oracle
from dart_pytorch_b200.apps.servers import load_hf_model
from dart_pytorch_b200.io.pozalorn_loader import PozalornLoader
from dart_pytorch_b200.io.safetensors import SafeTensors
from dart_pytorch_b200.models import registry
from dart_pytorch_b200.models.pozalorn import Pozalorn, PozalornConfig
from dart_pytorch_b200.nn.hybrid import HybridCache
from dart_pytorch_b200.nn.mixers import MatrixState, PairState, RotaryTable, WindowState, row_layout

SCALING = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}


def gla(mlp=None, **kw):
    return {"type": "gla", "mixer": dict(dict(heads=3, dim=16, vdim=24, tau=8.0), **kw), "mlp": mlp}


def window(size=9, pool=None, **kw):
    mask = {"size": size}
    if pool:
        mask["pool"] = pool
    rot = {"base": kw.pop("base", 10000.0), "dims": kw.pop("rot", 8)}
    if kw.pop("scaled", True):
        rot["scaling"] = SCALING
    return dict(dict(heads=4, kv_heads=2, dim=16, vdim=24, mask=mask, rot=rot, scale=0.4), **kw)


def attention(mlp=None, size=9, pool=4, **kw):
    return {"type": "attention", "mixer": window(size, pool, **kw), "mlp": mlp}


def parallel(mlp=None, left_scale=0.7, right_scale=1.1, heads=3, dim=16, vdim=8, decay=None, **left):
    decay = decay or [math.exp(-2.0 ** (-i)) for i in range(heads)]
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": window(**left), "left_scale": left_scale, "right_scale": right_scale,
                      "right": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def config(layers=None, width=40, vocab=97, eps=1e-5):
    layers = layers or [gla(dense()), attention(), parallel(dense(24))]
    return {"architecture": "Pozalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def write_model(path, cfg, weights):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    SafeTensors.save_file(weights, str(path / "model.safetensors"), dtype="BF16")


def test_registry_and_configuration():
    assert registry.family_of({"architecture": "Pozalorn"}) == "pozalorn"
    cfg = config()
    c = PozalornConfig.from_json(cfg, oracle.random_weights(cfg, 0, rank=7))
    assert (c.vocab_size, c.width, c.norm_eps, c.num_heads, c.num_layers) == (97, 40, 1e-5, 4, 3)
    assert c.layers[0].rank == 7
    for path, key in ((("layers", 0, "mixer"), "tau"), (("layers", 1, "mixer"), "rot"), (("layers", 2, "mixer"), "left_scale"),
                      (("layers", 2, "mixer", "right"), "decay"), (("layers", 2, "mixer", "left"), "mask"),
                      (("layers", 0, "mlp"), "ff")):
        bad = copy.deepcopy(cfg)
        at = bad
        for p in path:
            at = at[p]
        del at[key]
        with pytest.raises(ValueError, match=key):
            PozalornConfig.from_json(bad)
    bad = config()
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError):
        PozalornConfig.from_json(bad)


@pytest.mark.parametrize("rank", [1, 5, 16])
def test_checkpoint_round_trip(tmp_path, rank):
    cfg = config([gla(dense(), dim=10, vdim=6), attention(rot=16), parallel(dense(21)), gla()])
    w = oracle.random_weights(cfg, 3, rank)
    write_model(tmp_path / "m", cfg, w)
    model, tok, report = load_hf_model("auto", str(tmp_path / "m"), device="cpu")
    assert isinstance(model, Pozalorn) and tok is None and report.unused_keys == []
    back = PozalornLoader.dump(model)
    assert set(back) == set(w)
    for k in w:
        assert back[k].shape == w[k].shape and torch.equal(back[k], w[k]), k
    missing = dict(w)
    del missing["l2.mix.left.sink"]
    with pytest.raises(ValueError, match="l2.mix.left.sink"):
        PozalornLoader.load_map(model, missing)
    wrong = dict(w)
    wrong["l1.dwa"] = torch.zeros(4)
    with pytest.raises(ValueError, match="l1.dwa"):
        PozalornLoader.load_map(model, wrong)


def test_no_cpu_path():
    model = Pozalorn(PozalornConfig.from_json(config()))
    with pytest.raises(RuntimeError, match="CUDA"):
        model.step(model.new_cache(8), torch.zeros(1, 3, dtype=torch.long))


def test_row_layout_is_aligned():
    cols, n = row_layout(q=30, k=8, v=1)
    assert cols == {"q": 0, "k": 32, "v": 40} and n == 48


@pytest.mark.parametrize("scaling", [None, SCALING, {"factor": 2.0, "low": 0.5, "high": 20.0, "original": 100}])
@pytest.mark.parametrize("base,dims", [(10000.0, 16), (500.0, 6), (30000.0, 48)])
def test_rotary_table(scaling, base, dims):
    t = RotaryTable(base, dims, scaling)
    f = oracle.frequencies({"base": base, "dims": dims, "scaling": scaling})
    assert torch.allclose(t.frequencies(), f, rtol=1e-12)
    rows = t.rows(50, "cpu")
    assert rows.shape[0] >= 50
    x = torch.randn(50, 2, dims + 3, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    want = oracle.rotate(x, torch.arange(50), f)
    c, s = rows[:50, :, 0].double()[:, None], rows[:50, :, 1].double()[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    assert torch.allclose(want[..., 0:dims:2], u * c - v * s, atol=1e-6)
    assert torch.allclose(want[..., 1:dims:2], v * c + u * s, atol=1e-6)
    assert torch.equal(want[..., dims:], x[..., dims:])
    longer = RotaryTable(base, dims, scaling).rows(rows.shape[0] + 1, "cpu")       # shared tables grow, old ones stay valid
    assert longer.shape[0] >= 2 * rows.shape[0] and torch.equal(longer[:50], rows[:50])


def test_states():
    states = [WindowState(6, 4, 9, 4, RotaryTable(100.0, 2), None), MatrixState(2, 3, 5),
              PairState(WindowState(2, 2, 70, 0, None, None), MatrixState(1, 2, 2))]
    cache = HybridCache(states, 0, 2, 100, torch.float32, "cpu")
    w, m, p = states
    assert w.ring % 8 == 0 and w.ring >= 9 + 31 and p.left.ring >= 70 + 31
    assert w.k.shape == (2, w.ring, 6) and w.v.shape == (2, w.ring, 4) and w.k_pool.shape == (2, 32, 6)
    assert w.rot.shape[0] >= cache.capacity and p.left.k_pool is None
    assert m.s.shape == (2, 2, 3, 5) and p.right.s.shape == (2, 1, 2, 2) and p.right.s.data_ptr() % 16 == 0
    w.k[:] = 1.0
    w.k_pool[:] = 2.0
    m.s.fill_(3.0)
    k = w.k
    cache.advance(128)
    cache.graph = object()
    cache.ensure(200)
    assert cache.graph is None and w.k is k and w.k_pool.shape == (2, cache.capacity // 4, 6)
    assert bool((w.k_pool[:, :32] == 2).all()) and bool((w.k_pool[:, 32:] == 0).all())
    cache.reset()
    assert float(m.s.abs().sum()) == 0.0 and cache.seq_len == 0


@pytest.mark.parametrize("pos,hist", [(0, 0), (3, 3), (8, 8), (39, 9), (40, 8), (47, 9), (100, 9), (1000, 4)])
def test_history_of_a_ring(pos, hist):
    s = WindowState(1, 1, 9, 4, None, None)
    s.grow(1, 128, 0, torch.float32, "cpu")
    for p in range(max(0, pos - s.ring), pos):
        s.k[0, p % s.ring] = float(p)
    got = s.history(s.k, 1, pos, hist, 5)
    assert got.shape == (1, hist + 5, 1) and got[0, :hist, 0].tolist() == [float(p) for p in range(pos - hist, pos)]


def test_oracle_mechanisms():
    # decays of 1 add up, decays of 0 keep the last token only
    q = k = torch.ones(4, 1, 2, dtype=torch.float64)
    v = torch.arange(1.0, 5.0, dtype=torch.float64).view(4, 1, 1)
    assert oracle.linear_attention(q, k, v, torch.ones_like(q)).flatten().tolist() == [2, 6, 12, 20]
    assert oracle.linear_attention(q, k, v, torch.zeros_like(q)).flatten().tolist() == [2, 4, 6, 8]
    # window of 5, blocks of 3: the block (3, 4, 5) is seen from position 10 on, (0, 1, 2) from 7 on
    assert oracle.visible(6, 5, 3) == ([2, 3, 4, 5, 6], [])
    assert oracle.visible(7, 5, 3) == ([3, 4, 5, 6, 7], [0])
    assert oracle.visible(9, 5, 3) == ([5, 6, 7, 8, 9], [0])
    assert oracle.visible(10, 5, 3) == ([6, 7, 8, 9, 10], [0, 1])
    assert oracle.visible(2, 5, None) == ([0, 1, 2], [])


def test_oracle_is_causal_and_notices_mistakes():
    cfg = config()
    w = oracle.random_weights(cfg, 0)
    tokens = torch.randint(0, 97, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = oracle.run(cfg, w, tokens)
    assert torch.allclose(full[:14], oracle.run(cfg, w, tokens[:14]), atol=1e-10)
    for plant, first in (("loses_state", 10), ("window_long", 9), ("window_short", 8), ("pool_early", 11), ("pool_none", 12),
                         ("no_sink", 0), ("no_average", 0), ("values_stay_turned", 1)):
        d = (oracle.run(cfg, w, tokens, plant=plant) - full).abs().amax(-1)
        assert float(d[first:].max()) > 1e-3, plant
        assert first == 0 or float(d[:first].max()) < 1e-9, plant
    assert oracle.greedy(cfg, w, tokens[:4], 3)[:4] == tokens[:4]
