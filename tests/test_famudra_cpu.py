"""Famudra without a GPU: configuration, registry, checkpoint loading, state bookkeeping, the trace replay's protocol, and
the plain implementation the GPU tests compare against (checked against itself and for the mistakes it should expose)."""
import copy
import json

import pytest
import torch

import famudra_oracle as oracle
from dart_pytorch_b200.apps.servers import load_hf_model
from dart_pytorch_b200.apps.trace_run import TraceRunner
from dart_pytorch_b200.io.famudra_loader import FamudraLoader
from dart_pytorch_b200.io.safetensors import SafeTensors
from dart_pytorch_b200.models import registry
from dart_pytorch_b200.models.famudra import Famudra, FamudraConfig
from dart_pytorch_b200.nn.hybrid import CachePool, HybridCache, LatentState, RecurrentState


def attention(**kw):
    return dict(dict(heads=2, dim=12, vdim=20, q_rank=24, kv_rank=32, scale=0.3), **kw)


def moe(experts=5, top=2, ff=16, shared=24):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers=None, loop=None, width=40, vocab=97):
    layers = layers or [{"type": "rglru", "mixer": {"width": 24, "blocks": 3, "conv": 3}, "mlp": moe()},
                        {"type": "latent_attention", "mixer": attention(), "mlp": None}]
    out = {"architecture": "Famudra", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers}
    if loop:
        out["loop"] = loop
    return out


def write_model(path, cfg, weights):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    SafeTensors.save_file(weights, str(path / "model.safetensors"), dtype="BF16")


def test_registry_names_families():
    assert registry.family_of({"architecture": "Famudra"}) == "famudra"
    assert registry.family_of({"model_type": "gpt_neox"}) == "pythia"
    with pytest.raises(ValueError):
        registry.family_of({"model_type": "unheard_of"})


def test_config_reads_everything_and_validates():
    c = FamudraConfig.from_json(config(loop={"start": 0, "stop": 1, "times": 3}))
    assert c.schedule == [(0, False), (0, True), (0, True), (1, False)]
    assert (c.vocab_size, c.width, c.norm_eps, c.num_heads) == (97, 40, 1e-5, 2)
    assert FamudraConfig.from_json(config()).schedule == [(0, False), (1, False)]
    with pytest.raises(ValueError):
        FamudraConfig.from_json(config(loop={"start": 1, "stop": 3, "times": 2}))
    bad = config()
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError):
        FamudraConfig.from_json(bad)
    lacks = config()
    del lacks["layers"][1]["mixer"]["scale"]
    with pytest.raises(ValueError, match="scale"):
        FamudraConfig.from_json(lacks)


def test_checkpoint_round_trip(tmp_path):
    cfg = config(loop={"start": 0, "stop": 2, "times": 2})
    w = oracle.random_weights(cfg, 3)
    write_model(tmp_path / "m", cfg, w)
    model, tok, report = load_hf_model("auto", str(tmp_path / "m"), device="cpu")
    assert isinstance(model, Famudra) and tok is None and report.unused_keys == []
    back = FamudraLoader.dump(model)
    assert set(back) == set(w)
    for k in w:
        assert back[k].shape == w[k].shape and torch.equal(back[k], w[k]), k
    missing = dict(w)
    del missing["l0.mix.lam"]
    with pytest.raises(ValueError, match="l0.mix.lam"):
        FamudraLoader.load_map(model, missing)
    wrong = dict(w)
    wrong["l1.mix.uk"] = torch.zeros(24, 31)
    with pytest.raises(ValueError, match="l1.mix.uk"):
        FamudraLoader.load_map(model, wrong)


def test_no_cpu_path():
    model = Famudra(FamudraConfig.from_json(config()))
    cache = model.new_cache(8)
    with pytest.raises(RuntimeError, match="CUDA"):
        model.step(cache, torch.zeros(1, 3, dtype=torch.long))


def test_cache_growth_reset_and_pool():
    states = [LatentState(8), RecurrentState(6, 4)]
    cache = HybridCache(states, 5, 2, 100, torch.float32, "cpu", counters=4)
    assert cache.capacity == 128 and states[0].buf.shape == (2, 128, 8)
    assert states[1].conv.shape == (2, 3, 6) and states[1].s.shape == (2, 6) and len(cache.shift) == 2
    assert all(s.data_ptr() % 16 == 0 for s in cache.shift)
    states[0].buf[:, :128] = 1.0
    states[1].s.fill_(2.0)
    cache.shift[1].fill_(3.0)
    cache.advance(128)
    cache.graph = object()
    cache.ensure(129)
    assert cache.capacity == 256 and cache.graph is None            # a captured step addresses the old buffers
    assert bool((states[0].buf[:, :128] == 1).all()) and bool((states[0].buf[:, 128:] == 0).all())
    assert int(cache.pos) == 128
    cache.reset()
    assert cache.seq_len == 0 and int(cache.pos) == 0 and float(cache.flat.abs().sum()) == 0.0
    pool = CachePool(lambda b, n: HybridCache([LatentState(8)], 5, b, n, torch.float32, "cpu"), keep=2)
    a, b = pool.acquire(1, 100), pool.acquire(1, 300)
    pool.release(a)
    pool.release(b)
    assert pool.acquire(2, 10) not in (a, b)                         # another batch
    assert pool.acquire(1, 200) is b                                 # the one that is large enough
    assert pool.acquire(1, 50) is a


class _FakeModel:
    """Counts tokens per request; the 'logits' of a place are (tokens before it, its token)."""
    device = torch.device("cpu")

    def __init__(self):
        self.freed, self.made = [], 0

    def new_cache(self, n):
        self.made += 1
        return {"n": 0, "id": self.made}

    def free_cache(self, c):
        self.freed.append(c["id"])

    def step(self, cache, tokens, rows):
        out = [[float(cache["n"] + r), float(tokens[0, r])] for r in rows]
        cache["n"] += tokens.shape[1]
        return torch.tensor(out).reshape(-1, 2)


def test_trace_replay_protocol(tmp_path):
    m = _FakeModel()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [9], "want": [0]}, {"id": "b", "tokens": [1, 2], "want": [1]}],
              "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [3], "want": [0]}], "end": ["a", "b"]}]
    said = []
    TraceRunner(m).run([json.dumps(s) for s in steps] + [""], str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 2)  # noqa: E731
    assert read(0).tolist() == [[0, 5], [2, 7]]
    assert not (tmp_path / "1.f32").exists()
    assert read(2).tolist() == [[4, 9], [1, 2]]
    assert read(3).tolist() == [[0, 3]]                               # a new request of the same name starts over
    assert m.made == 3 and sorted(m.freed) == [1, 2, 3]


def test_oracle_is_causal_and_notices_mistakes():
    cfg = config(loop={"start": 1, "stop": 2, "times": 2})
    w = oracle.random_weights(cfg, 0)
    tokens = torch.randint(0, 97, (20,), generator=torch.Generator().manual_seed(1)).tolist()
    full = oracle.run(cfg, w, tokens)
    head = oracle.run(cfg, w, tokens[:9])
    assert torch.allclose(full[:9], head, atol=1e-10)
    for plant in ("misses_own_key", "misses_first_key", "loop_without_embedding"):
        assert (oracle.run(cfg, w, tokens, plant=plant)[1:] - full[1:]).abs().amax(-1).min() > 1e-3, plant
    no_shift = copy.copy(w)
    no_shift["l1.shift"] = torch.zeros(40)
    assert (oracle.run(cfg, no_shift, tokens) - full).abs().max() > 1e-2
    assert oracle.greedy(cfg, w, tokens[:4], 3)[:4] == tokens[:4]
