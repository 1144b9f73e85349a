"""Pozalorn on the GPU: every mechanism's kernel against plain formulas, and the model through its own step function, cache
pool, generation and services against the plain implementation in ``pozalorn_oracle``."""
import json
import math

import pytest
import torch

import pozalorn_oracle as oracle
from test_pozalorn_cpu import SCALING, attention, config, dense, gla, parallel, write_model

pytestmark = pytest.mark.gpu

DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def mixers():
    from dart_pytorch_b200.ops import mixers as X
    return X


def rand(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(DEV, dtype)


def close(got, want, rel):
    want = want.to(torch.float64).to(got.device)
    err = (got.to(torch.float64) - want).abs().max() / want.abs().max().clamp_min(1e-30)
    assert float(err) <= rel, float(err)


# ------------------------------------------------------------------------------------------- linear attention --
def linear_case(dtype, B, T, H, dk, dv, rank, bias, silu=False, seed=1):
    """Projected rows, decay weights and the plain result (outputs, final state)."""
    from dart_pytorch_b200.nn.mixers import row_layout
    cols, n = row_layout(q=H * dk, k=H * dk, v=H * dv, r=max(rank, 1))
    p = rand(B * T, n + 8, seed=seed, dtype=dtype)
    w2 = rand(H * dk, rank, seed=seed + 1, dtype=dtype) if rank else None
    b2 = (rand(H * dk, seed=seed + 2) + bias).to(dtype) if rank else None
    return cols, p, w2, b2


def linear_want(cols, p, w2, b2, B, T, H, dk, dv, tau, q_scale, decay=None, silu=False):
    P = p.double().cpu().view(B, T, -1)
    act = oracle.silu if silu else (lambda z: z)
    outs, S = [], []
    for b in range(B):
        q = act(P[b, :, cols["q"]:cols["q"] + H * dk]).view(T, H, dk) * q_scale
        k = act(P[b, :, cols["k"]:cols["k"] + H * dk]).view(T, H, dk)
        v = act(P[b, :, cols["v"]:cols["v"] + H * dv]).view(T, H, dv)
        if decay is None:
            r = P[b, :, cols["r"]:cols["r"] + w2.shape[1]]
            z = r @ w2.double().cpu().t() + b2.double().cpu()
            a = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, H, dk)
        else:
            a = torch.tensor(decay, dtype=torch.float64).view(1, H, 1).expand(T, H, dk)
        outs.append(oracle.linear_attention(q, k, v, a).reshape(T, H * dv))
        s = torch.zeros(H, dk, dv, dtype=torch.float64)
        for t in range(T):
            s = a[t].unsqueeze(-1) * s + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        S.append(s)
    return torch.stack(outs), torch.stack(S)


def decay_table(decay):
    d = torch.tensor(decay, dtype=torch.float64)
    return torch.stack([d.log(), d - 1.0], 1).float().to(DEV)


def run_linear(cols, p, state, B, T, cut, H, dk, dv, **kw):
    X = mixers()
    P, at, outs = p.view(B, T, -1), 0, []
    for n in cut:
        n = min(n, T - at)
        if n <= 0:
            break
        rows = P[:, at:at + n].reshape(B * n, -1)
        outs.append(X.linear_attn(rows, cols, state, B, n, H, dk, dv, **kw).view(B, n, H * dv))
        at += n
    assert at == T
    return torch.cat(outs, 1)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,dk,dv,rank", [(1, 8, 8, 1), (3, 16, 24, 5), (2, 32, 64, 16), (2, 48, 136, 3), (1, 64, 40, 7),
                                          (2, 128, 72, 4), (1, 200, 64, 16), (2, 64, 128, 200), (3, 12, 6, 9), (1, 256, 128, 2), (2, 33, 16, 4)])
def test_gated_linear_attention(dtype, H, dk, dv, rank):
    B, T, tau, qs = 2, 150, 4.0, 0.3
    cols, p, w2, b2 = linear_case(dtype, B, T, H, dk, dv, rank, 2.0)
    want, S = linear_want(cols, p, w2, b2, B, T, H, dk, dv, tau, qs)
    for cut in ([T], [1] * T, [2] * 75, [15, 16, 17, 1, 63, 99], [64, 65, 99]):
        state = torch.zeros(B, H, dk, dv, device=DEV)
        o = run_linear(cols, p, state, B, T, cut, H, dk, dv, w2=w2, b2=b2, tau=tau, q_scale=qs)
        close(o, want, 2e-5 if dtype == F32 else 6e-3)
        close(state, S, 1e-5 if dtype == F32 else 5e-5)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("bias,tau,scale", [(9.0, 16.0, 1.0), (-6.0, 1.0, 3.0), (-30.0, 1.0, 10.0), (0.0, 0.25, 4.0)])
def test_long_and_short_memories(dtype, bias, tau, scale):
    """Decays next to 1, decays that wipe the state at once, and both in one piece."""
    B, T, H, dk, dv, rank = 1, 200, 2, 32, 16, 4
    cols, p, w2, b2 = linear_case(dtype, B, T, H, dk, dv, rank, bias)
    w2 = (w2.float() * scale).to(dtype)
    want, S = linear_want(cols, p, w2, b2, B, T, H, dk, dv, tau, 1.0)
    for cut in ([T], [1] * T, [100, 100]):
        state = torch.zeros(B, H, dk, dv, device=DEV)
        o = run_linear(cols, p, state, B, T, cut, H, dk, dv, w2=w2, b2=b2, tau=tau)
        close(o, want, 3e-5 if dtype == F32 else 6e-3)
        close(state, S, 3e-5 if dtype == F32 else 1e-4)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("decay", [[0.3], [0.9, 0.99999], [1.0, 0.6, 1e-3]])
def test_constant_decay(dtype, decay):
    B, T, H, dk, dv = 2, 170, len(decay), 24, 16
    cols, p, _, _ = linear_case(dtype, B, T, H, dk, dv, 0, 0.0)
    want, S = linear_want(cols, p, None, None, B, T, H, dk, dv, 1.0, 1.0, decay, silu=True)
    for cut in ([T], [1] * T, [31, 1, 64, 74]):
        state = torch.zeros(B, H, dk, dv, device=DEV)
        o = run_linear(cols, p, state, B, T, cut, H, dk, dv, decay=decay_table(decay), silu=True)
        close(o, want, 3e-5 if dtype == F32 else 1e-2)
        close(state, S, 3e-5 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("segments", [1, 2, 3, 7])
def test_segments_agree(segments):
    X = mixers()
    B, T, H, dk, dv, rank = 2, 64 * 7 - 5, 2, 32, 72, 4
    cols, p, w2, b2 = linear_case(BF, B, T, H, dk, dv, rank, 4.0)
    want, S = linear_want(cols, p, w2, b2, B, T, H, dk, dv, 8.0, 1.0)
    first = rand(B, H, dk, dv, seed=9)
    a = torch.exp(torch.nn.functional.logsigmoid((p[:, cols["r"]:cols["r"] + rank].double() @ w2.double().t() +
                                                  b2.double())) / 8.0).view(B, T, H, dk)
    state, fresh = first.clone(), torch.zeros_like(first)
    seg = -(-T // segments // 64) * 64
    n = -(-T // seg)
    kw = dict(w2=w2, b2=b2, tau=8.0, chunked=True, segments=n)
    close(X.linear_attn(p, cols, fresh, B, T, H, dk, dv, **kw).view(B, T, -1), want, 6e-3)
    close(fresh, S, 5e-5)
    # a state that was there before fades by the product of the decays and adds to every output
    o = X.linear_attn(p, cols, state, B, T, H, dk, dv, **kw).view(B, T, H, dv).double()
    fade = a.cumprod(1)
    q = p[:, :H * dk].double().view(B, T, H, dk)
    old = torch.einsum("bthd,bhde->bthe", q * fade, first.double())
    close(o, want.to(DEV).view(B, T, H, dv) + old, 6e-3)
    close(state, S.to(DEV) + fade[:, -1, :, :, None] * first.double(), 5e-5)


def test_a_single_key_stands_out_across_pieces():
    """One token's key is large and matches one query: the value comes back however far away, faded by the decay."""
    X = mixers()
    T, dk, dv = 400, 32, 16
    decay = 0.99
    for j in (0, 1, 63, 64, 65, 127, 128, 255):
        p = torch.zeros(T, 2 * dk + dv, device=DEV, dtype=BF)
        v = rand(dv, seed=j, dtype=BF)
        p[j, dk:2 * dk] = 1.0
        p[j, 2 * dk:] = v
        p[:, :dk] = 1.0 / dk
        state = torch.zeros(1, 1, dk, dv, device=DEV)
        o = X.linear_attn(p, {"q": 0, "k": dk, "v": 2 * dk}, state, 1, T, 1, dk, dv, decay=decay_table([decay]))
        for i in (j, j + 1, j + 63, j + 64, T - 1):
            close(o[i], v.double() * decay ** (i - j), 6e-3)
        assert j == 0 or float(o[:j].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("gate", ["silu", "sigmoid"])
@pytest.mark.parametrize("groups,n", [(3, 24), (1, 200), (4, 64), (2, 7), (1, 2056), (1, 5000), (2, 131)])
def test_head_norm_gate(dtype, gate, groups, n):
    rows, eps = 5, 1e-2
    o, w, g = rand(rows, groups * n, seed=1, dtype=dtype), rand(n, seed=2, dtype=dtype), rand(rows, groups * n + 8, seed=3, dtype=dtype)
    act = oracle.silu if gate == "silu" else torch.sigmoid
    want = (oracle.rms(o.double().view(rows, groups, n), eps) * w.double()).view(rows, -1) * act(g[:, :groups * n].double())
    close(mixers().head_norm_gate(o, w, g[:, :groups * n], eps, gate), want, 3e-6 if dtype == F32 else 5e-3)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("ff", [64, 21])
def test_gelu_gated_unit(dtype, ff):
    from dart_pytorch_b200.ops import kernels as K
    g, u = rand(9, ff, seed=1, dtype=dtype, scale=3.0), rand(9, ff, seed=2, dtype=dtype)
    close(K.geglu_fwd(g, u), oracle.gelu_tanh(g.double()) * u.double(), 2e-6 if dtype == F32 else 5e-3)


# ------------------------------------------------------------------------------------------- windowed attention --
def plain_window(q, k, v, pos, scale, size, pool, sink=None, turn=None):
    """``q [S, H, d]`` at positions ``pos ...`` over all keys so far; the pooled blocks are means of the given rows."""
    T = k.shape[0]
    full = torch.zeros(T, *q.shape[1:], dtype=torch.float64)
    full[pos:pos + q.shape[0]] = q.double().cpu()
    kd, vd = k.double().cpu(), v.double().cpu()
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[2], dtype=torch.float64)
    for s in range(q.shape[0]):
        i = pos + s
        js, bs = oracle.visible(i, size, pool)
        ks = torch.cat([kd[js]] + [kd[b * pool:(b + 1) * pool].mean(0, keepdim=True) for b in bs])
        vs = torch.cat([vd[js]] + [vd[b * pool:(b + 1) * pool].mean(0, keepdim=True) for b in bs])
        for h in range(H):
            z = ks[:, h // (H // G)] @ full[i, h] * scale
            m = z.max() if sink is None else torch.maximum(z.max(), sink[h].double().cpu())
            p = torch.exp(z - m)
            den = p.sum() + (torch.exp(sink[h].double().cpu() - m) if sink is not None else 0.0)
            out[s, h] = (p / den) @ vs[:, h // (H // G)]
    return out if turn is None else oracle.rotate(out, -torch.arange(pos, pos + q.shape[0]), turn)


class Windowed:
    """A WindowState fed with finished keys and values, and the three kernels over it."""

    def __init__(self, dtype, B, T, G, dk, dv, size, pool, turn_base=None, seed=1):
        from dart_pytorch_b200.nn.mixers import RotaryTable, WindowState
        self.dims = (G, dk, dv)
        self.k, self.v = rand(B, T, G * dk, seed=seed, dtype=dtype), rand(B, T, G * dv, seed=seed + 1, dtype=dtype)
        self.B, self.T, self.size, self.pool = B, T, size, pool
        self.rotary_v = RotaryTable(turn_base, dv) if turn_base else None
        self.state = WindowState(G * dk, G * dv, size, pool, None, self.rotary_v)
        self.state.grow(B, T, 0, dtype, DEV)

    def fill_ring(self, n):
        """The rings as they are once positions below ``n`` have been written; other rows hold garbage."""
        s = self.state
        s.k.fill_(float("nan"))
        s.v.fill_(float("nan"))
        for p in range(max(0, n - s.ring), n):
            s.k[:, p % s.ring], s.v[:, p % s.ring] = self.k[:, p], self.v[:, p]

    def pooled(self, n):
        X = mixers()
        if self.pool:
            s = self.state
            s.k_pool.fill_(77.0)
            s.v_pool.fill_(77.0)
            X.pool_blocks(self.k, self.v, s.k_pool, s.v_pool, self.B, pool=self.pool, first=0, count=n // self.pool)

    def ring_keys(self, n):
        self.fill_ring(n)
        self.pooled(n)
        s = self.state
        return mixers().WindowKeys(s.k, s.v, self.size, ring=True, pool=self.pool, k_pool=s.k_pool, v_pool=s.v_pool)

    def linear_keys(self, pos, S):
        self.pooled(pos + S)
        s = self.state
        lin0 = pos - min(pos, max(self.size - 1, self.pool))
        return mixers().WindowKeys(self.k[:, lin0:pos + S].contiguous(), self.v[:, lin0:pos + S].contiguous(), self.size,
                                   lin0=lin0, pool=self.pool, k_pool=s.k_pool, v_pool=s.v_pool)


WINDOW_SIZES = [(BF, 2, 1, 64, 64), (BF, 4, 2, 32, 48), (BF, 3, 3, 96, 128), (BF, 8, 1, 128, 40), (BF, 4, 2, 64, 8), (BF, 2, 2, 20, 12),
                (F32, 4, 2, 24, 40), (F32, 3, 1, 130, 6), (BF, 9, 1, 16, 16)]


@pytest.mark.parametrize("dtype,H,G,dk,dv", WINDOW_SIZES)
@pytest.mark.parametrize("size,pool,sink,turned", [(9, 4, False, True), (40, 0, True, False), (1, 1, True, True), (70, 16, True, True),
                                                   (5, 11, False, False)])
def test_window_kernels_in_decoding(dtype, H, G, dk, dv, size, pool, sink, turned):
    X = mixers()
    B, T = 2, 300
    w = Windowed(dtype, B, T, G, dk, dv, size, pool, 300.0 if turned else None)
    sk = rand(H, seed=5, dtype=dtype, scale=2.0) if sink else None
    turn = w.rotary_v.frequencies() if turned else None
    scale = 1.5 / math.sqrt(dk)
    for pos, S in ((0, 1), (3, 1), (size - 1, 1), (size, 1), (size + pool, 2), (100, 7), (255, 32), (299, 1)):
        keys = w.ring_keys(pos + S)
        q = rand(B * S, H * dk, seed=pos, dtype=dtype)
        want = torch.stack([plain_window(q.view(B, S, H, dk)[b], w.k[b].view(T, G, dk), w.v[b].view(T, G, dv), pos, scale, size,
                                         pool, sk, turn) for b in range(B)])
        rel = 2e-5 if dtype == F32 else 1.2e-2           # pooled rows are rounded to bf16
        args = (q, keys, B, S, H, G, dk, dv, pos, scale)
        close(X.window_attn(*args, sink=sk, rot=w.state.rot_v).view(want.shape), want, rel)
        if X.window_decode_ok(dtype, H, G, dk, dv):
            for splits in (1, 3, X.window_decode_plan(B * S, H, G, dk, dv, 400)[0]):
                ws = torch.full((B * S * H * splits * 130,), float("nan"), device=DEV)
                o = X.window_attn_decode(*args, sink=sk, rot=w.state.rot_v, splits=splits, ws=ws)
                close(o.view(want.shape), want, rel)
            if S == 1:
                at = torch.tensor([pos], dtype=torch.int32, device=DEV)
                o = X.window_attn_decode(q, keys, B, 1, H, G, dk, dv, 0, scale, sink=sk, rot=w.state.rot_v, pos_ptr=at)
                close(o.view(want.shape), want, rel)


@pytest.mark.parametrize("dtype,H,G,dk,dv", WINDOW_SIZES)
@pytest.mark.parametrize("size,pool,sink,turned", [(9, 4, False, True), (130, 0, True, False), (70, 16, True, True), (300, 3, True, False),
                                                   (5, 11, False, False)])
@pytest.mark.parametrize("pos,S", [(0, 33), (0, 300), (37, 129), (200, 257)])
def test_window_kernels_in_prompts(dtype, H, G, dk, dv, size, pool, sink, turned, pos, S):
    X = mixers()
    B, T = 2, pos + S
    w = Windowed(dtype, B, T, G, dk, dv, size, pool, 300.0 if turned else None)
    sk = rand(H, seed=5, dtype=dtype, scale=2.0) if sink else None
    turn = w.rotary_v.frequencies() if turned else None
    scale = 1.5 / math.sqrt(dk)
    keys = w.linear_keys(pos, S)
    q = rand(B * S, H * dk, seed=3, dtype=dtype)
    rows = sorted({r for r in (0, 1, size - 1, size, size + pool - 1, S // 2, 63, 64, 127, 128, 255, 256, S - 1) if r < S})
    args = (q, keys, B, S, H, G, dk, dv, pos, scale)
    want = torch.stack([torch.cat([plain_window(q.view(B, S, H, dk)[b, r:r + 1], w.k[b].view(T, G, dk), w.v[b].view(T, G, dv),
                                                pos + r, scale, size, pool, sk, turn) for r in rows]) for b in range(B)])
    outs = [X.window_attn(*args, sink=sk, rot=w.state.rot_v)]
    if X.window_flash_ok(dtype, dk, dv, scale):
        outs.append(X.window_attn_fwd(*args, sink=sk, rot=w.state.rot_v))
    for o in outs:
        close(o.view(B, S, H, dv)[:, rows], want, 2e-5 if dtype == F32 else 1.2e-2)
    if len(outs) > 1:                                    # every row, against the generic kernel
        close(outs[1], outs[0], 1.2e-2)


@pytest.mark.parametrize("dtype,dk,pool", [(BF, 64, 8), (F32, 48, 8), (BF, 128, 5), (BF, 20, 3)])
def test_single_keys_at_the_edges_stand_out(dtype, dk, pool):
    """A query aligned with one key returns its value while the key is in the window, a share of it as part of a pooled block,
    and nothing in between: one token inside and outside of every edge, in prompts and in decoding."""
    X = mixers()
    T, size = 220, 37
    w = Windowed(dtype, 1, T, 1, dk, dk, size, pool)
    w.k[:] = 0.0
    w.v[:] = 0.0
    for j in (0, 1, pool - 1, pool, 40, 63, 64, 100, 127, 128, 150):
        w.k[0, j], w.v[0, j] = 1.0, 1.0
        q = torch.ones(T, dk, device=DEV, dtype=dtype)
        scale = 600.0 / dk                               # 600 against the key, 600 / pool against its block
        keys = w.linear_keys(0, T)
        outs = [X.window_attn(q, keys, 1, T, 1, 1, dk, dk, 0, scale)[:, 0]]
        if X.window_flash_ok(dtype, dk, dk, scale):
            outs.append(X.window_attn_fwd(q, keys, 1, T, 1, 1, dk, dk, 0, scale)[:, 0])
        seen = j // pool * pool + pool - 1 + size        # first query that sees the key's block
        for i in sorted({j - 1, j, j + 1, j + size - 1, j + size, seen - 1, seen, seen + 1, T - 1}):
            if not 0 <= i < T:
                continue
            want = 1.0 if j <= i < j + size else 1.0 / pool if i >= seen else 0.0
            got = [float(o[i]) for o in outs]
            ring = w.ring_keys(i + 1)
            got.append(float(X.window_attn(q[:1], ring, 1, 1, 1, 1, dk, dk, i, scale)[0, 0]))
            if X.window_decode_ok(dtype, 1, 1, dk, dk):
                ws = torch.empty(4 * 130, device=DEV)
                got.append(float(X.window_attn_decode(q[:1], ring, 1, 1, 1, 1, dk, dk, i, scale)[0, 0]))
                got.append(float(X.window_attn_decode(q[:1], ring, 1, 1, 1, 1, dk, dk, i, scale, splits=4, ws=ws)[0, 0]))
            assert all(abs(x - want) < 0.01 for x in got), (i, j, want, got)
        w.k[0, j], w.v[0, j] = 0.0, 0.0


@pytest.mark.parametrize("sink", [-30.0, 0.0, 5.0, 40.0])
def test_sink_takes_its_share(sink):
    """Equal scores: every output is a known share of the values."""
    X = mixers()
    T, dk, size = 100, 64, 20
    w = Windowed(BF, 1, T, 1, dk, dk, size, 0)
    w.k[:] = 0.0
    w.v[:] = 1.0
    sk = torch.tensor([sink], device=DEV, dtype=BF)
    q = rand(T, dk, dtype=BF)
    n = torch.arange(1, T + 1).clamp(max=size).double()
    want = n / (n + math.exp(sink))
    for o in (X.window_attn_fwd(q, w.linear_keys(0, T), 1, T, 1, 1, dk, dk, 0, 1.0, sink=sk),
              X.window_attn(q, w.linear_keys(0, T), 1, T, 1, 1, dk, dk, 0, 1.0, sink=sk)):
        assert float((o[:, 0].double().cpu() / want - 1.0).abs().max()) < 6e-3
    for splits in (1, 3):
        o = X.window_attn_decode(q[:1], w.ring_keys(T), 1, 1, 1, 1, dk, dk, T - 1, 1.0, sink=sk, splits=splits,
                                 ws=torch.empty(splits * 130, device=DEV))
        assert abs(float(o[0, 0]) / float(want[-1]) - 1.0) < 6e-3


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 16, 24, 8), (3, 1, 18, 10, 18), (2, 2, 40, 8, 2), (6, 3, 64, 64, 64)])
@pytest.mark.parametrize("norm", [None, "head", "together"])
def test_norms_and_rotations_of_a_row(dtype, H, G, dk, dv, rot, norm):
    from dart_pytorch_b200.nn.mixers import RotaryTable, row_layout
    X = mixers()
    B, S, pos, ring, eps = 2, 6, 5, 16, 1e-2
    cols, n = row_layout(q=H * dk, k=G * dk, v=G * dv)
    p = rand(B * S, n, seed=1, dtype=dtype)
    tab, tab_v = RotaryTable(500.0, rot, SCALING), RotaryTable(500.0, dv)
    gq = rand(H * dk if norm == "together" else dk, seed=2, dtype=dtype) if norm else None
    gk = rand(G * dk if norm == "together" else dk, seed=3, dtype=dtype) if norm else None
    rings = [torch.zeros(B, ring, G * d, device=DEV, dtype=dtype) for d in (dk, dv)]
    lin = [torch.zeros(B, 3 + S, G * d, device=DEV, dtype=dtype) for d in (dk, dv)]
    at = torch.tensor([pos], dtype=torch.int32, device=DEV)
    q = X.qkv_prep(p, cols, B, S, H, G, dk, dv, eps=eps, gq=gq, gk=gk, whole=norm == "together", rot=tab.rows(64, DEV),
                   rot_v=tab_v.rows(64, DEV), k_ring=rings[0], v_ring=rings[1], pos=0, pos_ptr=at, k_lin=lin[0], v_lin=lin[1], hist=3)
    P = p.double().cpu()

    def part(name, heads, d, g):
        x = P[:, cols[name]:cols[name] + heads * d]
        if g is not None:
            g = g.double().cpu()
            x = oracle.rms(x, eps) * g if norm == "together" else oracle.rms(x.view(-1, heads, d), eps) * g
        return x.reshape(B, S, heads, d)
    where = torch.arange(pos, pos + S)
    turn = lambda x, f: torch.stack([oracle.rotate(x[b], where, f) for b in range(B)])  # noqa: E731
    rel = 2e-6 if dtype == F32 else 5e-3
    close(q.view(B, S, H, dk), turn(part("q", H, dk, gq), tab.frequencies()), rel)
    for i, (name, d, g, f) in enumerate((("k", dk, gk, tab.frequencies()), ("v", dv, None, tab_v.frequencies()))):
        want = turn(part(name, G, d, g), f).reshape(B, S, G * d)
        close(rings[i][:, pos:pos + S], want, rel)
        assert torch.equal(lin[i][:, 3:], rings[i][:, pos:pos + S]) and float(lin[i][:, :3].abs().sum()) == 0
        assert float(rings[i][:, :pos].abs().sum()) == 0 and float(rings[i][:, pos + S:].abs().sum()) == 0


# ------------------------------------------------------------------------------------------- residual stream --
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("D", [40, 37, 1032, 2048, 4096])
def test_branch_norm(dtype, D):
    X = mixers()
    M, eps = 7, 1e-2
    x, m1, m2, w, wf = rand(M, D, seed=1), *(rand(M, D, seed=s, dtype=dtype) for s in (2, 3)), *(rand(D, seed=s, dtype=dtype) for s in (4, 5))
    stack, avg = rand(6, M, D, seed=6), rand(5, seed=7, dtype=dtype)
    d = lambda t: t.double()  # noqa: E731
    want = d(x) + oracle.rms(0.7 * d(m1) - 0.2 * d(m2), eps) * d(w)
    mean = sum(d(avg[j]) * d(stack[j]) for j in range(4)) + d(avg[4]) * want
    result, x_out = torch.empty(M, D, device=DEV), torch.empty(M, D, device=DEV)
    h = X.branch_norm(x, M, D, dtype, eps, m1=m1, m2=m2, c1=0.7, c2=-0.2, w=w, stack=stack, n=4, avg=avg, result=result, x_out=x_out)
    rel = 3e-6 if dtype == F32 else 5e-3
    close(result, want, 3e-6)
    close(x_out, mean, 3e-6)
    close(h, mean, rel)
    pick = torch.tensor([5, 0, 2], dtype=torch.int32, device=DEV)
    h = X.branch_norm(x, 3, D, dtype, eps, m1=m1, m2=m2, c1=0.7, c2=-0.2, w=w, stack=stack, n=4, avg=avg, wf=wf, pick=pick)
    close(h, (oracle.rms(mean, eps) * d(wf))[pick.long()], rel)
    table, tokens = rand(11, D, seed=8, dtype=dtype), torch.randint(0, 11, (M,), device=DEV)
    h = X.branch_norm(None, M, D, dtype, eps, embed=table, tokens=tokens, result=result)
    assert torch.equal(h, table[tokens]) and torch.equal(result, table[tokens].float())


# ------------------------------------------------------------------------------------------- the model --
CONFIGS = {
    "mixed": config([gla(dense()), attention(dense(56)), gla(), parallel(dense(24), size=21), attention(size=30, pool=7)], width=64,
                    vocab=130),
    "linear_only": config([gla(dense(), heads=2, dim=32, vdim=48), gla(heads=5, dim=8, vdim=8, tau=1.0)], width=48),
    "windows_only": config([attention(dense(), size=33, pool=1, heads=2, kv_heads=2, dim=64, vdim=64, rot=64),
                            attention(size=1, pool=2, heads=6, kv_heads=1, dim=24, vdim=40, rot=6, scaled=False)], width=56),
    "parallel_only": config([parallel(dense(), size=1, heads=1), parallel(size=65, heads=4, dim=40, vdim=48, left_scale=1.0,
                                                                          right_scale=-0.5, decay=[0.2, 0.9, 0.99, 1.0])], width=72),
    "odd_sizes": config([gla(dense(21), heads=3, dim=10, vdim=6), attention(heads=3, kv_heads=3, dim=10, vdim=14, rot=4, size=12, pool=5),
                         parallel(dense(10), heads=2, dim=6, vdim=10, size=7)], width=38, vocab=75),
    "wide_heads": config([attention(dense(128), heads=4, kv_heads=2, dim=128, vdim=96, rot=64, size=50, pool=16),
                          gla(dense(128), heads=2, dim=128, vdim=128), parallel(heads=2, dim=64, vdim=128, size=100)], width=128,
                         vocab=256),
}


def build(name, dtype, seed=0, cfg=None, weights=None):
    from dart_pytorch_b200.io.pozalorn_loader import PozalornLoader
    from dart_pytorch_b200.models.pozalorn import Pozalorn, PozalornConfig
    cfg = cfg or CONFIGS[name]
    w = weights or oracle.random_weights(cfg, seed)
    m = Pozalorn(PozalornConfig.from_json(cfg, w, device=DEV, dtype=dtype))
    PozalornLoader.load_map(m, w)
    return cfg, w, m


def prompt(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cut(m, tokens, cut):
    cache = m.new_cache(len(tokens))
    at, outs = 0, []
    for n in cut:
        n = min(n, len(tokens) - at)
        if n <= 0:
            break
        outs.append(m.step(cache, torch.tensor([tokens[at:at + n]], device=DEV)).clone())
        at += n
    m.free_cache(cache)
    assert at == len(tokens)
    return torch.cat(outs)


def errors(got, want):
    """rms of the difference per position over the rms of the logits."""
    want = want.to(got.device).double()
    return (got.double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def check_model(got, want, dtype):
    e = errors(got, want)
    if dtype == F32:
        assert float(e.max()) < 5e-5, float(e.max())
    else:
        assert float(e.median()) < 0.03 and float(e.max()) < 0.12, (float(e.median()), float(e.max()))


CUTS = {"whole": [999], "one_by_one": [1] * 200, "twos": [2] * 100, "portions": [3, 31, 32, 33, 1, 1, 64, 7, 999],
        "prompt_then_decode": [96] + [1] * 100, "sixty_fives": [65] * 9, "fifteens": [15, 16, 17] * 9}


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_model_against_plain(name, dtype):
    cfg, w, m = build(name, dtype)
    tokens = prompt(cfg, 140)
    want = oracle.run(cfg, w, tokens)
    for cut in CUTS.values():
        check_model(run_cut(m, tokens, cut), want, dtype)


@pytest.mark.parametrize("plant,first", [("loses_state", 10), ("window_long", 21), ("window_short", 9), ("pool_early", 12),
                                         ("pool_none", 12), ("no_sink", 0), ("no_average", 0), ("values_stay_turned", 1)])
def test_model_differs_from_planted_mistakes(plant, first):
    cfg, w, m = build("mixed", F32)
    tokens = prompt(cfg, 60)
    got = run_cut(m, tokens, [45] + [1] * 40)
    check_model(got, oracle.run(cfg, w, tokens), F32)
    assert float(errors(got, oracle.run(cfg, w, tokens, plant=plant))[first:].max()) > 1e-3


@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_bf16_cuts_agree_closely(name):
    """The same weights and tokens cut differently: no further apart than rounding."""
    cfg, _, m = build(name, BF)
    tokens = prompt(cfg, 140)
    whole = run_cut(m, tokens, CUTS["whole"])
    for cut_name, cut in CUTS.items():
        e = errors(run_cut(m, tokens, cut), whole)
        assert float(e.max()) < 0.1 and float(e.median()) < 0.03, cut_name


def test_batches_against_each_alone():
    for dtype in (F32, BF):
        cfg, _, m = build("mixed", dtype)
        rows = [prompt(cfg, 80, seed=s) for s in (3, 4, 5)]
        for cut in ([80], [33, 47], [40] + [1] * 40, [2] * 40):
            cache = m.new_cache(80, batch=3)
            t = torch.tensor(rows, device=DEV)
            at, outs = 0, []
            for n in cut:
                outs.append(m.step(cache, t[:, at:at + n]).view(3, n, -1).clone())
                at += n
            m.free_cache(cache)
            got = torch.cat(outs, 1)
            for b in range(3):
                e = errors(got[b], run_cut(m, rows[b], cut))
                assert float(e.max()) < (2e-5 if dtype == F32 else 0.08)


def test_reused_state_starts_clean():
    cfg, w, m = build("mixed", F32)
    a, b = prompt(cfg, 120, seed=8), prompt(cfg, 60, seed=9)
    fresh = run_cut(m, b, [45] + [1] * 15)
    run_cut(m, a, [100] + [1] * 20)
    c1 = m.new_cache(120)
    m.step(c1, torch.tensor([a], device=DEV))
    m.free_cache(c1)
    c2 = m.new_cache(60)
    assert c2 is c1 and c2.seq_len == 0
    m.free_cache(c2)
    again = run_cut(m, b, [45] + [1] * 15)
    assert torch.equal(fresh, again)
    check_model(again, oracle.run(cfg, w, b), F32)


def test_two_requests_interleaved():
    cfg, w, m = build("mixed", F32)
    a, b = prompt(cfg, 70, seed=10), prompt(cfg, 70, seed=11)
    ca, cb = m.new_cache(70), m.new_cache(70)
    assert ca is not cb
    got = {0: [], 1: []}
    for lo, hi in ((0, 40), (40, 41), (41, 42), (42, 61), (61, 62), (62, 70)):
        for k, (c, t) in enumerate(((ca, a), (cb, b))):
            got[k].append(m.step(c, torch.tensor([t[lo:hi]], device=DEV)).clone())
    check_model(torch.cat(got[0]), oracle.run(cfg, w, a), F32)
    check_model(torch.cat(got[1]), oracle.run(cfg, w, b), F32)


def test_cache_grows_under_a_captured_step():
    cfg, w, m = build("mixed", F32)
    tokens = prompt(cfg, 150)
    cache = m.new_cache(4)
    assert cache.capacity == 128
    outs = [m.step(cache, torch.tensor([tokens[:120]], device=DEV))]
    for t in tokens[120:]:
        outs.append(m.step(cache, torch.tensor([[t]], device=DEV)).clone())
    assert cache.capacity == 256
    check_model(torch.cat(outs), oracle.run(cfg, w, tokens), F32)


@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_captured_and_direct_decode_agree(monkeypatch, name):
    cfg, _, m = build(name, BF)
    tokens = prompt(cfg, 90)
    a = run_cut(m, tokens, [40] + [1] * 50)
    monkeypatch.setenv("DPTB200_DECODE_GRAPH", "0")
    assert float(errors(a, run_cut(m, tokens, [40] + [1] * 50)).max()) < 1e-2


@pytest.mark.parametrize("dtype", [F32, BF])
def test_long_decoding(dtype):
    """Memories of thousands of tokens, windows that pass over decoded tokens many times, pooled rows far back."""
    cfg = config([gla(dense(), heads=2, dim=16, vdim=16, tau=16.0), attention(size=20, pool=6, heads=2, dim=16, vdim=16),
                  parallel(heads=2, dim=16, vdim=16, decay=[0.9999, 0.99], size=50)], width=32, vocab=50)
    w = oracle.random_weights(cfg, 0)
    w["l0.mix.a2.b"] = torch.full((32,), 8.0)
    cfg, w, m = build(None, dtype, cfg=cfg, weights=w)
    tokens = prompt(cfg, 700)
    want = oracle.run(cfg, w, tokens)
    check_model(run_cut(m, tokens, [10] + [1] * 690), want, dtype)
    check_model(run_cut(m, tokens, [700]), want, dtype)


def test_far_token_shows():
    """A changed first token changes the last logits through states and pooled rows, and the model follows the change."""
    cfg, w, m = build("mixed", F32)
    tokens = prompt(cfg, 200)
    other = [(tokens[0] + 1) % cfg["vocab"]] + tokens[1:]
    want = oracle.run(cfg, w, tokens)[-1:], oracle.run(cfg, w, other)[-1:]
    moved = float(errors(want[1].to(DEV), want[0]))
    for cut in ([200], [150] + [1] * 50, [64] * 4):
        for t, x in zip((tokens, other), want):
            e = errors(run_cut(m, t, cut)[-1:], x)
            assert float(e.max()) < 5e-5 and float(e.max()) < 0.2 * moved


def test_first_tokens_alone():
    cfg, w, m = build("mixed", F32)
    for n in (1, 2, 3):
        tokens = prompt(cfg, n)
        for cut in ([n], [1] * n):
            check_model(run_cut(m, tokens, cut), oracle.run(cfg, w, tokens), F32)


def test_wanted_rows_only():
    cfg, _, m = build("mixed", F32)
    t = torch.tensor([prompt(cfg, 50)], device=DEV)
    c = m.new_cache(60)
    full = m.step(c, t).clone()
    m.free_cache(c)
    c = m.new_cache(60)
    assert float(errors(m.step(c, t[:, :40], [39, 3]), full[[39, 3]]).max()) < 1e-5
    assert m.step(c, t[:, 40:45], []).shape == (0, cfg["vocab"])
    assert float(errors(m.step(c, t[:, 45:], [4]), full[49:]).max()) < 1e-5
    m.free_cache(c)


def test_generation_and_services(tmp_path):
    """Greedy ids through generate, generate_batch and the service equal the plain implementation's."""
    from dart_pytorch_b200.apps.servers import GenerationService, load_hf_model
    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 21, rank=9)
    write_model(tmp_path / "m", cfg, w)
    m, _, _ = load_hf_model("auto", str(tmp_path / "m"), device=DEV, dtype=F32)
    p = prompt(cfg, 9)
    want = oracle.greedy(cfg, w, p, 14)
    assert [int(t) for t in m.generate(p, 14, temperature=0.0)] == want
    assert [int(t) for t in m.generate(p, 14, temperature=0.0, use_cache=False)] == want
    q = prompt(cfg, 9, seed=2)
    both = m.generate_batch(torch.tensor([p, q]), 14)
    assert both.tolist() == [want, oracle.greedy(cfg, w, q, 14)]
    code, out = GenerationService(m).run({"tokens": p, "maxNewTokens": 14})
    assert code == 200 and out["tokens"] == want
    assert GenerationService(m).info()["vocabSize"] == cfg["vocab"]
    sampled = m.generate(p, 5, temperature=0.8, top_k=4)
    assert len(sampled) == 14 and all(0 <= t < cfg["vocab"] for t in sampled)
    assert torch.isfinite(m.hidden(torch.tensor(p))).all() and m(torch.tensor(p)).shape == (9, cfg["vocab"])


def test_command_line(tmp_path, capsys):
    from dart_pytorch_b200.apps.__main__ import main
    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 22)
    write_model(tmp_path / "m", cfg, w)
    p = prompt(cfg, 6)
    main(["pozalorn", str(tmp_path / "m"), "--tokens", ",".join(map(str, p)), "--max-new-tokens", "4"])
    text = capsys.readouterr().out
    assert json.loads(text[text.index("{"):text.rindex("}") + 1])["tokens"] == oracle.greedy(cfg, w, p, 4)


def test_trace_replay(tmp_path):
    from dart_pytorch_b200.apps.servers import load_hf_model
    from dart_pytorch_b200.apps.trace_run import TraceRunner
    cfg = CONFIGS["odd_sizes"]
    w = oracle.random_weights(cfg, 23)
    write_model(tmp_path / "m", cfg, w)
    m, _, _ = load_hf_model("auto", str(tmp_path / "m"), device=DEV, dtype=F32)
    a, b = prompt(cfg, 60), prompt(cfg, 7, seed=5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:43], "want": [42]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[43:44], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[44:], "want": [0, 15]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [6]}], "end": ["b"]}]
    TraceRunner(m, 60).run([json.dumps(s) for s in steps], str(tmp_path), lambda s: None)
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=F32).view(-1, cfg["vocab"])  # noqa: E731
    wa, wb = oracle.run(cfg, w, a), oracle.run(cfg, w, b)
    for n, want in ((0, wa[[42]]), (1, wa[[43]]), (2, wa[[44, 59]]), (3, wb[[6]])):
        check_model(read(n), want, F32)
