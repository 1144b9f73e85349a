"""Plain, slow implementation of the Pozalorn equations (one function per mechanism, fp32 or fp64 on the CPU).

The oracle of the Pozalorn tests.  It shares no code with the package: it reads the same flat ``{name: tensor}`` weights and
the same configuration dictionary and processes one whole sequence at a time, recurrences token by token and attention
query by query.  ``run(..., plant=...)`` plants one of a few mistakes, for tests that check that a test would notice it.
"""
import math

import torch


def rms(x, eps):
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------- linear attention --
def linear_attention(q, k, v, decay):
    """``S_t = diag(decay_t) S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t``; ``q, k, decay [T, H, d]``, ``v [T, H, e]``."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = (S * q[t].unsqueeze(-1)).sum(1)
    return out


def key_channel_decay(h, a1, a2, bias, tau):
    """``sigmoid(a2 (a1 h) + bias)^(1 / tau)``."""
    z = (h @ a1.t()) @ a2.t() + bias
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gla(h, w, m, eps, plant=None):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].t()).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].t()).view(T, H, d)
    v = (h @ w["v"].t()).view(T, H, e)
    decay = key_channel_decay(h, w["a1"], w["a2"], w["a2.b"], m["tau"]).view(T, H, d)
    if plant == "loses_state" and T > 10:
        o = torch.cat([linear_attention(q[:10], k[:10], v[:10], decay[:10]),
                       linear_attention(q[10:], k[10:], v[10:], decay[10:])])
    else:
        o = linear_attention(q, k, v, decay)
    o = (rms(o, eps) * w["norm"]).reshape(T, H * e)
    return (o * silu(h @ w["g"].t())) @ w["o"].t()


def lightning(h, w, m, eps, plant=None):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = silu(h @ w["q"].t()).view(T, H, d), silu(h @ w["k"].t()).view(T, H, d), silu(h @ w["v"].t()).view(T, H, e)
    decay = torch.tensor(m["decay"], dtype=h.dtype).view(1, H, 1).expand(T, H, d)
    o = linear_attention(q, k, v, decay).reshape(T, H * e)
    return (rms(o, eps) * w["norm"] * torch.sigmoid(h @ w["g"].t())) @ w["o"].t()


# ------------------------------------------------------------------------------------------------- attention --
def frequencies(rot):
    """Angle per position of every pair, with the wavelength-dependent scaling when the configuration has one."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, pos, freq):
    """Turns the pairs ``(2i, 2i + 1)`` of ``x [T, H, d]`` by ``pos[t] * freq[i]``; further dimensions pass."""
    n = 2 * len(freq)
    a = (pos.to(torch.float64)[:, None] * freq[None]).to(torch.float64)
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def visible(i, size, pool, plant=None):
    """(positions, blocks) that a query at ``i`` sees."""
    if plant == "window_long":
        size = size + 1
    if plant == "window_short":
        size = size - 1
    lo = max(0, i - size + 1)
    blocks = []
    if pool:
        last = i - size if plant != "pool_early" else i - size + 1
        b = 0
        while b * pool + pool - 1 <= last:
            blocks.append(b)
            b += 1
        if plant == "pool_none":
            blocks = []
    return list(range(lo, i + 1)), blocks


def windowed_attention(q, k, v, scale, size, pool=None, sink=None, plant=None):
    """``q [T, H, d]`` against ``k [T, G, d]``, ``v [T, G, e]``: the window, means of ``pool`` keys and values for the blocks
    before it, and ``exp(sink_h)`` in the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    nb = T // pool if pool else 0
    pk = [k[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]
    pv = [v[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]
    for i in range(T):
        js, bs = visible(i, size, pool, plant)
        ks = torch.stack([k[j] for j in js] + [pk[b] for b in bs])
        vs = torch.stack([v[j] for j in js] + [pv[b] for b in bs])
        for h in range(H):
            g = h // (H // G)
            s = ks[:, g] @ q[i, h] * scale
            m = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - m)
            den = p.sum() + (torch.exp(sink[h] - m) if sink is not None and plant != "no_sink" else 0.0)
            out[i, h] = (p / den) @ vs[:, g]
    return out


def attention(h, w, m, eps, *, whole_norm, rotated_values, sink, plant=None):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[n].t() + w[n + ".b"] for n in "qkv")
    if whole_norm:
        q, k = rms(q, eps) * w["q.norm"], rms(k, eps) * w["k.norm"]
        q, k = q.view(T, H, d), k.view(T, G, d)
    else:
        q, k = rms(q.view(T, H, d), eps) * w["q.norm"], rms(k.view(T, G, d), eps) * w["k.norm"]
    v = v.view(T, G, e)
    pos = torch.arange(T)
    f = frequencies(m["rot"])
    q, k = rotate(q, pos, f), rotate(k, pos, f)
    if rotated_values:
        fv = torch.tensor([m["rot"]["base"] ** (-2.0 * i / e) for i in range(e // 2)], dtype=torch.float64)
        v = rotate(v, pos, fv)
    o = windowed_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"].get("pool"), w["sink"] if sink else None, plant)
    if rotated_values and plant != "values_stay_turned":
        o = rotate(o, -pos, fv)
    out = o.reshape(T, H * e) @ w["o"].t()
    return out + w["o.b"] if "o.b" in w else out


# ------------------------------------------------------------------------------------------------- the model --
def mixer(h, kind, w, m, eps, plant=None):
    if kind == "gla":
        return gla(h, w, m, eps, plant)
    if kind == "attention":
        return attention(h, w, m, eps, whole_norm=True, rotated_values=True, sink=False, plant=plant)
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}  # noqa: E731
    left = attention(h, sub("left."), m["left"], eps, whole_norm=False, rotated_values=False, sink=True, plant=plant)
    return m["left_scale"] * left + m["right_scale"] * lightning(h, sub("right."), m["right"], eps, plant)


def feed_forward(h, w):
    return (gelu_tanh(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


def shapes(config, rank=5):
    """``{tensor name: shape}`` of a model whose decay projections have rank ``rank``."""
    D = config["width"]
    out = {"embed": [config["vocab"], D], "final.norm": [D], "head": [config["vocab"], D]}

    def linear(m, p, norm):
        H, d, e = m["heads"], m["dim"], m["vdim"]
        return {p + "q": [H * d, D], p + "k": [H * d, D], p + "v": [H * e, D], p + "g": [H * e, D], p + "o": [D, H * e],
                p + "norm": [norm]}

    def att(m, p, whole):
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        s = {p + "o": [D, H * e]}
        for n, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
            s.update({p + n: [rows, D], p + n + ".b": [rows]})
        s.update({p + "q.norm": [H * d if whole else d], p + "k.norm": [G * d if whole else d]})
        return s
    for i, spec in enumerate(config["layers"]):
        m = spec["mixer"]
        s = {"norm1": [D], "dwa": [i + 2]}
        if spec["type"] == "gla":
            s.update(linear(m, "mix.", m["vdim"]))
            n = m["heads"] * m["dim"]
            s.update({"mix.a1": [rank, D], "mix.a2": [n, rank], "mix.a2.b": [n]})
        elif spec["type"] == "attention":
            s.update(att(m, "mix.", True))
        else:
            s.update(att(m["left"], "mix.left.", False))
            s.update({"mix.left.sink": [m["left"]["heads"]], "mix.left.o.b": [D]})
            s.update(linear(m["right"], "mix.right.", m["right"]["heads"] * m["right"]["vdim"]))
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            s.update({"norm2": [D], "mlp.gate": [ff, D], "mlp.up": [ff, D], "mlp.down": [D, ff]})
        out.update({f"l{i}.{k}": v for k, v in s.items()})
    return out


def random_weights(config, seed, rank=5):
    """bf16-representable random weights; the gains keep scores spread out, decays between a few and hundreds of tokens, and
    every earlier result in the averages."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(config, rank).items():
        leaf = name.split(".", 1)[-1]
        r = torch.randn(*shape, generator=g)
        if leaf.endswith("dwa"):
            t = 0.15 * r
            t[-1] += 1.0
            t[0] += 0.3
        elif "norm" in leaf:
            t = 1.0 + 0.25 * r
        elif leaf.endswith("sink"):
            t = 1.0 + r
        elif leaf.endswith("a2.b"):
            t = 1.0 + 2.0 * r
        elif len(shape) == 1:
            t = 0.3 * r
        elif name == "embed":
            t = r
        elif leaf.endswith("a2"):
            t = 2.0 * r / math.sqrt(shape[-1])
        else:
            t = r / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).float()
    return out


def run(config, weights, tokens, dtype=torch.float64, plant=None, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    results = [x]
    for i, spec in enumerate(config["layers"]):
        x = x + rms(mixer(x, spec["type"], sub(f"l{i}.mix."), spec["mixer"], eps, plant), eps) * W[f"l{i}.norm1"]
        if spec["mlp"]:
            x = x + rms(feed_forward(x, sub(f"l{i}.mlp.")), eps) * W[f"l{i}.norm2"]
        results.append(x)
        dwa = W[f"l{i}.dwa"]
        x = sum(dwa[j] * results[j] for j in range(i + 2)) if plant != "no_average" else x
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps) * W["final.norm"] @ W["head"].t()


def greedy(config, weights, prompt, n, dtype=torch.float64):
    """``prompt`` followed by ``n`` tokens of largest logit, every step from scratch."""
    out = list(prompt)
    for _ in range(n):
        out.append(int(run(config, weights, out, dtype)[-1].argmax()))
    return out
