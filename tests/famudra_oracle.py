"""Plain, slow implementation of the Famudra equations (one function per mechanism, fp32 or fp64 on the CPU).

The oracle of the Famudra tests.  It shares no code with the package: it reads the same flat ``{name: tensor}`` weights
and the same configuration dictionary and processes one whole sequence at a time, position by position where a mechanism
is recurrent.  ``run(..., plant=...)`` plants one of a few mistakes, for tests that check that a test would notice it.
"""
import math

import torch


def rms(x, eps):
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(n, mu, first=None):
    """``n_t + (n_{t-1} - n_t) * mu`` with ``n_{-1} = first`` (zeros when None); ``n [T, D]``."""
    out = torch.empty_like(n)
    prev = torch.zeros_like(n[0]) if first is None else first
    for t in range(n.shape[0]):
        out[t] = n[t] + (prev - n[t]) * mu
        prev = n[t]
    return out


def causal_conv(x, taps, bias):
    """Depthwise causal convolution, the last tap multiplies the current row; ``x [T, C]``, ``taps [C, K]``."""
    K = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        acc = bias.clone()
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                acc = acc + taps[:, k] * x[s]
        out[t] = acc
    return out


def block_gate(u, w, b):
    """``sigmoid(w[g] u_g + b[g])`` for every one of the equal parts ``u_g`` of ``u [T, C]``; ``w [G, n, n]``."""
    G, n, _ = w.shape
    parts = [torch.sigmoid(u[:, g * n:(g + 1) * n] @ w[g].t() + b[g]) for g in range(G)]
    return torch.cat(parts, dim=1)


def gated_linear_recurrence(u, r, i, lam, c=8.0, state=None):
    """``S_t = a_t S_{t-1} + sqrt(1 - a_t^2) i_t u_t`` with ``log a_t = -c r_t softplus(lam)``; returns all ``S_t``."""
    sp = torch.log1p(torch.exp(-lam.abs())) + torch.clamp(lam, min=0)
    S = torch.zeros_like(u[0]) if state is None else state
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        log_a = -c * r[t] * sp
        a = torch.exp(log_a)
        S = a * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru(h, w, mixer, eps):
    y = gelu_tanh(h @ w["y"].t() + w["y.b"])
    u = causal_conv(h @ w["x"].t() + w["x.b"], w["conv"], w["conv.b"])
    S = gated_linear_recurrence(u, block_gate(u, w["ra"], w["ra.b"]), block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return (S * y) @ w["o"].t()


def latent_attention(h, w, mixer, eps, plant=None):
    H, dk, dv = mixer["heads"], mixer["dim"], mixer["vdim"]
    T = h.shape[0]
    c_q = rms(h @ w["dq"].t(), eps) * w["dq.norm"]
    c = rms(h @ w["dkv"].t(), eps) * w["dkv.norm"]
    q = (c_q @ w["uq"].t()).reshape(T, H, dk)
    k = (c @ w["uk"].t()).reshape(T, H, dk)
    v = (c @ w["uv"].t()).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        n = t + 1
        if plant == "misses_own_key" and t > 0:
            n = t
        lo = 1 if plant == "misses_first_key" and t > 0 else 0
        s = torch.einsum("hd,nhd->hn", q[t], k[lo:n]) * mixer["scale"]
        p = torch.softmax(s, dim=-1)
        out[t] = torch.einsum("hn,nhd->hd", p, v[lo:n])
    return out.reshape(T, H * dv) @ w["o"].t()


def expert(h, up, down):
    return torch.relu(h @ up.t()) ** 2 @ down.t()


def route(h, router, top):
    """Chosen experts ``[T, top]`` (largest logits) and the softmax over their logits alone."""
    z = h @ router.t()
    val, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    return idx[:, :top], torch.softmax(val[:, :top], dim=-1)


def moe(h, w, mlp):
    idx, wt = route(h, w["router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = int(idx[t, j])
            out[t] += wt[t, j] * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if mlp.get("shared"):
        out = out + expert(h, w["shared.up"], w["shared.down"])
    return out


def shapes(config):
    """``{tensor name: shape}`` of a model."""
    D = config["width"]
    out = {"embed": [config["vocab"], D], "final.norm": [], "head": [config["vocab"], D]}
    for i, spec in enumerate(config["layers"]):
        m, mlp = spec["mixer"], spec["mlp"]
        s = {"norm1": [], "shift": [D]}
        if spec["type"] == "rglru":
            C, G = m["width"], m["blocks"]
            n = C // G
            s.update({"mix.y": [C, D], "mix.y.b": [C], "mix.x": [C, D], "mix.x.b": [C], "mix.conv": [C, m["conv"]],
                      "mix.conv.b": [C], "mix.ra": [G, n, n], "mix.ra.b": [G, n], "mix.ri": [G, n, n], "mix.ri.b": [G, n],
                      "mix.lam": [C], "mix.o": [D, C]})
        else:
            H, R = m["heads"], m["kv_rank"]
            s.update({"mix.dq": [m["q_rank"], D], "mix.dq.norm": [m["q_rank"]], "mix.dkv": [R, D], "mix.dkv.norm": [R],
                      "mix.uq": [H * m["dim"], m["q_rank"]], "mix.uk": [H * m["dim"], R], "mix.uv": [H * m["vdim"], R],
                      "mix.o": [D, H * m["vdim"]]})
        if mlp:
            s.update({"norm2": [], "mlp.router": [mlp["router"]["experts"], D]})
            for e in range(mlp["router"]["experts"]):
                s.update({f"mlp.e{e}.up": [mlp["expert"]["ff"], D], f"mlp.e{e}.down": [D, mlp["expert"]["ff"]]})
            if mlp.get("shared"):
                s.update({"mlp.shared.up": [mlp["shared"]["ff"], D], "mlp.shared.down": [D, mlp["shared"]["ff"]]})
        out.update({f"l{i}.{k}": v for k, v in s.items()})
    return out


def random_weights(config, seed, gain=1.0):
    """bf16-representable random weights that keep every branch's output of the order of the stream."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(config).items():
        leaf = name.split(".", 1)[-1]
        r = torch.randn(*shape, generator=g) if shape else torch.randn(1, generator=g).reshape(())
        if not shape or leaf.endswith(".norm"):
            t = 1.0 + 0.2 * r
        elif name.endswith(".shift"):
            t = torch.sigmoid(r)
        elif name.endswith(".lam"):
            t = -4.0 + 2.0 * r                       # decays between a few and thousands of tokens
        elif len(shape) == 1 or leaf.endswith("ra.b") or leaf.endswith("ri.b"):
            t = 0.3 * r
        elif name == "embed":
            t = r
        elif leaf == "mix.conv":
            t = 0.6 * r
        elif leaf == "mlp.router":
            t = 3.0 * r / math.sqrt(shape[-1])
        else:
            t = gain * r / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).float()
    return out


def greedy(config, weights, prompt, n, dtype=torch.float64):
    """``prompt`` followed by ``n`` tokens of largest logit, every step from scratch."""
    out = list(prompt)
    for _ in range(n):
        out.append(int(run(config, weights, out, dtype)[-1].argmax()))
    return out


def layer_schedule(config):
    """Layer indices in the order they run, each with a flag: the embedding output is added before it."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for p in range(times):
        order += [(i, p > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def run(config, weights, tokens, dtype=torch.float64, plant=None, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` (a list) receives the residual stream after every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}
    emb = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = emb.clone()
    for i, add_emb in layer_schedule(config):
        spec = config["layers"][i]
        if add_emb and plant != "loop_without_embedding":
            x = x + emb
        h = rms(x, eps) * W[f"l{i}.norm1"]
        h = token_shift(h, W[f"l{i}.shift"])
        mix = sub(f"l{i}.mix.")
        if spec["type"] == "rglru":
            d = rglru(h, mix, spec["mixer"], eps)
        else:
            d = latent_attention(h, mix, spec["mixer"], eps, plant)
        if spec["mlp"]:
            d = d + moe(rms(x, eps) * W[f"l{i}.norm2"], sub(f"l{i}.mlp."), spec["mlp"])
        x = x + d
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps) * W["final.norm"] @ W["head"].t()
