"""Per-kernel timing at the GPT-2 124M training shapes (16 x 1024 tokens, d 768), one row per kernel.

Each case is timed with CUDA events on the launching stream after warm-up, with an L2 flush (a 256 MiB write) before
every timed launch and a short device-side sleep queued ahead of it (so host launch latency is hidden and the
events bracket device time only), and reported against the measured copy bandwidth / bf16 GEMM throughput of the machine
(``MEASURED_PEAKS.json`` at the repository root when present, else 6.65 TB/s and 1.59 PFLOP/s).

    python benchmarks/kernel_bench.py                       # table of all cases
    python benchmarks/kernel_bench.py --only norm_bwd --iters 1 --warmup 1     # what a profiler run wraps

``--json PATH`` also writes the rows as JSON.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from dart_pytorch_b200.ops import flash as A  # noqa: E402
from dart_pytorch_b200.ops import kernels as K  # noqa: E402


def peaks():
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    hbm, tf, src = 6650.0, 1590.0, "fallback"
    if os.path.exists(path):
        try:
            d = json.load(open(path))
            hbm = float(d.get("hbm_gbs", hbm))
            tf = float(d.get("bf16_tflops", tf))
            src = "measured"
        except Exception:
            pass
    return hbm, tf, src


def build_cases(dev, want=()):
    """Cases are built only when their group is selected, so a profiler run of one kernel holds little memory."""
    def on(group):
        return not want or any(w in group or group in w for w in want)
    M, D, H, hd, B, S, V = 16384, 768, 12, 64, 16, 1024, 50257
    VP = (V + 127) // 128 * 128
    bf = dict(device=dev, dtype=torch.bfloat16)
    x = torch.randn(M, D, **bf)
    dy = torch.randn(M, D, **bf)
    dres = torch.randn(M, D, **bf)
    gamma = torch.ones(D, **bf)
    beta = torch.zeros(D, **bf)
    cases = {}

    def gemm_case(name, m, n, k, ta, tb, **kw):
        if want and not any(w in name for w in want):
            return
        a = torch.randn((k, m) if ta else (m, k), **bf)
        b = torch.randn((n, k) if tb else (k, n), **bf)
        c = torch.empty(m, n, **bf)
        extra = {}
        nbytes = 2 * (m * k + n * k + m * n)
        if kw.get("bias"):
            extra["bias"] = torch.randn(n, **bf)
        if kw.get("residual"):
            extra["residual"] = torch.randn(m, n, **bf)
            nbytes += 2 * m * n
        if kw.get("act"):
            extra["act"] = kw["act"]
        if kw.get("aux_out"):          # pre-activation copy kept for the backward pass
            extra["aux_out"] = torch.empty(m, n, **bf)
            nbytes += 2 * m * n
        if kw.get("act_bwd"):          # multiply by act'(pre-activation) in the epilogue
            extra["aux_in"] = torch.randn(m, n, **bf)
            extra["act_bwd"] = kw["act_bwd"]
            nbytes += 2 * m * n
        if kw.get("accumulate"):       # weight gradients add into the flat gradient buffer
            extra["accumulate"] = True
            c.zero_()
            nbytes += 2 * m * n
        cases[name] = (lambda: K.gemm(a, b, c, trans_a=ta, trans_b=tb, **extra), nbytes, 2.0 * m * n * k)

    gemm_case("gemm_qkv_fwd", M, 3 * D, D, False, True, bias=True)
    gemm_case("gemm_proj_fwd", M, D, D, False, True, bias=True, residual=True)
    gemm_case("gemm_fc1_fwd_gelu", M, 4 * D, D, False, True, bias=True, act="gelu_tanh_d", aux_out=True)
    gemm_case("gemm_fc2_fwd", M, D, 4 * D, False, True, bias=True, residual=True)
    gemm_case("gemm_lmhead_fwd", M, VP, D, False, True)
    gemm_case("gemm_fc1_dgrad", M, D, 4 * D, False, False)
    gemm_case("gemm_fc2_dgrad", M, 4 * D, D, False, False, act_bwd="mul")
    gemm_case("gemm_qkv_dgrad", M, D, 3 * D, False, False)
    gemm_case("gemm_fc1_wgrad", 4 * D, D, M, True, False, accumulate=True)
    gemm_case("gemm_fc2_wgrad", D, 4 * D, M, True, False, accumulate=True)
    gemm_case("gemm_qkv_wgrad", 3 * D, D, M, True, False, accumulate=True)
    gemm_case("gemm_proj_wgrad", D, D, M, True, False, accumulate=True)
    gemm_case("gemm_8192", 8192, 8192, 8192, False, True)
    # decode-sized rows: the per-GPU projections of a Llama-3-8B layer at TP = 8, batch 32 (weight streaming)
    gemm_case("gemm_dec_qkv", 32, 768, 4096, False, True)
    gemm_case("gemm_dec_wo", 32, 4096, 512, False, True)
    gemm_case("gemm_dec_gateup", 32, 3584, 4096, False, True)
    gemm_case("gemm_dec_down", 32, 4096, 1792, False, True)
    gemm_case("gemm_dec_head", 32, 16032, 4096, False, True)

    if on("norm"):
      _, mean, rstd = K.layernorm_fwd(x, gamma, beta, 1e-5)
      _, rrstd = K.rmsnorm_fwd(x, gamma, 1e-5)
    else:
      mean = rstd = rrstd = None
    cases["norm_fwd"] = (lambda: K.layernorm_fwd(x, gamma, beta, 1e-5), 2 * 2 * M * D, 0.0)
    cases["norm_bwd"] = (lambda: K.layernorm_bwd(x, dy, gamma, mean, rstd, dres=dres), 4 * 2 * M * D, 0.0)
    cases["rmsnorm_fwd"] = (lambda: K.rmsnorm_fwd(x, gamma, 1e-5), 2 * 2 * M * D, 0.0)
    cases["rmsnorm_bwd"] = (lambda: K.rmsnorm_bwd(x, dy, gamma, rrstd, dres=dres), 4 * 2 * M * D, 0.0)

    if on("attn"):
        qkv = torch.randn(M, 3 * D, **bf)
        o = torch.empty(M, D, **bf)
        q2, k2, v2 = qkv[:, :D], qkv[:, D:2 * D], qkv[:, 2 * D:]
        _, lse = A.attn_fwd(q2, k2, v2, B, S, S, H, H, hd, True, out=o)
        do = torch.randn(M, D, **bf)
        dqkv = torch.empty(M, 3 * D, **bf)
        att_flops = 4.0 * B * H * S * S * hd / 2  # causal: half of the score matrix
        cases["attn_fwd"] = (lambda: A.attn_fwd(q2, k2, v2, B, S, S, H, H, hd, True, out=o), 2 * 4 * M * D, att_flops)
        cases["attn_bwd"] = (lambda: A.attn_bwd(q2, k2, v2, o, do, lse, dqkv[:, :D], dqkv[:, D:2 * D], dqkv[:, 2 * D:],
                                                B, S, S, H, H, hd, True), 2 * 8 * M * D, 2.5 * att_flops)
    if on("ce"):
        logits = torch.randn(M, VP, **bf)
        tgt = torch.randint(0, V, (M,), device=dev)
        _, lse_ce = K.ce_fwd(logits, tgt, V)
        gone = torch.ones(1, device=dev, dtype=torch.float32)
        cases["ce_fwd"] = (lambda: K.ce_fwd(logits, tgt, V), 2 * M * VP, 0.0)
        cases["ce_bwd"] = (lambda: K.ce_bwd(logits, tgt, lse_ce, gone, 1.0 / M, V, out=logits, pad_to=VP), 4 * M * VP, 0.0)

    for cols in (D, 3 * D, 4 * D) if on("colsum") else ():
        src = torch.randn(M, cols, **bf)
        dst = torch.zeros(cols, **bf)
        cases[f"colsum_{cols}"] = (lambda src=src, dst=dst: K.colsum(src, dst, accumulate=True), 2 * M * cols, 0.0)

    if on("embedding"):
        table = torch.randn(V, D, **bf)
        pos = torch.randn(S, D, **bf)
        idx = torch.randint(0, V, (M,), device=dev)
        dtable = torch.zeros(V, D, **bf)
        cases["embedding_fwd"] = (lambda: K.embedding_fwd(table, idx, pos, 0, S), 2 * 2 * M * D, 0.0)
        cases["embedding_bwd"] = (lambda: K.embedding_bwd(dtable, idx, dy), 2 * 2 * M * D, 0.0)
    if on("adam") or on("grad_norm"):
        n = 124_500_000
        p = torch.randn(n, device=dev)           # fp32 master
        shadow = p.to(torch.bfloat16)            # bf16 working copy
        g = torch.randn(n, **bf)
        m1 = torch.zeros(n, device=dev)
        v1 = torch.zeros(n, device=dev)
        ctrl = torch.zeros(4, device=dev)
        ctrl[1] = 1.0
        ctrl[2] = 1.0
        cases["grad_norm"] = (lambda: K.grad_norm(g, ctrl, 1.0), 2 * n, 0.0)
        cases["adam_flat"] = (lambda: K.adam_flat(p, shadow, g, m1, v1, ctrl, 1e-4, 0.9, 0.95, 1e-8, 0.1, 0.1, 0.05),
                              n * (2 + 2 + 4 * 6), 0.0)
    if on("swiglu") or on("softmax"):
        gate = torch.randn(M, 4 * D, **bf)
        up = torch.randn(M, 4 * D, **bf)
        sw = torch.empty(M, 4 * D, **bf)
        cases["swiglu_fwd"] = (lambda: K.swiglu_fwd(gate, up, sw), 3 * 2 * M * 4 * D, 0.0)
        sm = torch.randn(B * H * 64, S, **bf)
        cases["softmax_fwd"] = (lambda: K.softmax_fwd(sm), 2 * 2 * sm.numel(), 0.0)
    if on("decode"):
        from dart_pytorch_b200.ops import decode as Dk
        Bd, Sk, Hq, Hkv, hdd = 32, 2304, 4, 1, 128                    # one rank of Llama-8B TP=8, batch 32
        qd = torch.randn(Bd, Hq * hdd, **bf)
        kc = torch.randn(Bd, Sk, Hkv * hdd, **bf)
        vc = torch.randn(Bd, Sk, Hkv * hdd, **bf)
        od = torch.empty(Bd, Hq * hdd, **bf)
        cases["attn_decode"] = (lambda: Dk.attn_decode(qd, kc, vc, Bd, 1, Sk, Hq, Hkv, hdd, Sk - 1, out=od),
                                2 * 2 * Bd * Sk * Hkv * hdd, 0.0)
    if on("hybrid"):
        cases.update(build_hybrid_cases(dev))
    if on("pozalorn"):
        cases.update(build_pozalorn_cases(dev))
    return cases


def build_pozalorn_cases(dev):
    """Serving kernels of Pozalorn at the "medium" size of ``hybrid_bench.py``, 4 x 2048 prompt tokens and 32 decode rows after
    2303 tokens, and (``pozalorn_like_*``) the kernels that play the same part in Llama at that width.  Bytes are what a kernel
    has to read and write once, products what the equations need (a state update and an output per token, visible keys only)."""
    from dart_pytorch_b200.nn.mixers import RotaryTable, row_layout
    from dart_pytorch_b200.ops import decode as Dk
    from dart_pytorch_b200.ops import mixers as X
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    D, H, Gk, hd, W, P, LH, dk, dv, ff, layers = 2048, 16, 4, 128, 1024, 16, 16, 64, 128, 5504, 6
    B, S = 4, 2048
    M, Bd, at = B * S, 32, 2303
    rn = lambda *s: torch.randn(*s, **bf)  # noqa: E731
    cases = {}

    def add(name, fn, nbytes, flops=0.0):
        cases["pozalorn_" + name] = (fn, nbytes, flops)
    rot, rot_v = RotaryTable(5e5, hd).rows(4096, dev), RotaryTable(5e5, hd).rows(4096, dev)
    decays = torch.tensor([0.5 ** (2.0 ** -(8.0 * i / LH)) for i in range(LH)], dtype=torch.float64)
    decays = torch.stack([decays.log(), decays - 1], 1).float().to(dev)
    w2, b2 = rn(LH * dk, 16) * 0.1, rn(LH * dk) + 4.0
    for tag, seqs, rows in (("", B, M), ("dec_", Bd, Bd)):
        n = rows // seqs
        # ---- linear attention
        cols, width = row_layout(q=LH * dk, k=LH * dk, v=LH * dv, g=LH * dv, r=16)
        p, state = rn(rows, width), torch.zeros(seqs, LH, dk, dv, **f32)
        nb = 2 * rows * LH * (2 * dk + 2 * dv) + 8 * seqs * LH * dk * dv
        fl = 4.0 * rows * LH * dk * dv
        add(tag + "linear_gated", lambda p=p, state=state, seqs=seqs, n=n, cols=cols: X.linear_attn(
            p, cols, state, seqs, n, LH, dk, dv, w2=w2, b2=b2, tau=16.0, q_scale=dk ** -0.5), nb + 32 * rows, fl)
        add(tag + "linear_constant", lambda p=p, state=state, seqs=seqs, n=n, cols=cols: X.linear_attn(
            p, cols, state, seqs, n, LH, dk, dv, decay=decays, silu=True), nb, fl)
        o, wh, wj = rn(rows, LH * dv), rn(dv), rn(LH * dv)
        g = p[:, cols["g"]:cols["g"] + LH * dv]
        add(tag + "norm_gate_head", lambda o=o, g=g: X.head_norm_gate(o, wh, g, 1e-6, "silu"), 6 * rows * LH * dv)
        add(tag + "norm_gate_joint", lambda o=o, g=g: X.head_norm_gate(o, wj, g, 1e-6, "sigmoid"), 6 * rows * LH * dv)
        # ---- windowed attention
        cols, width = row_layout(q=H * hd, k=Gk * hd, v=Gk * hd)
        p, ring = rn(rows, width), W + 32
        kr, vr = rn(seqs, ring, Gk * hd), rn(seqs, ring, Gk * hd)
        kp, vp = rn(seqs, 4096 // P, Gk * hd), rn(seqs, 4096 // P, Gk * hd)
        kl, vl = (rn(seqs, n, Gk * hd), rn(seqs, n, Gk * hd)) if n > 1 else (None, None)
        gq, gk = rn(H * hd), rn(Gk * hd)
        add(tag + "qkv_prep", lambda p=p, seqs=seqs, n=n, kr=kr, vr=vr, kl=kl, vl=vl, cols=cols: X.qkv_prep(
            p, cols, seqs, n, H, Gk, hd, hd, eps=1e-6, gq=gq, gk=gk, whole=True, rot=rot, rot_v=rot_v, k_ring=kr, v_ring=vr,
            pos=0 if n > 1 else at, k_lin=kl, v_lin=vl), 4 * rows * width)
        q, sink = rn(rows, H * hd), rn(H)
        if n > 1:
            pairs = sum(min(i + 1, W) + max(0, (i - W + 1) // P) for i in range(n)) * seqs
            keys = X.WindowKeys(kl, vl, W, pool=P, k_pool=kp, v_pool=vp)
            add("window_attn_pooled", lambda: X.window_attn_fwd(q0, keys0, B, S, H, Gk, hd, hd, 0, hd ** -0.5, rot=rot_v),
                4 * rows * (H + Gk) * hd, 4.0 * pairs * H * hd)
            q0, keys0 = q, keys
            plain = sum(min(i + 1, W) for i in range(n)) * seqs
            add("window_attn_sink", lambda: X.window_attn_fwd(q0, X.WindowKeys(keys0.k, keys0.v, W), B, S, H, Gk, hd, hd, 0,
                                                              hd ** -0.5, sink=sink0), 4 * rows * (H + Gk) * hd, 4.0 * plain * H * hd)
            sink0 = sink
            add("pool_blocks", lambda: X.pool_blocks(keys0.k, keys0.v, kp0, vp0, B, pool=P, first=0, count=S // P),
                4 * rows * Gk * hd)
            kp0, vp0 = kp, vp
        else:
            keys = X.WindowKeys(kr, vr, W, ring=True, pool=P, k_pool=kp, v_pool=vp)
            count = W + (at - W + 1) // P
            splits, floats = X.window_decode_plan(Bd, H, Gk, hd, hd, count)
            ws = torch.empty(max(1, floats), **f32)
            add("dec_window_attn", lambda: X.window_attn_decode(qd, kd, Bd, 1, H, Gk, hd, hd, at, hd ** -0.5, rot=rot_v,
                                                                splits=splits, ws=ws), 4 * Bd * count * Gk * hd)
            qd, kd = q, keys
        # ---- stream and feed-forward
        x, m, w, stack = torch.randn(rows, D, **f32), rn(rows, D), rn(D), torch.randn(layers, rows, D, **f32)
        avg, y, res = rn(4), torch.empty(rows, D, **f32), torch.empty(rows, D, **f32)
        add(tag + "stream_mixer", lambda x=x, m=m, w=w, y=y, rows=rows: X.branch_norm(
            x, rows, D, torch.bfloat16, 1e-6, m1=m, m2=m, w=w, x_out=y), rows * D * (4 + 4 + 4 + 2))
        add(tag + "stream_average", lambda x=x, m=m, w=w, y=y, rows=rows, stack=stack, res=res: X.branch_norm(
            x, rows, D, torch.bfloat16, 1e-6, m1=m, w=w, stack=stack, n=3, avg=avg, result=res, x_out=y),
            rows * D * (4 + 2 + 12 + 4 + 4 + 2))
        gu = rn(rows, 2 * ff)
        add(tag + "geglu", lambda gu=gu: K.geglu_fwd(gu[:, :ff], gu[:, ff:]), 6 * rows * ff)
        add("like_" + tag + "swiglu", lambda gu=gu: K.swiglu_fwd(gu[:, :ff], gu[:, ff:]), 6 * rows * ff)
        add("like_" + tag + "rmsnorm", lambda m=m, w=w: K.rmsnorm_fwd(m, w, 1e-5), 4 * rows * D)
    # ---- Llama's attention
    qf, kf, vf, of = rn(M, H * hd), rn(M, Gk * hd), rn(M, Gk * hd), torch.empty(M, H * hd, **bf)
    add("like_attn_fwd", lambda: A.attn_fwd(qf, kf, vf, B, S, S, H, Gk, hd, True, out=of, need_lse=False),
        4 * M * (H + Gk) * hd, 2.0 * B * S * S * H * hd)
    kc, vc, od, qs = rn(Bd, at + 1, Gk * hd), rn(Bd, at + 1, Gk * hd), torch.empty(Bd, H * hd, **bf), rn(Bd, H * hd)
    add("like_dec_attn", lambda: Dk.attn_decode(qs, kc, vc, Bd, 1, at + 1, H, Gk, hd, at, out=od), 4 * Bd * (at + 1) * Gk * hd)
    qkv, qkvd = rn(M, (H + 2 * Gk) * hd), rn(Bd, (H + 2 * Gk) * hd)
    kq, vq = rn(B, S, Gk * hd), rn(B, S, Gk * hd)
    add("like_rope_append", lambda: Dk.rope_kv_append(qkv, kq, vq, B, S, H, Gk, hd, 0), 4 * M * (H + 2 * Gk) * hd)
    add("like_dec_rope_append", lambda: Dk.rope_kv_append(qkvd, kc, vc, Bd, 1, H, Gk, hd, at), 4 * Bd * (H + 2 * Gk) * hd)
    return cases


def build_hybrid_cases(dev):
    """Serving kernels of the hybrid decoder (Famudra) at the "medium" size of ``hybrid_bench.py``, 4 x 2048 prompt tokens and
    32 decode rows over 2304 tokens, and (``hybrid_like_*``) the kernels that play the same part in Llama at that width."""
    from dart_pytorch_b200.nn.hybrid import DroplessMoE
    from dart_pytorch_b200.ops import decode as Dk
    from dart_pytorch_b200.ops import hybrid as Y
    from dart_pytorch_b200.parallel import ep as EP
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    D, H, hd, Rq, R, C, G, E, top, ff, sff, V = 2048, 16, 128, 768, 512, 2560, 10, 64, 6, 1024, 2048, 32768
    B, S = 4, 2048
    M, Bd, Sk = B * S, 32, 2304
    rn = lambda *s: torch.randn(*s, **bf)  # noqa: E731
    cases = {}

    def add(name, fn, nbytes, flops=0.0):
        cases["hybrid_" + name] = (fn, nbytes, flops)

    def gemm(name, m, n, k):
        a, w, c = rn(m, k), rn(n, k), torch.empty(m, n, **bf)
        add(name, lambda: K.gemm(a, w, c, trans_b=True), 2 * (m * k + n * k + m * n), 2.0 * m * n * k)
    # ---- prompts
    gemm("like_gemm_gate_up", M, 2 * 5464 // 8 * 8, D)
    gemm("gemm_dq_dkv", M, Rq + R, D)
    q2, k2, v2, o2 = rn(M, H * hd), rn(M, H * hd), rn(M, H * hd), torch.empty(M, H * hd, **bf)
    fl = 4.0 * B * H * S * S * hd / 2
    for name, precise in (("like_attn_fwd", False), ("attn_fwd_precise", True)):
        add(name, lambda precise=precise: A.attn_fwd(q2, k2, v2, B, S, S, H, H, hd, True, out=o2, need_lse=False,
                                                     precise=precise), 2 * 4 * M * H * hd, fl)
    moe = {}
    for tag, rows in (("", M), ("dec_", Bd)):
        m = DroplessMoE(8, E, top, 8, 0, device=dev, dtype=torch.bfloat16)
        router, x = rn(E, D), rn(rows, D)
        ctr = torch.zeros(2 * E, dtype=torch.int32, device=dev)
        idx, w = Y.moe_route(x, router, top, ctr)
        base = ctr.clone()
        xs, off, slot = Y.moe_place(x, idx, ctr, E)
        if tag == "":
            wu, wd, su, sd = rn(E * ff, D), rn(E * D, ff), rn(sff, D), rn(D, sff)
        up, y, s_up, sh = torch.empty(rows * top, ff, **bf), rn(rows * top, D), torch.empty(rows, sff, **bf), rn(rows, D)
        hint = (rows * top + E - 1) // E
        live = int((base[:E] > 0).sum())
        seg = Y.grouped_segment

        def run_up(x=x, xs=xs, up=up, off=off, s_up=s_up, hint=hint):
            Y.grouped_gemm(seg(xs, wu, up, groups=E, N_=ff, K=D, offsets=off, act="relu2", rows_hint=hint),
                           seg(x, su, s_up, groups=1, N_=sff, K=D, act="relu2"))

        def run_down(up=up, y=y, off=off, s_up=s_up, sh=sh, hint=hint):
            Y.grouped_gemm(seg(up, wd, y, groups=E, N_=D, K=ff, offsets=off, rows_hint=hint),
                           seg(s_up, sd, sh, groups=1, N_=D, K=sff))
        wb = 2 * (live * ff * D + sff * D)
        flops = 2.0 * rows * D * (top * ff + sff)
        add(tag + "experts_up", run_up, wb + 2 * rows * (top * (D + ff) + D + sff), flops)
        add(tag + "experts_down", run_down, wb + 2 * rows * (top * (D + ff) + D + sff), flops)
        like_logits = torch.empty(rows, E, **bf)

        def like_route(x=x, like_logits=like_logits, rows=rows):    # the expert-parallel MoE layer's router
            K.gemm(x, router, like_logits, trans_b=True)
            EP.slots(EP.route(like_logits, top)[1], E, rows)
        add("like_" + tag + "route", like_route, 2 * rows * D)
        add(tag + "route", lambda x=x, ctr=ctr: Y.moe_route(x, router, top, ctr), 2 * rows * D)

        def place(x=x, idx=idx, ctr=ctr, base=base):
            ctr.copy_(base)
            Y.moe_place(x, idx, ctr, E)
        add(tag + "place", place, 2 * rows * D * (1 + top))
        xr, mix, g, mu, st = torch.randn(rows, D, **f32), rn(rows, D), rn(1), rn(D), torch.zeros(B if tag == "" else rows, D, **f32)
        t = Y.LayerTerms(mix, sh, y, slot, w)
        add(tag + "stream_norm", lambda xr=xr, t=t, rows=rows, g=g, mu=mu, st=st: Y.stream_norm(
            xr, t, rows, rows // st.shape[0], g, 1e-6, g2=g, shift=mu, shift_state=st), rows * D * (4 + 2 + 2 + 2 * top + 4 + 4))
        gamma = rn(D)
        add("like_" + tag + "rmsnorm", lambda x=x, gamma=gamma: K.rmsnorm_fwd(x, gamma, 1e-5), 4 * rows * D)
        # ---- recurrence
        seqs = B if tag == "" else rows
        n = C // G
        yx, taps, bias = rn(rows, 2 * C), rn(C, 4), rn(C)
        cs, ss = torch.zeros(seqs, 3, C, **f32), torch.zeros(seqs, C, **f32)
        u = Y.conv_state(yx[:, C:], taps, bias, cs, seqs, rows // seqs, G)
        wg, z = rn(G * 2 * n, 2 * n), torch.empty(rows, 2 * C, **f32)
        add(tag + "conv", lambda yx=yx, cs=cs, seqs=seqs, rows=rows: Y.conv_state(yx[:, C:], taps, bias, cs, seqs,
                                                                                 rows // seqs, G), rows * C * 6)
        add(tag + "gates", lambda u=u, z=z: Y.grouped_gemm(seg(u, wg, z, groups=G, N_=2 * n, K=2 * n, x_col_stride=2 * n,
                                                               out_col_stride=2 * n)),
            rows * C * 12 + 8 * C * n, 8.0 * rows * C * n)
        add(tag + "lru_scan", lambda u=u, z=z, yx=yx, ss=ss, seqs=seqs, rows=rows: Y.lru_scan(
            u, z, bias, bias, bias, yx[:, :C], ss, seqs, rows // seqs, G, 8.0), rows * C * 16)
        # ---- latent attention
        d, gq, gc = rn(rows, Rq + R), rn(Rq), rn(R)
        cache = rn(seqs, Sk, R)
        pos = 0 if tag == "" else Sk - 1
        add(tag + "latent_append", lambda d=d, cache=cache, seqs=seqs, rows=rows, pos=pos: Y.latent_norm_append(
            d, gq, gc, cache, seqs, rows // seqs, pos, 1e-6), 4 * rows * (Rq + R))
    ql, ukt, uv = rn(Bd, H * hd), rn(H * R, hd), rn(H * hd, R)
    qa, ol, oo = torch.empty(Bd, H * R, **bf), rn(Bd, H * R), torch.empty(Bd, H * hd, **bf)
    add("dec_absorb_q", lambda: Y.grouped_gemm(seg(ql, ukt, qa, groups=H, N_=R, K=hd, x_col_stride=hd, out_col_stride=R)),
        2 * (H * R * hd + Bd * H * (hd + R)))
    add("dec_absorb_v", lambda: Y.grouped_gemm(seg(ol, uv, oo, groups=H, N_=hd, K=R, x_col_stride=R, out_col_stride=hd)),
        2 * (H * R * hd + Bd * H * (hd + R)))
    splits, wsn = Y.latent_attn_plan(Bd, H, R, Sk, False)
    ws = torch.empty(max(1, wsn), **f32)
    add("dec_latent_attn", lambda: Y.latent_attn(ol, cache, Bd, 1, H, Sk - 1, 0.05, splits=splits, ws=ws),
        2 * Bd * (Sk * R + 2 * H * R))
    kc, vc, od = rn(Bd, Sk, 4 * hd), rn(Bd, Sk, 4 * hd), torch.empty(Bd, H * hd, **bf)
    add("like_dec_attn", lambda: Dk.attn_decode(ql, kc, vc, Bd, 1, Sk, H, 4, hd, Sk - 1, out=od), 4 * Bd * Sk * 4 * hd)
    qkv = rn(M, (H + 8) * hd)
    kp, vp = rn(B, S, 4 * hd), rn(B, S, 4 * hd)
    add("like_rope_append", lambda: Dk.rope_kv_append(qkv, kp, vp, B, S, H, 4, hd, 0), 4 * M * (H + 8) * hd)
    hh, hw, hl = rn(Bd, D), rn(V, D), torch.empty(Bd, V, **f32)
    add("dec_head", lambda: Y.grouped_gemm(seg(hh, hw, hl, groups=1, N_=V, K=D)), 2 * V * D + 4 * Bd * V)
    gemm("like_dec_gate_up", Bd, 2 * 5464 // 8 * 8, D)
    gemm("like_dec_down", Bd, D, 5464 // 8 * 8)
    gemm("like_dec_qkv", Bd, (H + 8) * hd, D)
    gemm("like_dec_head", Bd, V, D)
    gemm("dec_dq_dkv", Bd, Rq + R, D)
    return cases


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--only", default="", help="comma-separated substrings of case names")
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--json", default="")
    args = ap.parse_args()
    dev = torch.device("cuda", 0)
    torch.manual_seed(0)
    hbm, tf, src = peaks()
    want = [w for w in args.only.split(",") if w]
    cases = build_cases(dev, want)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows = []
    print(f"{'kernel':24s} {'us':>9s} {'GB/s':>8s} {'TF/s':>8s}  frac of {src} peak")
    for name, (fn, nbytes, flops) in cases.items():
        if want and not any(w in name for w in want):
            continue
        for _ in range(args.warmup):
            fn()
        ts = []
        for _ in range(args.iters):
            flush.fill_(1)
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            torch.cuda._sleep(400_000)   # the GPU idles ~0.2 ms while the host queues the launches behind it
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1) * 1e3)
        ts.sort()
        us = ts[len(ts) // 2]
        gbs = nbytes / us / 1e3
        tfs = flops / us / 1e6
        frac = max(gbs / hbm, tfs / tf)
        bound = "mem" if gbs / hbm >= tfs / tf else "mma"
        print(f"{name:24s} {us:9.1f} {gbs:8.0f} {tfs:8.0f}  {frac:5.2f} ({bound})")
        rows.append(dict(kernel=name, us=us, gbs=gbs, tflops=tfs, frac=frac, bound=bound, peaks=src))
    K.N.raise_on_device_error()
    if args.json:
        with open(args.json, "w") as f:
            json.dump(rows, f, indent=1)


if __name__ == "__main__":
    main()
