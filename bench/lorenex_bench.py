"""Lorenex beside Kudonex (the framework's closest design: paged attention, a state space and a matrix memory with
mixture-of-experts feed-forwards on an fp32 stream) at equal layer sizes, random weights: prefill and decode throughput through
each model's own generator, and the time of each Lorenex kernel next to the kernel that does the like job in Kudonex, Duratar
or Gorozen, as fractions of the measured roofline (``MEASURED_PEAKS.json``: copy bandwidth and cuBLAS bf16 rate of this pool's
B200). Scans are given against the nominal fp32 FMA rate, the selective scan against the slower of that and the nominal rate of
the special-function units (16 exponentials per SM and clock), which its decays need.

    python bench.py --workload lorenex [--steps K --warmup W]

Timing: CUDA events on the launching stream, W >= 3 warm-up iterations; the single-kernel rows (all designs) are replayed
from a CUDA graph with an L2 flush (a 256 MB write) between timed iterations; the end-to-end rows run steps whose weights and
caches together exceed L2.
"""
from __future__ import annotations

import json
import time

import torch

from duratar_bench import FP32_TFLOPS
from gorozen_bench import Timer, _peaks
from kudonex_bench import kudonex_config
from segorax_bench import GraphTimer

EXP_RATE = 148 * 16 * 1.965e9 / 1e12      # nominal exponentials per second of the special-function units, in units of 1e12

SIZES = {
    # name: (width, attention heads, kv heads, head size, matrix-memory heads, key size, value size, decay rank,
    #        state-space inner size, states, step rank, taps, dense ff, experts, identity experts, top, vocab)
    "2k wide, 16 heads": (2048, 16, 4, 128, 16, 128, 128, 16, 4096, 16, 128, 4, 6144, 8, 2, 4, 32768),
    "4k wide, 16 attention heads, 32 scan heads": (4096, 16, 4, 128, 32, 128, 128, 16, 8192, 16, 256, 4, 12288, 8, 2, 4, 32768),
}


def lorenex_config(W, H, G, D, SH, SD, SDv, rank, inner, N, R, taps, F, E, X, top, V):
    par = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "conv": taps, "scale": D ** -0.5, "q_temp": {"coef": 0.1, "every": 8192}},
           "right": {"inner": inner, "state": N, "dt_rank": R, "conv": taps}, "left_scale": 1.0, "right_scale": 1.0}
    gla = {"heads": SH, "dim": SD, "vdim": SDv, "tau": 16.0}
    dense = {"kind": "dense", "ff": F}
    # the feed-forward multiplies as much per token as a dense one of F: `top` experts of F / top (fewer where identity experts win)
    moe = {"kind": "moe", "expert": {"ff": F // top, "limit": 7.0}, "router": {"experts": E, "identity": X, "top": top}}
    layers = [{"type": "parallel", "mixer": par, "mlp": dense}, {"type": "gla", "mixer": gla, "mlp": moe},
              {"type": "parallel", "mixer": par, "mlp": dense}, {"type": "gla", "mixer": gla, "mlp": moe}]
    return {"architecture": "Lorenex", "layers": layers, "norm": {"eps": 1e-6}, "embedding": {"scale": W ** 0.5}, "residual_mult": 0.3,
            "max_positions": 8192, "vocab": V, "width": W}


def build_models(size, dev):
    from llm_in_practise_b200.models.kudonex import KudonexConfig, KudonexForCausalLM
    from llm_in_practise_b200.models.lorenex import LorenexConfig, LorenexForCausalLM
    W, H, G, D, SH, SD, SDv, rank, inner, N, R, taps, F, E, X, top, V = SIZES[size]
    torch.manual_seed(0)
    lx = LorenexForCausalLM(LorenexConfig.from_dict(lorenex_config(*SIZES[size])), dtype=torch.bfloat16, device=dev,
                            decay_ranks={1: rank, 3: rank}).eval()
    kx = KudonexForCausalLM(KudonexConfig.from_dict(kudonex_config(W, H, G, D, 0, SH, SD, SDv, max(1, SH // 4), taps, F, E, 2, V)),
                            dtype=torch.bfloat16, device=dev).eval()
    for model in (lx, kx):
        for n, p in model.named_parameters():
            leaf = n.split(".")[-1]
            if p.dtype == torch.bfloat16 and p.dim() >= 2 and leaf != "embed_tokens":
                p.data.normal_(std=p.shape[-1] ** -0.5)
            elif leaf in ("canon", "conv_w", "qkv_conv", "router", "a2"):
                p.data.normal_(std=0.3)
            elif leaf == "act":
                p.data.fill_(0.5)
            elif leaf == "a2_bias":
                p.data.fill_(2.0)
            elif leaf in ("r1", "r2"):
                p.data.uniform_(0.1, 1.0)
            elif leaf == "talk":
                p.data.add_(torch.randn_like(p) * 0.1)
    return lx, kx


@torch.no_grad()
def end_to_end(size, dev, steps, warmup, prompt=2048, batch=32, ctx=1024):
    """tokens/s of (a) one prompt of ``prompt`` tokens, (b) one decode step of ``batch`` sequences at context ``ctx``."""
    from llm_in_practise_b200.inference import RaggedGenerator
    t = Timer(dev, flush=False)
    out = {}
    V = SIZES[size][-1]
    toks = torch.randint(0, V, (prompt,)).tolist()
    for name, model in zip(("lorenex", "kudonex"), build_models(size, dev)):
        g = RaggedGenerator(model, None, max(prompt, ctx + 64))
        per = -(-max(prompt, ctx + 64) // 64)
        cache = g.make_cache(batch * per, 64, batch, per * 64)
        for b in range(batch):
            g.set_block_row(cache, b, list(range(1 + b * per, 1 + (b + 1) * per)))
        ms = t(lambda: g.step([(0, 0, toks, [prompt - 1])], cache), steps, warmup)
        out[f"{name}_prefill_tok_s"] = prompt / ms * 1e3
        out[f"{name}_prefill_ms"] = ms
        last = [1] * batch
        ms = t(lambda: g.decode(last, [ctx] * batch, list(range(batch)), cache), steps * 4, warmup)
        out[f"{name}_decode_tok_s"] = batch / ms * 1e3
        out[f"{name}_decode_ms"] = ms
        out[f"{name}_kv_bytes_per_token"] = g.kv_token_bytes()
        out[f"{name}_state_bytes_per_sequence"] = g.state_bytes()
        out[f"{name}_parameters"] = model.num_parameters()
        del g, cache, model
        torch.cuda.empty_cache()
    return out


@torch.no_grad()
def kernel_rows(size, dev, steps, warmup, root):
    """Single kernels at the layer sizes: (name, Lorenex ms, fraction of roofline, like kernel or None, ms, fraction, bound)."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops import elementwise as ew
    from llm_in_practise_b200.ops.hyper import xielu
    from llm_in_practise_b200.ops.linear_scan import (delta_gates, linear_scan, lowrank_decay, scan_readout, selective_scan, short_conv)
    from llm_in_practise_b200.ops.moe import dispatch, gather_rows, moe_combine, route_grouped
    from llm_in_practise_b200.ops.multimap_attention import conv_qknorm_store, multimap_attention, qknorm_rope_store
    from llm_in_practise_b200.ops.norm import poly_norm, sandwich_norm
    from llm_in_practise_b200.ops.paged_attention import paged_attention
    hbm, tf, which = _peaks(root)
    W, H, G, D, SH, SD, SDv, rank, inner, N, R, taps, F, E, X, top, V = SIZES[size]
    t = GraphTimer(dev)
    rows = []
    bf, f32 = torch.bfloat16, torch.float32
    T, Bq, ctx, BS = 4096, 64, 4032, 64

    def frac_bw(nbytes, ms):
        return nbytes / (ms * 1e-3) / 1e9 / hbm

    def frac_fl(flops, ms):
        return flops / (ms * 1e-3) / 1e12 / tf

    def frac_fma(flops, ms):
        return flops / (ms * 1e-3) / 1e12 / FP32_TFLOPS

    rnd = lambda *s: torch.randn(*s, device=dev)                                                  # noqa: E731
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    pd, sd_ = torch.full((Bq,), ctx, dtype=torch.int32, device=dev), torch.arange(Bq, dtype=torch.int32, device=dev)
    pieces = make_pieces([(0, T, 0, 0)], dev)
    runs = pieces.runs
    # --- norm of the branch + scaled residual + cast vs Kudonex's layer-norm sandwich
    y32, res, wn = rnd(T, W), rnd(T, W), torch.ones(W, device=dev)
    ms_k = t(lambda: sandwich_norm(y32, wn, res, None, 1e-6, 0.0, bf, branch_mult=0.3, cast_next=True), steps, warmup)
    ms_l = t(lambda: sandwich_norm(y32, wn, res, wn, 1e-6, 0.0, f32, center=True), steps, warmup)
    rows.append(("output RMS norm + scaled residual + bf16 copy of the stream", ms_k, frac_bw(T * W * 14, ms_k),
                 "Kudonex: post layer norm + residual + pre layer norm (fp32 out)", ms_l, frac_bw(T * W * 16, ms_l), "HBM"))
    # --- power-norm activation vs Duratar's xIELU
    z = rnd(T, F).to(bf)
    act, pq = torch.full((4,), 0.5, device=dev), torch.full((2,), 0.5, device=dev)
    ms_k = t(lambda: poly_norm(z, act, 1e-6), steps, warmup)
    ms_l = t(lambda: xielu(z, pq), steps, warmup)
    rows.append((f"power-norm activation, {F} columns", ms_k, frac_bw(T * F * 4, ms_k), "Duratar: xIELU (no reduction)", ms_l, frac_bw(T * F * 4, ms_l), "HBM"))
    # --- convolution + norms + page store vs Duratar's norm + rotary + store
    C = (H + 2 * G) * D
    nb = T // BS
    ck, cv = (torch.zeros(nb + 1, G, BS, D, dtype=bf, device=dev) for _ in range(2))
    table = torch.arange(1, nb + 1, dtype=torch.int32, device=dev).view(1, nb)
    proj = rnd(T, C + 2 * inner).to(bf)
    bias, cw, tail = rnd(C), rnd(C, taps) * 0.5, torch.zeros(Bq + 1, taps - 1, C, device=dev)
    ms_k = t(lambda: conv_qknorm_store(proj[:, :C], bias, cw, tail, pos, slot, runs, 1, ck, cv, table, H, G, D, D, 1e-6, bf, temp=(0.1, 8192.0),
                                       norm_v=True), steps, warmup)
    Dm = D // 2
    dk, dv_ = torch.zeros(nb + 1, G * 2, BS, Dm, dtype=bf, device=dev), torch.zeros(nb + 1, G, BS, D, dtype=bf, device=dev)
    p32 = rnd(T, C)
    wq = torch.ones(Dm, device=dev)
    cos, sin = ew.rope_tables_partial(T, Dm, 1e6, dev)
    ms_l = t(lambda: qknorm_rope_store(p32, wq, wq, cos, sin, pos, slot, dk, dv_, table, H, G, 2, Dm, D, Dm, 1e-6, bf), steps, warmup)
    rows.append((f"q | k | v: bias, {taps}-tap convolution, row norms, temperature, page store, tail", ms_k, frac_bw(T * C * 4, ms_k),
                 "Duratar: q/k norm + rotary + K/V page store (fp32 in)", ms_l, frac_bw(T * C * 6, ms_l), "HBM"))
    # --- the state space's convolution vs Kudonex's (fp32 in and out)
    u_in = proj[:, C:C + inner]
    cw2, cb2, tail2 = rnd(inner, taps) * 0.5, rnd(inner), torch.zeros(Bq + 1, taps - 1, inner, device=dev)
    ms_k = t(lambda: short_conv(u_in, cw2, tail2, pos, slot, runs, 1, act=True, bias=cb2, out_dtype=bf), steps, warmup)
    x32 = rnd(T, inner + 8)
    ms_l = t(lambda: short_conv(x32[:, :inner], cw2, tail2, pos, slot, runs, 1, act=True, bias=cb2), steps, warmup)
    rows.append((f"state-space convolution + bias + silu + tail, {inner} channels, bf16", ms_k, frac_bw(T * inner * 4, ms_k),
                 "Kudonex: the same in fp32", ms_l, frac_bw(T * inner * 8, ms_l), "HBM"))
    del x32, p32
    # --- prompt attention, causal vs Gorozen's
    ck.normal_()
    cv.normal_()
    q = rnd(T, H * D).to(bf)
    fl = 4 * H * D * T * T / 2
    ms_k = t(lambda: multimap_attention(q, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, pieces=pieces, max_pos=T - 1), steps, warmup)
    ms_l = t(lambda: paged_attention(q, ck, cv, table, pos, slot, H, G, D, D ** -0.5, max_pos=T - 1, pieces=pieces), steps, warmup)
    rows.append((f"prompt attention, causal, {T} tokens (mma.sync)", ms_k, frac_fl(fl, ms_k), "Gorozen: prompt attention (mma.sync)", ms_l, frac_fl(fl, ms_l),
                 "bf16 tensor"))
    # --- decode attention: 64 sequences at context 4032
    nbd = Bq * (ctx // BS + 1)
    ckd, cvd = (rnd(nbd + 1, G, BS, D).to(bf) for _ in range(2))
    tabd = torch.arange(1, nbd + 1, dtype=torch.int32, device=dev).view(Bq, -1)
    qd = rnd(Bq, H * D).to(bf)
    by = Bq * G * (ctx + 1) * D * 4
    ms_k = t(lambda: multimap_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, 1, D, D, D ** -0.5, max_pos=ctx), steps, warmup)
    ms_l = t(lambda: paged_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, D, D ** -0.5, max_pos=ctx), steps, warmup)
    rows.append((f"decode attention, {Bq} sequences at {ctx}", ms_k, frac_bw(by, ms_k), "Gorozen: decode attention", ms_l, frac_bw(by, ms_l), "HBM"))
    del ckd, cvd
    # --- decays of the matrix memory vs Duratar's gates
    a1, a2, ab = rnd(T, rank), rnd(SH * SD, rank), torch.full((SH * SD,), 2.0, device=dev)
    ms_k = t(lambda: lowrank_decay(a1, a2, ab, 16.0, fast=True), steps, warmup)
    SG = max(1, SH // 4)
    qs, ks, aa, bb = rnd(T, SG * SD), rnd(T, SG * SD), rnd(T, SH * SD), rnd(T, SH)
    dtb, alog = torch.zeros(SH * SD, device=dev), torch.zeros(SH, device=dev)
    ms_l = t(lambda: delta_gates(qs, ks, aa, bb, dtb, alog, SG, SH, SD, 1.0), steps, warmup)
    roof = max(frac_bw(T * SH * SD * 4, ms_k), 3 * T * SH * SD / (ms_k * 1e-3) / 1e12 / EXP_RATE)     # two exponentials, one logarithm
    rows.append((f"per-channel decays from a rank-{rank} input, {SH * SD} channels", ms_k, roof,
                 "Duratar: unit q / k, decays, beta", ms_l, frac_bw(T * (2 * SG * SD + SH * SD + SH) * 8, ms_l),
                 "slower of HBM and special-function rate; Duratar: HBM"))
    # --- matrix memory: prompt and decode batch
    g = lowrank_decay(a1, a2, ab, 16.0, fast=True)
    q16, k16, vs = rnd(T, SH * SD) * SD ** -0.5, rnd(T, SH * SD) * SD ** -0.5, rnd(T, SH * SDv)
    st0 = torch.zeros(Bq + 1, SH, SD, SDv, device=dev)
    ga, gb = torch.rand(T, SH, device=dev) * 0.1 + 0.9, torch.rand(T, SH, device=dev)
    fl = SH * 2 * 2 * SD * SDv * T
    ms_k = t(lambda: linear_scan(q16, k16, vs, st0, pos, slot, runs, 1, SH, SH, SD, SDv, "channel", g=g, pieces=pieces), steps, warmup)
    ms_l = t(lambda: linear_scan(q16, k16, vs, st0, pos, slot, runs, 1, SH, SH, SD, SDv, "gated", g=ga, beta=gb), steps, warmup)
    rows.append((f"scan with a decay per key channel, one prompt of {T} tokens, {SH} heads of {SD} x {SDv}", ms_k, frac_fma(fl, ms_k),
                 "Kudonex: gated scan (decay per head)", ms_l, frac_fma(fl, ms_l), "nominal fp32 FMA rate"))
    by = Bq * SH * SD * SDv * 8
    ms_k = t(lambda: linear_scan(q16[:Bq], k16[:Bq], vs[:Bq], st0, pd, sd_, None, Bq, SH, SH, SD, SDv, "channel", g=g[:Bq]), steps, warmup)
    ms_l = t(lambda: linear_scan(q16[:Bq], k16[:Bq], vs[:Bq], st0, pd, sd_, None, Bq, SH, SH, SD, SDv, "gated", g=ga[:Bq], beta=gb[:Bq]), steps, warmup)
    rows.append((f"scan with a decay per key channel, decode batch of {Bq}", ms_k, frac_bw(by, ms_k), "Kudonex: gated scan, decode batch", ms_l,
                 frac_bw(by, ms_l), "HBM"))
    # --- selective scan: prompt and decode batch
    u, dt = rnd(T, inner).to(bf), rnd(T, inner) - 3
    bc, gate = rnd(T, 2 * N).to(bf), rnd(T, inner).to(bf)
    A, Dk, db = -torch.rand(N, inner, device=dev) * 4 - 0.1, torch.ones(inner, device=dev), torch.zeros(inner, device=dev)
    st2 = torch.zeros(Bq + 1, N, inner, device=dev)
    ms_s = t(lambda: selective_scan(u, dt, db, bc[:, :N], bc[:, N:], A, Dk, st2, pos, slot, runs, 1, gate=gate, pieces=pieces), steps, warmup)
    roof = max(T * inner * N / (ms_s * 1e-3) / 1e12 / EXP_RATE, frac_fma(8 * T * inner * N, ms_s))
    rows.append((f"selective scan, one prompt of {T} tokens, {inner} channels x {N} states", ms_s, roof,
                 "Kudonex: gated scan (one decay per head and token)", rows[-2][4], rows[-2][5],
                 "slower of special-function and fp32 FMA rate; Kudonex: fp32 FMA rate"))
    by2 = Bq * (N * inner * 8 + inner * (4 + 2 + 2 + 2))
    ms_k = t(lambda: selective_scan(u[:Bq], dt[:Bq], db, bc[:Bq, :N], bc[:Bq, N:], A, Dk, st2, pd, sd_, None, Bq, gate=gate[:Bq]), steps, warmup)
    rows.append((f"selective scan, decode batch of {Bq}", ms_k, frac_bw(by2, ms_k), "Kudonex: gated scan, decode batch", ms_l, frac_bw(by, ms_l), "HBM"))
    # --- read-out vs Kudonex's
    o32, wv, wfull = rnd(T, SH * SDv), torch.ones(SDv, device=dev), torch.ones(SH * SDv, device=dev)
    post = rnd(T, SH * SDv)
    ms_k = t(lambda: scan_readout(o32, SH, SDv, wv, SH, 1e-6, bf, oscale=SD ** -0.5, post=post, post_act="silu"), steps, warmup)
    o1, e1 = rnd(T, SH * (SDv + 1)), torch.rand(T, SH, device=dev)
    ms_l = t(lambda: scan_readout(o1, SH, SDv, wfull, SH, 1e-6, bf, e=e1, den_eps=1e-6, oscale=SD ** -0.5, post=post), steps, warmup)
    rows.append(("read-out: per-head norm, shared weight, silu gate", ms_k, frac_bw(T * SH * SDv * 10, ms_k),
                 "Kudonex: normaliser, per-head norm, weight, sigmoid gate", ms_l, frac_bw(T * SH * SDv * 10, ms_l), "HBM"))
    # --- router, gather and combine with identity experts vs Kudonex's
    hb = rnd(T, W).to(bf)
    wr, corr = rnd(E + X, W) * 0.05, torch.zeros(E + X, device=dev)
    ms_k = t(lambda: route_grouped(hb, wr, corr, top, softmax=True), steps, warmup)
    ms_l = t(lambda: route_grouped(hb, wr[:E].contiguous(), corr[:E].contiguous(), 2, 2, 1, 1, softmax=True), steps, warmup)
    rows.append((f"router: softmax over {E} + {X}, correction, top {top}", ms_k, frac_bw(T * W * 2, ms_k),
                 f"Kudonex: router over {E}, best group of 2, top 2", ms_l, frac_bw(T * W * 2, ms_l), "HBM"))
    ti, tp, _ = route_grouped(hb, wr, corr, top, softmax=True)
    ti2, tp2, _ = route_grouped(hb, wr[:E].contiguous(), corr[:E].contiguous(), 2, 2, 1, 1, softmax=True)
    d, d2 = dispatch(ti, E), dispatch(ti2, E)
    n_real = int((ti < E).sum())
    ms_k = t(lambda: gather_rows(hb, d), steps, warmup)
    ms_l = t(lambda: torch.zeros(d2.rows, W, dtype=bf, device=dev).index_copy(0, d2.dest, hb.index_select(0, d2.tok)), steps, warmup)
    rows.append((f"expert rows gathered ({n_real} of {T * top} assignments have one)", ms_k, frac_bw(T * W * 2 + n_real * W * 2, ms_k),
                 f"library gather and copy ({T * 2} assignments)", ms_l, frac_bw(T * W * 2 + T * 2 * W * 2, ms_l), "HBM"))
    ye, ye2 = rnd(d.rows, W).to(bf), rnd(d2.rows, W).to(bf)
    ms_k = t(lambda: moe_combine(ye, d.dest, tp, identity=res), steps, warmup)
    ms_l = t(lambda: moe_combine(ye2, d2.dest, tp2), steps, warmup)
    rows.append(("expert combination with identity rows (fp32)", ms_k, frac_bw(T * W * 8 + n_real * W * 2, ms_k),
                 "Kudonex: expert combination", ms_l, frac_bw(T * W * 4 + T * 2 * W * 2, ms_l), "HBM"))
    return rows, which


def run(args, root):
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    from llm_in_practise_b200.ops import _native as nv
    nv.lib()
    n0 = nv.launch_count
    t0 = time.time()
    res = {"metric": "Lorenex vs Kudonex at equal layer sizes: prefill / decode tok/s", "unit": "tok/s", "n_gpus": 1,
           "steps": args.steps, "warmup": max(3, args.warmup), "dtype": "bf16", "data": "synthetic", "sizes": {}, "kernels": {}}
    first = next(iter(SIZES))
    for size in SIZES:
        res["sizes"][size] = {k: round(v, 3) for k, v in end_to_end(size, dev, args.steps, args.warmup).items()}
        torch.cuda.empty_cache()
    for size in SIZES:
        rows, which = kernel_rows(size, dev, args.steps, args.warmup, root)
        res["kernels"][size] = [{"lorenex": a, "ms": round(b, 4), "of_roofline": round(c, 3), "like": d, "like_ms": round(e, 4),
                                 "like_of_roofline": round(f, 3), "bound": g, "gap_ratio": round(f / c, 2) if c and d else None}
                                for a, b, c, d, e, f, g in rows]
        res["roofline"] = which
        torch.cuda.empty_cache()
    res["gpu_launches"] = nv.launch_count - n0
    res["seconds"] = round(time.time() - t0, 1)
    res["value"] = res["sizes"][first]["lorenex_decode_tok_s"]
    res["config"] = {"model": "lorenex: two parallel layers (attention beside a selective state space, dense feed-forward) and two matrix-memory "
                              "layers (MoE with identity experts); kudonex: attention, mamba2, attention, mlstm with MoE of the same active size",
                     "sizes": {k: list(v) for k, v in SIZES.items()},
                     "l2": "single kernels: replayed from a CUDA graph, 256 MB flush between iterations; steps: weights + cache exceed L2"}
    print(json.dumps(res))
    return 0
