"""Nedesun beside Lorenex (the framework's closest design: attention beside a recurrence in one layer, a matrix memory with a
decay per key channel in the next) at equal layer sizes, random weights: prefill and decode throughput through each model's
own generator, and the time of each Nedesun kernel next to the kernel that does the like job in Lorenex, Duratar or Gorozen,
as fractions of the measured roofline (``MEASURED_PEAKS.json``: copy bandwidth and cuBLAS bf16 rate of this pool's B200).
Scans are given against the nominal fp32 FMA rate, decays against the slower of HBM and the special-function rate.

    python bench.py --workload nedesun [--steps K --warmup W]

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
from lorenex_bench import EXP_RATE, lorenex_config
from segorax_bench import GraphTimer

SIZES = {
    # name: (width, attention heads, kv heads, head size, window, kept, chunk, scan heads, key size, value size, delta q/k heads, taps,
    #        decay rank, gated ff, vocab)
    "2k wide, 16 heads": (2048, 16, 4, 128, 1024, 4, 2048, 16, 128, 128, 4, 4, 16, 4096, 32768),
    "4k wide, 16 attention heads, 32 scan heads": (4096, 16, 4, 128, 1024, 4, 2048, 32, 128, 128, 8, 4, 16, 8192, 32768),
}


def nedesun_config(W, H, G, D, win, keep, chunk, SH, SD, SDv, SG, taps, rank, F, V):
    mlp = {"kind": "dense", "ff": F}
    par = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "mask": {"size": win, "keep_first": keep}, "scale": D ** -0.5},
           "right": {"heads": SH, "kv_heads": SG, "dim": SD, "vdim": SDv, "conv": taps}}
    att = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "mask": {"size": chunk}, "rot": {"base": 1e6, "dims": D}, "scale": D ** -0.5,
           "softcap": 50.0, "v_mix": True}
    wkv = {"heads": SH, "dim": SD}
    layers = [{"type": "parallel", "mixer": par, "mlp": mlp}, {"type": "wkv", "mixer": wkv, "mlp": mlp},
              {"type": "attention", "mixer": att, "mlp": mlp}, {"type": "wkv", "mixer": wkv, "mlp": mlp}]
    return {"architecture": "Nedesun", "layers": layers, "norm": {"eps": 1e-6}, "embedding": {"scale": W ** 0.5}, "residual_mult": 0.3,
            "vocab": V, "width": W}


def build_models(size, dev):
    from llm_in_practise_b200.models.lorenex import LorenexConfig, LorenexForCausalLM
    from llm_in_practise_b200.models.nedesun import NedesunConfig, NedesunForCausalLM
    W, H, G, D, win, keep, chunk, SH, SD, SDv, SG, taps, rank, F, V = SIZES[size]
    torch.manual_seed(0)
    nd = NedesunForCausalLM(NedesunConfig.from_dict(nedesun_config(*SIZES[size])), dtype=torch.bfloat16, device=dev,
                            decay_ranks={1: rank, 3: rank}).eval()
    # the ungated feed-forward of equal size has half as many more rows; a state space of twice the width beside the attention
    lx = LorenexForCausalLM(LorenexConfig.from_dict(lorenex_config(W, H, G, D, SH, SD, SDv, rank, 2 * W, 16, W // 16, taps, 3 * F // 2, 8, 2, 4, V)),
                            dtype=torch.bfloat16, device=dev, decay_ranks={1: rank, 3: rank}).eval()
    for model in (nd, lx):
        for n, p in model.named_parameters():
            leaf = n.split(".")[-1]
            if p.dtype == torch.bfloat16 and p.dim() >= 2 and leaf != "embed_tokens":
                p.data.normal_(std=p.shape[-1] ** -0.5)
            elif leaf in ("conv_w", "qkv_conv", "router", "a2", "w2", "mu", "u"):
                p.data.normal_(std=0.3)
            elif leaf == "act":
                p.data.fill_(0.5)
            elif leaf == "a2_bias":
                p.data.fill_(2.0)
            elif leaf == "w0":
                p.data.fill_(-4.0)
            elif leaf == "dt_bias" and model is nd:
                p.data.fill_(-3.0)
    return nd, lx


@torch.no_grad()
def end_to_end(size, dev, steps, warmup, prompt=2048, batch=32, ctx=1024):
    """tokens/s of (a) one prompt of ``prompt`` tokens, (b) one decode step of ``batch`` sequences at context ``ctx``."""
    from llm_in_practise_b200.inference import RaggedGenerator
    t = Timer(dev, flush=False)
    out = {}
    V = SIZES[size][-1]
    toks = torch.randint(0, V, (prompt,)).tolist()
    for name, model in zip(("nedesun", "lorenex"), build_models(size, dev)):
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
    """Single kernels at the layer sizes: (name, Nedesun ms, fraction of roofline, like kernel, ms, fraction, bound)."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops import elementwise as ew
    from llm_in_practise_b200.ops.gemm import linear_each, linear_exact
    from llm_in_practise_b200.ops.linear_scan import delta_gates, linear_scan, lowrank_decay, scan_readout, short_conv, token_shift
    from llm_in_practise_b200.ops.multimap_attention import conv_qknorm_store, multimap_attention, qkv_store
    from llm_in_practise_b200.ops.norm import sandwich_norm
    from llm_in_practise_b200.ops.paged_attention import paged_attention
    hbm, tf, which = _peaks(root)
    W, H, G, D, win, keep, chunk, SH, SD, SDv, SG, taps, rank, F, V = SIZES[size]
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
    run = lambda f: t(f, steps, warmup)                                                           # noqa: E731
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    slot = torch.zeros(T, dtype=torch.int32, device=dev)
    pd, sd_ = torch.full((Bq,), ctx, dtype=torch.int32, device=dev), torch.arange(Bq, dtype=torch.int32, device=dev)
    pieces = make_pieces([(0, T, 0, 0)], dev)
    runs = pieces.runs
    # --- norm steps
    y32, y33, res, wn = rnd(T, W), rnd(T, W), rnd(T, W), torch.ones(W, device=dev)
    ms_l = run(lambda: sandwich_norm(y32, wn, res, None, 1e-6, 0.0, bf, branch_mult=0.3, cast_next=True))
    like = ("Lorenex: output norm + residual + bf16 copy", ms_l, frac_bw(T * W * 14, ms_l))
    ms = run(lambda: sandwich_norm(y32, None, res, wn, 1e-6, 0.0, bf, branch_mult=0.3))
    rows.append(("scaled residual + next norm", ms, frac_bw(T * W * 14, ms), *like, "HBM"))
    ms = run(lambda: sandwich_norm(y32, wn, res, wn, 1e-6, 0.0, bf, branch_mult=0.15, y2=y33, post_w2=wn))
    rows.append(("two normed branches + residual + next norm", ms, frac_bw(T * W * 18, ms), *like, "HBM"))
    # --- stores
    C = (H + 2 * G) * D
    nb = T // BS
    ck, cv, c1 = (torch.zeros(nb + 1, G, BS, D, dtype=bf, device=dev) for _ in range(3))
    table = torch.arange(1, nb + 1, dtype=torch.int32, device=dev).view(1, nb)
    proj = rnd(T, C + 2 * W).to(bf)
    bias, cw, tail = rnd(C), rnd(C, taps) * 0.5, torch.zeros(Bq + 1, taps - 1, C, device=dev)
    ms_l = run(lambda: conv_qknorm_store(proj[:, :C], bias, cw, tail, pos, slot, runs, 1, ck, cv, table, H, G, D, D, 1e-6, bf, temp=(0.1, 8192.0),
                                         norm_v=True))
    like = ("Lorenex: bias, convolution, row norms, page store, tail", ms_l, frac_bw(T * C * 4, ms_l))
    wq = torch.ones(D, device=dev)
    ms = run(lambda: qkv_store(proj[:, :C], None, wq, wq, None, pos, slot, ck, cv, table, H, G, D, D, 0, 1e-6, bf))
    rows.append(("q / k norms + page store", ms, frac_bw(T * C * 4, ms), *like, "HBM"))
    rope, lam = ew.rope_tables_partial(T, D, 1e6, dev), torch.full((1,), 0.3, device=dev)
    ms = run(lambda: qkv_store(proj[:, :C], bias, None, None, rope, pos, slot, ck, cv, table, H, G, D, D, D, 1e-6, bf, v_first=c1, v_lambda=lam))
    rows.append(("bias, rotary, mixed values + page store", ms, frac_bw(T * (C * 4 + G * D * 2 + D * 4), ms), *like, "HBM"))
    # --- prompt attention
    ck.normal_()
    cv.normal_()
    q = rnd(T, H * D).to(bf)
    sink, gate = torch.zeros(H, device=dev), rnd(T, H)
    fl = lambda keys: 4 * H * D * keys                                                            # noqa: E731
    full = T * (T + 1) / 2
    ms_l = run(lambda: multimap_attention(q, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, pieces=pieces, max_pos=T - 1))
    like = ("Lorenex: prompt attention, causal (mma.sync)", ms_l, frac_fl(fl(full), ms_l))
    seen = sum(min(p + 1, win) + max(0, min(keep, p + 1 - win)) for p in range(T))
    ms_w = run(lambda: multimap_attention(q, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, win, keep, pieces=pieces, max_pos=T - 1))
    ms = run(lambda: multimap_attention(q, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, win, keep, pieces=pieces, max_pos=T - 1, sink=sink))
    rows.append((f"prompt attention, window {win} + {keep} kept, sink, {T} tokens (mma.sync)", ms, frac_fl(fl(seen), ms),
                 "the same window without a sink", ms_w, frac_fl(fl(seen), ms_w), "bf16 tensor"))
    seen = sum(p % chunk + 1 for p in range(T))
    ms = run(lambda: multimap_attention(q, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, pieces=pieces, max_pos=T - 1, softcap=50.0, chunk=chunk,
                                        gate=gate))
    rows.append((f"prompt attention, chunks of {chunk}, capped scores, head gates (mma.sync)", ms, frac_fl(fl(seen), ms), *like, "bf16 tensor"))
    ms = run(lambda: multimap_attention(q * 8, ck, cv, table, pos, slot, H, G, 1, D, D, D ** -0.5, pieces=pieces, max_pos=T - 1, softcap=50.0, chunk=chunk,
                                        gate=gate))
    rows.append(("the same with scores near the cap", ms, frac_fl(fl(seen), ms), *like, "bf16 tensor"))
    # --- decode attention: 64 sequences at context 4032
    nbd = Bq * (ctx // BS + 1)
    ckd, cvd = (rnd(nbd + 1, G, BS, D).to(bf) for _ in range(2))
    tabd = torch.arange(1, nbd + 1, dtype=torch.int32, device=dev).view(Bq, -1)
    qd, gd = rnd(Bq, H * D).to(bf), rnd(Bq, H)
    sz = torch.zeros(H, device=dev)
    ms_l = run(lambda: paged_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, D, D ** -0.5, sinks=sz, window=win, max_pos=ctx))
    ms = run(lambda: multimap_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, 1, D, D, D ** -0.5, win, keep, max_pos=ctx, sink=sz))
    by = Bq * G * D * 4
    rows.append((f"decode attention, {Bq} sequences at {ctx}, window {win} + {keep}, sink", ms, frac_bw(by * (win + keep), ms),
                 f"Gorozen: decode attention, window {win}, sinks", ms_l, frac_bw(by * win, ms_l), "HBM"))
    ms_l = run(lambda: multimap_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, 1, D, D, D ** -0.5, max_pos=ctx))
    ms = run(lambda: multimap_attention(qd, ckd, cvd, tabd, pd, sd_, H, G, 1, D, D, D ** -0.5, max_pos=ctx, softcap=50.0, chunk=2 * chunk, gate=gd))
    rows.append((f"decode attention, {Bq} sequences at {ctx} of one chunk, capped scores, gates", ms, frac_bw(by * (ctx + 1), ms),
                 "Lorenex: decode attention", ms_l, frac_bw(by * (ctx + 1), ms_l), "HBM"))
    del ckd, cvd
    # --- the delta rule's inputs and scan
    CC = 2 * SG * SD + SH * SDv
    u_in = rnd(T, CC + 64).to(bf)[:, :CC]
    cw2, tail2 = rnd(CC, taps) * 0.5, torch.zeros(Bq + 1, taps - 1, CC, device=dev)
    x32 = rnd(T, CC + 8)
    ms = run(lambda: short_conv(u_in, cw2, tail2, pos, slot, runs, 1, act=True))
    ms_l = run(lambda: short_conv(x32[:, :CC], cw2, tail2, pos, slot, runs, 1, act=True))
    rows.append((f"convolution + silu + tail, {CC} channels, bf16 in, fp32 out", ms, frac_bw(T * CC * 6, ms), "Duratar: the same, fp32 in", ms_l,
                 frac_bw(T * CC * 8, ms_l), "HBM"))
    del x32
    qs = rnd(T, SG * SD) * SD ** -0.5
    ks = torch.nn.functional.normalize(rnd(T, SG, SD), dim=-1).view(T, -1)
    vs = rnd(T, SH * SDv)
    ah, bb, ac = rnd(T, SH), rnd(T, SH), rnd(T, SH * SD)
    z1, zc, alog = torch.zeros(SH, device=dev), torch.zeros(SH * SD, device=dev), torch.zeros(SH, device=dev)
    q2, k2 = qs.clone(), ks.clone()
    ms = run(lambda: delta_gates(q2, k2, ah, bb, z1, alog, SG, SH, SD, 1.0))
    ms_l = run(lambda: delta_gates(q2, k2, ac, bb, zc, alog, SG, SH, SD, 1.0))
    rows.append(("unit q / k, decays per head, beta (in place)", ms, frac_bw(T * (2 * SG * SD + 2 * SH) * 8, ms),
                 "Duratar: the same with decays per channel", ms_l, frac_bw(T * (2 * SG * SD + SH * SD + SH) * 8, ms_l), "HBM"))
    gh, gc, be = torch.rand(T, SH, device=dev) * 0.1 + 0.9, torch.rand(T, SH * SD, device=dev) * 0.1 + 0.9, torch.rand(T, SH, device=dev)
    st = torch.zeros(Bq + 1, SH, SD, SDv, device=dev)
    fl_tok = SH * 3 * 2 * SD * SDv
    ms = run(lambda: linear_scan(qs, ks, vs, st, pos, slot, runs, 1, SH, SG, SD, SDv, "head_delta", g=gh, beta=be, pieces=pieces))
    ms_l = run(lambda: linear_scan(qs, ks, vs, st, pos, slot, runs, 1, SH, SG, SD, SDv, "delta", g=gc, beta=be))
    rows.append((f"delta scan, a decay per head, one prompt of {T} tokens, {SH} heads of {SD} x {SDv}", ms, frac_fma(fl_tok * T, ms),
                 "Duratar: delta scan (decay per channel)", ms_l, frac_fma(fl_tok * T, ms_l), "nominal fp32 FMA rate"))
    by = Bq * SH * SD * SDv * 8
    ms = run(lambda: linear_scan(qs[:Bq], ks[:Bq], vs[:Bq], st, pd, sd_, None, Bq, SH, SG, SD, SDv, "head_delta", g=gh[:Bq], beta=be[:Bq]))
    ms_l = run(lambda: linear_scan(qs[:Bq], ks[:Bq], vs[:Bq], st, pd, sd_, None, Bq, SH, SG, SD, SDv, "delta", g=gc[:Bq], beta=be[:Bq]))
    rows.append((f"delta scan, decode batch of {Bq}", ms, frac_bw(by, ms), "Duratar: delta scan, decode batch", ms_l, frac_bw(by, ms_l), "HBM"))
    del gc, ac
    # --- wkv: shifts, products, decays, scan
    h = rnd(T, W).to(bf)
    mu, prev = rnd(5, W), torch.zeros(Bq + 1, 1, W, device=dev)
    cw3, tail3 = rnd(W, taps) * 0.5, torch.zeros(Bq + 1, taps - 1, W, device=dev)
    ms = run(lambda: token_shift(h, mu, prev, pos, slot, runs, 1))
    ms_l = run(lambda: short_conv(h, cw3, tail3, pos, slot, runs, 1, act=True, out_dtype=bf))
    rows.append((f"five token shifts + carry, {W} columns", ms, frac_bw(T * W * 12, ms), "Lorenex: convolution + silu + tail, bf16", ms_l,
                 frac_bw(T * W * 4, ms_l), "HBM"))
    N = SH * SD
    x4, w4 = rnd(4, T, W).to(bf), (rnd(4, N, W) * W ** -0.5).to(bf)
    wcat = w4.view(4 * N, W)
    ms = run(lambda: linear_each(x4, w4))
    ms_l = run(lambda: linear_exact(h, wcat, out_dtype=f32))
    rows.append((f"r, k, v, g products of their own inputs, {T} tokens", ms, frac_fl(8 * T * N * W, ms), "Lorenex: one product of one input", ms_l,
                 frac_fl(8 * T * N * W, ms_l), "bf16 tensor"))
    x16, h16 = x4[:, :16].contiguous(), h[:16].contiguous()
    ms = run(lambda: linear_each(x16, w4))
    ms_l = run(lambda: linear_exact(h16, wcat, out_dtype=f32))
    rows.append(("the same, decode batch of 16", ms, frac_bw(8 * N * W, ms), "Lorenex: one product of one input", ms_l, frac_bw(8 * N * W, ms_l), "HBM"))
    del x4
    a1, a2, ab = rnd(T, rank), rnd(N, rank), torch.full((N,), -4.0, device=dev)
    roof = lambda ms, n: max(frac_bw(T * N * 4, ms), n * T * N / (ms * 1e-3) / 1e12 / EXP_RATE)   # noqa: E731
    ms = run(lambda: lowrank_decay(a1, a2, ab, fast=True, form="exp_exp"))
    ms_l = run(lambda: lowrank_decay(a1, a2, ab, 16.0, fast=True))
    rows.append((f"decays exp(-exp(.)) from a rank-{rank} input, {N} channels", ms, roof(ms, 2), "Lorenex: decays sigmoid(.)^(1/tau)", ms_l,
                 roof(ms_l, 3), "slower of HBM and special-function rate"))
    w = lowrank_decay(a1, a2, ab, fast=True, form="exp_exp")
    r16, k16, vv, bonus = rnd(T, N) * SD ** -0.5, rnd(T, N) * SD ** -0.5, rnd(T, N), rnd(SH, SD)
    st = torch.zeros(Bq + 1, SH, SD, SD, device=dev)
    fl_tok = SH * 2 * 2 * SD * SD
    ms = run(lambda: linear_scan(r16, k16, vv, st, pos, slot, runs, 1, SH, SH, SD, SD, "channel", g=w, pieces=pieces, u=bonus))
    ms_l = run(lambda: linear_scan(r16, k16, vv, st, pos, slot, runs, 1, SH, SH, SD, SD, "channel", g=w, pieces=pieces))
    rows.append((f"wkv scan with a bonus, one prompt of {T} tokens, {SH} heads of {SD} x {SD}", ms, frac_fma(fl_tok * T, ms),
                 "Lorenex: scan with a decay per key channel", ms_l, frac_fma(fl_tok * T, ms_l), "nominal fp32 FMA rate"))
    by = Bq * SH * SD * SD * 8
    ms = run(lambda: linear_scan(r16[:Bq], k16[:Bq], vv[:Bq], st, pd, sd_, None, Bq, SH, SH, SD, SD, "channel", g=w[:Bq], u=bonus))
    ms_l = run(lambda: linear_scan(r16[:Bq], k16[:Bq], vv[:Bq], st, pd, sd_, None, Bq, SH, SH, SD, SD, "channel", g=w[:Bq]))
    rows.append((f"wkv scan with a bonus, decode batch of {Bq}", ms, frac_bw(by, ms), "Lorenex: scan, decode batch", ms_l, frac_bw(by, ms_l), "HBM"))
    # --- read-outs
    o32, post, wh, wc = rnd(T, N), rnd(T, N), torch.ones(SD, device=dev), torch.ones(N, device=dev)
    postb = post.to(bf)
    ms_l = run(lambda: scan_readout(o32, SH, SD, wh, SH, 1e-6, bf, post=post, post_act="silu"))
    like = ("Lorenex: read-out (shared weight, fp32 gate)", ms_l, frac_bw(T * N * 10, ms_l))
    ms = run(lambda: scan_readout(o32, SH, SD, wc, SH, 1e-6, bf, post=post, post_act="silu"))
    rows.append(("wkv read-out: per-head norm, a weight per column, silu gate", ms, frac_bw(T * N * 10, ms), *like, "HBM"))
    ms = run(lambda: scan_readout(o32, SH, SD, wh, SH, 1e-6, bf, post=postb, post_act="silu"))
    rows.append(("delta read-out: per-head norm, shared weight, bf16 silu gate", ms, frac_bw(T * N * 8, ms), *like, "HBM"))
    # --- gated unit
    gu = rnd(T, 2 * F).to(bf)
    ms = run(lambda: ew.act_glu(gu, "silu"))
    ms_l = run(lambda: ew.clamped_glu(gu, 7.0, 1.702, 1.0))
    rows.append((f"silu gated unit, {F} columns", ms, frac_bw(T * F * 6, ms), "Gorozen: clamped gated unit", ms_l, frac_bw(T * F * 6, ms_l), "HBM"))
    return rows, which


def run(args, root):
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    from llm_in_practise_b200.ops import _native as nv
    nv.lib()
    n0 = nv.launch_count
    t0 = time.time()
    res = {"metric": "Nedesun vs Lorenex at equal layer sizes: prefill / decode tok/s", "unit": "tok/s", "n_gpus": 1,
           "steps": args.steps, "warmup": max(3, args.warmup), "dtype": "bf16", "data": "synthetic", "sizes": {}, "kernels": {}}
    first = next(iter(SIZES))
    for size in SIZES:
        res["sizes"][size] = {k: round(v, 3) for k, v in end_to_end(size, dev, args.steps, args.warmup).items()}
        torch.cuda.empty_cache()
    for size in SIZES:
        rows, which = kernel_rows(size, dev, args.steps, args.warmup, root)
        res["kernels"][size] = [{"nedesun": a, "ms": round(b, 4), "of_roofline": round(c, 3), "like": d, "like_ms": round(e, 4),
                                 "like_of_roofline": round(f, 3), "bound": g, "gap_ratio": round(f / c, 2)} for a, b, c, d, e, f, g in rows]
        res["roofline"] = which
        torch.cuda.empty_cache()
    res["gpu_launches"] = nv.launch_count - n0
    res["seconds"] = round(time.time() - t0, 1)
    res["value"] = res["sizes"][first]["nedesun_decode_tok_s"]
    res["config"] = {"model": "nedesun: parallel (window attention with a sink beside a delta rule), wkv, chunked attention, wkv, gated feed-forwards; "
                              "lorenex: parallel, matrix memory, parallel, matrix memory with feed-forwards of the same active size",
                     "sizes": {k: list(v) for k, v in SIZES.items()},
                     "l2": "single kernels: replayed from a CUDA graph, 256 MB flush between iterations; steps: weights + cache exceed L2"}
    print(json.dumps(res))
    return 0
