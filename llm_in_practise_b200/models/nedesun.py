"""Nedesun: a decoder-only language model whose layers mix tokens in one of three ways: sink attention in a window beside a
gated delta rule, softly capped attention in chunks with values shared along the depth, or a matrix memory over shifted
tokens with a bonus for the current one.

The stream x (fp32) starts as ``embed[token] * s_e``. RMS(y) = y / sqrt(mean(y^2) + eps). Layer i (tensors ``l<i>.*``),
m = ``residual_mult``:

    x <- x + m mixer(RMS(x) * g_1)          x <- x + m ff(RMS(x) * g_2)     (the second line only if the layer has a feed-forward)

* ``parallel``: 0.5 (RMS(left(h)) * g_l + RMS(right(h)) * g_r).
  left: grouped-query attention without rotation; q and k rows RMS-normed with a weight; position i sees j <= i if i - j < size
  or j < keep_first; exp(sink_h) joins the softmax's denominator.
  right: q, k, v pass a short causal convolution and silu; q, k become unit vectors (q also / sqrt(dim)); per head
  beta = sigmoid(W_b h), g = exp(-exp(A_log) softplus(W_a h + dt_bias)); S <- g S, u = beta (v - S^T k), S <- S + k u^T,
  o = S^T q; every head RMS-normed with a weight shared by the heads, times silu(W_g h), then W_o.
* ``attention``: biased q, k, v, o; split-half rotary on the first ``rot.dims`` dims; scores c tanh(s / c); position i sees
  j <= i of its own chunk (i // size == j // size); in layers with ``v_mix``, v <- (1 - lambda) v + lambda v_1 with v_1 the values
  of the first such layer (the mixed v is cached, the first layer's own v are its cached ones); head h times sigmoid(W_g h)_h.
* ``wkv``: r, k, v, g, w each read h + (h' - h) mu_s, h' the previous token's h; w = exp(-exp(W_2 tanh(W_1 .) + w_0)) per head and
  key channel; o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T; every head RMS-normed, times a weight per column,
  times silu(g), then W_o.
* feed-forward: W_down (silu(W_gate h) * W_up h).

The output is ``embed @ (RMS(x) * g)`` (the embedding table without its scale). What is fp32 whatever the model dtype: the
stream, every norm, rotary tables and arithmetic, attention scores and softmax, unit norms, decays, beta, the states and
tails, the scans and their read-outs, the head gates' and the scans' gate projections, the logits.

Keys and values live in the paged cache (``kv_layout``), recurrent states, convolution tails and the previous token's h in its
per-sequence state rows (``state_layout``). ``inference/ragged.RaggedGenerator`` and ``serve/engine.LLMEngine`` drive
``forward_ragged``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

import torch
from torch import nn

from ..ops import elementwise as ew
from ..ops.gemm import linear_each, linear_exact
from ..ops.linear_scan import delta_gates, linear_scan, lowrank_decay, scan_readout, short_conv, token_shift
from ..ops.multimap_attention import multimap_attention, qkv_store
from ..ops.norm import sandwich_norm

MIXERS = ("parallel", "attention", "wkv")
UNIT_EPS = 1e-6                             # inside the root of the delta rule's unit norm: fixed by the design
BRANCH = 0.5                                # weight of each half of a parallel mixer: fixed by the design
SHIFTS = ("r", "k", "v", "g", "w")          # the mixes of a wkv layer; the first four are projected to heads x dim


@dataclass
class NedesunParallel:
    heads: int                                  # left: attention
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int
    rheads: int                                 # right: delta rule
    rkv_heads: int
    rdim: int
    rvdim: int
    conv: int


@dataclass
class NedesunAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    chunk: int
    rot_dims: int
    rot_base: float
    v_mix: bool
    v_from: Optional[int] = None                # the first layer with v_mix, for the later ones


@dataclass
class NedesunWKV:
    heads: int
    dim: int


@dataclass
class NedesunLayerSpec:
    type: str
    mixer: object
    ff: int = 0                                 # 0: the layer has no feed-forward


@dataclass
class NedesunConfig:
    vocab_size: int
    hidden_size: int
    layers: List[NedesunLayerSpec]
    norm_eps: float
    residual_mult: float = 1.0
    embed_scale: float = 1.0
    model_type: str = "nedesun"
    raw: dict = field(default_factory=dict, repr=False)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def to_dict(self) -> dict:
        return dict(self.raw)

    @classmethod
    def from_dict(cls, d: dict) -> "NedesunConfig":
        layers: List[NedesunLayerSpec] = []
        first_mix: Optional[int] = None
        for i, L in enumerate(d["layers"]):
            kind, m = L["type"], L["mixer"]
            if kind not in MIXERS:
                raise ValueError(f"Nedesun has no mixer {kind!r}")
            if kind == "parallel":
                a, r = m["left"], m["right"]
                mask = a.get("mask") or {}
                mx = NedesunParallel(heads=int(a["heads"]), kv_heads=int(a.get("kv_heads", a["heads"])), dim=int(a["dim"]),
                                     vdim=int(a.get("vdim", a["dim"])), scale=float(a["scale"]), window=int(mask.get("size", 0)),
                                     keep_first=int(mask.get("keep_first", 0)), rheads=int(r["heads"]),
                                     rkv_heads=int(r.get("kv_heads", r["heads"])), rdim=int(r["dim"]), rvdim=int(r.get("vdim", r["dim"])),
                                     conv=int(r.get("conv", 1)))
                if mx.heads % mx.kv_heads or mx.rheads % mx.rkv_heads or mx.conv < 1:
                    raise ValueError(f"layer {i}: bad parallel mixer sizes")
            elif kind == "attention":
                rot, mask = m.get("rot") or {}, m.get("mask") or {}
                mx = NedesunAttention(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads", m["heads"])), dim=int(m["dim"]),
                                      vdim=int(m.get("vdim", m["dim"])), scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                                      chunk=int(mask.get("size", 0)), rot_dims=int(rot.get("dims", 0)),
                                      rot_base=float(rot.get("base", 10000.0)), v_mix=bool(m.get("v_mix", False)))
                if mx.heads % mx.kv_heads or mx.rot_dims % 2 or mx.rot_dims > mx.dim:
                    raise ValueError(f"layer {i}: bad attention sizes")
                if mx.v_mix:
                    if first_mix is None:
                        first_mix = i
                    else:
                        o = layers[first_mix].mixer
                        if (o.kv_heads, o.vdim) != (mx.kv_heads, mx.vdim):
                            raise ValueError(f"layer {i}: its values are not shaped like those of layer {first_mix}, which they are mixed with")
                        mx.v_from = first_mix
            else:
                mx = NedesunWKV(heads=int(m["heads"]), dim=int(m["dim"]))
            f = L.get("mlp")
            if f is not None and f.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
            layers.append(NedesunLayerSpec(kind, mx, int(f["ff"]) if f is not None else 0))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                   residual_mult=float(d.get("residual_mult", 1.0)), embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), raw=d)


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class NedesunLayer(nn.Module):
    def __init__(self, cfg: NedesunConfig, spec: NedesunLayerSpec, dtype, device, decay_rank: int):
        super().__init__()
        m, W = spec.mixer, cfg.hidden_size
        self.spec = spec
        f32 = lambda *n, v=0.0: nn.Parameter(torch.full(n, v, dtype=torch.float32, device=device))       # noqa: E731
        wt = lambda *n: nn.Parameter(torch.zeros(*n, dtype=dtype, device=device))                        # noqa: E731
        self.norm1 = f32(W, v=1.0)
        # projections that read the mixer's input are one weight: rows that may leave it in the model dtype (``parts``), then
        # gates and step sizes, which stay fp32 (``tail``); both start on a multiple of 8 rows
        parts, tail = [], []
        if spec.type == "wkv":
            H, D = m.heads, m.dim
            self.mu = f32(len(SHIFTS), W)
            self.rkvg = wt(4, _pad8(H * D), W)
            self.rank = decay_rank
            self.w1 = wt(_pad8(decay_rank), W)
            self.w2, self.w0 = f32(H * D, decay_rank), f32(H * D)
            self.u = f32(H, D)
            self.mix_norm = f32(H * D, v=1.0)
            self.o_proj = wt(W, H * D)
        elif spec.type == "attention":
            H, G, D, Dv = m.heads, m.kv_heads, m.dim, m.vdim
            parts, tail = [("q", H * D), ("k", G * D), ("v", G * Dv)], [("g", H)]
            self.qkv_bias = f32((H + G) * D + G * Dv)
            self.vmix = f32(1)
            self.o_proj, self.o_bias = wt(W, H * Dv), wt(W)
        else:
            H, G, D, Dv = m.heads, m.kv_heads, m.dim, m.vdim
            RH, RG, RD, RDv = m.rheads, m.rkv_heads, m.rdim, m.rvdim
            parts = [("left.q", H * D), ("left.k", G * D), ("left.v", G * Dv), ("right.q", RG * RD), ("right.k", RG * RD),
                     ("right.v", RH * RDv), ("right.g", RH * RDv)]
            tail = [("right.b", RH), ("right.a", RH)]
            self.q_norm, self.k_norm, self.sink = f32(D, v=1.0), f32(D, v=1.0), f32(H)
            self.conv_w = f32(2 * RG * RD + RH * RDv, m.conv)
            self.A_log, self.dt_bias, self.mix_norm = f32(RH), f32(RH), f32(RDv, v=1.0)
            self.left_o, self.right_o = wt(W, H * Dv), wt(W, RH * RDv)
            self.left_out, self.right_out = f32(W, v=1.0), f32(W, v=1.0)
        self.parts = {}
        lo = 0
        for group in (parts, tail):
            for n, r in group:
                self.parts[n] = (lo, lo + r)
                lo += r
            lo = _pad8(lo)
            if group is parts:
                self.main = lo
        if lo:
            self.in_proj = wt(lo, W)
        if spec.ff:
            self.norm2 = f32(W, v=1.0)
            self.gate_up, self.down_proj = wt(2 * spec.ff, W), wt(W, spec.ff)

    def project(self, h: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """(rows that may be in the model dtype, fp32 gate rows). A few tokens take one product written in fp32, many tokens two
        so that the wide rows move in 16 bits."""
        if h.dtype == torch.float32 or h.shape[0] <= 64:
            p = linear_exact(h, self.in_proj, out_dtype=torch.float32)
            return p[:, :self.main], p[:, self.main:]
        return linear_exact(h, self.in_proj[:self.main]), linear_exact(h, self.in_proj[self.main:], out_dtype=torch.float32)

    def cols(self, main: torch.Tensor, tail: torch.Tensor, name: str) -> torch.Tensor:
        lo, hi = self.parts[name]
        return main[:, lo:hi] if hi <= self.main else tail[:, lo - self.main:hi - self.main]

    # ------------------------------------------------------------------ mixers: h [T, W] (model dtype) -> fp32 [T, W] (parallel: one per half)
    def parallel(self, h, pos, slot, state, cache, li: int, pieces, eps: float, max_pos: int):
        m = self.spec.mixer
        dt = h.dtype
        runs, n_runs = (pieces.runs, pieces.n_runs) if pieces is not None else (None, h.shape[0])
        main, tail = self.project(h)
        H, G, D, Dv = m.heads, m.kv_heads, m.dim, m.vdim
        q = qkv_store(main, None, self.q_norm, self.k_norm, None, pos, slot, cache.k[li], cache.v[li], cache.table, H, G, D, Dv, 0, eps, dt)
        ctx = multimap_attention(q, cache.k[li], cache.v[li], cache.table, pos, slot, H, G, 1, D, Dv, m.scale, m.window, m.keep_first,
                                 pieces=pieces, max_pos=max_pos, sink=self.sink)
        left = linear_exact(ctx, self.left_o, out_dtype=torch.float32)
        H, G, D, Dv = m.rheads, m.rkv_heads, m.rdim, m.rvdim
        c0, c1 = self.parts["right.q"][0], self.parts["right.v"][1]
        qkv = short_conv(main[:, c0:c1], self.conv_w, state[1], pos, slot, runs, n_runs, act=True)
        q, k, v = qkv[:, :G * D], qkv[:, G * D:2 * G * D], qkv[:, 2 * G * D:]
        a, b = self.cols(main, tail, "right.a"), self.cols(main, tail, "right.b")
        delta_gates(q, k, a, b, self.dt_bias, self.A_log, G, H, D, D ** -0.5, UNIT_EPS)
        o = linear_scan(q, k, v, state[0], pos, slot, runs, n_runs, H, G, D, Dv, "head_delta", g=a, beta=b)
        z = scan_readout(o, H, Dv, self.mix_norm, H, eps, dt, post=self.cols(main, tail, "right.g"), post_act="silu")
        return left, linear_exact(z, self.right_o, out_dtype=torch.float32)

    def attention(self, h, rope, pos, slot, cache, li: int, pieces, eps: float, max_pos: int):
        m = self.spec.mixer
        H, G, D, Dv = m.heads, m.kv_heads, m.dim, m.vdim
        main, tail = self.project(h)
        mixed = m.v_from is not None
        q = qkv_store(main, self.qkv_bias, None, None, rope, pos, slot, cache.k[li], cache.v[li], cache.table, H, G, D, Dv, m.rot_dims, eps,
                      h.dtype, v_first=cache.v[m.v_from] if mixed else None, v_lambda=self.vmix if mixed else None)
        ctx = multimap_attention(q, cache.k[li], cache.v[li], cache.table, pos, slot, H, G, 1, D, Dv, m.scale, pieces=pieces,
                                 max_pos=max_pos, softcap=m.softcap, chunk=m.chunk, gate=self.cols(main, tail, "g"))
        return linear_exact(ctx, self.o_proj, out_dtype=torch.float32, bias=self.o_bias)

    def wkv(self, h, pos, slot, state, pieces, eps: float):
        m = self.spec.mixer
        H, D = m.heads, m.dim
        runs, n_runs = (pieces.runs, pieces.n_runs) if pieces is not None else (None, h.shape[0])
        mixes = token_shift(h, self.mu, state[1], pos, slot, runs, n_runs)
        n = self.rkvg.shape[1]
        p = linear_each(mixes[:4], self.rkvg)
        r, k, v, g = (p[:, j * n:j * n + H * D] for j in range(4))
        w = lowrank_decay(linear_exact(mixes[4], self.w1, out_dtype=torch.float32)[:, :self.rank], self.w2, self.w0,
                          fast=h.dtype != torch.float32, form="exp_exp")
        o = linear_scan(r, k, v, state[0], pos, slot, runs, n_runs, H, H, D, D, "channel", g=w, pieces=pieces, u=self.u)
        z = scan_readout(o, H, D, self.mix_norm, H, eps, h.dtype, post=g, post_act="silu")
        return linear_exact(z, self.o_proj, out_dtype=torch.float32)

    def feed_forward(self, h: torch.Tensor) -> torch.Tensor:
        return linear_exact(ew.act_glu(linear_exact(h, self.gate_up), "silu"), self.down_proj, out_dtype=torch.float32)


class NedesunForCausalLM(nn.Module):
    """``forward_ragged`` is the serving step; ``forward(input_ids)`` runs whole sequences through the same step."""
    ragged = True                                   # served by inference.ragged.RaggedGenerator

    def __init__(self, cfg: NedesunConfig, dtype=torch.bfloat16, device=None, init_std: float = 0.02, decay_ranks=None):
        super().__init__()
        self.config = cfg
        self.dtype_ = dtype
        W, V = cfg.hidden_size, cfg.vocab_size
        self.embed_tokens = nn.Parameter(torch.empty(V, W, dtype=dtype, device=device).normal_(std=init_std))
        # the ranks of the decays' low-rank projections come from the checkpoint's shapes: {layer: rank}
        self.layers = nn.ModuleList([NedesunLayer(cfg, s, dtype, device, int((decay_ranks or {}).get(i, 16)))
                                     for i, s in enumerate(cfg.layers)])
        self.norm = nn.Parameter(torch.ones(W, dtype=torch.float32, device=device))
        self._rope = {}

    @property
    def device(self) -> torch.device:
        return self.embed_tokens.device

    def head_weight(self) -> torch.Tensor:
        return self.embed_tokens                    # the output projection is the embedding table

    def kv_layout(self):
        """(key rows, key row size, value row size) per layer: attention, alone or as half of a parallel mixer, has a pool."""
        return [(s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim) if s.type != "wkv" else (0, 0, 0) for s in self.config.layers]

    def state_layout(self):
        """Per layer, the shapes of the fp32 tensors a sequence carries from token to token. wkv: the matrix state per head and
        the last token's h. parallel: the matrix state per head and the last inputs of the q | k | v convolution."""
        out = []
        for s in self.config.layers:
            m = s.mixer
            if s.type == "wkv":
                out.append([(m.heads, m.dim, m.dim), (1, self.config.hidden_size)])
            elif s.type == "parallel":
                out.append([(m.rheads, m.rdim, m.rvdim), (m.conv - 1, 2 * m.rkv_heads * m.rdim + m.rheads * m.rvdim)])
            else:
                out.append([])
        return out

    def rope(self, m: NedesunAttention, device, need: int):
        if not m.rot_dims:
            return None
        key = (m.rot_dims, m.rot_base, str(device))
        t = self._rope.get(key)
        if t is None or t[0].shape[0] < need:
            t = self._rope[key] = ew.rope_tables_partial(max(need, 4096), m.rot_dims, m.rot_base, device)
        return t

    @torch.no_grad()
    def forward_ragged(self, ids: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, cache, want: Optional[torch.Tensor] = None,
                       max_pos: int = 0, pieces=None, layer_outputs: Optional[list] = None) -> torch.Tensor:
        """One serving step over a flat token list: ``ids`` long [T], ``pos`` / ``slot`` int32 [T] (position in its sequence
        and cache / state row of every token), ``cache`` a ``PagedKVCache`` whose table rows cover those positions and whose
        state rows belong to the same sequences. Returns fp32 logits of the rows ``want`` (long [n]; default all).
        ``pieces`` describes the runs of consecutive tokens (None: every token is a sequence of its own step, a decode
        batch). ``layer_outputs``: a list that receives the residual stream after every layer."""
        cfg = self.config
        dt = self.embed_tokens.dtype
        eps, mult = cfg.norm_eps, cfg.residual_mult
        need = max(int(max_pos) + 1, cache.max_len)
        reads = [layer.norm1 for layer in self.layers] + [self.norm]       # what norms the stream in front of each layer, and the head
        h, x = sandwich_norm(ew.embedding_pos(ids, self.embed_tokens, cfg.embed_scale), None, None, reads[0], eps, 0.0, dt)
        for li, layer in enumerate(self.layers):
            nxt = layer.norm2 if layer.spec.ff else reads[li + 1]
            if layer.spec.type == "parallel":
                left, right = layer.parallel(h, pos, slot, cache.state[li], cache, li, pieces, eps, max_pos)
                h, x = sandwich_norm(left, layer.left_out, x, nxt, eps, 0.0, dt, branch_mult=BRANCH * mult, y2=right, post_w2=layer.right_out)
            else:
                if layer.spec.type == "attention":
                    y = layer.attention(h, self.rope(layer.spec.mixer, ids.device, need), pos, slot, cache, li, pieces, eps, max_pos)
                else:
                    y = layer.wkv(h, pos, slot, cache.state[li], pieces, eps)
                h, x = sandwich_norm(y, None, x, nxt, eps, 0.0, dt, branch_mult=mult)
            if layer.spec.ff:
                h, x = sandwich_norm(layer.feed_forward(h), None, x, reads[li + 1], eps, 0.0, dt, branch_mult=mult)
            if layer_outputs is not None:
                layer_outputs.append(x)
        if want is not None:
            h = h.index_select(0, want)
        return linear_exact(h.contiguous(), self.embed_tokens, out_dtype=torch.float32)

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor, labels=None, **_) -> dict:
        """Whole sequences [B, S] through the serving step with a throw-away cache: ``{"logits": [B, S, V]}`` (fp32)."""
        if labels is not None:
            raise NotImplementedError("Nedesun is an inference model here: no loss / backward")
        from ..inference.ragged import RaggedGenerator
        B, S = input_ids.shape
        gen = RaggedGenerator(self, None, max_len=S)
        per = -(-S // 64)
        cache = gen.make_cache(num_blocks=B * per, block_size=64, max_seqs=B, max_len=S)
        for b in range(B):
            gen.set_block_row(cache, b, list(range(1 + b * per, 1 + (b + 1) * per)))
        logits = gen.step([(b, 0, input_ids[b].tolist(), list(range(S))) for b in range(B)], cache)
        return {"logits": logits.view(B, S, -1)}

    @torch.no_grad()
    def generate(self, input_ids: torch.Tensor, max_new_tokens: int = 256, **kw) -> torch.Tensor:
        from ..inference.ragged import RaggedGenerator
        g = self.__dict__.get("_generator")
        need = input_ids.shape[1] + int(max_new_tokens)
        if g is None or g.max_len < need:
            g = self.__dict__["_generator"] = RaggedGenerator(self, None, max(need, 4096))
        return g.generate(input_ids.to(self.device), max_new_tokens=max_new_tokens, **kw)

    def num_parameters(self, only_trainable: bool = False) -> int:
        return sum(p.numel() for p in self.parameters() if p.requires_grad or not only_trainable)


# ------------------------------------------------------------------------------------------------------------------
# checkpoint: config.json + model.safetensors with the design's own tensor names
# ------------------------------------------------------------------------------------------------------------------
def _tensor_map(model: NedesunForCausalLM):
    """(checkpoint name, the view of a parameter that holds it) per tensor."""
    out = [("embed", model.embed_tokens), ("final.norm", model.norm)]
    for i, layer in enumerate(model.layers):
        spec = layer.spec
        p, m = f"l{i}.", spec.mixer
        q = p + "mix."
        out.append((p + "norm1", layer.norm1))
        out += [(q + n, layer.in_proj[lo:hi]) for n, (lo, hi) in layer.parts.items()]
        if spec.type == "wkv":
            out += [(f"{q}mu.{s}", layer.mu[j]) for j, s in enumerate(SHIFTS)]
            out += [(q + s, layer.rkvg[j, :m.heads * m.dim]) for j, s in enumerate(SHIFTS[:4])]
            out += [(q + "w1", layer.w1[:layer.rank]), (q + "w2", layer.w2), (q + "w0", layer.w0), (q + "u", layer.u),
                    (q + "norm", layer.mix_norm), (q + "o", layer.o_proj)]
        elif spec.type == "attention":
            out += [(f"{q}{n}.b", layer.qkv_bias[lo:hi]) for n, (lo, hi) in layer.parts.items() if n != "g"]
            out += [(q + "vmix", layer.vmix[0]), (q + "o", layer.o_proj), (q + "o.b", layer.o_bias)]
        else:
            c0 = layer.parts["right.q"][0]
            out += [(f"{q}right.{n}.conv", layer.conv_w[lo - c0:hi - c0]) for n in "qkv" for lo, hi in [layer.parts["right." + n]]]
            out += [(q + "left.q.norm", layer.q_norm), (q + "left.k.norm", layer.k_norm), (q + "left.sink", layer.sink),
                    (q + "left.o", layer.left_o), (q + "left.out", layer.left_out), (q + "right.A_log", layer.A_log),
                    (q + "right.dt_bias", layer.dt_bias), (q + "right.norm", layer.mix_norm), (q + "right.o", layer.right_o),
                    (q + "right.out", layer.right_out)]
        if spec.ff:
            out += [(p + "norm2", layer.norm2), (p + "mlp.gate", layer.gate_up[:spec.ff]), (p + "mlp.up", layer.gate_up[spec.ff:]),
                    (p + "mlp.down", layer.down_proj)]
    return out


@torch.no_grad()
def load_nedesun_weights(model: NedesunForCausalLM, path: str) -> None:
    from ..io.safetensors import safe_open
    with safe_open(os.path.join(path, "model.safetensors")) as f:
        names = set(f.keys())
        used = set()
        for name, dst in _tensor_map(model):
            if name not in names and name.endswith("mix.vmix"):
                continue                                       # a layer that mixes no values may come without its factor
            used.add(name)
            t = f.get_tensor(name)
            dst.copy_(t.to(dst.device, dst.dtype).reshape(dst.shape))
        missing = names - used
        if missing:
            raise ValueError(f"checkpoint tensors the model has no place for: {sorted(missing)[:8]}")


def _decay_ranks(path: str, cfg: NedesunConfig) -> dict:
    from ..io.safetensors import safe_open
    with safe_open(os.path.join(path, "model.safetensors")) as f:
        return {i: int(f.info(f"l{i}.mix.w1")[1][0]) for i, s in enumerate(cfg.layers) if s.type == "wkv"}


def nedesun_from_pretrained(path: str, dtype=torch.bfloat16, device=None) -> NedesunForCausalLM:
    with open(os.path.join(path, "config.json")) as f:
        cfg = NedesunConfig.from_dict(json.load(f))
    model = NedesunForCausalLM(cfg, dtype=dtype, device=device, decay_ranks=_decay_ranks(path, cfg))
    load_nedesun_weights(model, path)
    model.name_or_path = path
    return model.eval()


@torch.no_grad()
def nedesun_state_dict(model: NedesunForCausalLM) -> dict:
    """Tensors under the checkpoint's names (the inverse of ``load_nedesun_weights``)."""
    return {name: t.detach().contiguous() for name, t in _tensor_map(model)}
