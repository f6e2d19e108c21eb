"""Lorenex: a decoder-only language model whose layers read the residual stream as it is and norm only what they add to it; a
layer's mixer is either a gated linear attention with a decay per key channel, or softmax attention and a selective state
space side by side over the same input.

The stream x (fp32) starts as ``embed[token] * s_e + pos[p]`` with a learned position table. RMS(y) = y / sqrt(mean(y^2) + eps).
Layer i (tensors ``l<i>.*``), m = ``residual_mult``:

    x <- x + m RMS(mixer(x)) * g_1
    x <- x + m RMS(ff(x)) * g_2                 only if the layer has a feed-forward

* ``gla``: q = W_q x / sqrt(dim), k = W_k x, v = W_v x per head; decays a = sigmoid(W_a2 W_a1 x + b)^(1 / tau) per key channel;
  S' = diag(a) S + k v^T, o = S'^T q; every head RMS-normed with a weight shared by the heads, times silu(W_g x), then W_o.
* ``parallel``: ``left_scale`` * left(x) + ``right_scale`` * right(x).
  left: grouped-query attention without rotation; q, k, v (with biases) pass a short causal convolution, then every q, k and v
  row is divided by its root mean square; q is multiplied by 1 + c ln(floor((p + 1) / every) + 1) at position p.
  right: W_in x = [u | z]; u passes a causal convolution with bias and silu; W_x u = [dt | B | C];
  dt = softplus(W_dt dt + b); per channel c and state n: S'[c, n] = exp(-dt_c exp(A_log[c, n])) S[c, n] + dt_c u_c B_n;
  y_c = sum_n S'[c, n] C_n + D_c u_c; y silu(z), then W_o.
* feed-forward: dense ``W_down act(W_up x)`` with act(z) = a RMS(z) + b RMS(z^2) + c RMS(z^3) + e over a token's values, or a
  mixture of experts: s = softmax(W_r x) in fp32 over experts and identity experts; the ``top`` largest of s + correction,
  weighted by s as it is; an expert is W_down (g sigmoid(1.702 g) (u + 1)) with clamped g and u, an identity expert is x.

A layer with ``weights_of: j`` runs layer j's tensors again with pages and state of its own. The output is
``embed @ (RMS(x) * g)`` (the embedding table without its scale). What is fp32 whatever the model dtype: the stream, every
norm, attention scores and softmax, the router, the recurrent states and tails, decays, step sizes, the scans and their
read-outs. Projections, the rows that leave a short convolution, B and C are in the model dtype where they do not feed the
matrix memory (whose projections are written in fp32).

Keys and values live in the paged cache (``kv_layout``), convolution tails and recurrent states in its per-sequence state rows
(``state_layout``). ``inference/ragged.RaggedGenerator`` and ``serve/engine.LLMEngine`` drive ``forward_ragged``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

import torch
from torch import nn

from ..ops import elementwise as ew
from ..ops.gemm import linear_exact
from ..ops.linear_scan import linear_scan, lowrank_decay, scan_readout, selective_scan, short_conv
from ..ops.moe import gated_moe_ffn, route_grouped
from ..ops.multimap_attention import conv_qknorm_store, multimap_attention
from ..ops.norm import poly_norm, sandwich_norm

MIXERS = ("gla", "parallel")
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0           # the experts' gated unit: fixed by the design


@dataclass
class LorenexGLA:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass
class LorenexParallel:
    heads: int                                  # left: attention
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    temp_coef: float
    temp_every: float
    inner: int                                  # right: selective state space
    state: int
    dt_rank: int
    rconv: int
    left_scale: float
    right_scale: float


@dataclass
class LorenexFF:
    kind: str                                   # "dense" | "moe"
    ff: int
    experts: int = 0
    identity: int = 0
    top: int = 0
    limit: float = 0.0


@dataclass
class LorenexLayerSpec:
    type: str
    mixer: object
    mlp: Optional[LorenexFF]
    source: int                                 # the layer whose tensors it runs (its own index unless ``weights_of``)


@dataclass
class LorenexConfig:
    vocab_size: int
    hidden_size: int
    layers: List[LorenexLayerSpec]
    norm_eps: float
    max_positions: int
    residual_mult: float = 1.0
    embed_scale: float = 1.0
    model_type: str = "lorenex"
    raw: dict = field(default_factory=dict, repr=False)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def to_dict(self) -> dict:
        return dict(self.raw)

    @classmethod
    def from_dict(cls, d: dict) -> "LorenexConfig":
        layers: List[LorenexLayerSpec] = []
        for i, L in enumerate(d["layers"]):
            kind, m = L["type"], L["mixer"]
            if kind not in MIXERS:
                raise ValueError(f"Lorenex has no mixer {kind!r}")
            if kind == "gla":
                mx = LorenexGLA(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
                if not mx.tau > 0:
                    raise ValueError(f"layer {i}: tau must be positive")
            else:
                a, r = m["left"], m["right"]
                t = a.get("q_temp") or {}
                mx = LorenexParallel(heads=int(a["heads"]), kv_heads=int(a.get("kv_heads", a["heads"])), dim=int(a["dim"]),
                                     vdim=int(a.get("vdim", a["dim"])), conv=int(a.get("conv", 1)), scale=float(a["scale"]),
                                     temp_coef=float(t.get("coef", 0.0)), temp_every=float(t.get("every", 1)),
                                     inner=int(r["inner"]), state=int(r["state"]), dt_rank=int(r["dt_rank"]),
                                     rconv=int(r.get("conv", 1)), left_scale=float(m.get("left_scale", 1.0)),
                                     right_scale=float(m.get("right_scale", 1.0)))
                if mx.heads % mx.kv_heads or mx.conv < 1 or mx.rconv < 1 or not mx.temp_every > 0:
                    raise ValueError(f"layer {i}: bad parallel mixer sizes")
            f = L.get("mlp")
            ff = None
            if f is not None:
                fk = f.get("kind", "dense")
                if fk == "dense":
                    ff = LorenexFF("dense", int(f["ff"]))
                elif fk == "moe":
                    r, e = f["router"], f["expert"]
                    ff = LorenexFF("moe", int(e["ff"]), experts=int(r["experts"]), identity=int(r.get("identity", 0)), top=int(r["top"]),
                                   limit=float(e["limit"]))
                    if not 1 <= ff.top <= ff.experts + ff.identity or ff.experts < 1:
                        raise ValueError(f"layer {i}: bad router sizes")
                else:
                    raise ValueError(f"unknown feed-forward kind {fk!r}")
            source, j = i, L.get("weights_of")
            if j is not None:
                if not 0 <= int(j) < len(d["layers"]) or int(j) == i:
                    raise ValueError(f"layer {i}: weights_of must name another layer")
                seen = {i}
                source = int(j)
                while d["layers"][source].get("weights_of") is not None:        # a layer that borrows may itself be borrowed from
                    if source in seen:
                        raise ValueError(f"layer {i}: weights_of goes round in a circle")
                    seen.add(source)
                    source = int(d["layers"][source]["weights_of"])
            layers.append(LorenexLayerSpec(kind, mx, ff, source))
        for i, s in enumerate(layers):
            o = layers[s.source]
            if (s.type, s.mixer, s.mlp) != (o.type, o.mixer, o.mlp):
                raise ValueError(f"layer {i}: differs from layer {s.source}, whose weights it runs")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                   max_positions=int(d["max_positions"]), residual_mult=float(d.get("residual_mult", 1.0)),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), raw=d)


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class LorenexLayer(nn.Module):
    def __init__(self, cfg: LorenexConfig, spec: LorenexLayerSpec, dtype, device, decay_rank: int):
        super().__init__()
        m, f, W = spec.mixer, spec.mlp, cfg.hidden_size
        self.spec = spec
        f32 = lambda *n, v=0.0: nn.Parameter(torch.full(n, v, dtype=torch.float32, device=device))       # noqa: E731
        wt = lambda *n: nn.Parameter(torch.zeros(*n, dtype=dtype, device=device))                        # noqa: E731
        self.norm1 = f32(W, v=1.0)
        # projections that read the mixer's input are one weight; parts = name -> (first row, end row); rows padded to 8
        if spec.type == "gla":
            H, D, Dv = m.heads, m.dim, m.vdim
            parts = [("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv), ("a1", decay_rank)]
            self.a2, self.a2_bias = f32(H * D, decay_rank), f32(H * D)
            self.mix_norm = f32(Dv, v=1.0)
            self.o_proj = wt(W, H * Dv)
        else:
            H, G, D, Dv, inner, N, R = m.heads, m.kv_heads, m.dim, m.vdim, m.inner, m.state, m.dt_rank
            C = (H + G) * D + G * Dv
            parts = [("left.q", H * D), ("left.k", G * D), ("left.v", G * Dv), ("right.in", 2 * inner)]
            self.qkv_bias, self.qkv_conv = f32(C), f32(C, m.conv)
            self.conv_w, self.conv_b = f32(inner, m.rconv), f32(inner)
            # rows of the second projection: step-size rank | B | C, each starting on a multiple of 8 (padding rows are zero)
            self.x_parts = {"dt": (0, R), "B": (_pad8(R), _pad8(R) + N), "C": (_pad8(R) + _pad8(N), _pad8(R) + _pad8(N) + N)}
            self.x_proj = wt(_pad8(R) + 2 * _pad8(N), inner)
            self.dt_proj, self.dt_bias = wt(inner, _pad8(R)), f32(inner)
            self.A_log, self.D_skip = f32(inner, N), f32(inner)
            # both output projections as one: its operand is [attention output | state-space output], already scaled
            self.o_cols = {"left": (0, H * Dv), "right": (_pad8(H * Dv), _pad8(H * Dv) + inner)}
            self.o_proj = wt(W, _pad8(_pad8(H * Dv) + inner))
            self._A = None
        self.parts = {}
        lo = 0
        for n, r in parts:
            self.parts[n] = (lo, lo + r)
            lo += r
        self.in_proj = wt(_pad8(lo), W)
        if f is not None:
            self.norm2 = f32(W, v=1.0)
            if f.kind == "dense":
                self.up_proj, self.down_proj, self.act = wt(f.ff, W), wt(W, f.ff), f32(4)
            else:
                self.router, self.correction = f32(f.experts + f.identity, W), f32(f.experts + f.identity)
                self.experts_gate_up = wt(f.experts, 2 * f.ff, W)
                self.experts_down = wt(f.experts, W, f.ff)

    def rates(self) -> torch.Tensor:
        """A = -exp(A_log), laid out [state, inner] like the recurrent state: a function of the weights only, formed once."""
        if self._A is None:
            self._A = (-torch.exp(self.A_log)).t().contiguous()
        return self._A

    # ------------------------------------------------------------------ mixers: h [T, W] (model dtype) -> fp32 [T, W]
    def gla(self, h, pos, slot, state, pieces, eps: float):
        m = self.spec.mixer
        H, D, Dv = m.heads, m.dim, m.vdim
        proj = linear_exact(h, self.in_proj, out_dtype=torch.float32)
        sl = lambda n: proj[:, self.parts[n][0]:self.parts[n][1]]             # noqa: E731
        a = lowrank_decay(sl("a1"), self.a2, self.a2_bias, m.tau, fast=h.dtype != torch.float32)
        runs, n_runs = (pieces.runs, pieces.n_runs) if pieces is not None else (None, h.shape[0])
        o = linear_scan(sl("q"), sl("k"), sl("v"), state[0], pos, slot, runs, n_runs, H, H, D, Dv, "channel", g=a, pieces=pieces)
        # the queries' 1 / sqrt(dim) is a factor of o: it is applied where the heads are normed
        z = scan_readout(o, H, Dv, self.mix_norm, H, eps, h.dtype, oscale=D ** -0.5, post=sl("g"), post_act="silu")
        return linear_exact(z, self.o_proj, out_dtype=torch.float32)

    def parallel(self, h, pos, slot, state, cache, li: int, pieces, eps: float, max_pos: int):
        m = self.spec.mixer
        H, G, D, Dv, inner = m.heads, m.kv_heads, m.dim, m.vdim, m.inner
        dt = h.dtype
        runs, n_runs = (pieces.runs, pieces.n_runs) if pieces is not None else (None, h.shape[0])
        proj = linear_exact(h, self.in_proj)
        c0 = self.parts["right.in"][0]
        K = self.o_proj.shape[1]
        y = torch.empty(h.shape[0], K, dtype=dt, device=h.device)
        (l0, l1), (r0, r1) = self.o_cols["left"], self.o_cols["right"]
        if l1 < r0:
            y[:, l1:r0].zero_()
        if r1 < K:
            y[:, r1:].zero_()
        q = conv_qknorm_store(proj[:, :c0], self.qkv_bias, self.qkv_conv, state[0], pos, slot, runs, n_runs, cache.k[li], cache.v[li],
                              cache.table, H, G, D, Dv, eps, dt, temp=(m.temp_coef, m.temp_every), norm_v=True)
        multimap_attention(q, cache.k[li], cache.v[li], cache.table, pos, slot, H, G, 1, D, Dv, m.scale, post=m.left_scale,
                           pieces=pieces, max_pos=max_pos, out=y[:, l0:l1])
        u = short_conv(proj[:, c0:c0 + inner], self.conv_w, state[1], pos, slot, runs, n_runs, act=True, bias=self.conv_b, out_dtype=dt)
        p = linear_exact(u, self.x_proj)
        ps = lambda n: p[:, self.x_parts[n][0]:self.x_parts[n][1]]            # noqa: E731
        step = linear_exact(p[:, :self.dt_proj.shape[1]], self.dt_proj, out_dtype=torch.float32)
        selective_scan(u, step, self.dt_bias, ps("B"), ps("C"), self.rates(), self.D_skip, state[2], pos, slot, runs, n_runs,
                       gate=proj[:, c0 + inner:c0 + 2 * inner], scale=m.right_scale, out=y[:, r0:r1], pieces=pieces)
        return linear_exact(y, self.o_proj, out_dtype=torch.float32)

    def feed_forward(self, h: torch.Tensor, x: torch.Tensor, eps: float) -> torch.Tensor:
        """``h`` [T, W] is the stream in the model dtype, ``x`` the stream itself (fp32) -> the sublayer's output, fp32."""
        f = self.spec.mlp
        if f.kind == "dense":
            return linear_exact(poly_norm(linear_exact(h, self.up_proj), self.act, eps), self.down_proj, out_dtype=torch.float32)
        top_i, top_p, _ = route_grouped(h, self.router, self.correction, f.top, softmax=True)
        return gated_moe_ffn(h, top_i, top_p, self.experts_gate_up, self.experts_down,
                             lambda gu: ew.clamped_glu(gu, f.limit, GLU_ALPHA, GLU_SHIFT), identity=x)


class LorenexForCausalLM(nn.Module):
    """``forward_ragged`` is the serving step; ``forward(input_ids)`` runs whole sequences through the same step."""
    ragged = True                                   # served by inference.ragged.RaggedGenerator

    def __init__(self, cfg: LorenexConfig, dtype=torch.bfloat16, device=None, init_std: float = 0.02, decay_ranks=None):
        super().__init__()
        self.config = cfg
        self.dtype_ = dtype
        W, V = cfg.hidden_size, cfg.vocab_size
        self.embed_tokens = nn.Parameter(torch.empty(V, W, dtype=dtype, device=device).normal_(std=init_std))
        self.pos_table = nn.Parameter(torch.zeros(cfg.max_positions, W, dtype=torch.float32, device=device))
        # one module per set of tensors; the ranks of the decays' low-rank projections come from the checkpoint's shapes
        own = {i: LorenexLayer(cfg, s, dtype, device, int((decay_ranks or {}).get(i, 16)))
               for i, s in enumerate(cfg.layers) if s.source == i}
        self.own_layers = nn.ModuleDict({str(i): layer for i, layer in own.items()})
        self.norm = nn.Parameter(torch.ones(W, dtype=torch.float32, device=device))

    @property
    def layers(self) -> List[LorenexLayer]:
        """The module of every layer in running order (a module appears as often as its weights are run)."""
        return [self.own_layers[str(s.source)] for s in self.config.layers]

    @property
    def max_positions(self) -> int:
        return self.config.max_positions            # the position table ends there: no sequence may be longer

    @property
    def device(self) -> torch.device:
        return self.embed_tokens.device

    def head_weight(self) -> torch.Tensor:
        return self.embed_tokens                    # the output projection is the embedding table

    def kv_layout(self):
        """(key rows, key row size, value row size) per layer: only the attention half of a parallel layer has a pool."""
        return [(s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim) if s.type == "parallel" else (0, 0, 0) for s in self.config.layers]

    def state_layout(self):
        """Per layer, the shapes of the fp32 tensors a sequence carries from token to token. gla: the matrix state per head.
        parallel: the last inputs of the q | k | v convolution, the last inputs of the state space's convolution, and the
        state-space state, laid out [state, inner] so that neighbouring channels are neighbours in memory."""
        out = []
        for s in self.config.layers:
            m = s.mixer
            if s.type == "gla":
                out.append([(m.heads, m.dim, m.vdim)])
            else:
                out.append([(m.conv - 1, (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim), (m.rconv - 1, m.inner), (m.state, m.inner)])
        return out

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
        layers = self.layers
        x0 = ew.embedding_pos(ids, self.embed_tokens, cfg.embed_scale, pos, self.pos_table)
        h, x = sandwich_norm(x0, None, None, None if layers else self.norm, eps, 0.0, dt, cast_next=True)
        for li, layer in enumerate(layers):
            state = cache.state[li]
            if layer.spec.type == "gla":
                y = layer.gla(h, pos, slot, state, pieces, eps)
            else:
                y = layer.parallel(h, pos, slot, state, cache, li, pieces, eps, max_pos)
            nxt = self.norm if li + 1 == len(layers) else None        # the sublayers read the stream itself, the head its norm
            if layer.spec.mlp is None:
                h, x = sandwich_norm(y, layer.norm1, x, nxt, eps, 0.0, dt, branch_mult=mult, cast_next=True)
            else:
                h, x = sandwich_norm(y, layer.norm1, x, None, eps, 0.0, dt, branch_mult=mult, cast_next=True)
                h, x = sandwich_norm(layer.feed_forward(h, x, eps), layer.norm2, x, nxt, eps, 0.0, dt, branch_mult=mult, cast_next=True)
            if layer_outputs is not None:
                layer_outputs.append(x)
        if want is not None:
            h = h.index_select(0, want)
        return linear_exact(h.contiguous(), self.embed_tokens, out_dtype=torch.float32)

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor, labels=None, **_) -> dict:
        """Whole sequences [B, S] through the serving step with a throw-away cache: ``{"logits": [B, S, V]}`` (fp32)."""
        if labels is not None:
            raise NotImplementedError("Lorenex is an inference model here: no loss / backward")
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
            g = self.__dict__["_generator"] = RaggedGenerator(self, None, min(max(need, 4096), self.max_positions))
        return g.generate(input_ids.to(self.device), max_new_tokens=max_new_tokens, **kw)

    def num_parameters(self, only_trainable: bool = False) -> int:
        return sum(p.numel() for p in self.parameters() if p.requires_grad or not only_trainable)


# ------------------------------------------------------------------------------------------------------------------
# checkpoint: config.json + model.safetensors with the design's own tensor names
# ------------------------------------------------------------------------------------------------------------------
def _tensor_map(model: LorenexForCausalLM):
    """(checkpoint name, the view of a parameter that holds it) per tensor."""
    out = [("embed", model.embed_tokens), ("pos", model.pos_table), ("final.norm", model.norm)]
    for i, spec in enumerate(model.config.layers):
        if spec.source != i:
            continue
        layer = model.own_layers[str(i)]
        p, m, f = f"l{i}.", spec.mixer, spec.mlp
        out.append((p + "norm1", layer.norm1))
        for n, (lo, hi) in layer.parts.items():
            out.append((f"{p}mix.{n}", layer.in_proj[lo:hi]))
        if spec.type == "gla":
            out += [(p + "mix.a2", layer.a2), (p + "mix.a2.b", layer.a2_bias), (p + "mix.norm", layer.mix_norm), (p + "mix.o", layer.o_proj)]
        else:
            lq, rq = p + "mix.left.", p + "mix.right."
            for n in ("q", "k", "v"):
                lo, hi = layer.parts["left." + n]
                out += [(f"{lq}{n}.b", layer.qkv_bias[lo:hi]), (f"{lq}{n}.conv", layer.qkv_conv[lo:hi])]
            (l0, l1), (r0, r1) = layer.o_cols["left"], layer.o_cols["right"]
            xp = layer.x_parts
            out += [(lq + "o", layer.o_proj[:, l0:l1]), (rq + "o", layer.o_proj[:, r0:r1]), (rq + "conv", layer.conv_w),
                    (rq + "conv.b", layer.conv_b), (rq + "x", [layer.x_proj[lo:hi] for lo, hi in (xp["dt"], xp["B"], xp["C"])]),
                    (rq + "dt", layer.dt_proj[:, :m.dt_rank]), (rq + "dt.b", layer.dt_bias), (rq + "A_log", layer.A_log), (rq + "D", layer.D_skip)]
        if f is None:
            continue
        out.append((p + "norm2", layer.norm2))
        if f.kind == "dense":
            out += [(p + "mlp.up", layer.up_proj), (p + "mlp.down", layer.down_proj), (p + "mlp.act", layer.act)]
            continue
        out += [(p + "mlp.router", layer.router), (p + "mlp.correction", layer.correction)]
        for e in range(f.experts):
            q = f"{p}mlp.e{e}."
            out += [(q + "gate", layer.experts_gate_up[e, :f.ff]), (q + "up", layer.experts_gate_up[e, f.ff:]),
                    (q + "down", layer.experts_down[e])]
    return out


@torch.no_grad()
def load_lorenex_weights(model: LorenexForCausalLM, path: str) -> None:
    from ..io.safetensors import safe_open
    with safe_open(os.path.join(path, "model.safetensors")) as f:
        names = set(f.keys())
        used = set()
        for name, dst in _tensor_map(model):
            used.add(name)
            t = f.get_tensor(name)
            parts = dst if isinstance(dst, list) else [dst]        # a tensor whose rows are spread over padded sections
            for d, s in zip(parts, t.split([d.shape[0] for d in parts]) if len(parts) > 1 else [t]):
                d.copy_(s.to(d.device, d.dtype).reshape(d.shape))
        missing = names - used
        if missing:
            raise ValueError(f"checkpoint tensors the model has no place for: {sorted(missing)[:8]}")
    for layer in model.own_layers.values():
        layer._A = None


def _decay_ranks(path: str, cfg: LorenexConfig) -> dict:
    from ..io.safetensors import safe_open
    with safe_open(os.path.join(path, "model.safetensors")) as f:
        return {i: int(f.info(f"l{i}.mix.a1")[1][0]) for i, s in enumerate(cfg.layers) if s.type == "gla" and s.source == i}


def lorenex_from_pretrained(path: str, dtype=torch.bfloat16, device=None) -> LorenexForCausalLM:
    with open(os.path.join(path, "config.json")) as f:
        cfg = LorenexConfig.from_dict(json.load(f))
    model = LorenexForCausalLM(cfg, dtype=dtype, device=device, decay_ranks=_decay_ranks(path, cfg))
    load_lorenex_weights(model, path)
    model.name_or_path = path
    return model.eval()


@torch.no_grad()
def lorenex_state_dict(model: LorenexForCausalLM) -> dict:
    """Tensors under the checkpoint's names (the inverse of ``load_lorenex_weights``)."""
    return {name: (torch.cat(t, 0) if isinstance(t, list) else t).detach().contiguous() for name, t in _tensor_map(model)}
