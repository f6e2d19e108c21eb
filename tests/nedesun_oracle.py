"""A plain float64 statement of the Nedesun equations: one function per mechanism, whole sequences, token by token where
there is a state. It shares nothing with the package (no ops, no cache, no batching) and is what the tests compare the
serving step against.

Weights are a dict name -> tensor under the checkpoint's names (``l<i>.mix.q`` ...); ``cfg`` is the parsed config.json.
"""
import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def unit(x):
    """A unit vector along the last dim."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def causal_conv(u, w):
    """u [n, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), nothing before t = 0."""
    n, C = u.shape
    taps = w.shape[1]
    y = torch.zeros(n, C, dtype=F64)
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j].to(F64) * u[s]
    return y


def rotate(x, base, dims):
    """x [n, R, D]: position p turns dim i against dim i + dims / 2 (i < dims / 2) by p base^(-2 i / dims)."""
    n, half = x.shape[0], dims // 2
    y = x.clone()
    for i in range(half):
        ang = torch.arange(n, dtype=F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = x[..., i], x[..., i + half]
        y[..., i] = a * c - b * s
        y[..., i + half] = b * c + a * s
    return y


def window_visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def chunk_visible(i, j, size):
    return j <= i and i // size == j // size


def attend(q, k, v, scale, visible, softcap=None, sink=None):
    """q [n, H, D], k [n, G, D], v [n, G, Dv] -> [n, H, Dv]. ``visible(i, j)``: does position i see j; ``softcap``: scores pass
    c tanh(s / c); ``sink`` [H]: one more term exp(sink_h) in the softmax's denominator."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    mask = torch.tensor([[visible(i, j) for j in range(n)] for i in range(n)])
    outs = []
    for a in range(H):
        s = q[:, a] @ k[:, a // rep].T * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~mask, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[a].to(F64).expand(n, 1)], 1)
        outs.append(torch.softmax(s, -1)[:, :n] @ v[:, a // rep])
    return torch.stack(outs, 1)


# ---------------------------------------------------------------------------------------------------- parallel, left half
def windowed_attention(h, P, m, eps):
    n, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda name: h @ P[name].to(F64).T                                  # noqa: E731
    q = rms(lin("q").view(n, H, D), eps) * P["q.norm"].to(F64)
    k = rms(lin("k").view(n, G, D), eps) * P["k.norm"].to(F64)
    v = lin("v").view(n, G, Dv)
    keep = m["mask"].get("keep_first", 0)
    o = attend(q, k, v, float(m["scale"]), lambda i, j: window_visible(i, j, m["mask"]["size"], keep), sink=P["sink"])
    return o.reshape(n, H * Dv) @ P["o"].to(F64).T


# --------------------------------------------------------------------------------------------------- parallel, right half
def gated_delta_scan(q, k, v, g, beta):
    """q, k [n, H, D], v [n, H, Dv], g, beta [n, H] -> (o [n, H, Dv], S [H, D, Dv])."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    o = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, q[t])
    return o, S


def delta_inputs(h, P, m):
    """(q, k, v, g, beta) of the scan, q and k already repeated for the heads that share them."""
    n, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda name: h @ P[name].to(F64).T                                  # noqa: E731
    q, k, v = (silu(causal_conv(lin(x), P[x + ".conv"])) for x in ("q", "k", "v"))
    q, k = unit(q.view(n, G, D)) * D ** -0.5, unit(k.view(n, G, D))
    g = torch.exp(-torch.exp(P["A_log"].to(F64)) * softplus(lin("a") + P["dt_bias"].to(F64)))
    rep = H // G
    return q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), v.view(n, H, Dv), g, torch.sigmoid(lin("b"))


def gated_delta(h, P, m, eps):
    n, H, Dv = h.shape[0], m["heads"], m["vdim"]
    o, _ = gated_delta_scan(*delta_inputs(h, P, m))
    o = rms(o, eps) * P["norm"].to(F64) * silu(h @ P["g"].to(F64).T).view(n, H, Dv)
    return o.reshape(n, H * Dv) @ P["o"].to(F64).T


def parallel(h, P, m, eps):
    left = rms(windowed_attention(h, _sub(P, "left."), m["left"], eps), eps) * P["left.out"].to(F64)
    right = rms(gated_delta(h, _sub(P, "right."), m["right"], eps), eps) * P["right.out"].to(F64)
    return 0.5 * (left + right)


# -------------------------------------------------------------------------------------------------------------- attention
def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def chunked_attention(h, P, m, v_first):
    """(output, this layer's own values before any mixing)."""
    n, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda name: h @ P[name].to(F64).T + P[name + ".b"].to(F64)         # noqa: E731
    rot = m["rot"]
    q = rotate(lin("q").view(n, H, D), rot["base"], rot["dims"])
    k = rotate(lin("k").view(n, G, D), rot["base"], rot["dims"])
    own = lin("v").view(n, G, Dv)
    v = mix_values(own, v_first, float(P["vmix"])) if m.get("v_mix") and v_first is not None else own
    o = attend(q, k, v, float(m["scale"]), lambda i, j: chunk_visible(i, j, m["mask"]["size"]), softcap=float(m["softcap"]))
    o = o * torch.sigmoid(h @ P["g"].to(F64).T)[:, :, None]
    return o.reshape(n, H * Dv) @ P["o"].to(F64).T + P["o.b"].to(F64), own


# -------------------------------------------------------------------------------------------------------------------- wkv
def token_shift(h, mu):
    prev = torch.cat([torch.zeros(1, h.shape[1], dtype=F64), h[:-1]], 0)
    return h + (prev - h) * mu.to(F64)


def wkv_scan(r, k, v, w, u):
    """r, k, w [n, H, D], v [n, H, D], u [H, D] -> (o [n, H, D], S [H, D, D])."""
    n, H, D = r.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    o = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return o, S


def wkv_decay(mix, P):
    z = torch.tanh(mix @ P["w1"].to(F64).T) @ P["w2"].to(F64).T + P["w0"].to(F64)
    return torch.exp(-torch.exp(z))


def wkv(h, P, m, eps):
    n, H, D = h.shape[0], m["heads"], m["dim"]
    mix = {s: token_shift(h, P["mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ P[s].to(F64).T).view(n, H, D) for s in "rkv")
    o, _ = wkv_scan(r, k, v, wkv_decay(mix["w"], P).view(n, H, D), P["u"].to(F64))
    gate = silu(mix["g"] @ P["g"].to(F64).T)
    return (rms(o, eps).reshape(n, H * D) * P["norm"].to(F64) * gate) @ P["o"].to(F64).T


# ------------------------------------------------------------------------------------------------------------------ model
def _sub(P, prefix):
    return {k[len(prefix):]: v for k, v in P.items() if k.startswith(prefix)}


def feed_forward(h, P):
    return (silu(h @ P["gate"].to(F64).T) * (h @ P["up"].to(F64).T)) @ P["down"].to(F64).T


def forward(cfg, W, tokens):
    """(logits [n, vocab], the stream after every layer)."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    table = W["embed"].to(F64)
    x = table[torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    streams, v_first = [], None
    for i, L in enumerate(cfg["layers"]):
        P, m = _sub(W, f"l{i}."), L["mixer"]
        mix = _sub(P, "mix.")
        h = rms(x, eps) * P["norm1"].to(F64)
        if L["type"] == "parallel":
            y = parallel(h, mix, m, eps)
        elif L["type"] == "wkv":
            y = wkv(h, mix, m, eps)
        else:
            y, own = chunked_attention(h, mix, m, v_first)
            if m.get("v_mix") and v_first is None:
                v_first = own
        x = x + mult * y
        if L["mlp"] is not None:
            x = x + mult * feed_forward(rms(x, eps) * P["norm2"].to(F64), _sub(P, "mlp."))
        streams.append(x)
    return (rms(x, eps) * W["final.norm"].to(F64)) @ table.T, streams


def greedy(cfg, W, prompt, new):
    toks = list(prompt)
    for _ in range(new):
        toks.append(int(forward(cfg, W, toks)[0][-1].argmax()))
    return toks


# ------------------------------------------------------------------------------------------------------------------
# small configurations and random weights
# ------------------------------------------------------------------------------------------------------------------
def dense_spec(ff):
    return {"kind": "dense", "ff": ff}


def wkv_layer(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def attention_layer(heads, kv, dim, vdim, size, rot_dims=None, base=5000.0, softcap=20.0, v_mix=True, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "softcap": softcap, "v_mix": v_mix,
        "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims}, "scale": scale or dim ** -0.5}}


def parallel_layer(heads, kv, dim, vdim, size, keep, rheads, rkv, rdim, rvdim, conv=3, scale=None, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                 "scale": scale or dim ** -0.5},
        "right": {"heads": rheads, "kv_heads": rkv, "dim": rdim, "vdim": rvdim, "conv": conv}}}


def make_config(width, vocab, layers, eps=1e-5, residual_mult=0.4, embed_scale=3.0):
    return {"architecture": "Nedesun", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "residual_mult": residual_mult, "embedding": {"scale": embed_scale}}


def random_weights(cfg, seed=0, rank=5):
    """bfloat16 tensors under the checkpoint's names."""
    g = torch.Generator().manual_seed(seed)
    width = cfg["width"]
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        t = torch.randn(*shape, generator=g, dtype=torch.float32) * (std if std is not None else shape[-1] ** -0.5) + mean
        W[name] = t.to(torch.bfloat16)

    put("embed", cfg["vocab"], width, std=0.5)
    put("final.norm", width, std=0.2, mean=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        put(p + "norm1", width, std=0.2, mean=1.0)
        if L["type"] == "wkv":
            N = m["heads"] * m["dim"]
            for s in "rkvgw":
                put(q + "mu." + s, width, std=0.3, mean=0.5)
            for s in "rkvg":
                put(q + s, N, width)
            put(q + "w1", rank, width)
            put(q + "w2", N, rank, std=1.0)
            put(q + "w0", N, std=1.5, mean=-3.0)
            put(q + "u", m["heads"], m["dim"], std=0.6)
            put(q + "norm", N, std=0.2, mean=1.0)
            put(q + "o", width, N)
        elif L["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for s, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                put(q + s, rows, width, std=1.5 * width ** -0.5)
                put(q + s + ".b", rows, std=0.5)
            W[q + "vmix"] = torch.tensor(0.25 + 0.1 * (i % 4)).to(torch.bfloat16)
            put(q + "g", H, width, std=1.5 * width ** -0.5)
            put(q + "o", width, H * Dv)
            put(q + "o.b", width, std=0.3)
        else:
            a, r = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for s, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                put(f"{q}left.{s}", rows, width)
            put(q + "left.q.norm", D, std=0.3, mean=1.3)
            put(q + "left.k.norm", D, std=0.3, mean=1.3)
            put(q + "left.sink", H, std=1.0, mean=1.0)
            put(q + "left.o", width, H * Dv)
            H, G, D, Dv = r["heads"], r["kv_heads"], r["dim"], r["vdim"]
            for s, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                put(f"{q}right.{s}", rows, width)
                put(f"{q}right.{s}.conv", rows, r["conv"], std=0.6)
            put(q + "right.a", H, width)
            put(q + "right.b", H, width)
            put(q + "right.A_log", H, std=0.5)
            put(q + "right.dt_bias", H, std=1.0, mean=-2.0)
            put(q + "right.norm", Dv, std=0.2, mean=1.0)
            put(q + "right.g", H * Dv, width)
            put(q + "right.o", width, H * Dv)
            put(q + "left.out", width, std=0.2, mean=1.0)
            put(q + "right.out", width, std=0.2, mean=1.0)
        if L["mlp"] is not None:
            put(p + "norm2", width, std=0.2, mean=1.0)
            put(p + "mlp.gate", L["mlp"]["ff"], width)
            put(p + "mlp.up", L["mlp"]["ff"], width)
            put(p + "mlp.down", width, L["mlp"]["ff"])
    return W
