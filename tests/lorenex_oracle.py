"""A plain float64 statement of the Lorenex equations: one function per mechanism, whole sequences, token by token where
there is a state. It shares nothing with the package (no ops, no cache, no batching) and is what the tests compare the
serving step against.

Weights are a dict name -> tensor under the checkpoint's names (``l<i>.mix.q`` ...); ``cfg`` is the parsed config.json.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def embed(tokens, W, scale):
    return W["embed"].to(F64)[torch.as_tensor(tokens)] * scale + W["pos"].to(F64)[:len(tokens)]


def causal_conv(u, w, bias=None):
    """u [n, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), nothing before t = 0."""
    n, C = u.shape
    taps = w.shape[1]
    y = torch.zeros(n, C, dtype=F64)
    for j in range(taps):
        back = taps - 1 - j                        # w[:, j] weighs the input `back` tokens ago
        if back < n:
            y[back:] += w[:, j].to(F64) * u[:n - back]
    return y if bias is None else y + bias.to(F64)


def gla_decay(z, tau):
    """sigmoid(z)^(1 / tau)."""
    return torch.sigmoid(z) ** (1.0 / tau)


def channel_decay_scan(q, k, v, a):
    """q, k, a [n, H, D], v [n, H, Dv] -> (o [n, H, Dv], S [H, D, Dv]): S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    o = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, q[t])
    return o, S


def gla(h, P, m, eps):
    """h [n, W] -> [n, W]. P: the mixer's tensors by short name."""
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    lin = lambda name: h @ P[name].to(F64).T                                  # noqa: E731
    q = (lin("q") * D ** -0.5).view(n, H, D)
    k, v = lin("k").view(n, H, D), lin("v").view(n, H, Dv)
    z = lin("a1") @ P["a2"].to(F64).T + P["a2.b"].to(F64)
    o, _ = channel_decay_scan(q, k, v, gla_decay(z, float(m["tau"])).view(n, H, D))
    o = rms(o, eps) * P["norm"].to(F64)
    return (o.reshape(n, H * Dv) * silu(lin("g"))) @ P["o"].to(F64).T


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


def qkv_after_conv(h, P, m, eps):
    """Queries (normed, with their temperature), keys and values (normed) of every position: [n, H, D], [n, G, D], [n, G, Dv]."""
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    out = []
    for name, rows, size in (("q", H, D), ("k", G, D), ("v", G, Dv)):
        u = h @ P[name].to(F64).T + P[name + ".b"].to(F64)
        out.append(rms(causal_conv(u, P[name + ".conv"]).view(n, rows, size), eps))
    t = m["q_temp"]
    temp = torch.tensor([query_temperature(p, float(t["coef"]), int(t["every"])) for p in range(n)], dtype=F64)
    return out[0] * temp[:, None, None], out[1], out[2]


def attend(q, k, v, scale):
    """q [n, H, D], k [n, G, D], v [n, G, Dv] -> [n, H * Dv]: every position over itself and all before it."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    mask = torch.ones(n, n, dtype=torch.bool).tril()
    outs = []
    for a in range(H):
        s = (q[:, a] @ k[:, a // rep].T * scale).masked_fill(~mask, float("-inf"))
        outs.append(torch.softmax(s, -1) @ v[:, a // rep])
    return torch.cat(outs, -1)


def attention(h, P, m, eps):
    q, k, v = qkv_after_conv(h, P, m, eps)
    return attend(q, k, v, float(m["scale"])) @ P["o"].to(F64).T


def selective_scan(x, dt, B, C, A, D):
    """x, dt [n, I], B, C [n, N], A [I, N], D [I] -> (y [n, I], S [I, N])."""
    n, inner = x.shape
    S = torch.zeros(inner, A.shape[1], dtype=F64)
    y = torch.zeros(n, inner, dtype=F64)
    for t in range(n):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba(h, P, m):
    inner, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = h @ P["in"].to(F64).T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, P["conv"], P["conv.b"]))
    p = x @ P["x"].to(F64).T
    dt = softplus(p[:, :R] @ P["dt"].to(F64).T + P["dt.b"].to(F64))
    y, _ = selective_scan(x, dt, p[:, R:R + N], p[:, R + N:R + 2 * N], -torch.exp(P["A_log"].to(F64)), P["D"].to(F64))
    return (y * silu(z)) @ P["o"].to(F64).T


def _sub(P, prefix):
    return {k[len(prefix):]: v for k, v in P.items() if k.startswith(prefix)}


def parallel(h, P, m, eps):
    return float(m["left_scale"]) * attention(h, _sub(P, "left."), m["left"], eps) + \
        float(m["right_scale"]) * mamba(h, _sub(P, "right."), m["right"])


def poly_norm(z, act, eps):
    a, b, c, e = (float(x) for x in act)
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def route(h, P, f):
    """Per token: the chosen experts in falling order of their choice score and their weights."""
    s = torch.softmax(h @ P["router"].to(F64).T, -1)
    choice = s + P["correction"].to(F64)
    idx = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :f["router"]["top"]]
    return idx.tolist(), s.gather(1, idx).tolist()


def expert(x, P, e, limit):
    g = (P[f"e{e}.gate"].to(F64) @ x).clamp(max=limit)
    u = (P[f"e{e}.up"].to(F64) @ x).clamp(-limit, limit)
    return P[f"e{e}.down"].to(F64) @ (g * torch.sigmoid(1.702 * g) * (u + 1))


def feed_forward(h, P, f, eps):
    if f["kind"] == "dense":
        return poly_norm(h @ P["up"].to(F64).T, P["act"].to(F64), eps) @ P["down"].to(F64).T
    idx, wts = route(h, P, f)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(idx[t], wts[t]):
            out[t] += w * (expert(h[t], P, e, float(f["expert"]["limit"])) if e < f["router"]["experts"] else h[t])
    return out


def forward(cfg, W, tokens):
    """(logits [n, vocab], the stream after every layer)."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = embed(tokens, W, float(cfg["embedding"]["scale"]))
    streams = []
    for i, L in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = cfg["layers"][j]["weights_of"]
        P = _sub(W, f"l{j}.")
        mix = gla if L["type"] == "gla" else parallel
        x = x + m * rms(mix(x, _sub(P, "mix."), L["mixer"], eps), eps) * P["norm1"].to(F64)
        if L["mlp"] is not None:
            x = x + m * rms(feed_forward(x, _sub(P, "mlp."), L["mlp"], eps), eps) * P["norm2"].to(F64)
        streams.append(x)
    return (rms(x, eps) * W["final.norm"].to(F64)) @ W["embed"].to(F64).T, streams


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


def moe_spec(experts, top, ff, identity=0, limit=2.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "identity": identity}}


def gla_layer(heads, dim, vdim, tau=8.0, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def parallel_layer(heads, kv, dim, vdim, inner, state, dt_rank, conv=2, rconv=3, scale=None, coef=0.4, every=16, ls=0.7, rs=0.6, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or dim ** -0.5,
                 "q_temp": {"coef": coef, "every": every}},
        "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": rconv}, "left_scale": ls, "right_scale": rs}}


def same_as(layers, j):
    """An entry that runs layer j's weights again."""
    return {**layers[j], "weights_of": j}


def make_config(width, vocab, layers, max_positions=512, eps=1e-5, residual_mult=0.4, embed_scale=3.0):
    return {"architecture": "Lorenex", "width": width, "vocab": vocab, "layers": layers, "max_positions": max_positions,
            "norm": {"eps": eps}, "residual_mult": residual_mult, "embedding": {"scale": embed_scale}}


def random_weights(cfg, seed=0, a_rank=6, decisive=True):
    """bfloat16 tensors under the checkpoint's names. Router rows are large, so that a choice seldom hangs on rounding."""
    g = torch.Generator().manual_seed(seed)
    width = cfg["width"]
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        t = torch.randn(*shape, generator=g, dtype=torch.float32) * (std if std is not None else shape[-1] ** -0.5) + mean
        W[name] = t.to(torch.bfloat16)

    put("embed", cfg["vocab"], width, std=0.5)
    put("pos", cfg["max_positions"], width, std=0.5)
    put("final.norm", width, std=0.2, mean=1.0)
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m, f = f"l{i}.", L["mixer"], L["mlp"]
        put(p + "norm1", width, std=0.2, mean=1.0)
        if L["type"] == "gla":
            H, D, Dv = m["heads"], m["dim"], m["vdim"]
            for n, r in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv), ("a1", a_rank)):
                put(f"{p}mix.{n}", r, width)
            put(p + "mix.a2", H * D, a_rank, std=1.5 * a_rank ** -0.5)
            put(p + "mix.a2.b", H * D, std=2.0)
            put(p + "mix.norm", Dv, std=0.2, mean=1.0)
            put(p + "mix.o", width, H * Dv)
        else:
            a, r = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                put(f"{p}mix.left.{n}", rows, width)
                put(f"{p}mix.left.{n}.b", rows, std=0.5)
                put(f"{p}mix.left.{n}.conv", rows, a["conv"], std=0.6)
            put(p + "mix.left.o", width, H * Dv)
            inner, N, R = r["inner"], r["state"], r["dt_rank"]
            put(p + "mix.right.in", 2 * inner, width)
            put(p + "mix.right.conv", inner, r["conv"], std=0.6)
            put(p + "mix.right.conv.b", inner, std=0.5)
            put(p + "mix.right.x", R + 2 * N, inner)
            put(p + "mix.right.dt", inner, R)
            put(p + "mix.right.dt.b", inner, std=1.5, mean=-2.0)
            put(p + "mix.right.A_log", inner, N, std=0.8)
            put(p + "mix.right.D", inner, std=0.5, mean=1.0)
            put(p + "mix.right.o", width, inner)
        if f is None:
            continue
        put(p + "norm2", width, std=0.2, mean=1.0)
        if f["kind"] == "dense":
            put(p + "mlp.up", f["ff"], width)
            put(p + "mlp.down", width, f["ff"])
            put(p + "mlp.act", 4, std=0.5, mean=0.3)
        else:
            E, X = f["router"]["experts"], f["router"].get("identity", 0)
            put(p + "mlp.router", E + X, width, std=(2.0 if decisive else 1.0) * width ** -0.5)
            put(p + "mlp.correction", E + X, std=0.05)
            for e in range(E):
                put(f"{p}mlp.e{e}.gate", f["expert"]["ff"], width, std=1.5 * width ** -0.5)
                put(f"{p}mlp.e{e}.up", f["expert"]["ff"], width, std=1.5 * width ** -0.5)
                put(f"{p}mlp.e{e}.down", width, f["expert"]["ff"])
    return W
