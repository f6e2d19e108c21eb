"""Lorenex against the plain float64 oracle in ``lorenex_oracle.py``: every mechanism alone, then the model through the ragged
step, the serving engine's block / slot / state pools and its scheduler. Small random models of several shapes; the same
tests run on the CPU path and (marked ``gpu``) on the CUDA kernels in fp32 and bf16."""
import json
import math

import pytest
import torch

import lorenex_oracle as O

CASES = [("cpu", torch.float32), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu)]
F32_CASES = [("cpu", torch.float32), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu)]


def tol(dtype):
    return 2e-4 if dtype == torch.float32 else 6e-2


def row_errs(got, want):
    """Per row: RMS difference over RMS of the oracle, means over the last axis removed."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def rel_err(got, want):
    return float(row_errs(got.reshape(1, -1), want.reshape(1, -1))[0])


def assert_rows(got, want, dtype, what=""):
    """Every position against the oracle. In fp32 each row must agree. In 16 bits a router score that the oracle decides by a
    hair can fall the other way and move that token's row (and, through the recurrent states, later ones a little) by more
    than rounding, so there nine rows in ten are held to the tolerance and the median to half of it."""
    e = row_errs(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < tol(dtype), (what, float(e.max()), int(e.argmax()))
    else:
        assert float(e.quantile(0.9)) < tol(dtype) and float(e.median()) < tol(dtype) / 2, (what, float(e.quantile(0.9)), float(e.median()))


def build(tmp_path, cfg, W, device, dtype, name="m"):
    from llm_in_practise_b200.io.hf import from_pretrained
    from llm_in_practise_b200.io.safetensors import save_file
    d = tmp_path / name
    d.mkdir(exist_ok=True)
    (d / "config.json").write_text(json.dumps(cfg))
    save_file(W, str(d / "model.safetensors"))
    return from_pretrained(str(d), dtype=dtype, device=torch.device(device))


def fresh_cache(gen, n_seqs, max_len, block=64, poison=True):
    """A cache whose rows list their blocks in a scrambled physical order and whose state rows hold garbage: a sequence that
    starts at position 0 must not read what an earlier user of its row left."""
    per = -(-max_len // block)
    cache = gen.make_cache(n_seqs * per, block, n_seqs, per * block)
    ids = list(range(1, n_seqs * per + 1))[::-1]
    for s in range(n_seqs):
        gen.set_block_row(cache, s, ids[s::n_seqs][:per])
    if poison:
        for layer in cache.state:
            for t in layer:
                t.fill_(37.0)
        for k in cache.k + cache.v:
            k.fill_(9.0)
    return cache


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _i32(x, device):
    return torch.tensor(x, dtype=torch.int32, device=device)


def _mixed():
    layers = [O.parallel_layer(4, 2, 16, 32, inner=40, state=12, dt_rank=5, conv=3, rconv=4, mlp=O.dense_spec(80)),
              O.gla_layer(3, 24, 16, tau=8.0, mlp=O.moe_spec(6, 3, 24, identity=2))]
    layers += [O.same_as(layers, 1), O.same_as(layers, 0), O.gla_layer(2, 8, 40, tau=3.0, mlp=None)]
    return O.make_config(64, 96, layers)


VARIANTS = {
    # both mixers, weights run again in another order, a layer without feed-forward, values wider than keys
    "mixed": _mixed,
    # gla first; as many kv heads as heads; keys wider than values; one tap (no convolution tails); MoE behind the attention
    # without identity experts, every expert chosen; a borrowed layer that is borrowed from again
    "gla_first": lambda: O.make_config(48, 80, (lambda L: L + [O.same_as(L, 0), {**L[0], "weights_of": 3}])([
        O.gla_layer(1, 40, 24, tau=16.0, mlp=O.dense_spec(56)),
        O.parallel_layer(2, 2, 48, 32, inner=24, state=3, dt_rank=1, conv=1, rconv=1, scale=0.3, coef=0.9, every=7, ls=1.0, rs=1.0,
                         mlp=O.moe_spec(3, 3, 16)),
        O.parallel_layer(3, 1, 16, 16, inner=64, state=40, dt_rank=8, conv=2, rconv=2, coef=0.0, every=1, ls=0.3, rs=1.4, mlp=None)]),
        eps=1e-3, residual_mult=1.0, embed_scale=1.0),
    # more identity experts than experts, one expert per token, a tight limit; a state space whose inner size is below the width
    "identity": lambda: O.make_config(40, 64, [
        O.parallel_layer(6, 3, 32, 64, inner=16, state=16, dt_rank=16, conv=5, rconv=3, coef=0.2, every=50,
                         mlp=O.moe_spec(2, 1, 8, identity=5, limit=0.3)),
        O.gla_layer(4, 16, 16, tau=1.0, mlp=O.moe_spec(4, 2, 32, identity=1, limit=7.0))], residual_mult=0.7),
}

# sizes that are not multiples of the kernels' vector widths
ODD = {
    "w72": lambda: O.make_config(72, 75, [
        O.parallel_layer(5, 5, 20, 28, inner=36, state=7, dt_rank=3, conv=4, rconv=5, every=33, mlp=O.dense_spec(92)),
        O.gla_layer(3, 10, 14, tau=12.0, mlp=O.moe_spec(5, 2, 36, identity=2))]),
    "w100": lambda: O.make_config(100, 130, [
        O.gla_layer(2, 36, 72, tau=5.0, mlp=O.moe_spec(4, 2, 52, identity=1)),
        O.parallel_layer(3, 3, 13, 9, inner=50, state=21, dt_rank=7, conv=2, rconv=2, every=5, mlp=O.dense_spec(60)),
        O.parallel_layer(4, 1, 80, 112, inner=10, state=65, dt_rank=9, conv=6, rconv=7, every=64, mlp=None)], residual_mult=0.25),
}


# ------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("W", [40, 72, 100, 256])
def test_output_norm_scaled_residual_and_stream_read(device, dtype, W):
    """x + m norm(y) g on an fp32 stream, the next sublayer reading x itself; after the last layer the head's norm."""
    from llm_in_practise_b200.ops.norm import sandwich_norm
    g = torch.Generator().manual_seed(W)
    n, eps, m = 5, 1e-3, 0.3
    y, x = torch.randn(n, W, generator=g) * 3, torch.randn(n, W, generator=g) * 2
    w1, w2 = torch.randn(W, generator=g), torch.randn(W, generator=g)
    want = x.double() + m * O.rms(y.double(), eps) * w1.double()
    h, xn = sandwich_norm(y.to(device), w1.to(device), x.to(device), None, eps, 0.0, dtype, branch_mult=m, cast_next=True)
    torch.testing.assert_close(xn.cpu().double(), want, rtol=1e-5, atol=1e-5)
    assert h.dtype == dtype and torch.equal(h, xn.to(dtype))
    h, xn = sandwich_norm(y.to(device), w1.to(device), x.to(device), w2.to(device), eps, 0.0, dtype, branch_mult=m, cast_next=True)
    t = tol(dtype) / 4
    torch.testing.assert_close(h.cpu().double(), O.rms(want, eps) * w2.double(), rtol=t, atol=t)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("rows,F", [(3, 8), (5, 100), (2, 4096), (4, 2049)])
def test_power_norm_activation(device, dtype, rows, F):
    from llm_in_practise_b200.ops.norm import poly_norm
    g = torch.Generator().manual_seed(F)
    z = (torch.randn(rows, F, generator=g) * torch.logspace(-2, 1, rows)[:, None]).to(dtype)     # rows where eps matters, too
    for act, eps in (([0.7, -0.4, 1.3, 0.2], 1e-5), ([0.0, 1.0, 0.0, 0.0], 1e-2), ([0.0, 0.0, 1.0, -0.5], 1e-6)):
        a = torch.tensor(act)
        got = poly_norm(z.to(device), a.to(device), eps)
        assert got.dtype == dtype
        t = 2e-5 if dtype == torch.float32 else 1e-2
        torch.testing.assert_close(got.cpu().double(), O.poly_norm(z.double(), a, eps), rtol=t, atol=t)


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("C,rank,tau", [(24, 16, 16.0), (130, 5, 1.0), (7, 33, 4.0), (256, 4, 64.0), (300, 16, 2.0)])
def test_lowrank_decay(device, dtype, C, rank, tau):
    from llm_in_practise_b200.ops.linear_scan import lowrank_decay
    g = torch.Generator().manual_seed(C)
    n = {24: 19, 130: 600, 7: 2100, 256: 1, 300: 2077}[C]                            # a decode batch, and the blockings of long prompts
    buf = torch.randn(n, rank + 3, generator=g)
    w, b = torch.randn(C, rank, generator=g) * 3, torch.randn(C, generator=g) * 8          # far into both tails of the sigmoid
    fast = lowrank_decay(buf.to(device)[:, 3:], w.to(device), b.to(device), tau, fast=True)
    got = lowrank_decay(buf.to(device)[:, 3:], w.to(device), b.to(device), tau)
    want = O.gla_decay(buf[:, 3:].double() @ w.double().T + b.double(), tau)
    torch.testing.assert_close(got.cpu().double(), want, rtol=2e-5, atol=1e-12)
    torch.testing.assert_close(fast.cpu().double(), want, rtol=1e-4, atol=3e-7)


def _cut_runs(lens, plans, rows):
    """Yield per step (parts, runs, pos, slot) for sequences cut by `plans` (one list of counts per sequence)."""
    done = [0] * len(lens)
    for step in range(len(plans[0])):
        parts, runs, pos, slot = [], [], [], []
        for s in range(len(lens)):
            c = plans[s][step]
            if c:
                runs.append([len(pos), c, done[s], rows[s]])
                parts.append((s, done[s], c))
                pos += list(range(done[s], done[s] + c))
                slot += [rows[s]] * c
                done[s] += c
        yield parts, runs, pos, slot
    assert done == list(lens)


# runs of several tiles beside short ones, tiles that start in the middle of a sequence, single tokens
LENS = [330, 85]
PLANS = [[33, 1, 1, 2, 64, 200, 1, 28], [0, 0, 1, 16, 65, 0, 1, 2]]


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("H,G,D,Dv", [(3, 3, 16, 32), (2, 2, 40, 12), (1, 1, 128, 128), (4, 2, 16, 24), (6, 3, 8, 8), (5, 5, 14, 10),
                                      (2, 2, 72, 37), (1, 1, 200, 20)])
def test_channel_decay_scan_across_cuts(device, dtype, H, G, D, Dv):
    """S <- diag(g) S + k v^T in reused rows that hold garbage, however the sequences are cut; a second sequence in the same
    steps has its own state. Decays reach from almost 0 to almost 1, so that far tokens matter."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.linear_scan import linear_scan
    g = torch.Generator().manual_seed(D + Dv)
    data, refs = [], []
    for L in LENS:
        q, k = torch.randn(L, G, D, generator=g) * D ** -0.5, torch.randn(L, G, D, generator=g)
        v = torch.randn(L, H, Dv, generator=g)
        a = torch.sigmoid(torch.randn(L, H, D, generator=g) * 2 + 2) ** (1 / 16)
        a[:, :, 0] = 0.9999
        a[::7, :, 1 % D] = 1e-4
        data.append((q, k, v, a))
        rep = H // G
        refs.append(O.channel_decay_scan(q.double().repeat_interleave(rep, 1), k.double().repeat_interleave(rep, 1), v.double(), a.double()))
    state = torch.full((3, H, D, Dv), 5.0, device=device)
    rows = [2, 0]
    outs = [[], []]
    for parts, runs, pos, slot in _cut_runs(LENS, PLANS, rows):
        cat = lambda i: torch.cat([data[s][i][p:p + c].reshape(c, -1) for s, p, c in parts], 0).to(device)      # noqa: E731
        single = all(c == 1 for _, _, c in parts)
        pieces = None if single else make_pieces(runs, device)
        o = linear_scan(cat(0), cat(1), cat(2), state, _i32(pos, device), _i32(slot, device), None if single else pieces.runs,
                        len(runs), H, G, D, Dv, "channel", g=cat(3), pieces=pieces)
        i = 0
        for s, _, c in parts:
            outs[s].append(o[i:i + c])
            i += c
    for s in range(2):
        got = torch.cat(outs[s], 0).cpu().double().view(LENS[s], H, Dv)
        assert rel_err(got, refs[s][0]) < 1e-4, s
        assert rel_err(state[rows[s]].cpu(), refs[s][1]) < 1e-4


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("inner,N,gated", [(40, 16, True), (24, 3, True), (130, 8, False), (16, 20, True), (9, 40, True), (33, 130, False)])
def test_selective_scan_across_cuts(device, dtype, inner, N, gated):
    """A decay per channel and state, the softplus step, the skip term, the gate and the output factor, written into a column
    slice, in reused rows that hold garbage, however the sequences are cut."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.linear_scan import selective_scan
    g = torch.Generator().manual_seed(inner + N)
    A = -torch.exp(torch.randn(inner, N, generator=g))
    A[:, 0] = -1e-3                                                       # one state that remembers the whole sequence
    D, bias = torch.randn(inner, generator=g), torch.randn(inner, generator=g) - 2
    data, refs = [], []
    for L in LENS:
        u, z = torch.randn(L, inner, generator=g).to(dtype), torch.randn(L, inner, generator=g).to(dtype)
        B, C = torch.randn(L, N, generator=g).to(dtype), (torch.randn(L, N, generator=g) * N ** -0.5).to(dtype)
        dt = torch.randn(L, inner, generator=g) * 2
        data.append((u, dt, B, C, z))
        y, S = O.selective_scan(u.double(), O.softplus(dt.double() + bias.double()), B.double(), C.double(), A.double(), D.double())
        refs.append(((y * O.silu(z.double()) if gated else y) * 0.6, S))
    state = torch.full((3, N, inner), 5.0, device=device)
    rows = [2, 0]
    outs = [[], []]
    for parts, runs, pos, slot in _cut_runs(LENS, PLANS, rows):
        u, dt, B, C, z = (torch.cat([data[s][i][p:p + c] for s, p, c in parts], 0).to(device) for i in range(5))
        single = all(c == 1 for _, _, c in parts)
        pieces = None if single else make_pieces(runs, device)
        buf = torch.full((len(pos), inner + 11), 7.0, dtype=dtype, device=device)
        selective_scan(u, dt, bias.to(device), B, C, A.t().contiguous().to(device), D.to(device), state, _i32(pos, device), _i32(slot, device),
                       None if single else pieces.runs, len(runs), gate=z if gated else None, scale=0.6, out=buf[:, 5:5 + inner], pieces=pieces)
        assert float((buf[:, :5] - 7).abs().max()) == 0 and float((buf[:, 5 + inner:] - 7).abs().max()) == 0
        i = 0
        for s, _, c in parts:
            outs[s].append(buf[i:i + c, 5:5 + inner])
            i += c
    for s in range(2):
        e = row_errs(torch.cat(outs[s], 0), refs[s][0])
        assert float(e.max()) < (1e-4 if dtype == torch.float32 else 2e-2), s
        assert rel_err(state[rows[s]].cpu(), refs[s][1].T) < (1e-4 if dtype == torch.float32 else 1e-3)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("C,taps", [(24, 4), (10, 1), (36, 3), (7, 5), (16, 2)])
def test_short_conv_in_the_model_dtype(device, dtype, C, taps):
    """The state space's convolution reads its inputs in the model dtype; decode steps advance the tail in the same launch."""
    from llm_in_practise_b200.ops.linear_scan import short_conv
    g = torch.Generator().manual_seed(C + taps)
    xs = [torch.randn(L, C, generator=g).to(dtype) for L in LENS]
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    refs = [O.silu(O.causal_conv(x.double(), w, b)) for x in xs]
    tail = torch.full((3, taps - 1, C), 5.0, device=device)
    rows = [2, 0]
    outs = [[], []]
    for parts, runs, pos, slot in _cut_runs(LENS, PLANS, rows):
        x = torch.cat([xs[s][p:p + c] for s, p, c in parts], 0).to(device)
        single = all(c == 1 for _, _, c in parts)
        y = short_conv(x, w.to(device), tail, _i32(pos, device), _i32(slot, device), None if single else _i32(runs, device), len(runs),
                       act=True, bias=b.to(device), out_dtype=dtype)
        i = 0
        for s, _, c in parts:
            outs[s].append(y[i:i + c])
            i += c
    for s in range(2):
        t = 1e-5 if dtype == torch.float32 else 2e-2
        torch.testing.assert_close(torch.cat(outs[s], 0).cpu().double(), refs[s], rtol=t, atol=t)
        if taps > 1:
            torch.testing.assert_close(tail[rows[s]].cpu(), xs[s][-(taps - 1):].float())


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("H,G,D,Dv,taps", [(4, 2, 16, 32, 3), (3, 3, 48, 20, 1), (6, 1, 128, 96, 4), (2, 2, 13, 9, 2), (2, 1, 256, 200, 5),
                                           (2, 2, 24, 24, 6)])
def test_convolved_normed_qkv_store(device, dtype, H, G, D, Dv, taps):
    """Bias, convolution, row norms, query temperature (its steps at multiples of `every`) and page writes, across cuts in
    reused tail rows: what lies before a sequence's start is zero, not the bias."""
    from llm_in_practise_b200.inference.generate import PagedKVCache
    from llm_in_practise_b200.ops.multimap_attention import conv_qknorm_store
    g = torch.Generator().manual_seed(D + taps)
    C, eps, coef, every = (H + G) * D + G * Dv, 1e-3, 0.6, 16
    xs = [torch.randn(L, C, generator=g).to(dtype) for L in LENS]
    bias, w = torch.randn(C, generator=g) * 2, torch.randn(C, taps, generator=g)
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "q_temp": {"coef": coef, "every": every}}
    eye = torch.eye(C, dtype=torch.float64)
    cols = {"q": (0, H * D), "k": (H * D, (H + G) * D), "v": ((H + G) * D, C)}
    P = {}
    for n, (lo, hi) in cols.items():
        P[n], P[n + ".b"], P[n + ".conv"] = eye[lo:hi], bias[lo:hi], w[lo:hi]
    refs = [O.qkv_after_conv(x.double(), P, m, eps) for x in xs]
    cache = PagedKVCache(1, 9, [G], 64, [D], dtype, torch.device(device), 3, 384, Dv=[Dv])
    rows = [2, 0]
    blocks = [[5, 3, 8, 1, 7, 2], [6, 4]]
    for s in range(2):
        cache.set_row(rows[s], blocks[s])
    tail = torch.full((3, taps - 1, C), 5.0, device=device)
    outs = [[], []]
    for parts, runs, pos, slot in _cut_runs(LENS, PLANS, rows):
        x = torch.cat([xs[s][p:p + c] for s, p, c in parts], 0).to(device)
        single = all(c == 1 for _, _, c in parts)
        wide = torch.cat([x, x[:, :4]], 1)                                # rows longer than q | k | v, as in a fused projection
        q = conv_qknorm_store(wide[:, :C], bias.to(device), w.to(device), tail, _i32(pos, device), _i32(slot, device),
                              None if single else _i32(runs, device), len(runs), cache.k[0], cache.v[0], cache.table, H, G, D, Dv, eps,
                              dtype, temp=(coef, float(every)), norm_v=True)
        i = 0
        for s, _, c in parts:
            outs[s].append(q[i:i + c])
            i += c
    t = 1e-4 if dtype == torch.float32 else 3e-2
    for s in range(2):
        n = LENS[s]
        torch.testing.assert_close(torch.cat(outs[s], 0).cpu().double().view(n, H, D), refs[s][0], rtol=t, atol=t)
        k, v = cache.seq_view(0, rows[s], n)
        torch.testing.assert_close(k[:, :n].cpu().double().transpose(0, 1), refs[s][1], rtol=t, atol=t)
        torch.testing.assert_close(v[:, :n].cpu().double().transpose(0, 1), refs[s][2], rtol=t, atol=t)
    assert O.query_temperature(14, coef, every) == 1.0 and abs(O.query_temperature(15, coef, every) - 1 - coef * math.log(2)) < 1e-12


def _pages(device, dtype, k, v, G, D, Dv):
    """Keys and values [n, G, .] in scrambled pages of one cache row."""
    from llm_in_practise_b200.inference.generate import PagedKVCache
    n = k.shape[0]
    nb = -(-n // 64)
    cache = PagedKVCache(1, nb + 1, [G], 64, [D], dtype, torch.device(device), 3, nb * 64, Dv=[Dv])
    cache.k[0].fill_(50.0)
    cache.v[0].fill_(-50.0)
    cache.set_row(1, list(range(nb, 0, -1)))
    pos = torch.arange(n, device=device)
    cache.store(0, torch.full((n,), 1, dtype=torch.long, device=device), pos, k.to(device), v.to(device))
    return cache


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 32, 64), (3, 3, 96, 32), (8, 2, 128, 128), (2, 1, 16, 48), (5, 5, 20, 28), (4, 1, 112, 80),
                                      (6, 2, 13, 9), (2, 2, 64, 256)])
def test_one_map_attention_tokens_and_pieces(device, dtype, H, G, D, Dv):
    """Key and value rows of different sizes, an output factor, output rows inside a wider buffer; single tokens (few tokens
    over many keys are cut into key ranges), and pieces that start anywhere."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.multimap_attention import multimap_attention
    n, scale = 1300, 0.9 * D ** -0.5
    g = torch.Generator().manual_seed(H * D + Dv)
    q, k, v = (torch.randn(n, r, d, generator=g).to(dtype) for r, d in ((H, D), (G, D), (G, Dv)))
    cache = _pages(device, dtype, k, v, G, D, Dv)
    kd, vd = k.double(), v.double()

    def want(rows):
        out = torch.zeros(len(rows), H * Dv, dtype=torch.float64)
        for x, i in enumerate(rows):
            for h in range(H):
                a = torch.softmax(kd[:i + 1, h // (H // G)] @ q[i, h].double() * scale, 0)
                out[x, h * Dv:(h + 1) * Dv] = a @ vd[:i + 1, h // (H // G)]
        return out * 0.8

    plans = [([0, 1, 63, 64, 65, 511, 1023, 1299], False), ([700], False)]
    plans += [(list(range(f, f + c)), True) for f, c in ((0, 130), (37, 100), (60, 9), (126, 2), (1200, 70))]
    for rows, piece in plans:
        T = len(rows)
        pieces = make_pieces([(0, T, rows[0], 1)], device) if piece else None
        buf = torch.full((T, H * Dv + 6), 3.0, dtype=dtype, device=device)
        multimap_attention(q[rows].reshape(T, -1).to(device), cache.k[0], cache.v[0], cache.table, _i32(rows, device), _i32([1] * T, device),
                           H, G, 1, D, Dv, scale, post=0.8, pieces=pieces, max_pos=max(rows), out=buf[:, 2:2 + H * Dv])
        assert float((buf[:, :2] - 3).abs().max()) == 0 and float((buf[:, 2 + H * Dv:] - 3).abs().max()) == 0
        e = row_errs(buf[:, 2:2 + H * Dv], want(rows))
        assert float(e.max()) < tol(dtype), (rows[:3], piece, float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("as_piece", [False, True])
def test_one_dominant_key_far_back_and_at_page_borders(device, dtype, as_piece):
    """One key is made to dominate a query's scores: the output is that key's value, from the first token of the sequence on
    and across page borders; a key one place in the future must leave no trace."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.multimap_attention import multimap_attention
    H, G, D, Dv, n = 4, 2, 32, 64, 720
    g = torch.Generator().manual_seed(5)
    for qi, kj, seen in ((700, 0, True), (700, 1, True), (700, 63, True), (700, 64, True), (700, 127, True), (700, 700, True), (700, 701, False),
                         (63, 0, True), (64, 63, True), (128, 127, True), (5, 6, False), (0, 0, True), (191, 192, False), (192, 192, True)):
        q, k, v = (torch.randn(n, r, d, generator=g) for r, d in ((H, D), (G, D), (G, Dv)))
        unit = torch.nn.functional.normalize(torch.randn(D, generator=g), dim=0)
        k[kj], q[qi] = unit * 10, unit * 60
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        cache = _pages(device, dtype, k, v, G, D, Dv)
        first = max(0, qi - 20) if as_piece else qi
        rows = list(range(first, qi + 1))
        pieces = make_pieces([(0, len(rows), first, 1)], device) if as_piece else None
        got = multimap_attention(q[rows].reshape(len(rows), -1).to(device), cache.k[0], cache.v[0], cache.table, _i32(rows, device),
                                 _i32([1] * len(rows), device), H, G, 1, D, Dv, D ** -0.5, pieces=pieces, max_pos=qi)[-1]
        key = v[kj].float().repeat_interleave(H // G, 0).reshape(-1)
        assert (float((got.float().cpu() - key).abs().max()) < 0.05) == seen, (qi, kj, seen)


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("E,X,top", [(8, 3, 4), (4, 0, 2), (2, 6, 1), (5, 5, 10)])
def test_router_chooses_by_corrected_scores_and_weighs_by_scores(device, dtype, E, X, top):
    from llm_in_practise_b200.ops.moe import route_grouped
    g = torch.Generator().manual_seed(E * 7 + X)
    n, W = 40, 24
    h, wr, corr = torch.randn(n, W, generator=g), torch.randn(E + X, W, generator=g) * 0.5, torch.randn(E + X, generator=g) * 0.3
    want_i, want_p = O.route(h.double(), {"router": wr, "correction": corr}, O.moe_spec(E, top, 8, X))
    ti, tp, _ = route_grouped(h.to(device), wr.to(device), corr.to(device), top, softmax=True)
    assert ti.tolist() == want_i
    torch.testing.assert_close(tp.cpu().double(), torch.tensor(want_p, dtype=torch.float64), rtol=1e-4, atol=1e-7)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("n,W,E,X,top,ff", [(50, 64, 4, 3, 3, 24), (3, 40, 2, 2, 2, 16), (300, 48, 5, 1, 2, 20), (1, 72, 3, 4, 1, 12)])
def test_experts_and_identity_experts(device, dtype, n, W, E, X, top, ff):
    """The weighted sum over experts with clamped gated units and identity experts (which return the fp32 row itself): tokens
    that choose only identity experts, only experts, and both."""
    from llm_in_practise_b200.ops import elementwise as ew
    from llm_in_practise_b200.ops.moe import dispatch, gated_moe_ffn
    g = torch.Generator().manual_seed(n + W)
    f = O.moe_spec(E, top, ff, X, limit=0.8)
    x = torch.randn(n, W, generator=g)
    h = x.to(dtype)
    P = {}
    for e in range(E):
        P[f"e{e}.gate"], P[f"e{e}.up"] = (torch.randn(ff, W, generator=g) * W ** -0.5 * 2).to(dtype), (torch.randn(ff, W, generator=g) * W ** -0.5 * 2).to(dtype)
        P[f"e{e}.down"] = (torch.randn(W, ff, generator=g) * ff ** -0.5).to(dtype)
    ti = torch.stack([torch.randperm(E + X, generator=g)[:top] for _ in range(n)])
    ti[0] = torch.arange(E + X - 1, E + X - 1 - top, -1)                   # the last indices first: identity experts as far as there are
    tp = torch.rand(n, top, generator=g)
    gu = torch.stack([torch.cat([P[f"e{e}.gate"], P[f"e{e}.up"]]) for e in range(E)])
    down = torch.stack([P[f"e{e}.down"] for e in range(E)])
    got = gated_moe_ffn(h.to(device), ti.to(device), tp.to(device), gu.to(device), down.to(device),
                        lambda z: ew.clamped_glu(z, 0.8, 1.702, 1.0), identity=x.to(device))
    want = torch.zeros(n, W, dtype=torch.float64)
    for t in range(n):
        for e, w in zip(ti[t].tolist(), tp[t].tolist()):
            want[t] += w * (O.expert(h[t].double(), P, e, 0.8) if e < E else x[t].double())
    assert got.dtype == torch.float32
    assert float(row_errs(got, want).max()) < (1e-4 if dtype == torch.float32 else 2e-2)
    d = dispatch(ti.to(device), E)
    flat = ti.reshape(-1)
    assert torch.equal(d.dest.cpu() < 0, flat >= E) and d.counts.tolist() == [int((flat == e).sum()) for e in range(E)]
    used = d.dest[d.dest >= 0]
    assert used.unique().numel() == used.numel()
    assert torch.equal(d.tile_map[used // 128].cpu().long(), flat[flat < E])
    assert f["router"]["identity"] == X


# ------------------------------------------------------------------------------------------------------------------
# the model through the ragged step
# ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("variant", list(VARIANTS))
def test_whole_prompt_and_residuals(tmp_path, device, dtype, variant):
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = VARIANTS[variant]()
    W = O.random_weights(cfg, seed=11)
    model = build(tmp_path, cfg, W, device, dtype)
    toks = _tokens(150, cfg["vocab"], 1)
    ref, res_ref = O.forward(cfg, W, toks)
    gen = RaggedGenerator(model, None, 192)
    cache = fresh_cache(gen, 1, 192)
    res = []
    got = gen.step([(0, 0, toks, list(range(len(toks))))], cache, layer_outputs=res)
    assert got.dtype == torch.float32 and all(r.dtype == torch.float32 for r in res)
    for i, L in enumerate(cfg["layers"]):                        # only parallel layers hold pages
        assert (cache.k[i].numel() > 0) == (L["type"] == "parallel")
        assert len(cache.state[i]) == (3 if L["type"] == "parallel" else 1)
    for li, (a, b) in enumerate(zip(res, res_ref)):
        assert_rows(a, b, dtype, (variant, li))
    assert_rows(got, ref, dtype, variant)
    # the first tokens of a sequence: a one-token request and the start of a longer one agree with the oracle row by row
    one = gen.step([(0, 0, toks[:1], [0])], fresh_cache(gen, 1, 64))
    assert rel_err(one, ref[:1]) < 2 * tol(dtype)
    assert rel_err(got[:3], ref[:3]) < 2 * tol(dtype)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("name", list(ODD))
def test_odd_sizes(tmp_path, device, dtype, name):
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = ODD[name]()
    W = O.random_weights(cfg, seed=3, a_rank=5)
    model = build(tmp_path, cfg, W, device, dtype)
    n = 220
    toks = _tokens(n, cfg["vocab"], 2)
    ref = O.forward(cfg, W, toks)[0]
    gen = RaggedGenerator(model, None, 256)
    cache = fresh_cache(gen, 2, 256)
    p, outs = 0, []
    for c in [30, 34, 2, 3, 141, 1, 1, 1, 7]:
        outs.append(gen.step([(1, p, toks[p:p + c], list(range(c)))], cache))
        p += c
    assert_rows(torch.cat(outs, 0), ref, dtype, name)


@pytest.mark.parametrize("device,dtype", CASES)
def test_portions_decode_and_long_decode(tmp_path, device, dtype):
    """Whatever way a sequence is cut into steps — whole, portions down to two tokens that straddle page borders, one token at
    a time for 150 tokens — every position's logits equal the oracle's for the whole sequence."""
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=12)
    model = build(tmp_path, cfg, W, device, dtype)
    n = 230
    toks = _tokens(n, cfg["vocab"], 2)
    ref = O.forward(cfg, W, toks)[0]
    gen = RaggedGenerator(model, None, 256)
    for cuts in ([60, 2, 2, 3, 61, 1, 2, 64, 35], [63, 2, 65, 100], [80] + [1] * 150, [1, 1, 2, 36, 2, 188], [230]):
        assert sum(cuts) == n
        cache = fresh_cache(gen, 1, 256)
        p, outs = 0, []
        for c in cuts:
            outs.append(gen.step([(0, p, toks[p:p + c], list(range(c)))], cache))
            p += c
        assert_rows(torch.cat(outs, 0), ref, dtype, cuts[:4])


@pytest.mark.parametrize("device,dtype", CASES)
def test_mixed_batch_equals_each_alone(tmp_path, device, dtype):
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = VARIANTS["gla_first"]()
    W = O.random_weights(cfg, seed=13)
    model = build(tmp_path, cfg, W, device, dtype)
    lens = [250, 9, 170, 1]
    seqs = [_tokens(L, cfg["vocab"], 20 + i) for i, L in enumerate(lens)]
    refs = [O.forward(cfg, W, s)[0] for s in seqs]
    gen = RaggedGenerator(model, None, 256)
    cache = fresh_cache(gen, 4, 256)
    plans = [[64, 2, 0, 150, 1, 1, 32], [0, 9, 0, 0, 0, 0, 0], [3, 1, 160, 1, 1, 2, 2], [0, 0, 1, 0, 0, 0, 0]]
    done = [0] * 4
    outs = [[] for _ in seqs]
    for step in range(7):
        entries, who = [], []
        for s, plan in enumerate(plans):
            c = plan[step]
            if c:
                entries.append((s, done[s], seqs[s][done[s]:done[s] + c], list(range(c))))
                who.append((s, c))
                done[s] += c
        got = gen.step(entries, cache)
        o = 0
        for s, c in who:
            outs[s].append(got[o:o + c])
            o += c
    assert done == lens
    for s in range(4):
        assert_rows(torch.cat(outs[s], 0), refs[s], dtype, s)


@pytest.mark.parametrize("device,dtype", CASES)
def test_engine_replay_reuses_pages_slots_and_state(tmp_path, device, dtype):
    """The engine's own slot pool (4 rows, each with its recurrent state) and block pool (sized for the live requests only):
    six requests come and go, so rows, their state and pages are handed out again while neighbours still use theirs."""
    from llm_in_practise_b200.serve.engine import EngineArgs, LLMEngine
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=14)
    model = build(tmp_path, cfg, W, device, dtype)
    lens = {"a": 130, "b": 64, "c": 65, "d": 20, "e": 128, "f": 70}
    seqs = {k: _tokens(L, cfg["vocab"], 30 + i) for i, (k, L) in enumerate(lens.items())}
    refs = {k: O.forward(cfg, W, s)[0] for k, s in seqs.items()}
    eng = LLMEngine(model, None, EngineArgs(max_num_seqs=4, max_model_len=192, block_size=64, num_kv_blocks=7,
                                            enable_prefix_caching=False, warmup=False))
    done = {k: 0 for k in lens}
    outs = {k: [] for k in lens}

    def run(parts, end=()):
        entries = []
        for k, c in parts:
            entries.append((k, seqs[k][done[k]:done[k] + c], list(range(c))))
            done[k] += c
        got = eng.replay_step(entries, end)
        o = 0
        for k, c in parts:
            outs[k].append(got[o:o + c])
            o += c

    run([("a", 100), ("b", 30)])
    run([("a", 30), ("b", 34), ("c", 65)], end=["b"])
    run([("d", 20), ("c", 0), ("e", 60)], end=["a"])
    run([("e", 68), ("d", 0)], end=["d", "c"])
    run([("f", 2)])
    run([("f", 62), ("e", 0)])
    run([("f", 6)], end=["e", "f"])
    assert done == lens
    for k in lens:
        assert_rows(torch.cat([o for o in outs[k] if o.shape[0]], 0), refs[k], dtype, k)
    assert len(eng.free) == 4 and len(eng._free_blocks) == 7


@pytest.mark.parametrize("device,dtype", F32_CASES)
def test_greedy_generation_through_engine_and_generate(tmp_path, device, dtype):
    from llm_in_practise_b200.inference import GenerationConfig
    from llm_in_practise_b200.serve.engine import EngineArgs, LLMEngine
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=15)
    model = build(tmp_path, cfg, W, device, dtype)
    prompts = [_tokens(L, cfg["vocab"], 40 + i) for i, L in enumerate([5, 70, 17, 33, 2, 64])]
    new = 10
    refs = [O.greedy(cfg, W, p, new) for p in prompts]
    # scheduler: 4 rows for 6 requests, 24 prompt tokens per iteration, so prompts are cut and mixed with decode tokens; the
    # engine is asked for prefix caching and must switch it off by itself (a recurrent state cannot restart mid-sequence)
    eng = LLMEngine(model, None, EngineArgs(max_num_seqs=4, max_model_len=128, max_prefill_tokens=24, block_size=64,
                                            enable_prefix_caching=True, warmup=False))
    assert not eng.args.enable_prefix_caching
    reqs = eng.generate(prompts, GenerationConfig(max_new_tokens=new, ignore_eos=True))
    for r, p, ref in zip(reqs, prompts, refs):
        assert r.finish_reason == "length"
        assert p + r.output_ids == ref
    again = eng.generate([prompts[1], prompts[5]], GenerationConfig(max_new_tokens=new, ignore_eos=True))
    assert prompts[1] + again[0].output_ids == refs[1] and prompts[5] + again[1].output_ids == refs[5]
    out = model.generate(torch.tensor([prompts[2], prompts[2][::-1]], device=device), max_new_tokens=new)
    assert out[0].tolist() == refs[2]
    assert out[1].tolist() == O.greedy(cfg, W, prompts[2][::-1], new)
    lg = model(torch.tensor([prompts[3]], device=device))["logits"][0]
    assert rel_err(lg, O.forward(cfg, W, prompts[3])[0]) < tol(dtype)


@pytest.mark.parametrize("device,dtype", F32_CASES)
def test_the_position_table_ends(tmp_path, device, dtype):
    """Rows of the engine stop at the model's last position, and a step past it is refused on the host."""
    from llm_in_practise_b200.inference import GenerationConfig
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    from llm_in_practise_b200.serve.engine import EngineArgs, LLMEngine
    cfg = O.make_config(32, 40, [O.parallel_layer(2, 1, 16, 16, inner=16, state=4, dt_rank=2, mlp=O.dense_spec(24))], max_positions=70)
    W = O.random_weights(cfg, seed=4)
    model = build(tmp_path, cfg, W, device, dtype)
    toks = _tokens(72, 40, 1)
    ref = O.forward(cfg, W, toks[:70])[0]
    gen = RaggedGenerator(model, None, 128)
    cache = fresh_cache(gen, 1, 128)
    got = gen.step([(0, 0, toks[:69], list(range(69)))], cache)
    assert_rows(torch.cat([got, gen.step([(0, 69, toks[69:70], [0])], cache)], 0), ref, dtype)
    with pytest.raises(ValueError):
        gen.step([(0, 70, toks[70:71], [0])], cache)
    with pytest.raises(ValueError):
        gen.step([(0, 69, toks[69:71], [0])], cache)
    eng = LLMEngine(model, None, EngineArgs(max_num_seqs=2, max_model_len=4096, block_size=64, warmup=False))
    assert eng.args.max_model_len == 70
    r = eng.generate([toks[:60]], GenerationConfig(max_new_tokens=64, ignore_eos=True))[0]
    assert 60 + len(r.output_ids) == 70


def test_checkpoint_names_round_trip_and_bad_configs(tmp_path):
    from llm_in_practise_b200.models.lorenex import LorenexConfig, lorenex_state_dict
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=16)
    model = build(tmp_path, cfg, W, "cpu", torch.bfloat16)
    sd = lorenex_state_dict(model)
    assert set(sd) == set(W)
    for k in W:
        assert sd[k].shape == W[k].shape, k
        assert torch.equal(sd[k].to(torch.bfloat16).cpu(), W[k]), k
    c = LorenexConfig.from_dict(cfg)
    assert [s.source for s in c.layers] == [0, 1, 1, 0, 4]
    assert model.layers[1] is model.layers[2] and model.layers[0] is model.layers[3]
    assert model.kv_layout() == [(2, 16, 32), (0, 0, 0), (0, 0, 0), (2, 16, 32), (0, 0, 0)]
    assert model.state_layout()[0] == [(2, 160), (3, 40), (12, 40)] and model.state_layout()[2] == [(3, 24, 16)]
    for breakage in (lambda b: b["layers"][0].__setitem__("type", "recurrent"), lambda b: b["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 3),
                     lambda b: b["layers"][1]["mlp"]["router"].__setitem__("top", 9), lambda b: b["layers"][2].__setitem__("weights_of", 0),
                     lambda b: b["layers"][2].__setitem__("weights_of", 2), lambda b: b["layers"][0]["mlp"].__setitem__("kind", "glu")):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            LorenexConfig.from_dict(bad)


def test_replay_builds_every_kernel_source_the_model_calls():
    """A fresh checkout compiles only the sources listed for the design: each entry point the model's ops call is in one."""
    import inspect
    import re
    from llm_in_practise_b200 import _build
    from llm_in_practise_b200.ops import elementwise, gemm, linear_scan, moe, multimap_attention, norm
    from llm_in_practise_b200.recipes.trace import NATIVE_SOURCES
    have = set()
    for stem in NATIVE_SOURCES["Lorenex"]:
        have |= set(re.findall(r"B200_API int (b200_\w+)\(", (_build.CSRC / f"{stem}.cu").read_text()))
    called = set()
    for fn in (elementwise.embedding_pos, elementwise.clamped_glu, gemm.gemm, gemm.gemv16, gemm.linear_exact, linear_scan.linear_scan,
               linear_scan.lowrank_decay, linear_scan.scan_readout, linear_scan.selective_scan, linear_scan.short_conv, linear_scan._conv_tail,
               moe.route_grouped, moe.dispatch, moe.gather_rows, moe._grouped_gemm, moe.moe_combine, multimap_attention.conv_qknorm_store,
               multimap_attention.multimap_attention, norm.poly_norm, norm.sandwich_norm):
        called |= set(re.findall(r"\b(b200_\w+)\b", inspect.getsource(fn)))
    called -= {"b200_gemm_args"}
    assert len(called) > 15 and called <= have, sorted(called - have)
