"""Nedesun against the plain float64 oracle in ``nedesun_oracle.py``: every mechanism alone, then the model through the ragged
step, the serving engine's block / slot / state pools and its scheduler. Small random models of several shapes; the same
tests run on the CPU path and (marked ``gpu``) on the CUDA kernels in fp32 and bf16."""
import json

import pytest
import torch

import nedesun_oracle as O

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
    e = row_errs(got, want)
    assert float(e.max()) < tol(dtype), (what, float(e.max()), int(e.argmax()))


def build(tmp_path, cfg, W, device, dtype, name="m"):
    from llm_in_practise_b200.io.hf import from_pretrained
    from llm_in_practise_b200.io.safetensors import save_file
    d = tmp_path / name
    d.mkdir(exist_ok=True)
    (d / "config.json").write_text(json.dumps(cfg))
    save_file(W, str(d / "model.safetensors"))
    return from_pretrained(str(d), dtype=dtype, device=torch.device(device))


def fresh_cache(gen, n_seqs, max_len, block=64):
    """A cache whose rows list their blocks in a scrambled physical order and whose pages and state rows hold garbage: a
    sequence that starts at position 0 must not read what an earlier user left."""
    per = -(-max_len // block)
    cache = gen.make_cache(n_seqs * per, block, n_seqs, per * block)
    ids = list(range(1, n_seqs * per + 1))[::-1]
    for s in range(n_seqs):
        gen.set_block_row(cache, s, ids[s::n_seqs][:per])
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
    return O.make_config(64, 96, [
        O.parallel_layer(4, 2, 16, 24, size=21, keep=3, rheads=4, rkv=2, rdim=16, rvdim=24, conv=3, mlp=O.dense_spec(80)),
        O.wkv_layer(3, 16, mlp=O.dense_spec(48)),
        O.attention_layer(6, 2, 24, 16, size=27, rot_dims=16, softcap=6.0, mlp=None),
        O.wkv_layer(2, 8),
        O.attention_layer(3, 1, 32, 32, size=50, base=800.0, softcap=15.0, v_mix=False, mlp=O.dense_spec(40)),
        O.attention_layer(4, 2, 16, 16, size=13, rot_dims=8, softcap=9.0, mlp=O.dense_spec(64))])


VARIANTS = {
    # all three mixers, layers with and without feed-forward, a layer between two that share values which shares none
    "mixed": _mixed,
    # attention first; one kv head per head; no kept tokens and windows larger than the prompt; one tap (no tails); values wider
    # than keys; a delta rule with one q/k head; chunks of one page; three layers of mixed values
    "attention_first": lambda: O.make_config(48, 80, [
        O.attention_layer(2, 2, 48, 8, size=64, rot_dims=4, softcap=30.0, scale=0.12, mlp=O.dense_spec(56)),
        O.parallel_layer(2, 2, 8, 40, size=400, keep=0, rheads=3, rkv=1, rdim=40, rvdim=8, conv=1, scale=0.5, mlp=None),
        O.attention_layer(4, 2, 16, 8, size=5, softcap=2.0, mlp=None),
        O.attention_layer(2, 2, 64, 8, size=128, rot_dims=32, base=100.0, softcap=50.0, mlp=O.dense_spec(24))],
        eps=1e-3, residual_mult=1.0, embed_scale=1.0),
    # windows of one token beside kept ones, more kept tokens than the window, a single wkv head wider than the model's width
    "narrow": lambda: O.make_config(40, 64, [
        O.wkv_layer(1, 64, mlp=None),
        O.parallel_layer(6, 3, 32, 16, size=1, keep=9, rheads=2, rkv=2, rdim=8, rvdim=56, conv=5, mlp=O.dense_spec(32)),
        O.parallel_layer(3, 1, 64, 64, size=6, keep=70, rheads=6, rkv=3, rdim=24, rvdim=16, conv=2, mlp=None)], residual_mult=0.7),
}

# sizes that are not multiples of the kernels' vector widths
ODD = {
    "w72": (lambda: O.make_config(72, 75, [
        O.wkv_layer(3, 10, mlp=O.dense_spec(92)),
        O.attention_layer(5, 5, 20, 28, size=33, rot_dims=6, mlp=O.dense_spec(36)),
        O.parallel_layer(5, 5, 20, 28, size=40, keep=5, rheads=3, rkv=3, rdim=10, rvdim=14, conv=4, mlp=O.dense_spec(20))]), 3),
    "w100": (lambda: O.make_config(100, 130, [
        O.parallel_layer(3, 3, 13, 9, size=17, keep=2, rheads=4, rkv=1, rdim=36, rvdim=72, conv=7, mlp=O.dense_spec(52)),
        O.attention_layer(4, 1, 80, 112, size=90, rot_dims=54, mlp=None),
        O.wkv_layer(2, 37, mlp=None),
        O.attention_layer(3, 1, 9, 112, size=70, rot_dims=2, mlp=O.dense_spec(60))], residual_mult=0.25), 11),
    "w128": (lambda: O.make_config(128, 256, [                                    # sizes the small-batch product kernels take
        O.attention_layer(2, 1, 96, 128, size=100, rot_dims=96, mlp=O.dense_spec(128)),
        O.wkv_layer(2, 64, mlp=O.dense_spec(128)),
        O.parallel_layer(2, 1, 128, 64, size=90, keep=4, rheads=2, rkv=1, rdim=64, rvdim=64, conv=4, mlp=O.dense_spec(256))]), 16),
}


# ------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("W", [40, 72, 100, 256])
def test_two_normed_branches_and_the_next_norm(device, dtype, W):
    """x + m (norm(y1) g1 + norm(y2) g2) on an fp32 stream and the norm behind it; branches of very different size."""
    from llm_in_practise_b200.ops.norm import sandwich_norm
    g = torch.Generator().manual_seed(W)
    n, eps, m = 5, 1e-3, 0.3
    y1, y2, x = torch.randn(n, W, generator=g) * 30, torch.randn(n, W, generator=g) * 0.02, torch.randn(n, W, generator=g) * 2
    w1, w2, w3 = (torch.randn(W, generator=g) for _ in range(3))
    want = x.double() + m * (O.rms(y1.double(), eps) * w1.double() + O.rms(y2.double(), eps) * w2.double())
    dev = lambda t: t.to(device)                                                                  # noqa: E731
    h, xn = sandwich_norm(dev(y1), dev(w1), dev(x), dev(w3), eps, 0.0, dtype, branch_mult=m, y2=dev(y2), post_w2=dev(w2))
    torch.testing.assert_close(xn.cpu().double(), want, rtol=1e-5, atol=1e-5)
    t = tol(dtype) / 4
    assert h.dtype == dtype
    torch.testing.assert_close(h.cpu().double(), O.rms(want, eps) * w3.double(), rtol=t, atol=t)


def test_embedding_scale_enters_the_stream_in_fp32():
    from llm_in_practise_b200.ops.elementwise import embedding_pos
    table = torch.randn(9, 7).to(torch.bfloat16)
    ids = torch.tensor([3, 3, 0, 8])
    torch.testing.assert_close(embedding_pos(ids, table, 11.3), table[ids].float() * 11.3)


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
ROWS = [2, 0]


def _walk(device, call):
    """Run ``call(parts, pos, slot, runs or None, n_runs, pieces)`` over the cuts; collect its rows per sequence."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    outs = [[], []]
    for parts, runs, pos, slot in _cut_runs(LENS, PLANS, ROWS):
        single = all(c == 1 for _, _, c in parts)
        pieces = None if single else make_pieces(runs, device)
        y = call(parts, _i32(pos, device), _i32(slot, device), None if single else pieces.runs, len(runs), pieces)
        i = 0
        for s, _, c in parts:
            outs[s].append(y[i:i + c])
            i += c
    return [torch.cat(o, 0).cpu().double() for o in outs]


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("W,S", [(24, 5), (7, 5), (130, 2), (64, 1)])
def test_token_shift_across_cuts(device, dtype, W, S):
    """The token before is the row before inside a piece, the carried one at its start, zeros (not what the state row held) at
    the start of a sequence."""
    from llm_in_practise_b200.ops.linear_scan import token_shift
    g = torch.Generator().manual_seed(W)
    xs = [torch.randn(L, W, generator=g).to(dtype) for L in LENS]
    mu = torch.randn(S, W, generator=g)
    prev = torch.full((3, 1, W), 5.0, device=device)

    def call(parts, pos, slot, runs, n_runs, pieces):
        x = torch.cat([xs[s][p:p + c] for s, p, c in parts], 0).to(device)
        y = token_shift(x, mu.to(device), prev, pos, slot, runs, n_runs)
        assert y.dtype == dtype and y.shape == (S, x.shape[0], W)
        return y.transpose(0, 1)

    for s, got in enumerate(_walk(device, call)):
        want = torch.stack([O.token_shift(xs[s].double(), mu[i]) for i in range(S)], 1)
        t = 1e-5 if dtype == torch.float32 else 2e-2
        torch.testing.assert_close(got, want, rtol=t, atol=t)
        assert torch.equal(prev[ROWS[s], 0].cpu(), xs[s][-1].float())


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("C,rank,n", [(24, 16, 19), (130, 5, 600), (7, 33, 2100), (256, 4, 1), (300, 16, 2077)])
def test_exponential_lowrank_decay(device, dtype, C, rank, n):
    """exp(-exp(W_2 tanh(x) + w_0)) from decays that forget at once to ones that are 1 but for 1e-4, whose power over a long
    reach must come out right."""
    from llm_in_practise_b200.ops.linear_scan import lowrank_decay
    g = torch.Generator().manual_seed(C)
    buf = torch.randn(n, rank + 3, generator=g) * 2
    w, b = torch.randn(C, rank, generator=g) * 0.6, torch.linspace(-9, 2, C)
    want = torch.exp(-torch.exp(torch.tanh(buf[:, 3:].double()) @ w.double().T + b.double()))
    P = {"w1": torch.eye(rank), "w2": w, "w0": b}
    torch.testing.assert_close(O.wkv_decay(buf[:, 3:].double(), P), want)
    run = lambda fast: lowrank_decay(buf.to(device)[:, 3:], w.to(device), b.to(device), fast=fast, form="exp_exp")      # noqa: E731
    got, fast = run(False), run(True)
    torch.testing.assert_close(got.cpu().double(), want, rtol=2e-5, atol=1e-9)
    torch.testing.assert_close(fast.cpu().double(), want, rtol=1e-4, atol=3e-7)
    slow = want.min(0).values > 0.999
    if n > 500 and bool(slow.any()):                    # the error of a product over all tokens, relative to 1
        err = (got.cpu().double().log().sum(0) - want.log().sum(0)).abs()[slow]
        assert float(err.max()) < 2e-5


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("G,H,D", [(2, 4, 16), (3, 3, 10), (1, 5, 72)])
def test_unit_rows_and_decay_per_head(device, dtype, G, H, D):
    from llm_in_practise_b200.ops.linear_scan import delta_gates
    g = torch.Generator().manual_seed(D)
    n = 9
    q, k = torch.randn(n, G * D, generator=g) * 3, torch.randn(n, G * D, generator=g)
    k[0] = 0.0                                                          # a zero row stays zero
    k[1] *= 1e-4                                                        # eps matters
    tail = torch.randn(n, 2 * H + 3, generator=g) * 4
    bias, A_log = torch.randn(H, generator=g), torch.randn(H, generator=g)
    qd, kd, td = (t.clone().to(device) for t in (q, k, tail))                                     # the gates are formed in place
    a, b = td[:, 3:3 + H], td[:, 3 + H:]
    delta_gates(qd, kd, a, b, bias.to(device), A_log.to(device), G, H, D, D ** -0.5, 1e-6)
    unit = lambda x: O.unit(x.double().view(n, G, D)).view(n, G * D)                             # noqa: E731
    torch.testing.assert_close(qd.cpu().double(), unit(q) * D ** -0.5, rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(kd.cpu().double(), unit(k), rtol=1e-5, atol=1e-6)
    want = torch.exp(-torch.exp(A_log.double()) * O.softplus(tail[:, 3:3 + H].double() + bias.double()))
    torch.testing.assert_close(a.cpu().double(), want, rtol=1e-5, atol=1e-7)
    torch.testing.assert_close(b.cpu().double(), torch.sigmoid(tail[:, 3 + H:].double()), rtol=1e-5, atol=1e-7)
    torch.testing.assert_close(td[:, :3].cpu(), tail[:, :3])


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("H,G,D,Dv", [(3, 3, 16, 32), (2, 2, 40, 12), (1, 1, 128, 128), (4, 2, 16, 24), (6, 3, 8, 8), (5, 1, 14, 10),
                                      (2, 2, 72, 37), (2, 1, 200, 20), (4, 2, 64, 64)])
def test_delta_scan_with_a_decay_per_head_across_cuts(device, dtype, H, G, D, Dv):
    """The gated delta rule in reused rows that hold garbage, however the sequences are cut; one head hardly forgets."""
    from llm_in_practise_b200.ops.linear_scan import linear_scan
    g = torch.Generator().manual_seed(D + Dv)
    data, refs = [], []
    rep = H // G
    for L in LENS:
        q, k = (O.unit(torch.randn(L, G, D, generator=g).double()).float() for _ in range(2))
        v = torch.randn(L, H, Dv, generator=g)
        a = torch.exp(-torch.exp(torch.randn(L, H, generator=g) * 2 - 4))
        a[:, 0] = 0.9999
        beta = torch.sigmoid(torch.randn(L, H, generator=g) * 2)
        data.append((q, k, v, a, beta))
        refs.append(O.gated_delta_scan(q.double().repeat_interleave(rep, 1), k.double().repeat_interleave(rep, 1), v.double(), a.double(),
                                       beta.double()))
    state = torch.full((3, H, D, Dv), 5.0, device=device)

    def call(parts, pos, slot, runs, n_runs, pieces):
        q, k, v, a, beta = (torch.cat([data[s][i][p:p + c].reshape(c, -1) for s, p, c in parts], 0).to(device) for i in range(5))
        return linear_scan(q, k, v, state, pos, slot, runs, n_runs, H, G, D, Dv, "head_delta", g=a, beta=beta, pieces=pieces)

    for s, got in enumerate(_walk(device, call)):
        e = row_errs(got, refs[s][0].reshape(LENS[s], -1))
        assert float(e.max()) < 1e-4, (s, float(e.max()), int(e.argmax()))
        assert rel_err(state[ROWS[s]].cpu(), refs[s][1]) < 1e-4


@pytest.mark.parametrize("device,dtype", F32_CASES)
@pytest.mark.parametrize("H,D,Dv", [(3, 16, 32), (2, 40, 12), (1, 128, 128), (6, 8, 8), (5, 14, 10), (2, 72, 37), (1, 200, 20), (2, 64, 64)])
def test_channel_scan_with_a_bonus_across_cuts(device, dtype, H, D, Dv):
    """The read-out sees the state before its decay and the token itself through the bonus alone; runs of several tiles."""
    from llm_in_practise_b200.ops.linear_scan import linear_scan
    g = torch.Generator().manual_seed(D + Dv)
    data, refs = [], []
    u = torch.randn(H, D, generator=g) * 2
    for L in LENS:
        q, k = torch.randn(L, H, D, generator=g) * D ** -0.5, torch.randn(L, H, D, generator=g)
        v = torch.randn(L, H, Dv, generator=g)
        a = torch.exp(-torch.exp(torch.randn(L, H, D, generator=g) * 2 - 3))
        a[:, :, 0] = 0.9999
        a[::7, :, 1 % D] = 1e-4
        data.append((q, k, v, a))
        refs.append(O.wkv_scan(q.double(), k.double(), v.double(), a.double(), u.double()))
    state = torch.full((3, H, D, Dv), 5.0, device=device)

    def call(parts, pos, slot, runs, n_runs, pieces):
        q, k, v, a = (torch.cat([data[s][i][p:p + c].reshape(c, -1) for s, p, c in parts], 0).to(device) for i in range(4))
        return linear_scan(q, k, v, state, pos, slot, runs, n_runs, H, H, D, Dv, "channel", g=a, pieces=pieces, u=u.to(device))

    for s, got in enumerate(_walk(device, call)):
        e = row_errs(got, refs[s][0].reshape(LENS[s], -1))
        assert float(e.max()) < 1e-4, (s, float(e.max()), int(e.argmax()))
        assert rel_err(state[ROWS[s]].cpu(), refs[s][1]) < 1e-4


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shared", [True, False])
def test_readout_with_a_silu_gate_in_the_model_dtype(device, dtype, shared):
    """Shared and per-column weights; the gate as a strided slice of fp32 rows or of rows in the model dtype."""
    from llm_in_practise_b200.ops.linear_scan import scan_readout
    H, Dv, n, eps = 3, 20, 6, 1e-2
    g = torch.Generator().manual_seed(3)
    o = torch.randn(n, H * Dv, generator=g) * 0.2
    w = torch.randn(Dv if shared else H * Dv, generator=g)
    for gate_dtype in {torch.float32, dtype}:
        gate = torch.randn(n, H * Dv + 8, generator=g).to(gate_dtype)
        got = scan_readout(o.to(device), H, Dv, w.to(device), H, eps, dtype, post=gate.to(device)[:, 8:], post_act="silu")
        z = (O.rms(o.double().view(n, H, Dv), eps).reshape(n, -1)) * (w.double().repeat(H) if shared else w.double())
        t = tol(dtype) / 4
        torch.testing.assert_close(got.cpu().double(), z * O.silu(gate[:, 8:].double()), rtol=t, atol=t)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("M", [1, 9, 16, 17, 150])
@pytest.mark.parametrize("N,K", [(64, 128), (40, 72), (24, 36), (256, 256)])
def test_products_with_bias_and_products_of_several_inputs(device, dtype, M, N, K):
    from llm_in_practise_b200.ops.gemm import linear_each, linear_exact
    g = torch.Generator().manual_seed(M + N)
    x, w, b = (torch.randn(*s, generator=g).to(dtype) for s in ((4, M, K), (4, N, K), (N,)))
    t = 1e-4 if dtype == torch.float32 else 2e-2
    got = linear_each(x.to(device), w.to(device))
    want = torch.einsum("bmk,bnk->mbn", x.double(), w.double()).reshape(M, 4 * N)
    assert got.dtype == torch.float32
    torch.testing.assert_close(got.cpu().double(), want, rtol=1e-4, atol=2e-4 * K ** 0.5)
    for out in (torch.float32, dtype):
        y = linear_exact(x[1].to(device), w[2].to(device), out_dtype=out, bias=b.to(device))
        torch.testing.assert_close(y.cpu().double(), x[1].double() @ w[2].double().T + b.double(), rtol=t, atol=t * K ** 0.5)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("H,G,D,Dv,rot", [(4, 2, 16, 32, 16), (3, 3, 48, 20, 20), (6, 1, 128, 96, 64), (2, 2, 13, 9, 6), (2, 1, 256, 200, 256),
                                          (5, 5, 20, 28, 0), (2, 1, 80, 300, 2), (1, 1, 70, 130, 34)])
def test_qkv_store(device, dtype, H, G, D, Dv, rot):
    """Bias, row norms, partial rotary, values mixed with another pool's, page writes — all together and each left out —, from
    rows longer than q | k | v, at positions that jump over pages of scrambled order, for a few tokens and for many."""
    from llm_in_practise_b200.inference.generate import PagedKVCache
    from llm_in_practise_b200.ops.elementwise import rope_tables_partial
    from llm_in_practise_b200.ops.multimap_attention import qkv_store
    g = torch.Generator().manual_seed(D + Dv)
    C, eps, L, base = (H + G) * D + G * Dv, 1e-3, 600, 300.0
    x = torch.randn(L, C + 4, generator=g).to(dtype)
    first = torch.randn(L, G, Dv, generator=g).to(dtype)
    bias, wq, wk = torch.randn(C, generator=g) * 2, torch.randn(D, generator=g), torch.randn(D, generator=g)
    lam = torch.tensor([0.3])
    rope = rope_tables_partial(640, rot, base, torch.device(device)) if rot else None
    for with_bias, norm, mix, n in ((True, True, True, L), (False, True, False, 40), (True, False, True, 40), (False, False, False, L)):
        cache = PagedKVCache(2, 11, [G, G], 64, [D, D], dtype, torch.device(device), 2, 640, Dv=[Dv, Dv])
        cache.set_row(1, [4, 9, 1, 10, 2, 7, 3, 8, 5, 6])
        p = torch.arange(L - n, L)
        cache.store(1, torch.ones(n, dtype=torch.long, device=device), p.to(device), torch.zeros(n, G, D, dtype=dtype, device=device),
                    first[p].to(device))
        dev = lambda t, on: t.to(device) if on else None                                          # noqa: E731
        q = qkv_store(x[p].to(device)[:, :C] if n < L else x.to(device)[:, :C], dev(bias, with_bias), dev(wq, norm), dev(wk, norm), rope,
                      _i32(p.tolist(), device), _i32([1] * n, device), cache.k[0], cache.v[0], cache.table, H, G, D, Dv, rot, eps, dtype,
                      v_first=cache.v[1] if mix else None, v_lambda=dev(lam, mix))
        y = x[:, :C].double() + (bias.double() if with_bias else 0.0)
        yq, yk, yv = y[:, :H * D].view(L, H, D), y[:, H * D:(H + G) * D].view(L, G, D), y[:, (H + G) * D:].view(L, G, Dv)
        if norm:
            yq, yk = O.rms(yq, eps) * wq.double(), O.rms(yk, eps) * wk.double()
        yq, yk = O.rotate(yq, base, rot), O.rotate(yk, base, rot)
        if mix:
            yv = O.mix_values(yv, first.double(), float(lam))
        t = 1e-4 if dtype == torch.float32 else 3e-2
        torch.testing.assert_close(q.cpu().double().view(n, H, D), yq[p], rtol=t, atol=t)
        k, v = cache.seq_view(0, 1, L)
        torch.testing.assert_close(k[:, p].cpu().double().transpose(0, 1), yk[p], rtol=t, atol=t)
        torch.testing.assert_close(v[:, p].cpu().double().transpose(0, 1), yv[p], rtol=t, atol=t)


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


OPTIONS = {
    "window and sink": dict(window=90, keep_first=7, sink=True),
    "wide window and sink": dict(window=1000, keep_first=130, sink=True),
    "capped chunks and gate": dict(softcap=3.0, chunk=100, gate=True),
    "capped long chunks": dict(softcap=40.0, chunk=1200),
    "everything": dict(softcap=2.0, window=333, keep_first=64, sink=True, gate=True),
}


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("options", list(OPTIONS))
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 32, 64), (3, 3, 96, 40), (8, 2, 128, 128), (2, 1, 16, 48), (5, 5, 20, 28), (4, 1, 112, 80),
                                      (6, 2, 13, 9), (2, 2, 24, 8), (2, 1, 64, 200)])
def test_attention_options_tokens_and_pieces(device, dtype, options, H, G, D, Dv):
    """Sinks, capped scores, chunks and gates on single tokens (few tokens over many keys are cut into key ranges) and on
    pieces that start anywhere and reach over windows' and chunks' edges."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.multimap_attention import multimap_attention
    opt = OPTIONS[options]
    n, scale = 1300, 2.0 * D ** -0.5
    g = torch.Generator().manual_seed(H * D + Dv)
    q, k, v = (torch.randn(n, r, d, generator=g).to(dtype) for r, d in ((H, D), (G, D), (G, Dv)))
    sink = torch.linspace(-3, 9, H) if opt.get("sink") else None
    gate = torch.randn(n, H + 3, generator=g) if opt.get("gate") else None
    cache = _pages(device, dtype, k, v, G, D, Dv)
    window, keep, chunk, cap = opt.get("window", 0), opt.get("keep_first", 0), opt.get("chunk", 0), opt.get("softcap", 0.0)
    rep = H // G
    kd, vd = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)

    def want(rows):
        out = torch.zeros(len(rows), H, Dv, dtype=torch.float64)
        for x, i in enumerate(rows):
            js = [j for j in range(i + 1) if (O.chunk_visible(i, j, chunk) if chunk else O.window_visible(i, j, window, keep))]
            s = torch.einsum("hd,nhd->hn", q[i].double(), kd[js]) * scale
            if cap:
                s = cap * torch.tanh(s / cap)
            if sink is not None:
                s = torch.cat([s, sink.double()[:, None]], 1)
            out[x] = torch.einsum("hn,nhe->he", torch.softmax(s, -1)[:, :len(js)], vd[js])
            if gate is not None:
                out[x] *= torch.sigmoid(gate[i, 3:].double())[:, None]
        return out.view(len(rows), -1)

    plans = [([0, 1, 63, 64, 65, 99, 100, 511, 1023, 1299], False), ([700], False), ([1199], False)]
    plans += [(list(range(f, f + c)), True) for f, c in ((0, 130), (37, 100), (60, 9), (126, 2), (1150, 70))]
    for rows, piece in plans:
        T = len(rows)
        pieces = make_pieces([(0, T, rows[0], 1)], device) if piece else None
        got = multimap_attention(q[rows].reshape(T, -1).to(device), cache.k[0], cache.v[0], cache.table, _i32(rows, device), _i32([1] * T, device),
                                 H, G, 1, D, Dv, scale, window, keep, pieces=pieces, max_pos=max(rows),
                                 sink=sink.to(device) if sink is not None else None, softcap=cap, chunk=chunk,
                                 gate=gate.to(device)[rows][:, 3:] if gate is not None else None)
        e = row_errs(got, want(rows))
        assert float(e.max()) < tol(dtype), (rows[:3], piece, float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("as_piece", [False, True])
def test_dominant_keys_at_every_edge(device, dtype, as_piece):
    """One key is made to dominate a query's scores: if the query sees it the output is that key's value, else the key leaves
    no trace — at the edges of windows, of the kept first tokens, of chunks and of pages, one place in the future, far away."""
    from llm_in_practise_b200.inference.ragged import make_pieces
    from llm_in_practise_b200.ops.multimap_attention import multimap_attention
    H, G, D, Dv, n = 4, 2, 32, 64, 720
    g = torch.Generator().manual_seed(5)
    win = dict(window=100, keep_first=20)
    cases = [(win, qi, kj, seen) for qi, kj, seen in (
        (700, 601, True), (700, 600, False), (700, 0, True), (700, 19, True), (700, 20, False), (700, 63, False), (700, 700, True),
        (700, 701, False), (119, 20, True), (120, 20, False), (120, 19, True), (120, 21, True), (99, 20, True), (163, 64, True),
        (164, 64, False), (192, 93, True), (192, 92, False))]
    cases += [(dict(window=1, keep_first=3), qi, kj, seen) for qi, kj, seen in ((500, 500, True), (500, 499, False), (500, 2, True), (500, 3, False))]
    chunk = dict(chunk=150, softcap=25.0)
    cases += [(chunk, qi, kj, seen) for qi, kj, seen in (
        (149, 0, True), (150, 149, False), (150, 150, True), (151, 150, True), (299, 150, True), (299, 149, False), (300, 299, False),
        (700, 600, True), (700, 599, False), (700, 0, False), (700, 701, False), (639, 600, True), (640, 639, True))]
    for opt, qi, kj, seen in cases:
        q, k, v = (torch.randn(n, r, d, generator=g) for r, d in ((H, D), (G, D), (G, Dv)))
        unit = torch.nn.functional.normalize(torch.randn(D, generator=g), dim=0)
        k[kj], q[qi] = unit * 10, unit * (12 if "softcap" in opt else 60)      # a capped score must stay apart from the others
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        cache = _pages(device, dtype, k, v, G, D, Dv)
        first = max(0, qi - 20) if as_piece else qi
        rows = list(range(first, qi + 1))
        pieces = make_pieces([(0, len(rows), first, 1)], device) if as_piece else None
        for sink in (-20.0, 60.0):                           # a sink far below the key's score, and one far above a capped score
            got = multimap_attention(q[rows].reshape(len(rows), -1).to(device), cache.k[0], cache.v[0], cache.table, _i32(rows, device),
                                     _i32([1] * len(rows), device), H, G, 1, D, Dv, D ** -0.5, pieces=pieces, max_pos=qi,
                                     sink=torch.full((H,), sink, device=device), **opt)[-1].float().cpu()
            key = v[kj].float().repeat_interleave(H // G, 0).reshape(-1)
            if sink > 0 and "softcap" in opt:
                assert float(got.abs().max()) < 1e-6, (opt, qi, kj, sink)
            else:
                assert (float((got - key).abs().max()) < 0.05) == seen, (opt, qi, kj, seen, sink)


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
    for i, L in enumerate(cfg["layers"]):
        assert (cache.k[i].numel() > 0) == (L["type"] != "wkv")
        assert len(cache.state[i]) == (0 if L["type"] == "attention" else 2)
    for li, (a, b) in enumerate(zip(res, res_ref)):
        assert_rows(a, b, dtype, (variant, li))
    assert_rows(got, ref, dtype, variant)
    # the first tokens of a sequence: a one-token request and the start of a longer one agree with the oracle row by row
    one = gen.step([(0, 0, toks[:1], [0])], fresh_cache(gen, 1, 64))
    assert rel_err(one, ref[:1]) < tol(dtype)
    assert rel_err(got[:3], ref[:3]) < tol(dtype)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("name", list(ODD))
def test_odd_sizes(tmp_path, device, dtype, name):
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    make, rank = ODD[name]
    cfg = make()
    W = O.random_weights(cfg, seed=3, rank=rank)
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
    """Whatever way a sequence is cut into steps — whole, portions down to two tokens that straddle page, window and chunk
    borders, one token at a time for 150 tokens — every position's logits equal the oracle's for the whole sequence."""
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=12)
    model = build(tmp_path, cfg, W, device, dtype)
    n = 230
    toks = _tokens(n, cfg["vocab"], 2)
    ref = O.forward(cfg, W, toks)[0]
    gen = RaggedGenerator(model, None, 256)
    for cuts in ([60, 2, 2, 3, 61, 1, 2, 64, 35], [26, 2, 22, 2, 62, 2, 114], [80] + [1] * 150, [1, 1, 2, 36, 2, 188], [230]):
        assert sum(cuts) == n
        cache = fresh_cache(gen, 1, 256)
        p, outs = 0, []
        for c in cuts:
            outs.append(gen.step([(0, p, toks[p:p + c], list(range(c)))], cache))
            p += c
        assert_rows(torch.cat(outs, 0), ref, dtype, cuts[:4])


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("variant", ["attention_first", "narrow"])
def test_mixed_batch_equals_each_alone(tmp_path, device, dtype, variant):
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    cfg = VARIANTS[variant]()
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


@pytest.mark.parametrize("device,dtype", CASES)
def test_a_far_token_shows_in_the_logits_until_it_may_not(tmp_path, device, dtype):
    """Two prompts that differ in one token. A model of attention layers alone forgets it when it leaves the window (but not
    when it is one of the kept first tokens) and when a chunk ends; the recurrent halves remember it."""
    from llm_in_practise_b200.inference.ragged import RaggedGenerator
    win = O.parallel_layer(4, 2, 16, 24, size=50, keep=4, rheads=2, rkv=1, rdim=16, rvdim=16, conv=2)
    cases = [(win, True, 3, [140], []), (win, True, 4, [53], [54, 140]), (win, True, 30, [79], [80, 140]), (win, False, 30, [79, 80, 140], []),
             (O.attention_layer(4, 2, 16, 16, size=40), True, 20, [39], [40, 140]), (O.attention_layer(4, 2, 16, 16, size=40), True, 40, [79], [80]),
             (O.wkv_layer(2, 16), False, 30, [31, 79], [])]
    for x, (layer, cut_right, at, seen, unseen) in enumerate(cases):
        cfg = O.make_config(32, 40, [layer])
        W = O.random_weights(cfg, seed=x)
        for name in W:
            if name.endswith("w0"):
                W[name] = torch.full_like(W[name], -7.0)                   # decays that remember
            if name.endswith("A_log"):
                W[name] = torch.full_like(W[name], -6.0)
            if cut_right and name.endswith("right.out"):
                W[name] = torch.zeros_like(W[name])                        # attention alone
        model = build(tmp_path, cfg, W, device, dtype, name=f"m{x}")
        a = _tokens(150, 40, 5)
        b = list(a)
        b[at] = (b[at] + 17) % 40
        gen = RaggedGenerator(model, None, 192)
        out = []
        for toks in (a, b):
            cache = fresh_cache(gen, 1, 192)
            parts = [gen.step([(0, 0, toks[:100], list(range(100)))], cache)]
            parts += [gen.step([(0, p, toks[p:p + 1], [0])], cache) for p in range(100, 150)]
            out.append(torch.cat(parts, 0).cpu())
        d = (out[0] - out[1]).abs().max(-1).values
        assert float(d[:at].max()) == 0.0 if at else True
        for p in seen:
            assert float(d[p]) > 0, (x, p)
        for p in unseen:
            assert float(d[p]) == 0.0, (x, p)
        assert_rows(out[0], O.forward(cfg, W, a)[0], dtype, x)


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


def test_checkpoint_names_round_trip_and_bad_configs(tmp_path):
    from llm_in_practise_b200.models.nedesun import NedesunConfig, nedesun_state_dict
    cfg = VARIANTS["mixed"]()
    W = O.random_weights(cfg, seed=16)
    model = build(tmp_path, cfg, W, "cpu", torch.bfloat16)
    sd = nedesun_state_dict(model)
    assert set(sd) == set(W)
    for k in W:
        assert sd[k].shape == W[k].shape, k
        assert torch.equal(sd[k].to(torch.bfloat16).cpu(), W[k]), k
    c = NedesunConfig.from_dict(cfg)
    assert [s.mixer.v_from for s in c.layers if s.type == "attention"] == [None, None, 2]
    assert model.kv_layout() == [(2, 16, 24), (0, 0, 0), (2, 24, 16), (0, 0, 0), (1, 32, 32), (2, 16, 16)]
    assert model.state_layout() == [[(4, 16, 24), (2, 160)], [(3, 16, 16), (1, 64)], [], [(2, 8, 8), (1, 64)], [], []]
    with pytest.raises(ValueError):                                # a tensor without a place
        build(tmp_path, cfg, {**W, "l0.mix.left.extra": W["final.norm"]}, "cpu", torch.float32, name="extra")
    for breakage in (lambda b: b["layers"][0].__setitem__("type", "recurrent"), lambda b: b["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 3),
                     lambda b: b["layers"][0]["mixer"]["right"].__setitem__("kv_heads", 3), lambda b: b["layers"][2]["mixer"]["rot"].__setitem__("dims", 26),
                     lambda b: b["layers"][2]["mixer"]["rot"].__setitem__("dims", 7), lambda b: b["layers"][5]["mixer"].__setitem__("vdim", 24),
                     lambda b: b["layers"][0]["mlp"].__setitem__("kind", "glu")):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            NedesunConfig.from_dict(bad)


def test_options_that_do_not_go_together_are_refused():
    from llm_in_practise_b200.ops.linear_scan import linear_scan
    from llm_in_practise_b200.ops.multimap_attention import multimap_attention
    z = torch.zeros
    with pytest.raises(ValueError):                                # chunks and a window
        multimap_attention(z(1, 8), z(2, 1, 64, 8), z(2, 1, 64, 8), z(1, 1, dtype=torch.int32), _i32([0], "cpu"), _i32([0], "cpu"), 1, 1, 1, 8, 8,
                           1.0, window=4, chunk=8)
    with pytest.raises(ValueError):                                # a bonus belongs to the channel scan
        linear_scan(z(1, 8), z(1, 8), z(1, 8), z(1, 1, 8, 8), _i32([0], "cpu"), _i32([0], "cpu"), None, 1, 1, 1, 8, 8, "decay", decay=z(1), u=z(1, 8))


def test_replay_builds_every_kernel_source_the_model_calls():
    """A fresh checkout compiles only the sources listed for the design: each entry point the model's ops call is in one."""
    import inspect
    import re
    from llm_in_practise_b200 import _build
    from llm_in_practise_b200.ops import elementwise, gemm, linear_scan, multimap_attention, norm
    from llm_in_practise_b200.recipes.trace import NATIVE_SOURCES
    have = set()
    for stem in NATIVE_SOURCES["Nedesun"]:
        have |= set(re.findall(r"B200_API int (b200_\w+)\(", (_build.CSRC / f"{stem}.cu").read_text()))
    called = set()
    for fn in (elementwise.embedding_pos, elementwise.act_glu, gemm.gemm, gemm.gemv16, gemm.linear_exact, gemm.linear_each,
               linear_scan.linear_scan, linear_scan.lowrank_decay, linear_scan.scan_readout, linear_scan.short_conv, linear_scan._conv_tail,
               linear_scan.delta_gates, linear_scan.token_shift, multimap_attention.qkv_store, multimap_attention.multimap_attention,
               norm.sandwich_norm):
        called |= set(re.findall(r"\b(b200_\w+)\b", inspect.getsource(fn)))
    called -= {"b200_gemm_args"}
    assert len(called) > 12 and called <= have, sorted(called - have)
