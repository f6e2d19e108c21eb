"""Multi-map attention over the paged KV cache (``csrc/multimap_attn.cu``): every head has M attention maps (own query and
key rows, one set of values), the mask is a sliding window that also keeps the first tokens of the sequence, and two maps
can be combined differentially:

    token at position p sees key j of its own cache row  iff  j <= p and (p - j < window or j < keep_first)
    a_m = softmax_j(scale q_{h,m} . k_{g,m,j}) V_g                     g = h // (H / G)
    o   = a_0 - lambda a_1;   o <- o / sqrt(mean(o^2) + eps) * post     (``combine``; M = 2)

Keys live in ``cache_k`` [blocks, G * M, block, D] (after norm and rotation), values in ``cache_v`` [blocks, G, block, Dv];
Dv need not equal D. A layer may attend over the pools another layer filled (shared K/V). ``qkv_store`` (``qknorm_rope_store``)
is the step in front: bias, per-row RMS norm with a weight, split-half rotary on the first ``rot`` dims, values mixed with
another layer's, the page writes. One-map attention has options: capped scores, chunks instead of a window, a sink per head,
a sigmoid gate per token and head. Beside
``ops.paged_attention`` (one map, values sized like keys, sinks) and ``ops.latent_attention`` (latent rows), which serve
the same ragged step (the reference reaches it through vLLM, LLM_on_Kubernetes/Inference_Platfrom/README.md:1504-1509).
"""
from __future__ import annotations

import ctypes
import os
from typing import Optional

import torch

from . import _native as nv
from .linear_scan import _conv_tail, short_conv

vp, i32, i64, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
_MMA_MAX = 128                                                     # largest key / value row of the tensor-core kernel
_CONV_TAPS = 5                                                     # taps of the fused convolution + norm + store
_SPLIT_KEYS = int(os.environ.get("B200_PAGED_SPLIT_KEYS", "512"))  # keys per range of a small batch with many visible keys


class _AttnOpts(ctypes.Structure):
    _fields_ = [("sink", vp), ("gate", vp), ("ld_gate", i64), ("softcap", f32), ("chunk", i32)]


def qkv_store(proj: torch.Tensor, bias: Optional[torch.Tensor], wq: Optional[torch.Tensor], wk: Optional[torch.Tensor],
              rope, pos: torch.Tensor, slot: torch.Tensor, cache_k: torch.Tensor, cache_v: torch.Tensor, table: torch.Tensor, H: int,
              G: int, D: int, Dv: int, rot: int, eps: float, dtype: torch.dtype, v_first: Optional[torch.Tensor] = None,
              v_lambda: Optional[torch.Tensor] = None) -> torch.Tensor:
    """What stands in front of one-map attention. ``proj`` [T, >= (H + G) D + G Dv] = q | k | v rows (fp32 or bf16) gets ``bias``
    (fp32 [(H + G) D + G Dv] or None); q and k rows are RMS-normed with ``wq`` / ``wk`` (fp32 [D]; None: not normed) and their
    first ``rot`` dims turned by the token's position (``rope`` = (cos, sin) fp32 [max_pos, rot / 2], split-half pairs; None
    with ``rot`` 0). ``v_first``: the value pool of an earlier layer that already holds these tokens; then
    v <- (1 - lambda) v + lambda v_first with ``v_lambda`` fp32 [1]. Returns q [T, H * D] in ``dtype``; keys and values are
    written at (slot, pos) of the pools."""
    T = proj.shape[0]
    q_out = torch.empty(T, H * D, dtype=dtype, device=proj.device)
    BS = cache_k.shape[2]
    if v_first is not None and (v_first.shape != cache_v.shape or v_lambda is None):
        raise ValueError("qkv_store: values can only be mixed with a pool of the same shape, by a lambda")
    if nv.use_native(proj):
        if proj.stride(1) != 1 or cache_k.dtype != dtype:
            raise ValueError("qkv_store: rows with a contiguous last dim, q in the cache dtype")
        cos, sin = rope if rope is not None else (None, None)
        fn = nv.proto("b200_qkv_store", [vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, vp, vp, vp, i32, i32, i32, i32, i32, i32,
                                         i32, i32, f32, i32, i32, i32, vp])
        nv.check(fn(nv.ptr(proj), proj.stride(0), nv.ptr(bias), nv.ptr(wq), nv.ptr(wk), nv.ptr(cos), nv.ptr(sin), nv.ptr(pos), nv.ptr(slot),
                    nv.ptr(table), table.shape[1], nv.ptr(q_out), nv.ptr(cache_k), nv.ptr(cache_v), nv.ptr(v_first), nv.ptr(v_lambda), T, H,
                    G, 1, D, Dv, rot, BS, float(eps), 1, nv.dtype_code(proj.dtype), nv.dtype_code(dtype), nv.stream()), "qkv_store")
        nv.count_launch()
        return q_out
    nq, nk = H * D, G * D
    x = proj[:, :nq + nk + G * Dv].float()
    if bias is not None:
        x = x + bias.float()
    pl, sl = pos.long(), slot.long()
    hr = rot // 2

    def prep(y, w):
        if w is not None:
            y = y * torch.rsqrt((y * y).mean(-1, keepdim=True) + eps) * w.float()
        if rot:
            c, s = rope[0][pl][:, None, :], rope[1][pl][:, None, :]
            a, b = y[..., :hr], y[..., hr:rot]
            y = torch.cat([a * c - b * s, b * c + a * s, y[..., rot:]], -1)
        return y

    q_out.copy_(prep(x[:, :nq].view(T, H, D), wq).reshape(T, nq).to(dtype))
    blk, off = table[sl, pl // BS].long(), pl % BS
    v = x[:, nq + nk:].reshape(T, G, Dv)
    if v_first is not None:
        lam = float(v_lambda)
        v = (1.0 - lam) * v + lam * v_first[blk, :, off].float()
    cache_k[blk, :, off] = prep(x[:, nq:nq + nk].view(T, G, D), wk).to(cache_k.dtype)
    cache_v[blk, :, off] = v.to(cache_v.dtype)
    return q_out


def qknorm_rope_store(proj: torch.Tensor, wq: torch.Tensor, wk: Optional[torch.Tensor], cos: torch.Tensor, sin: torch.Tensor,
                      pos: torch.Tensor, slot: torch.Tensor, cache_k: Optional[torch.Tensor], cache_v: Optional[torch.Tensor],
                      table: torch.Tensor, H: int, G: int, M: int, D: int, Dv: int, rot: int, eps: float,
                      dtype: torch.dtype) -> torch.Tensor:
    """``proj`` fp32 [T, >= (H M + G M) D + G Dv] = q rows | k rows | v rows (the k / v part is absent when ``cache_k`` is
    None: a layer that attends over another layer's pools). Returns q [T, H * M * D] in ``dtype``, normed and rotated; the
    token's keys and values are written at (slot, pos) of the pools."""
    T = proj.shape[0]
    has_kv = cache_k is not None
    q_out = torch.empty(T, H * M * D, dtype=dtype, device=proj.device)
    if nv.use_native(proj):
        if proj.dtype != torch.float32 or proj.stride(1) != 1:
            raise ValueError("qknorm_rope_store: fp32 rows with a contiguous last dim")
        BS = cache_k.shape[2] if has_kv else 1
        fn = nv.proto("b200_qknorm_rope_store", [vp, i64, vp, vp, vp, vp, vp, vp, vp, i32, vp, vp, vp, i32, i32, i32, i32, i32, i32,
                                                 i32, i32, f32, i32, i32, vp])
        nv.check(fn(nv.ptr(proj), proj.stride(0), nv.ptr(wq), nv.ptr(wk), nv.ptr(cos), nv.ptr(sin), nv.ptr(pos), nv.ptr(slot),
                    nv.ptr(table), table.shape[1], nv.ptr(q_out), nv.ptr(cache_k), nv.ptr(cache_v), T, H, G, M, D, Dv, rot, BS,
                    float(eps), int(has_kv), nv.dtype_code(dtype), nv.stream()), "qknorm_rope_store")
        nv.count_launch()
        return q_out
    pl, sl = pos.long(), slot.long()
    hr = rot // 2
    c, s = (cos[pl][:, None, :], sin[pl][:, None, :]) if rot else (None, None)

    def prep(x, w):
        x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * w.float()
        y = x.clone()
        if rot:
            u, v = x[..., :hr], x[..., hr:rot]
            y[..., :hr] = u * c - v * s
            y[..., hr:rot] = v * c + u * s
        return y

    nq, nk = H * M * D, G * M * D
    q_out.copy_(prep(proj[:, :nq].float().view(T, H * M, D), wq).reshape(T, nq).to(dtype))
    if has_kv:
        BS = cache_k.shape[2]
        blk = table[sl, pl // BS].long()
        off = pl % BS
        cache_k[blk, :, off] = prep(proj[:, nq:nq + nk].float().view(T, G * M, D), wk).to(cache_k.dtype)
        cache_v[blk, :, off] = proj[:, nq + nk:nq + nk + G * Dv].view(T, G, Dv).to(cache_v.dtype)
    return q_out


def conv_qknorm_store(proj: torch.Tensor, bias: Optional[torch.Tensor], w: torch.Tensor, tail: torch.Tensor, pos: torch.Tensor,
                      slot: torch.Tensor, runs: Optional[torch.Tensor], n_runs: int, cache_k: torch.Tensor, cache_v: torch.Tensor,
                      table: torch.Tensor, H: int, G: int, D: int, Dv: int, eps: float, dtype: torch.dtype, temp=(0.0, 1.0),
                      norm_qk: bool = True, norm_v: bool = False) -> torch.Tensor:
    """Convolved queries, keys and values of one-map attention. ``proj`` [T, >= (H + G) D + G Dv] = q | k | v rows (fp32 or bf16)
    gets ``bias`` (fp32 [C] or None), then every channel a causal convolution over time (``w`` fp32 [C, taps]; the last
    taps - 1 biased inputs of a sequence wait in ``tail`` fp32 [rows, taps - 1, C], advanced here); then each q and k row is
    divided by its root mean square (``norm_qk``), each v row too (``norm_v``), and q at position p is multiplied by
    1 + c ln(floor((p + 1) / every) + 1) with ``temp`` = (c, every). Returns q [T, H * D] in ``dtype``; keys and values are
    written at (slot, pos) of the pools."""
    T = proj.shape[0]
    C, taps = w.shape
    q_out = torch.empty(T, H * D, dtype=dtype, device=proj.device)
    BS = cache_k.shape[2]
    if nv.use_native(proj):
        if proj.dtype not in (torch.float32, torch.bfloat16) or proj.stride(1) != 1 or cache_k.dtype != dtype:
            raise ValueError("conv_qknorm_store: fp32 or bf16 rows with a contiguous last dim, q in the cache dtype")
        if taps > _CONV_TAPS:                            # more taps than the fused kernel holds in registers: convolve first
            u = proj[:, :C].float() + bias if bias is not None else proj[:, :C]
            proj, bias, taps = short_conv(u, w, tail, pos, slot, runs, n_runs, act=False, out_dtype=proj.dtype), None, 1
            w = torch.ones(C, 1, dtype=torch.float32, device=proj.device)
        fn = nv.proto("b200_conv_qknorm_store", [vp, i64, vp, vp, vp, vp, vp, vp, i32, vp, vp, vp, i32, i32, i32, i32, i32, i32, i32, f32,
                                                 f32, f32, i32, i32, i32, i32, vp])
        nv.check(fn(nv.ptr(proj), proj.stride(0), nv.ptr(bias), nv.ptr(w), nv.ptr(tail), nv.ptr(pos), nv.ptr(slot), nv.ptr(table),
                    table.shape[1], nv.ptr(q_out), nv.ptr(cache_k), nv.ptr(cache_v), T, H, G, D, Dv, taps, BS, float(eps),
                    float(temp[0]), float(temp[1]), int(norm_qk), int(norm_v), nv.dtype_code(proj.dtype), nv.dtype_code(dtype),
                    nv.stream()), "conv_qknorm_store")
        nv.count_launch()
        if taps > 1:
            _conv_tail(proj, bias, tail, runs, pos, slot, n_runs if runs is not None else T, C, taps)
        return q_out
    u = proj[:, :C].float()
    if bias is not None:
        u = u + bias.float()
    y = short_conv(u, w, tail, pos, slot, runs, n_runs, act=False)
    nq, nk = H * D, G * D
    unit = lambda x: x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps)                       # noqa: E731
    q, k, v = y[:, :nq].view(T, H, D), y[:, nq:nq + nk].view(T, G, D), y[:, nq + nk:].reshape(T, G, Dv)
    if norm_qk:
        q, k = unit(q), unit(k)
    if norm_v:
        v = unit(v)
    t = 1.0 + temp[0] * torch.log(torch.floor((pos.double() + 1) / temp[1]) + 1).float()
    q_out.copy_((q * t.view(T, 1, 1)).reshape(T, nq).to(dtype))
    pl, sl = pos.long(), slot.long()
    blk, off = table[sl, pl // BS].long(), pl % BS
    cache_k[blk, :, off] = k.to(cache_k.dtype)
    cache_v[blk, :, off] = v.to(cache_v.dtype)
    return q_out


def multimap_attention(q: torch.Tensor, cache_k: torch.Tensor, cache_v: torch.Tensor, table: torch.Tensor, pos: torch.Tensor,
                       slot: torch.Tensor, H: int, G: int, M: int, D: int, Dv: int, scale: float, window: int = 0,
                       keep_first: int = 0, combine: bool = False, lam: float = 0.0, post: float = 1.0, eps: float = 0.0,
                       pieces=None, max_pos: int = 0, out: Optional[torch.Tensor] = None, sink: Optional[torch.Tensor] = None,
                       softcap: float = 0.0, chunk: int = 0, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Context [T, H * Dv] (q's dtype) of ``q`` [T, H * M * D] over the pools; see the module docstring for the mask and the
    combination; ``post`` multiplies the result with and without it. ``out``: where to write it (rows may be strided). ``pieces`` (``inference.ragged.Pieces``): bf16 steps with a run of 8 or more tokens go through the tensor-core
    kernel; everything else (fp32, decode batches, sizes it is not built for) through the per-token kernels. ``max_pos``: an upper
    bound of ``pos`` known on the host (0 = unknown), used to cut the keys of a small batch into ranges.

    One-map options: ``softcap`` > 0: scores become c tanh(s / c); ``chunk`` > 0 (without a window): position p sees only keys
    j <= p with j // chunk == p // chunk; ``sink`` fp32 [H]: exp(sink_h) joins the softmax's denominator; ``gate`` fp32 [T, H]
    (rows may be strided): head h's output times sigmoid(gate[t, h])."""
    T = q.shape[0]
    BS = cache_k.shape[2]
    if out is None:
        out = torch.empty(T, H * Dv, dtype=q.dtype, device=q.device)
    options = sink is not None or gate is not None or softcap or chunk
    if options and (M != 1 or (chunk and window > 0)):
        raise ValueError("multimap_attention: options are for one map, chunks for attention without a window")
    if nv.use_native(q):
        opts = None
        if options:
            if (sink is not None and (sink.dtype != torch.float32 or sink.numel() != H)) or \
                    (gate is not None and (gate.dtype != torch.float32 or gate.stride(1) != 1)):
                raise ValueError("multimap_attention: sink fp32 [H], gate fp32 rows with a contiguous last dim")
            opts = ctypes.byref(_AttnOpts(nv.ptr(sink), nv.ptr(gate), gate.stride(0) if gate is not None else 0, float(softcap), int(chunk)))
        if cache_k.dtype != q.dtype or not q.is_contiguous():
            raise ValueError("multimap_attention: contiguous q in the cache dtype")
        if out.dtype != q.dtype or out.stride(1) != 1:
            raise ValueError("multimap_attention: out in q's dtype with a contiguous last dim")
        if (pieces is not None and pieces.longest >= 8 and q.dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0
                and max(D, Dv) <= _MMA_MAX and scale > 0
                and BS & (BS - 1) == 0 and out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0 and os.environ.get("B200_PAGED_MMA", "1") != "0"):
            fn = nv.proto("b200_multimap_attn_mma_ex", [vp, vp, vp, vp, i32, vp, i32, vp, i64, i32, i32, i32, i32, i32, i32, f32, i32, i32, i32,
                                                        f32, f32, f32, vp, i32, vp])
            nv.check(fn(nv.ptr(q), nv.ptr(cache_k), nv.ptr(cache_v), nv.ptr(pieces.tiles), pieces.n_tiles, nv.ptr(table),
                        table.shape[1], nv.ptr(out), out.stride(0), H, G, M, D, Dv, BS, float(scale), int(window), int(keep_first), int(combine),
                        float(lam), float(post), float(eps), opts, nv.dtype_code(q.dtype), nv.stream()), "multimap_attn_mma")
            nv.count_launch()
            return out
        # few tokens with many visible keys (a small decode batch with a wide window or none): cut the keys into ranges
        seen = max_pos + 1 if max_pos > 0 else 0
        if window > 0:
            seen = min(seen, window + max(keep_first, 0))
        if chunk > 0:
            seen = min(seen, chunk)
        nsplit = 1
        if seen > 2 * _SPLIT_KEYS and T * G < 296:
            nsplit = min(32, -(-seen // _SPLIT_KEYS), max(1, 592 // (T * G)))
        part = torch.empty(T * H * M * nsplit * (Dv + 2), dtype=torch.float32, device=q.device) if nsplit * M > 1 else None
        fn = nv.proto("b200_multimap_attn_ex", [vp, vp, vp, vp, vp, vp, i32, vp, i64, vp, i32, i32, i32, i32, i32, i32, i32, f32, i32, i32,
                                                i32, i32, f32, f32, f32, vp, i32, vp])
        nv.check(fn(nv.ptr(q), nv.ptr(cache_k), nv.ptr(cache_v), nv.ptr(pos), nv.ptr(slot), nv.ptr(table), table.shape[1],
                    nv.ptr(out), out.stride(0), nv.ptr(part), T, H, G, M, D, Dv, BS, float(scale), int(window), int(keep_first), nsplit, int(combine),
                    float(lam), float(post), float(eps), opts, nv.dtype_code(q.dtype), nv.stream()), "multimap_attn")
        nv.count_launch(2 if nsplit * M > 1 else 1)
        return out
    rep = H // G
    pl, sl = pos.tolist(), slot.tolist()
    qf = q.float().view(T, H, M, D)
    for t in range(T):
        p = pl[t]
        lo = max(0, p + 1 - window) if window > 0 else (p // chunk * chunk if chunk else 0)
        idx = list(range(min(max(keep_first, 0), lo) if window > 0 else 0)) + list(range(lo, p + 1))
        it = torch.tensor(idx, dtype=torch.long, device=q.device)
        blk = table[sl[t], it // BS].long()
        off = it % BS
        k = cache_k[blk, :, off].float().view(len(idx), G, M, D).repeat_interleave(rep, 1)        # [n, H, M, D]
        v = cache_v[blk, :, off].float().repeat_interleave(rep, 1)                                 # [n, H, Dv]
        sc = torch.einsum("hmd,nhmd->hmn", qf[t], k) * scale
        if softcap:
            sc = softcap * torch.tanh(sc / softcap)
        if sink is not None:
            sc = torch.cat([sc, sink.float().view(H, 1, 1)], -1)
        a = torch.einsum("hmn,nhe->hme", sc.softmax(-1)[:, :, :len(idx)], v)
        o = a[:, 0] - lam * a[:, 1] if M == 2 else a[:, 0]
        if combine:
            o = o * torch.rsqrt((o * o).mean(-1, keepdim=True) + eps)
        o = o * post
        if gate is not None:
            o = o * torch.sigmoid(gate[t].float())[:, None]
        out[t] = o.reshape(H * Dv).to(q.dtype)
    return out
