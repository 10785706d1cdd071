"""Pepulix on the GPU against the plain statement: each mechanism alone (with weights or inputs made so that a fault
shows), then whole models under every way of cutting the work, then generation through the engine's own entry point
and the replay program."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pepulix_models as pm
import plain_pepulix as plain
import scenarios
from helpers import make_ctx, make_runner, rel_err
from neurogrid_b200.engine import StepEntry

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 1e-4, torch.bfloat16: 3e-2}
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def ops():
    from neurogrid_b200.csrc import ops as o
    return o


def _close(got, want, dtype):
    """float32: within the tolerance everywhere.  bfloat16: rows are judged one by one against the largest logit: nine
    in ten within twice the tolerance of a single part and the median within it."""
    if dtype == torch.float32:
        return rel_err(got, want) < TOL[dtype]
    d = (got.double().cpu() - want.double().cpu()).abs().amax(-1) / want.double().cpu().abs().max()
    return float(torch.quantile(d, 0.9)) < 2 * TOL[dtype] and float(d.median()) < TOL[dtype]


def _x(shape, dtype, seed=1, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (scale * torch.randn(*shape, generator=g)).to(torch.bfloat16).to(dtype).to(DEV)


def _pages(n_tokens, ps, shapes, dtype, seed=0):
    """Pages in a scrambled order with stale content, one tensor per (heads, columns), and the block table of one request."""
    n_pages = -(-n_tokens // ps) + 3
    g = torch.Generator().manual_seed(seed)
    order = torch.randperm(n_pages, generator=g)[: -(-n_tokens // ps)]
    table = torch.full((1, n_pages), -1, dtype=torch.int32)
    table[0, : len(order)] = order.to(torch.int32)
    return [(5 * torch.randn(n_pages, h, ps, c, generator=g)).to(dtype).to(DEV) for h, c in shapes], table.to(DEV)


def _places(table, pos, ps):
    return table[0, (pos // ps).to(DEV)].long(), (pos % ps).to(DEV)


# ------------------------------------------------------------------------------------------ sigmoid attention: preparation
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_k,dim,vdim,rot,extra", [(4, 2, 20, 12, 16, 0), (3, 1, 9, 7, 0, 5), (6, 2, 64, 48, 64, 6), (2, 2, 128, 256, 32, 0), (8, 1, 7, 1, 4, 8)])
@pytest.mark.parametrize("T", [45, 300])
@pytest.mark.parametrize("mode", ["none", "source", "mix"])
def test_preparation_norms_rotates_and_mixes(dtype, n_q, n_k, dim, vdim, rot, extra, T, mode):
    """q and k rotated, then over their root mean square; values over theirs, mixed with another layer's; what is cached is
    the mixed value; columns behind the values are left alone."""
    ps, before, eps = 8, 61, 1e-3
    qkv = _x((T, (n_q + n_k) * dim + n_k * vdim + extra), dtype, scale=0.3)
    (kp, vp), table = _pages(before + T, ps, [(n_k, dim), (n_k, vdim)], dtype)
    ctx = make_ctx([T], [before], [0], dtype=dtype)
    rc = dict(base=100.0, dims=rot)
    inv = (plain.pair_frequencies(rc)[0]).float().to(DEV) if rot else None
    g = torch.Generator().manual_seed(9)
    other = torch.randn(T, n_k * vdim, generator=g)
    first = {"none": None, "source": torch.full((T, n_k * vdim), float("nan"), device=DEV), "mix": other.to(DEV)}[mode]
    q = torch.empty(T, n_q * dim, dtype=dtype, device=DEV)
    ops().qkv_prep(qkv, q, None, None, inv, kp, vp, table, ctx.positions, ctx.row_entry, n_q, n_k, n_k, dim, vdim, eps, ctx.status,
                   half_pairing=True, unit_norm=True, v_norm=True, v_first=first, v_lambda=0.3 if mode == "mix" else None)
    x = qkv.double().cpu()
    pad = torch.zeros(before, x.shape[1], dtype=F64)
    full = torch.cat([pad, x])                                       # the oracle's positions count from the first row
    qd = plain.rms_div(plain.rotate(full[:, : n_q * dim].view(-1, n_q, dim), rc if rot else None, False), eps)[before:]
    kd = plain.rms_div(plain.rotate(full[:, n_q * dim:(n_q + n_k) * dim].view(-1, n_k, dim), rc if rot else None, False), eps)[before:]
    vd = plain.rms_div(x[:, (n_q + n_k) * dim:(n_q + n_k) * dim + n_k * vdim].view(T, n_k, vdim), eps)
    if mode == "source":
        assert rel_err(first, vd.reshape(T, -1)) < 1e-5                # float32, not what the cache rounds
    if mode == "mix":
        vd = plain.mix_values(vd, other.double().view(T, n_k, vdim), 0.3)
    pg, at = _places(table, torch.arange(before, before + T), ps)
    assert rel_err(q, qd.reshape(T, -1)) < TOL[dtype]
    assert rel_err(kp[pg, :, at], kd) < TOL[dtype] and rel_err(vp[pg, :, at], vd) < TOL[dtype]
    assert int(ctx.status.item()) == 0


# ------------------------------------------------------------------------------------------ sigmoid attention: the cores
def _attend(kind, q, kp, vp, table, ctx, H, scale, bias, gate, n_splits=1, out_scale=0.6):
    """Every head times ``out_scale`` in the kernel; taken out again here.  The output is a block of columns."""
    n, vdim = q.shape[0], vp.shape[3]
    wide = torch.full((n, H * vdim + 8), 3.0, dtype=q.dtype, device=DEV)
    out = wide[:, 4:4 + H * vdim]
    args = (H, 1, None, 0, scale, 0.0, 0.0, False, 1.0, 1e-6)
    kw = dict(out_scale=out_scale, sigmoid=True, score_bias=bias, gate=gate)
    if kind == "rows":
        partial = torch.full((max(1, ops().mapped_attention_partial_floats(n, H, 1, vdim, n_splits)),), float("nan"), device=DEV) if n_splits > 1 else None
        ops().mapped_attention(q, kp, vp, table, ctx.positions, ctx.row_entry, out, *args, n_splits, partial, **kw)
    elif kind == "tiles":
        ops().mapped_attention_mma(q, kp, vp, table, ctx.cu_q, ctx.ctx_before, out, ctx.n_entries, ctx.max_q, *args, **kw)
    else:
        partial = torch.full((n * H * n_splits * (vdim + 2),), float("nan"), device=DEV)
        ops().mapped_attention_group(q, kp, vp, table, ctx.cu_q, ctx.ctx_before, ctx.row_entry, out, partial, ctx.n_entries, *args,
                                     n_splits, **kw)
    assert float(wide[:, :4].min()) == float(wide[:, -4:].max()) == 3.0
    return out.double() / out_scale


def _plain_attend(q, k, v, H, scale, bias, gate, rows):
    T, G, _ = k.shape
    out = torch.zeros(len(rows), H, v.shape[-1], dtype=F64)
    for h in range(H):
        w = plain.sigmoid_weights(q[:, h].double(), k[:, h // (H // G)].double(), scale, float(bias[h]))
        out[:, h] = (w @ v[:, h // (H // G)].double())[rows]
    if gate is not None:
        out = out * torch.sigmoid(gate.double().cpu())[:, :, None]
    return out.reshape(len(rows), -1)


KINDS = [("rows", torch.float32), ("rows", torch.bfloat16), ("tiles", torch.bfloat16), ("group", torch.bfloat16)]


@pytest.mark.parametrize("kind,dtype", KINDS)
@pytest.mark.parametrize("case", ["far key", "low scores", "high scores"])
@pytest.mark.parametrize("H,G,dim,vdim", [(8, 2, 64, 48), (3, 3, 128, 128), (16, 1, 16, 16)])
def test_attention_without_softmax(kind, dtype, case, H, G, dim, vdim):
    """"far key": one key far back (a page's first slot) weighs nearly one and the hundreds of others nearly nothing; "low
    scores": every weight is small and nothing normalises them; "high scores": every weight is nearly one, so the sum
    grows with the position.  The gate's logits are columns of a wider buffer."""
    T, ps = 420, 16
    g = torch.Generator().manual_seed(4)
    u = torch.randn(dim, generator=g)
    u = u / u.norm()
    q, k, v = 0.3 * torch.randn(T, H, dim, generator=g), 0.3 * torch.randn(T, G, dim, generator=g), torch.randn(T, G, vdim, generator=g)
    bias = torch.linspace(-6.0, -4.0, H)
    if case == "far key":
        q, k[48] = q + 3.0 * u, k[48] + 10.0 * u
        v[48] *= 4.0
    elif case == "low scores":
        q, k = q + 3.0 * u, k - 1.0 * u
    else:
        q, k, bias = q + 3.0 * u, k + 3.0 * u, bias + 6.0
    rnd = lambda t: t.to(torch.bfloat16).to(dtype)
    q, k, v = rnd(q), rnd(k), rnd(v)
    (kp, vp), table = _pages(T, ps, [(G, dim), (G, vdim)], dtype)
    pg, at = _places(table, torch.arange(T), ps)
    kp[pg, :, at], vp[pg, :, at] = k.to(DEV), v.to(DEV)
    scale = 0.4
    gates = _x((T, H + 5), dtype, seed=8, scale=2.0)[:, 3:3 + H]
    rows = list(range(T)) if kind != "group" else [0, 1, 15, 16, 47, 48, 49, 63, 64, 200, 300, 418, 419]
    want = _plain_attend(q, k, v, H, scale, bias, gates[rows], rows)
    bias = bias.to(DEV)
    if kind == "group":
        ctx = make_ctx([1] * len(rows), rows, list(range(len(rows))), dtype=dtype)
        tables = table.expand(len(rows), -1).contiguous()
        for n_splits in (1, 3, 16):
            got = _attend(kind, q[rows].reshape(len(rows), -1).to(DEV), kp, vp, tables, ctx, H, scale, bias, gates[rows].contiguous(), n_splits)
            assert rel_err(got, want) < TOL[dtype]
        return
    got, start = [], 0
    for n in (47, 2, 1, 100, T - 150):
        ctx = make_ctx([n], [start], [0], dtype=dtype)
        for n_splits in (1, 3) if kind == "rows" and n < 32 else (1,):
            part = _attend(kind, q[start:start + n].reshape(n, -1).to(DEV), kp, vp, table, ctx, H, scale, bias, gates[start:start + n], n_splits)
            assert rel_err(part, want[start:start + n]) < TOL[dtype] * (1 if dtype == torch.float32 else 1.5)
        got.append(part)
        start += n
    assert rel_err(torch.cat(got), want) < TOL[dtype]
    if case == "far key":                                # rows behind the key see it, rows before do not
        assert float(want[48].abs().max()) > 5 * float(want[47].abs().max())
    if case == "low scores":                             # a softmax would give the first row its value whole
        assert float(want[0].abs().max()) < 0.2 * float(v[0].double().abs().max())


@pytest.mark.parametrize("kind,dtype", KINDS)
def test_sigmoid_attention_batch_of_unequal_entries(kind, dtype):
    """Entries of several lengths and contexts in one launch, on pages of one pool in a scrambled order; no bias, no gate."""
    H, G, dim, vdim, ps, scale = 6, 2, 32, 16, 8, 0.5
    lens, before = ([1, 1, 1, 1], [0, 7, 130, 64]) if kind == "group" else ([1, 37, 2, 70], [5, 0, 40, 63])
    g = torch.Generator().manual_seed(2)
    seqs = [[(torch.randn(b + n, h, c, generator=g)).to(torch.bfloat16).to(dtype) for h, c in ((H, dim), (G, dim), (G, vdim))]
            for n, b in zip(lens, before)]
    per = -(-max(n + b for n, b in zip(lens, before)) // ps)
    kp, vp = (torch.full((per * 4, G, ps, c), 50.0, dtype=dtype, device=DEV) for c in (dim, vdim))
    table = torch.full((4, per + 2), -1, dtype=torch.int32, device=DEV)
    order = torch.randperm(per * 4, generator=g).tolist()
    want = []
    for e, (n, b) in enumerate(zip(lens, before)):
        table[e, : -(-(n + b) // ps)] = torch.tensor([order.pop() for _ in range(-(-(n + b) // ps))], dtype=torch.int32, device=DEV)
        q, k, v = seqs[e]
        pos = torch.arange(n + b)
        pg, at = table[e, (pos // ps).to(DEV)].long(), (pos % ps).to(DEV)
        kp[pg, :, at], vp[pg, :, at] = k.to(DEV), v.to(DEV)
        want.append(_plain_attend(q, k, v, H, scale, torch.zeros(H), None, list(range(b, n + b))))
    ctx = make_ctx(lens, before, [0, 1, 2, 3], dtype=dtype)
    q = torch.cat([s[0][b:].reshape(n, -1) for s, n, b in zip(seqs, lens, before)]).to(DEV)
    assert rel_err(_attend(kind, q, kp, vp, table, ctx, H, scale, None, None, 2 if kind == "group" else 1), torch.cat(want)) < TOL[dtype]


def test_sigmoid_kernels_refuse_what_they_do_not_do():
    q, (kp, vp), ctx = torch.zeros(2, 32, device=DEV), [torch.zeros(1, 1, 8, 16, device=DEV)] * 2, make_ctx([2], [0], [0], dtype=torch.float32)
    table, out, one = torch.zeros(1, 1, dtype=torch.int32, device=DEV), torch.zeros(2, 32, device=DEV), torch.zeros(2, device=DEV)
    args = (q, kp, vp, table, ctx.positions, ctx.row_entry, out, 2, 1, None, 0, 1.0, 0.0, 0.0, False, 1.0, 1e-6)
    for bad in (dict(sigmoid=True, sinks=one), dict(score_bias=one), dict(gate=torch.zeros(2, 3, device=DEV))):
        with pytest.raises(ops().KernelError):
            ops().mapped_attention(*args, **bad)


# ------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,rank,rot", [(3, 20, 8), (8, 48, 16), (2, 130, 2), (1, 7, 30)])
def test_latent_rows_and_queries_with_a_rescaled_rotation(dtype, H, rank, rot):
    """Cosines and sines of the rotated part carry a factor (the part grows, the latent does not); there is no gate."""
    T, before, ps, rq, eps = 40, 29, 8, 24, 1e-3
    rp = -(-(rank + rot) // 16) * 16
    rc = dict(base=500.0, dims=rot, scaling=dict(factor=5.0, original=64, fast=8.0, slow=0.5))
    f, mag = plain.pair_frequencies(rc)
    inv = f.float().to(DEV)
    x = _x((T, rq + rank + rot), dtype, scale=1.5)
    wq, wkv = (1 + 0.2 * torch.randn(rq)).to(DEV), (1 + 0.2 * torch.randn(rank)).to(DEV)
    (pages,), table = _pages(before + T, ps, [(1, rp)], dtype)
    ctx = make_ctx([T], [before], [0], dtype=dtype)
    cq = torch.empty(T, rq, dtype=dtype, device=DEV)
    ops().latent_prep(x, wq, wkv, cq, pages, None, table, ctx.positions, ctx.row_entry, 0, eps, ctx.status, rot=rot, inv_freq=inv,
                      rot_mag=mag)
    xd = x.double().cpu()
    turn = lambda t: plain.rotate(torch.cat([torch.zeros(before, *t.shape[1:], dtype=F64), t]), rc, True)[before:]
    assert rel_err(cq, plain.rms_norm(xd[:, :rq], wq.double().cpu(), eps)) < TOL[dtype]
    pg, at = _places(table, torch.arange(before, before + T), ps)
    row = pages[pg, 0, at]
    key = turn(xd[:, None, rq + rank:])[:, 0]
    assert rel_err(row[:, :rank], plain.rms_norm(xd[:, rq:rq + rank], wkv.double().cpu(), eps)) < TOL[dtype]
    assert rel_err(row[:, rank:rank + rot], key) < TOL[dtype]
    assert rp == rank + rot or float(row[:, rank + rot:].abs().max()) == 0
    assert rel_err(key.norm(dim=-1), mag * xd[:, rq + rank:].norm(dim=-1)) < 1e-9 and mag > 1.1
    q = _x((T, H * rp), dtype, seed=3)
    want = q.double().cpu().view(T, H, rp).clone()
    want[:, :, rank:rank + rot] = turn(want[:, :, rank:rank + rot])
    ops().latent_rope_q(q, ctx.positions, ctx.row_entry, inv, H, rank, rot_mag=mag)
    assert rel_err(q, want.reshape(T, -1)) < TOL[dtype] and int(ctx.status.item()) == 0


@pytest.mark.parametrize("H,rp", [(8, 64), (12, 32), (5, 256), (16, 160), (1, 96)])
@pytest.mark.parametrize("window", [None, 70])
@pytest.mark.parametrize("n_splits", [2, 7, 32])
def test_latent_core_in_runs_of_keys(H, rp, window, n_splits):
    """Rows of several requests, their keys cut into runs (more runs than some rows have tiles), with one key that towers
    over hundreds, padding rows among them; a gate per head."""
    ps, T = 16, 700
    g = torch.Generator().manual_seed(3)
    n_pages = 2 * (-(-T // ps)) + 4
    pages = (0.5 * torch.randn(n_pages, 1, ps, rp, generator=g)).to(torch.bfloat16)
    order = torch.randperm(n_pages, generator=g)[: 2 * (-(-T // ps))].view(2, -1)
    table = torch.cat([order, torch.full((2, 2), -1)], 1).to(torch.int32)
    pos = [0, 31, 32, 33, 699, 5, 300, 64, 640]
    entry = [0, 1, 0, 1, 0, -1, 1, 0, 1]
    q = (0.5 * torch.randn(len(pos), H * rp, generator=g)).to(torch.bfloat16)
    far = pages[table[0, 640 // ps].long(), 0, 640 % ps]
    q[4] = (4.0 * far / far.float().norm()).repeat(H).to(torch.bfloat16) + 0.1 * q[4]      # row 4 looks for key 640 of request 0
    pages[table[0, 640 // ps].long(), 0, 640 % ps] = 4 * far
    gate = torch.rand(len(pos), H, generator=g)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32)
    want = torch.zeros(len(pos), H, rp, dtype=F64)
    for r, (p, e) in enumerate(zip(pos, entry)):
        if e < 0:
            continue
        keys = torch.arange(max(0, p - window + 1) if window else 0, p + 1)
        C = pages[table[e, keys // ps].long(), 0, keys % ps].double()
        w = torch.softmax(q[r].double().view(H, rp) @ C.T * 0.4, -1)
        want[r] = (w @ C) * gate[r].double()[:, None]
    out = torch.full((len(pos), H * rp), 7.0, dtype=torch.bfloat16, device=DEV)
    partial = torch.full((ops().latent_core_partial_floats(len(pos), H, rp, n_splits),), float("nan"), device=DEV)
    ops().latent_core_mma(q.to(DEV), pages.to(DEV), table.to(DEV), i32(pos).to(DEV), i32(entry).to(DEV), gate.to(DEV), out, H, window,
                          0.4, n_splits, partial)
    assert rel_err(out, want.reshape(len(pos), -1)) < 1e-2 and float(out[5].abs().max()) == 0


def _part(spec, cls, dtype, seed, gains=None):
    part = cls(spec, dtype=dtype, device=DEV)
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, d in part.tensors().items():
        t = torch.randn(d.shape, generator=g)
        t = 1 + 0.2 * t if d.init == "norm" else t if d.init == "bias" else 1.3 * t / d.shape[-1] ** 0.5
        w[name] = ((gains or {}).get(name, 1.0) * t).to(torch.bfloat16).float()
    part.bind({k: v.to(DEV) for k, v in w.items()})
    return part, {k: v.double() for k, v in w.items()}


def _paged_view(part, n_tokens, ps, dtype, entries=1):
    from neurogrid_b200.parts import PagedView
    need = part.cache_need()
    shapes = [(need.n_kv_heads, need.head_dim)] + ([need.value_shape()] if need.values else [])
    pages, table = _pages(n_tokens, ps, shapes, dtype)
    return PagedView(pages[0], pages[1] if need.values else None, table)


def _whole(y):
    return y.double().sum(0) if y.dim() == 3 else y.double()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,rank,rot,scaling", [(5, 40, 16, True), (12, 24, 8, True), (3, 20, 8, False), (66, 30, 2, True), (2, 520, 6, True), (4, 31, 0, False)])
def test_latent_attention_part(dtype, H, rank, rot, scaling):
    """Whole, then decoded token by token, in every core (tensor-core tiles with two rows or one, rows, the plain kernel): a
    key far back stands out."""
    from neurogrid_b200.config.specs import LatentAttentionSpec, RopeSpec
    from neurogrid_b200.parts.latent_attention import LatentAttention
    T, Hd, d, dv, ps = 150, 64, 12, 10, 8
    sc = dict(factor=6.0, original=64, fast=8.0, slow=0.5) if scaling else None
    pos = RopeSpec(rot, 1000.0, "adjacent", rotary_dims=rot, yarn=tuple(sc.values()) if sc else None) if rot else None
    spec = LatentAttentionSpec(Hd, H, d, dv, 32, rank, 0.5, 1e-5, rope_dim=rot, position=pos, gate="none")
    part, w = _part(spec, LatentAttention, dtype, 3, {"uq": 1.5})
    x = _x((T, Hd), dtype, seed=5)
    x[20] = 3.0 * x[140] + x[20]                                     # token 140's query meets a key like its own
    m = dict(heads=H, dim=d, rot_dim=rot, vdim=dv, kv_rank=rank, scale=0.5)
    if rot:
        m["rot"] = dict(base=1000.0, dims=rot, **({"scaling": sc} if sc else {}))
    want = plain.latent_attention(x.double().cpu(), w, "", m, 1e-5)
    view = _paged_view(part, T, ps, dtype)
    got, at = [], 0
    for n in (90, 2, 1, 40) + (1,) * 17:
        ctx = make_ctx([n], [at], [0], dtype=dtype)
        got.append(_whole(part.forward(x[at:at + n].contiguous(), ctx, view)).clone())
        at += n
    assert at == T and rel_err(torch.cat(got), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,rot", [(8, 2, 32, 48, 24), (3, 1, 9, 7, 4), (34, 2, 16, 16, 16), (4, 4, 128, 64, 0)])
def test_attention_part_mixes_with_an_earlier_layer(dtype, H, G, d, dv, rot):
    """Two layers on one input, the second's values mixed with the first's: whole, portions, single tokens."""
    from neurogrid_b200.config.specs import MappedAttentionSpec, NoPositionSpec, RopeSpec
    from neurogrid_b200.parts.mapped_attention import MappedAttention
    T, Hd, ps = 120, 64, 8
    kw = dict(hidden=Hd, n_heads=H, n_kv_heads=G, key_dim=d, value_dim=dv, softmax_scale=6.0 / d, qk_norm=True, norm_weight=False,
              eps=1e-5, bias=True, o_bias=False, weights="sigmoid", score_bias=True, value_norm=True, head_gate=True,
              position=RopeSpec(d + d % 2, 300.0, "half", rotary_dims=rot) if rot else NoPositionSpec())
    parts = [_part(MappedAttentionSpec(value_mix=m, **kw), MappedAttention, dtype, s) for m, s in (("source", 3), ("mix", 4))]
    x = _x((T, Hd), dtype, seed=5)
    m = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=6.0 / d)
    if rot:
        m["rot"] = dict(base=300.0, dims=rot)
    h = x.double().cpu()
    y1, v1 = plain.attention(h, parts[0][1], "", m, 1e-5)
    y2, v2 = plain.attention(h, parts[1][1], "", m, 1e-5, v1)
    assert rel_err(plain.attention(h, parts[1][1], "", m, 1e-5)[0], y2) > 0.05            # the mixing shows
    views = [_paged_view(p, T, ps, dtype) for p, _ in parts]
    got, at = ([], []), 0
    for n in (70, 2, 1, 40) + (1,) * 7:
        ctx = make_ctx([n], [at], [0], dtype=dtype)
        for i, (part, _) in enumerate(parts):
            got[i].append(_whole(part.forward(x[at:at + n].contiguous(), ctx, views[i])).clone())
        at += n
    assert at == T
    for i, want in enumerate((y1, y2)):
        assert rel_err(torch.cat(got[i]), want) < TOL[dtype], i
    pg, s = _places(views[1].table, torch.arange(T), ps)
    assert rel_err(views[1].v_pages[pg, :, s], v2) < TOL[dtype]


# ------------------------------------------------------------------------------------------ feed-forward and the copies
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 64, 90])
@pytest.mark.parametrize("H,I", [(64, 88), (72, 200), (50, 30)])
def test_dense_feed_forward_with_biases(dtype, rows, H, I):
    from neurogrid_b200.config.specs import SwiGLUSpec
    from neurogrid_b200.parts.swiglu import SwiGLU
    spec = SwiGLUSpec(H, I, names=dict(gate="gate", up="up", down="down"), weight_suffix="", bias=True)
    part, w = _part(spec, SwiGLU, dtype, 2)
    x = _x((rows, H), dtype, seed=9)
    want = plain.dense_ff(x.double().cpu(), w, "")
    assert rel_err(_whole(part.forward(x, make_ctx([rows], [0], [0], dtype=dtype))), want) < TOL[dtype]
    part.defer_bias = True                                           # a block adds the last bias itself
    y = _whole(part.forward(x, make_ctx([rows], [0], [0], dtype=dtype))).cpu() + part.out_bias.double().cpu()
    assert rel_err(y, want) < TOL[dtype] and rel_err(part.out_bias, w["down.b"]) == 0


@pytest.mark.parametrize("M,K,I", [(1, 64, 40), (8, 192, 328), (33, 72, 56), (64, 128, 200)])
def test_biases_in_the_products_epilogue(M, K, I):
    """The epilogue rounds where the product and a pass over it would."""
    x, w = _x((M, K), torch.bfloat16), _x((2 * I, K), torch.bfloat16, seed=2, scale=2.0 / K ** 0.5)
    b = _x((2 * I,), torch.bfloat16, seed=3)
    fused, gu, out = (torch.empty(M, c, dtype=torch.bfloat16, device=DEV) for c in (I, 2 * I, I))
    ops().gemm_swiglu_sm100(x, w, fused, bias=b)
    ops().gemm_sm100(x, w, b, gu)
    ops().swiglu(gu, out)
    y = x.double() @ w.double().t() + b.double()
    assert rel_err(fused, out) < 1e-2 and rel_err(fused, plain.silu(y[:, :I]) * y[:, I:]) < TOL[torch.bfloat16] / 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,n_id,top,groups,keep,shared", [(14, 6, 3, 1, 1, False), (3, 5, 4, 1, 1, False), (1, 1, 1, 1, 1, False), (6, 2, 2, 4, 2, True), (40, 24, 8, 1, 1, False)])
def test_router_with_identity_experts(dtype, E, n_id, top, groups, keep, shared):
    rows, H = 37, 72
    x = _x((rows, H), dtype)
    wr, corr = _x((E + n_id, H), torch.float32, seed=2, scale=0.3), _x((E + n_id,), torch.float32, seed=3, scale=0.5 / (E + n_id))
    wsg = _x((H,), torch.float32, seed=4, scale=0.2) if shared else None
    out = torch.full((rows, E + shared + 1), float("nan"), device=DEV)
    ops().moe_router_sigmoid(x, wr, corr, wsg, out, top, groups, keep, softmax_scores=True, n_identity=n_id)
    if groups == 1:
        w = {"router": wr.double().cpu(), "correction": corr.double().cpu()}
        want = plain.routing_weights(x.double().cpu(), w, "", {"top": top})
        want = torch.cat([want[:, :E], want[:, E:].sum(-1, keepdim=True)], 1)
        assert float((want[:, -1] > 0).double().mean()) > 0.1 and float((want[:, -1] == 0).double().mean()) > (0.05 if E > 3 else -1)
        assert rel_err(out, want) < 1e-5
    else:
        import kernel_refs as refs
        want = torch.empty(rows, E + shared + 1)
        refs.moe_router_sigmoid(x.cpu(), wr.cpu(), corr.cpu(), wsg.cpu(), want, top, groups, keep, softmax_scores=True, n_identity=n_id)
        assert rel_err(out, want) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [5, 90])
@pytest.mark.parametrize("how", ["alone", "deferred", "into the stream"])
def test_moe_part_with_identity_experts(dtype, rows, how):
    from neurogrid_b200.config.specs import MoESpec
    from neurogrid_b200.parts.moe import MoE
    H, mlp = 64, dict(router=dict(experts=5, identity=3, top=3))
    part, w = _part(MoESpec(H, 5, 3, 24, scoring="softmax_all", correction=True, identity=3), MoE, dtype, 2, {"correction": 0.1})
    part.defer_identity = how == "deferred"
    x = _x((rows, H), dtype, seed=9)
    want = plain.moe_ff(x.double().cpu(), w, "", mlp)
    ctx = make_ctx([rows], [0], [0], dtype=dtype)
    h0 = torch.randn(rows, H, device=DEV)
    ctx.residual = h0.clone() if how == "into the stream" else None
    y = part.forward(x, ctx)
    y = _whole(y).cpu() if y is not None else (ctx.residual.double() - h0.double()).cpu()
    if how == "deferred":
        z, wts = part.identity
        assert rel_err(y, want) > 0.05
        y = y + (wts.double()[:, None] * z.double()).cpu()
    assert rel_err(y, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,H,n,parts", [(1, 40, 5, 0), (3, 56, 9, 2), (4, 2056, 3, 0), (5, 50, 4, 3), (3, 1024, 70, 1), (16, 31, 2, 0)])
def test_identity_experts_ride_in_the_update_of_the_copies(dtype, S, H, n, parts):
    g = torch.Generator().manual_seed(S)
    X = torch.randn(n, S * H, generator=g)
    mix, ow, iw = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    nw = torch.randn(H, generator=g)
    delta = torch.randn(parts, n, H, generator=g) if parts else _x((n, H), dtype, seed=3).cpu()
    z, wts = _x((n, H), dtype, seed=4), torch.rand(n, 7, generator=g).to(DEV)
    Xd, out, total = X.to(DEV), torch.empty(n, H, dtype=dtype, device=DEV), torch.empty(n, H, device=DEV)
    dev = {k: v.to(DEV) for k, v in dict(delta=delta, mix=mix, out_w=ow).items()}
    ops().hc_step(Xd, S, out=out, eps=1e-5, in_w=iw.to(DEV), norm_w=nw.to(DEV), sum_out=total, identity=(z, wts[:, 5]), **dev)
    y = (delta.double().sum(0) if parts else delta.double()) + wts[:, 5].double().cpu()[:, None] * z.double().cpu()
    xs = plain.connect(list(X.double().view(n, S, H).unbind(1)), y, mix.double(), ow.double())
    assert rel_err(Xd, torch.stack(xs, 1).reshape(n, -1)) < 1e-6 and rel_err(total, sum(xs)) < 1e-5
    assert rel_err(out, plain.rms_norm(sum(iw[s].double() * xs[s] for s in range(S)), nw.double(), 1e-5)) < TOL[dtype]


# ------------------------------------------------------------------------------------------ whole models
LENS = {"A": [1, 9, 40, 131, 64, 23, 77], "B": [3, 50, 97, 30, 64], "B0": [2, 41, 90], "C": [2, 17, 150, 33, 210],
        "D": [1, 45, 20, 100]}


def _folder(name, dtype):
    return name if dtype == torch.float32 else name + "_calm"


def _replay(runner, steps):
    got = []
    for s in steps:
        lg = runner.step([StepEntry(e["id"], e["tokens"], e["want"]) for e in s["entries"]])
        got.append(lg.clone())
        for r in s["end"]:
            runner.finish(r)
    runner.check_status()
    runner.cache.check()
    return scenarios.collect(steps, lambda i: got[i])


@pytest.fixture(scope="module")
def plain_logits(pepulix_dirs):
    out = {}
    for name in LENS:
        for folder in (name, name + "_calm"):
            cfg, w = pm.load_plain(pepulix_dirs[folder])
            reqs = scenarios.make_requests(LENS[name], cfg["vocab"], seed=7)
            out[folder] = (reqs, {r: plain.forward(cfg, w, t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("name", ["A", "B0", "C", "D"])
def test_stream_after_every_layer(pepulix_dirs, name):
    """float32, layer by layer: the sum of the stream's copies after every layer."""
    cfg, w = pm.load_plain(pepulix_dirs[name])
    toks = scenarios.make_requests([37], cfg["vocab"], seed=1)["r0"]
    _, after = plain.forward(cfg, w, toks, return_layers=True)
    runner = make_runner(pepulix_dirs[name], dtype=torch.float32, device="cuda", page_size=8, num_pages=16)
    seen = []
    model = runner.model
    run_entries, S = model.run_entries, cfg.get("streams") or 1

    def spy(ctx, caches, entries, h, pending):
        for e in entries:                              # one layer at a time; the update not yet written is folded in for the record
            pending = run_entries(ctx, caches, [e], h, pending)
            X = h.double().view(h.shape[0], S, -1)
            y = _whole(pending.y)
            if pending.bias is not None:
                y = y + pending.bias.double()
            if pending.identity is not None:
                y = y + pending.identity[1].double()[:, None] * pending.identity[0].double()
            X = torch.einsum("st,nsh->nth", pending.mix.double().view(S, S), X) + pending.out_w.double()[None, :, None] * y[:, None, :]
            seen.append(X.sum(1)[: len(toks)].cpu())
        return pending

    model.run_entries = spy
    runner.step([StepEntry("x", toks, [len(toks) - 1])])
    assert len(seen) == len(after) == len(cfg["layers"])
    for i, s in enumerate(seen):
        assert rel_err(s, after[i]) < 1e-4, i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "B0", "C", "D"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
def test_cuts_against_plain(pepulix_dirs, plain_logits, name, dtype, cut):
    reqs, want = plain_logits[_folder(name, dtype)]
    ps = pm.PAGE_SIZE[name]
    cap = 256 if cut == "mixed" else 512                     # tokens; mixed: pages and slots are used again
    runner = make_runner(pepulix_dirs[_folder(name, dtype)], dtype=dtype, device="cuda", page_size=ps, num_pages=cap // ps,
                         max_requests=4, max_seq_len=cap)
    steps = {"whole": scenarios.whole, "tail_decode": scenarios.tail_decode, "portions": scenarios.portions,
             "mixed": lambda r: scenarios.mixed(r, cap, round_to=ps)}[cut](reqs)
    got = _replay(runner, steps)
    allg, allw = torch.cat([got[r] for r in reqs]), torch.cat([want[r] for r in reqs])
    assert allg.shape == allw.shape
    assert _close(allg, allw, dtype), rel_err(allg, allw)
    if dtype == torch.float32:
        for r in reqs:
            assert rel_err(got[r], want[r]) < TOL[dtype], (r, rel_err(got[r], want[r]))
    assert all(f == cap // ps for f in runner.cache.pages_free()) and runner.cache.slots_free() == 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_first_tokens_and_long_decode(pepulix_dirs, name, dtype):
    """The first tokens one by one (empty states, a lone key), then decoding across many pages with graphs replayed."""
    folder = pepulix_dirs[_folder(name, dtype)]
    cfg, w = pm.load_plain(folder)
    toks = scenarios.make_requests([230], cfg["vocab"], seed=11)["r0"]
    want = plain.forward(cfg, w, toks)
    runner = make_runner(folder, dtype=dtype, device="cuda", page_size=8, num_pages=32, max_seq_len=256)
    got = torch.cat([runner.step([StepEntry("x", [t], [0])]).clone() for t in toks])
    runner.check_status()
    assert _close(got, want, dtype), rel_err(got, want)
    if dtype == torch.float32:
        assert rel_err(got[:14], want[:14]) < TOL[dtype]
    assert runner.graph_replays > 100 and runner.cache.pages_held("x") == [29] * len(runner.cache.pools)


@pytest.mark.parametrize("name", ["A", "C"])
def test_float32_cuts_agree_closely(pepulix_dirs, name):
    cfg, _ = pm.load_plain(pepulix_dirs[name])
    reqs = scenarios.make_requests([120], cfg["vocab"], seed=3)
    runner = make_runner(pepulix_dirs[name], dtype=torch.float32, device="cuda", num_pages=64, page_size=8)
    a = _replay(runner, scenarios.whole(reqs))["r0"]
    b = _replay(runner, scenarios.portions(reqs))["r0"]
    c = _replay(runner, scenarios.tail_decode(reqs))["r0"]
    assert rel_err(a, b) < 2e-5 and rel_err(a, c) < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_batch_of_unequal_requests_equals_each_alone(pepulix_dirs, name, dtype):
    folder = pepulix_dirs[_folder(name, dtype)]
    cfg, _ = pm.load_plain(folder)
    reqs = scenarios.make_requests([5, 70, 2, 33], cfg["vocab"], seed=5)
    runner = make_runner(folder, dtype=dtype, device="cuda", num_pages=64, page_size=8)
    alone = _replay(runner, scenarios.whole(reqs))
    lg = runner.step([StepEntry(r, t, list(range(len(t)))) for r, t in reqs.items()])
    at = 0
    for r, t in reqs.items():
        if dtype == torch.float32:
            assert rel_err(lg[at:at + len(t)], alone[r]) < 2e-5
        else:
            assert _close(lg[at:at + len(t)], alone[r], dtype)
        at += len(t)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_of_a_whole_model_shows_after_every_cut(dtype, tmp_path):
    """One token whose key one head of an attention layer looks for, 600 tokens back across pages and portions: the logits
    that read it agree with the oracle, and change when that token does."""
    cfg = {"architecture": "Pepulix", "vocab": 40, "width": 48, "streams": 2, "norm": {"eps": 1e-5},
           "layers": [{"type": "attention", "mlp": None, "mixer": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.5}}]}
    w = pm.draw_weights(cfg, 3)
    w["l0.mix.pb"] = torch.full((4,), -12.0, dtype=torch.bfloat16)          # only a key much like the query weighs
    w["l0.mix.k"] = w["l0.mix.q"][:64].clone()
    w["l0.mix.k.b"], w["l0.mix.q.b"] = torch.zeros(64, dtype=torch.bfloat16), torch.zeros(128, dtype=torch.bfloat16)
    folder = pm.write_model(cfg, 3, str(tmp_path / "m"), weights=w)
    cfg, wd = pm.load_plain(folder)
    toks = [t % 20 for t in scenarios.make_requests([700], 20, seed=4)["r0"]]
    toks[33], toks[640] = 31, 31                                            # the only two of their kind
    want = plain.forward(cfg, wd, toks)
    other = plain.forward(cfg, wd, toks[:33] + [32] + toks[34:])
    assert rel_err(other[640], want[640]) > 0.05 and rel_err(other[641:], want[641:]) < 0.01
    runner = make_runner(folder, dtype=dtype, device="cuda", page_size=8, num_pages=96, max_tokens_per_step=1024, max_seq_len=768)
    for cuts in ([700], [30, 4, 2, 600, 4] + [1] * 60, [33, 1, 2] + [64] * 9 + [2] * 44):
        got, at = [], 0
        for n in cuts:
            got.append(runner.step([StepEntry("x", toks[at:at + n], list(range(n)))]).clone())
            at += n
        runner.finish("x")
        assert at == 700 and rel_err(torch.cat(got), want) < TOL[dtype]


def test_greedy_generation_through_the_engine(pepulix_dirs):
    """Engine.generate (scheduler, portions, decode graphs, device sampler) against greedy decoding with the oracle."""
    from neurogrid_b200 import Engine
    cfg, w = pm.load_plain(pepulix_dirs["C"])
    prompts = list(scenarios.make_requests([12, 30, 5], cfg["vocab"], seed=9).values())
    eng = Engine(pepulix_dirs["C"], dtype="float32", max_seq_len=128, page_size=8, max_requests=2,
                 max_tokens_per_step=32, chunk_size=16)
    outs = eng.generate(prompts, max_new_tokens=24, ignore_eos=True)
    for p, o in zip(prompts, outs):
        lg = plain.forward(cfg, w, list(p) + o)                      # one pass: the oracle is causal
        assert len(o) == 24
        for j, tok in enumerate(o):
            row = lg[len(p) - 1 + j]
            top2 = torch.topk(row, 2).values
            assert tok == int(torch.argmax(row)) or float(top2[0] - top2[1]) < 1e-4 * float(row.abs().max())
    assert eng.stats()["slots_free"] == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(pepulix_dirs, tmp_path, dtype):
    folder = pepulix_dirs["A" if dtype == "float32" else "C_calm"]
    cfg, w = pm.load_plain(folder)
    V = cfg["vocab"]
    reqs = scenarios.make_requests([9, 70, 33, 120, 41], V, seed=5)
    cap = 256
    steps = scenarios.number(scenarios.portions(reqs) + scenarios.mixed(reqs, cap, round_to=64))
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder,
                           "--dtype", dtype, "--out", str(out), "--max-tokens", str(cap)],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = scenarios.collect(steps, lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V)))
    want = {r: plain.forward(cfg, w, t) for r, t in reqs.items()}
    assert _close(torch.cat([got[r] for r in reqs]), torch.cat([torch.cat([want[r], want[r]]) for r in reqs]),
                  torch.float32 if dtype == "float32" else torch.bfloat16)
