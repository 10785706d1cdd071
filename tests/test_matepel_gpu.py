"""Matepel on the GPU against the plain statement: each mechanism alone (with weights or inputs made so that a fault
shows), then whole models under every way of cutting the work, then generation through the engine's own entry point
and the replay program."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs as refs
import matepel_models as mm
import plain_matepel as plain
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


def _pages(n_tokens, ps, n_k, dim, dtype, seed=0):
    """Key and value pages in a scrambled order with stale content, and the block table of one request."""
    n_pages = -(-n_tokens // ps) + 3
    g = torch.Generator().manual_seed(seed)
    order = torch.randperm(n_pages, generator=g)[: -(-n_tokens // ps)]
    table = torch.full((1, n_pages), -1, dtype=torch.int32)
    table[0, : len(order)] = order.to(torch.int32)
    kp, vp = ((5 * torch.randn(n_pages, n_k, ps, dim, generator=g)).to(dtype).to(DEV) for _ in range(2))
    return kp, vp, table.to(DEV)


# ------------------------------------------------------------------------------------------ embedding, stream, gate
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [50, 72, 1024, 2056])
def test_embedding_and_its_norm(dtype, H):
    V, n = 37, 9
    table, w = _x((V, H), dtype, scale=0.02), (1 + 0.3 * torch.randn(H)).to(DEV)
    tok = torch.randint(0, V, (n,), dtype=torch.int32)
    out, status = torch.empty(n, H, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    ops().embed_norm(table, tok.to(DEV), w, out, status, 1e-3, 1.3)
    want = plain.rms_norm(table.double().cpu()[tok.long()] * 1.3, w.double().cpu(), 1e-3)
    assert rel_err(out, want) < 1e-6 and int(status) == 0
    tok[2] = V                                                       # outside the table: zeros and a status bit
    ops().embed_norm(table, tok.to(DEV), w, out, status, 1e-3, 1.3)
    assert int(status) == 1 and float(out[2].abs().max()) == 0 and rel_err(out[3:], want[3:]) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,H,n,parts", [(1, 40, 5, 0), (3, 56, 9, 2), (4, 2056, 3, 0), (5, 50, 4, 3), (16, 31, 2, 0)])
def test_bias_of_a_sublayer_rides_in_the_update_of_the_copies(dtype, S, H, n, parts):
    g = torch.Generator().manual_seed(S)
    X = torch.randn(n, S * H, generator=g)
    mix, ow, iw = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    nw, bias = torch.randn(H, generator=g), torch.randn(H, generator=g)
    delta = torch.randn(parts, n, H, generator=g) if parts else _x((n, H), dtype, seed=3).cpu()
    kw = dict(delta=delta, mix=mix, out_w=ow, in_w=iw, norm_w=nw, bias=bias)
    Xd, out = X.to(DEV), torch.empty(n, H, dtype=dtype, device=DEV)
    ops().hc_step(Xd, S, out=out, eps=1e-5, **{k: v.to(DEV) for k, v in kw.items()})
    y = (delta.double().sum(0) if parts else delta.double()) + bias.double()
    xs = plain.connect(list(X.double().view(n, S, H).unbind(1)), y, mix.double(), ow.double())
    assert rel_err(Xd, torch.stack(xs, 1).reshape(n, -1)) < 1e-6
    u = sum(iw[s].double() * xs[s] for s in range(S))
    assert rel_err(out, plain.rms_norm(u, nw.double(), 1e-5)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("I,limit", [(40, 0.9), (36, 2.0), (7, 0.3), (264, 1.3)])
def test_clamped_gate(dtype, I, limit):
    n = 13
    gu = _x((n, 2 * I), dtype, scale=1.5)
    wide = torch.zeros(n, I + 16, dtype=dtype, device=DEV)
    ops().swiglu(gu, wide[:, 8:8 + I], "clamped_glu", limit, 1.702)
    x = gu.double().cpu()
    g, u = x[:, :I].clamp(max=limit), x[:, I:].clamp(-limit, limit)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    assert rel_err(wide[:, 8:8 + I], want) < TOL[dtype] / 3 and float(wide[:, :8].abs().max()) == 0
    for hit in ((x[:, :I] > limit), (x[:, I:] > limit), (x[:, I:] < -limit)):        # every clamp bites
        assert hit.any()


@pytest.mark.parametrize("M,K,I", [(1, 64, 40), (8, 192, 328), (33, 72, 56), (64, 128, 200)])
def test_clamped_gate_in_the_products_epilogue(M, K, I):
    x, w = _x((M, K), torch.bfloat16), _x((2 * I, K), torch.bfloat16, seed=2, scale=2.0 / K ** 0.5)
    fused, gu, out = (torch.empty(M, c, dtype=torch.bfloat16, device=DEV) for c in (I, 2 * I, I))
    ops().gemm_swiglu_sm100(x, w, fused, activation="clamped_glu", limit=1.1, alpha=1.702)
    ops().gemm_sm100(x, w, None, gu)
    ops().swiglu(gu, out, "clamped_glu", 1.1, 1.702)
    assert torch.equal(fused, out)
    y = x.double() @ w.double().t()
    g, u = y[:, :I].clamp(max=1.1), y[:, I:].clamp(-1.1, 1.1)
    assert rel_err(fused, g * torch.sigmoid(1.702 * g) * (u + 1)) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [5, 90])
def test_dense_feed_forward(dtype, rows):
    from neurogrid_b200.config.specs import SwiGLUSpec
    from neurogrid_b200.parts.swiglu import SwiGLU
    H, I = 64, 88
    spec = SwiGLUSpec(H, I, names=dict(gate="gate", up="up", down="down"), weight_suffix="", activation="clamped_glu", limit=0.8)
    part = SwiGLU(spec, dtype=dtype, device=DEV)
    w = {k: _x(d.shape, torch.float32, seed=i, scale=1.5 / d.shape[1] ** 0.5) for i, (k, d) in enumerate(part.tensors().items())}
    part.bind(w)
    x = _x((rows, H), dtype, seed=9)
    ctx = make_ctx([rows], [0], [0], dtype=dtype)
    y = part.forward(x, ctx)
    y = y.double().sum(0) if y.dim() == 3 else y
    want = plain.clamped_ff(x.double().cpu(), {k: v.double().cpu() for k, v in w.items()}, "", {"limit": 0.8})
    assert rel_err(y, want) < TOL[dtype]


# ------------------------------------------------------------------------------------------ left: attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_k,dim,rot,extra", [(4, 2, 20, 16, 0), (3, 1, 10, 10, 6), (2, 2, 64, 32, 0), (6, 3, 7, 4, 3), (8, 2, 128, 0, 0)])
@pytest.mark.parametrize("T", [45, 300])
def test_keys_as_values_and_a_rescaled_rotation(dtype, n_q, n_k, dim, rot, extra, T):
    """Values are the keys as projected; cosine and sine carry a factor, so the rotated coordinates grow and the rest do
    not; columns behind the keys are left alone."""
    from neurogrid_b200.config.specs import RopeSpec
    from neurogrid_b200.parts.position import Rope
    ps, before = 8, 61
    qkv = _x((T, (n_q + n_k) * dim + extra), dtype, scale=2.0)
    cfg = dict(base=1000.0, dims=rot, scaling=dict(factor=6.0, original=64, fast=8.0, slow=0.5)) if rot else None
    inv, mag = None, 1.0
    if rot:
        pa = Rope(RopeSpec(dim + dim % 2, 1000.0, "half", rotary_dims=rot, yarn=(6.0, 64, 8.0, 0.5)), device=DEV).kernel_args()
        inv, mag = pa.inv_freq, pa.magnitude
    kp, vp, table = _pages(before + T, ps, n_k, dim, dtype)
    ctx = make_ctx([T], [before], [0], dtype=dtype)
    q = torch.empty(T, n_q * dim, dtype=dtype, device=DEV)
    ops().qkv_prep(qkv, q, None, None, inv, kp, vp, table, ctx.positions, ctx.row_entry, n_q, n_k, n_k, dim, dim, 1e-5,
                   ctx.status, half_pairing=True, v_is_k=True, rot_mag=mag)
    x = qkv.double().cpu()
    pos = torch.arange(before, before + T)
    k = x[:, n_q * dim:(n_q + n_k) * dim].view(T, n_k, dim)
    qd, kd = plain.rotate(x[:, : n_q * dim].view(T, n_q, dim), pos, cfg), plain.rotate(k, pos, cfg)
    assert rel_err(q, qd.reshape(T, -1)) < TOL[dtype]
    pg, at = table[0, (pos // ps).to(DEV)].long(), (pos % ps).to(DEV)
    assert rel_err(kp[pg, :, at].reshape(T, -1), kd.reshape(T, -1)) < TOL[dtype]
    assert torch.equal(vp[pg, :, at].double().cpu(), k)
    if rot:
        assert rel_err(plain.rotate(k, pos, {k2: v for k2, v in cfg.items() if k2 != "scaling"}), kd) > 0.1
    assert int(ctx.status.item()) == 0


def _attend(kind, q, kp, vp, table, ctx, H, scale, sinks, n_splits=1, out_scale=0.6):
    """Every head times ``out_scale`` in the kernel; taken out again here."""
    n, vdim = q.shape[0], vp.shape[3]
    out = torch.empty(n, H * vdim, dtype=q.dtype, device=DEV)
    args = (H, 1, None, 0, scale, 0.0, 0.0, False, 1.0, 1e-6)
    if kind == "rows":
        partial = torch.empty(max(1, ops().mapped_attention_partial_floats(n, H, 1, vdim, n_splits)), device=DEV) if n_splits > 1 else None
        ops().mapped_attention(q, kp, vp, table, ctx.positions, ctx.row_entry, out, *args, n_splits, partial, sinks=sinks,
                               out_scale=out_scale)
    elif kind == "tiles":
        ops().mapped_attention_mma(q, kp, vp, table, ctx.cu_q, ctx.ctx_before, out, ctx.n_entries, ctx.max_q, *args, sinks=sinks,
                                   out_scale=out_scale)
    else:
        partial = torch.empty(n * H * n_splits * (vdim + 2), device=DEV)
        ops().mapped_attention_group(q, kp, vp, table, ctx.cu_q, ctx.ctx_before, ctx.row_entry, out, partial, ctx.n_entries, *args,
                                     n_splits, sinks=sinks, out_scale=out_scale)
    return out.double() / out_scale


def _plain_attend(q, k, v, H, scale, rows):
    """Softmax with one more 1 in the denominator, float64, for the given query positions."""
    T, G, d = k.shape
    out = torch.zeros(len(rows), H, v.shape[-1], dtype=F64)
    for i, t in enumerate(rows):
        for h in range(H):
            g = h // (H // G)
            e = torch.exp((k[:t + 1, g].double() @ q[t, h].double()) * scale)
            out[i, h] = (e[:, None] * v[:t + 1, g].double()).sum(0) / (1 + e.sum())
    return out.reshape(len(rows), -1)


@pytest.mark.parametrize("kind,dtype", [("rows", torch.float32), ("rows", torch.bfloat16), ("tiles", torch.bfloat16), ("group", torch.bfloat16)])
@pytest.mark.parametrize("case", ["far key", "low scores"])
def test_attention_with_one_more_in_the_denominator(kind, dtype, case):
    """"far key": one key far back (on a page's first slot) towers over hundreds of others; "low scores": every score is
    well below the sink's 0, so the sink takes most of the weight, also at the first token, which sees it beside itself."""
    T, H, G, dim, ps = 420, 8, 2, 64, 16
    g = torch.Generator().manual_seed(4)
    u = torch.randn(dim, generator=g)
    u = u / u.norm()
    q, k, v = 0.3 * torch.randn(T, H, dim, generator=g), 0.3 * torch.randn(T, G, dim, generator=g), torch.randn(T, G, dim, generator=g)
    if case == "far key":
        q, k[48] = q + 3.0 * u, k[48] + 5.0 * u
    else:
        q, k = q + 3.0 * u, k - 3.0 * u
    rnd = lambda t: t.to(torch.bfloat16).to(dtype)
    q, k, v = rnd(q), rnd(k), rnd(v)
    kp, vp, table = _pages(T, ps, G, dim, dtype)
    pos = torch.arange(T)
    pg, at = table[0, (pos // ps).to(DEV)].long(), (pos % ps).to(DEV)
    kp[pg, :, at], vp[pg, :, at] = k.to(DEV), v.to(DEV)
    sinks = torch.zeros(H, device=DEV)
    scale = 0.4
    rows = list(range(T)) if kind != "group" else [0, 1, 15, 16, 47, 48, 49, 63, 64, 200, 300, 418, 419]
    want = _plain_attend(q, k, v, H, scale, rows)
    if kind == "group":
        ctx = make_ctx([1] * len(rows), rows, list(range(len(rows))), dtype=dtype)
        tables = table.expand(len(rows), -1).contiguous()
        for n_splits in (1, 3):
            got = _attend(kind, q[rows].reshape(len(rows), -1).to(DEV), kp, vp, tables, ctx, H, scale, sinks, n_splits)
            assert rel_err(got, want) < TOL[dtype]
        return
    got, start = [], 0
    for n in (47, 2, 1, T - 50):
        ctx = make_ctx([n], [start], [0], dtype=dtype)
        got.append(_attend(kind, q[start:start + n].reshape(n, -1).to(DEV), kp, vp, table, ctx, H, scale, sinks))
        start += n
    assert rel_err(torch.cat(got), want) < TOL[dtype]
    if case == "low scores":                                        # without the sink the first row would be v_0 whole
        assert float(want[0].abs().max()) < 0.5 * float(v[0].double().abs().max())


# ------------------------------------------------------------------------------------------ the recurrences
def _lightning_inputs(dtype, T, H, dk, dv, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t: t.to(torch.bfloat16).to(dtype).to(DEV)
    x = rnd(1.5 * torch.randn(T, 2 * H * (dk + dv), generator=g))
    return x, [0.97, 0.0, 1.0, 0.4, 0.999, 0.8][:H], (1 + 0.2 * torch.randn(H * dv, generator=g)).to(DEV)


def _mlstm_inputs(dtype, T, H, dk, dv, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t: t.to(torch.bfloat16).to(dtype).to(DEV)
    x = rnd(torch.randn(T, 2 * H * (dk + dv), generator=g))
    gates = 2.0 * torch.randn(T, 2 * H, generator=g)
    gates[::7, :H] += 25.0                       # input gates at the cap now and then: the running maximum jumps
    gates[3::11, H:] -= 40.0                     # forget gates that shut: log f about -cap
    gates[T // 2:, 0] -= 30.0                    # a head whose input gate shuts: exp(-m) rules the denominator
    bias = torch.cat([torch.randn(H, generator=g), torch.linspace(-1.0, 5.0, H)])
    return x, gates.to(DEV), bias.to(DEV), (1 + 0.2 * torch.randn(H * dv, generator=g)).to(DEV)


class _Recurrence:
    """One of the two recurrences on its own: inputs, the kernels, the plain statement, states."""

    def __init__(self, kind, dtype, T, H, dk, dv, seed=0, cap=6.0, parts=1):
        self.parts = parts
        self.kind, self.dtype, self.H, self.dk, self.dv, self.cap = kind, dtype, H, dk, dv, cap
        if kind == "lightning":
            self.x, self.decay, self.nw = _lightning_inputs(dtype, T, H, dk, dv, seed)      # (a decay per head)
        else:
            self.x, self.gates, self.bias, self.nw = _mlstm_inputs(dtype, T, H, dk, dv, seed)

    def states(self, slots, fill=None, seed=0):
        g = torch.Generator().manual_seed(seed)
        S = torch.randn(slots, self.H, self.dk, self.dv, generator=g)
        nm = torch.randn(slots, self.H, 1, self.dk + 1, generator=g).expand(-1, -1, -(-self.dv // 32), -1).contiguous()
        if fill is not None:
            S, nm = torch.full_like(S, fill), torch.full_like(nm, fill)
        return [S.to(DEV), nm.to(DEV)]

    def run(self, rows, ctx, states, out, scale=1.0, chunked=False):
        x = self.x[rows].contiguous()
        n = x.shape[0]
        raw = torch.full((n, self.H * self.dv), float("nan"), device=DEV)
        kw = {}
        if chunked:
            kw = dict(scratch=torch.full((ops().decayed_linear_scratch(n, ctx.n_entries, self.H, self.dk, self.dv),), float("nan"),
                                         device=DEV), max_q=max(ctx.q_lens))
        tail = (out, ctx.cu_q, ctx.ctx_before, ctx.slots, ctx.row_entry, ctx.n_entries, self.H, self.dk, self.dv, 1e-5, scale)
        if self.kind == "lightning":
            ops().lightning(x, ops().decay_powers(self.decay, DEV), self.nw, states[0], raw, *tail, **kw)
        else:
            gates = self.gates[rows].contiguous()
            if self.parts > 1:                             # the same numbers as a stack of partial sums
                cut = torch.randn(self.parts - 1, *gates.shape, generator=torch.Generator().manual_seed(1)).to(DEV)
                gates = torch.cat([cut, (gates - cut.sum(0))[None]]).contiguous()
            ops().mlstm(x, gates, self.bias, self.cap, self.nw, states[0], states[1], raw, *tail, **kw)

    def plain(self, rows, states=None, scale=1.0):
        """(output, states) of consecutive rows of one request, float64."""
        H, dk, dv = self.H, self.dk, self.dv
        x = self.x[rows].double().cpu()
        q, k = x[:, :H * dk].view(-1, H, dk), x[:, H * dk:2 * H * dk].view(-1, H, dk)
        v, g = x[:, 2 * H * dk:2 * H * dk + H * dv].view(-1, H, dv), x[:, 2 * H * dk + H * dv:]
        if self.kind == "lightning":
            act = lambda t: plain.silu(t).to(self.dtype).double()
            o, S = plain.decayed_sum(act(q), act(k), act(v), self.decay, None if states is None else states[0])
            o, new = plain.rms_norm(o.reshape(-1, H * dv), self.nw.double().cpu(), 1e-5), (S,)
        else:
            pre = self.cap * torch.tanh((self.gates[rows].double().cpu() + self.bias.double().cpu()) / self.cap)
            o, new = plain.matrix_memory(q * dk ** -0.5, k, v, pre[:, :H], torch.nn.functional.logsigmoid(pre[:, H:]), states)
            o = plain.rms_div(o, 1e-5).reshape(-1, H * dv) * self.nw.double().cpu()
        return o * torch.sigmoid(g) * scale, new

    def plain_state(self, states, slot):
        S, nm = states[0][slot].double().cpu(), states[1][slot, :, 0].double().cpu()
        return (S,) if self.kind == "lightning" else (S, nm[:, :-1], nm[:, -1])

    def same_state(self, states, slot, want, tol):
        ok = rel_err(states[0][slot], want[0]) < tol
        if self.kind == "mlstm":
            nm = states[1][slot]
            ok = ok and torch.equal(nm, nm[:, :1].expand_as(nm))                # every slice's copy
            ok = ok and rel_err(nm[:, 0, :-1], want[1]) < tol and rel_err(nm[:, 0, -1], want[2]) < tol
        return ok


@pytest.mark.parametrize("kind", ["lightning", "mlstm"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", [(2, 32, 48), (3, 8, 10), (1, 128, 64), (2, 17, 33), (1, 1, 1), (5, 24, 100), (1, 300, 7)])
def test_recurrence_whole_cut_and_token_by_token(kind, dtype, H, dk, dv):
    T = 150
    r = _Recurrence(kind, dtype, T, H, dk, dv)
    want, st = r.plain(slice(0, T), scale=0.9)
    for cuts in ([T], [1, 2, 60, 1, 1, 85], [1] * 20 + [9, 8, 7, 106]):
        states = r.states(4, fill=9.0)                                # stale: the first step must not read it
        wide = torch.zeros(T, H * dv + 6, dtype=dtype, device=DEV)    # the output as a block of columns
        at = 0
        for n in cuts:
            ctx = make_ctx([n], [at], [2], dtype=dtype)
            r.run(slice(at, at + n), ctx, states, wide[at:at + n, 3:3 + H * dv], 0.9)
            at += n
        assert rel_err(wide[:, 3:3 + H * dv], want) < TOL[dtype], cuts
        assert r.same_state(states, 2, st, TOL[torch.float32]) and float(wide[:, :3].abs().max()) == 0
        assert float((states[0][1] - 9.0).abs().max()) == 0 and float((states[1][3] - 9.0).abs().max()) == 0


@pytest.mark.parametrize("kind", ["lightning", "mlstm"])
@pytest.mark.parametrize("dtype,chunked", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
def test_recurrence_batch_of_unequal_entries(kind, dtype, chunked):
    H, dk, dv = 3, 32, 48
    lens, before, slots = [1, 37, 2, 200, 64], [5, 0, 40, 12, 0], [3, 0, 2, 1, 4]
    r = _Recurrence(kind, dtype, sum(lens), H, dk, dv, seed=4, parts=3)
    states = r.states(5, seed=8)
    first = [s.clone() for s in states]
    ctx = make_ctx(lens, before, slots, dtype=dtype)
    out = torch.empty(sum(lens), H * dv, dtype=dtype, device=DEV)
    r.run(slice(0, sum(lens)), ctx, states, out, chunked=chunked)
    at = 0
    for n, b, s in zip(lens, before, slots):
        want, st = r.plain(slice(at, at + n), r.plain_state(first, s) if b else None)
        assert rel_err(out[at:at + n], want) < TOL[dtype], (n, b)
        assert r.same_state(states, s, st, TOL[torch.float32]), (n, b)
        at += n


@pytest.mark.parametrize("kind", ["lightning", "mlstm"])
@pytest.mark.parametrize("H,dk,dv", [(2, 32, 16), (3, 16, 48), (1, 128, 128), (2, 80, 32), (1, 256, 64), (6, 48, 96)])
def test_recurrence_chunk_by_chunk(kind, H, dk, dv):
    """Lengths on, just under and just over a chunk's edge, down to two tokens, from states that are not zero, with heads
    that forget at once or never and gates at their caps: against the plain statement and, closer, against the
    token-by-token kernel."""
    dtype, C = torch.bfloat16, ops().DECAYED_CHUNK
    lens, before, slots = [2 * C, 3 * C - 1, C + 1, 2, C - 1, 5 * C + 17], [0, 7, 3, 90, 0, 100], [0, 3, 1, 2, 4, 5]
    N = sum(lens)
    r = _Recurrence(kind, dtype, N, H, dk, dv, seed=6)
    start = r.states(6, seed=8)
    ctx = make_ctx(lens, before, slots, dtype=dtype)
    a, b = torch.empty(N, H * dv, dtype=dtype, device=DEV), torch.empty(N, H * dv, dtype=dtype, device=DEV)
    sa, sb = [s.clone() for s in start], [s.clone() for s in start]
    r.run(slice(0, N), ctx, sa, a, 1.1)
    r.run(slice(0, N), ctx, sb, b, 1.1, chunked=True)
    assert rel_err(b, a) < 1e-2 and rel_err(sb[0], sa[0]) < 2e-5
    if kind == "mlstm":
        assert rel_err(sb[1], sa[1]) < 2e-5
    at = 0
    for n, bf, s in zip(lens, before, slots):
        want, st = r.plain(slice(at, at + n), r.plain_state(start, s) if bf else None, 1.1)
        assert rel_err(b[at:at + n], want) < TOL[dtype] / 3, (n, bf)
        assert r.same_state(sb, s, st, 2e-5), (n, bf)
        at += n


@pytest.mark.parametrize("kind", ["lightning", "mlstm"])
def test_recurrence_long_request_passes_between_the_two_forms(kind):
    """A request of several rounds of chunks, its portions alternating between the two forms: more than 32 chunks in one
    launch (the gates' scan works on 32 at a time), then single tokens, then portions."""
    H, dk, dv, dtype = 2, 16, 32, torch.bfloat16
    cuts = [35 * 64 + 5, 1, 1, 70, 1, 3, 128]
    T = sum(cuts)
    r = _Recurrence(kind, dtype, T, H, dk, dv, seed=3)
    want, st = r.plain(slice(0, T))
    states, got, at = r.states(2, fill=5.0), [], 0
    for n in cuts:
        out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
        r.run(slice(at, at + n), make_ctx([n], [at], [1], dtype=dtype), states, out, chunked=n >= 32)
        got.append(out)
        at += n
    assert rel_err(torch.cat(got), want) < TOL[dtype] / 3 and r.same_state(states, 1, st, 1e-4)


@pytest.mark.parametrize("kind,chunked", [("lightning", False), ("lightning", True), ("mlstm", False), ("mlstm", True)])
def test_a_key_far_back_shows(kind, chunked):
    """One token's key and value are large and a query 700 tokens later asks for them: what it reads is that value."""
    H, dk, dv, T, far = 1, 32, 16, 900, 130
    r = _Recurrence(kind, torch.bfloat16, T, H, dk, dv, seed=2)
    r.x *= 0.02
    r.x[far, dk:2 * dk] = 8.0 * torch.sign(torch.randn(dk, generator=torch.Generator().manual_seed(1))).to(DEV)
    r.x[far, 2 * dk:2 * dk + dv] = torch.linspace(-4, 4, dv).to(DEV)
    r.x[far + 700, :dk] = r.x[far, dk:2 * dk]
    if kind == "lightning":
        r.decay = [0.9995]
    else:
        r.gates[:, :H], r.gates[:, H:], r.bias[:] = -2.0, 9.0, 0.0
        r.gates[far, 0] = 5.0
    want, _ = r.plain(slice(0, T))
    out, states = torch.empty(T, H * dv, dtype=torch.bfloat16, device=DEV), r.states(1, fill=3.0)
    r.run(slice(0, T), make_ctx([T], [0], [0], dtype=torch.bfloat16), states, out, chunked=chunked)
    assert rel_err(out, want) < TOL[torch.bfloat16] / 3
    r.x[far, 2 * dk:2 * dk + dv] *= -1
    other, _ = r.plain(slice(0, T))
    assert float((other[far + 700] - want[far + 700]).abs().max()) > 0.3


# ------------------------------------------------------------------------------------------ parts
def _part(spec, cls, dtype, seed):
    part = cls(spec, dtype=dtype, device=DEV)
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, d in part.tensors().items():
        t = torch.randn(*d.shape, generator=g)
        t = 1 + 0.2 * t if d.init == "norm" else t if d.init == "bias" else 1.3 * t / d.shape[-1] ** 0.5
        w[name] = t.to(torch.bfloat16).float()
    part.bind({k: v.to(DEV) for k, v in w.items()})
    return part, {k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [9, 75])
def test_lightning_and_mlstm_parts(dtype, T):
    """Projections, gates' product and output projection around the recurrences."""
    from neurogrid_b200.config.specs import LightningSpec, MLSTMSpec
    from neurogrid_b200.parts import SlotView
    from neurogrid_b200.parts.decayed_linear import MLSTM, LightningAttention
    Hd = 64
    x = _x((T, Hd), dtype, seed=5)
    for spec, cls, m in ((LightningSpec(Hd, 2, 32, 16, (0.9, 0.99), 1e-5), LightningAttention, dict(heads=2, dim=32, vdim=16, decay=[0.9, 0.99])),
                         (MLSTMSpec(Hd, 3, 16, 48, 4.0, 1e-5), MLSTM, dict(heads=3, dim=16, vdim=48, gate_cap=4.0))):
        part, w = _part(spec, cls, dtype, seed=6)
        need = part.cache_need()
        views = [SlotView(torch.full((2,) + n.shape, 7.0, device=DEV)) for n in (need if isinstance(need, tuple) else (need,))]
        ctx = make_ctx([T], [0], [1], dtype=dtype)
        y = part.forward(x, ctx, tuple(views) if len(views) > 1 else views[0])
        y = y.double().sum(0) if y.dim() == 3 else y
        fn = plain.lightning if cls is LightningAttention else plain.mlstm
        want, _ = fn(x.double().cpu(), w, "", m, 1e-5)
        if dtype == torch.float32:
            assert rel_err(y, want) < TOL[dtype]
        else:                   # (the sign of q_0 . k_0 may be a rounding's: rows are judged one by one)
            assert _close(y, want, dtype)


# ------------------------------------------------------------------------------------------ whole models
LENS = {"A": [1, 9, 40, 131, 64, 23, 77], "B": [3, 50, 97, 30, 64], "B0": [2, 41, 90], "C": [2, 17, 150, 33, 210],
        "D": [1, 45, 20, 100]}


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
def plain_logits(matepel_dirs):
    out = {}
    for name in LENS:
        cfg, w = mm.load_plain(matepel_dirs[name])
        reqs = scenarios.make_requests(LENS[name], cfg["vocab"], seed=7)
        out[name] = (reqs, {r: plain.forward(cfg, w, t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("name", ["A", "B0", "C"])
def test_stream_after_every_layer(matepel_dirs, name):
    """float32, layer by layer: the sum of the stream's copies after every layer."""
    cfg, w = mm.load_plain(matepel_dirs[name])
    toks = scenarios.make_requests([37], cfg["vocab"], seed=1)["r0"]
    _, after = plain.forward(cfg, w, toks, return_layers=True)
    runner = make_runner(matepel_dirs[name], dtype=torch.float32, device="cuda", page_size=8, num_pages=16)
    seen = []
    model = runner.model
    run_entries, S = model.run_entries, cfg.get("streams") or 1

    def spy(ctx, caches, entries, h, pending):
        for e in entries:                              # one layer at a time; the update not yet written is folded in for the record
            pending = run_entries(ctx, caches, [e], h, pending)
            X = h.double().view(h.shape[0], S, -1)
            y = (pending.y.sum(0) if pending.y.dim() == 3 else pending.y).double()
            if pending.bias is not None:
                y = y + pending.bias.double()
            X = torch.einsum("st,nsh->nth", pending.mix.double().view(S, S), X) + pending.out_w.double()[None, :, None] * y[:, None, :]
            seen.append(X.sum(1)[: len(toks)].cpu())
        return pending

    model.run_entries = spy
    runner.step([StepEntry("x", toks, [len(toks) - 1])])
    assert len(seen) == len(after) == 4
    for i, s in enumerate(seen):
        assert rel_err(s, after[i]) < 1e-4, i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "B0", "C", "D"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
def test_cuts_against_plain(matepel_dirs, plain_logits, name, dtype, cut):
    reqs, want = plain_logits[name]
    ps = mm.PAGE_SIZE[name]
    cap = 256 if cut == "mixed" else 512                     # tokens; mixed: pages and slots are used again
    runner = make_runner(matepel_dirs[name], dtype=dtype, device="cuda", page_size=ps, num_pages=cap // ps,
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
def test_first_tokens_and_long_decode(matepel_dirs, name, dtype):
    """The first tokens one by one (empty states, the sink beside a lone key), then decoding across many pages with
    graphs replayed."""
    cfg, w = mm.load_plain(matepel_dirs[name])
    toks = scenarios.make_requests([230], cfg["vocab"], seed=11)["r0"]
    want = plain.forward(cfg, w, toks)
    runner = make_runner(matepel_dirs[name], dtype=dtype, device="cuda", page_size=8, num_pages=32, max_seq_len=256)
    got = torch.cat([runner.step([StepEntry("x", [t], [0])]).clone() for t in toks])
    runner.check_status()
    assert _close(got, want, dtype), rel_err(got, want)
    if dtype == torch.float32:
        assert rel_err(got[:14], want[:14]) < TOL[dtype]
    assert runner.graph_replays > 100 and runner.cache.pages_held("x") == [29] * len(runner.cache.pools)


@pytest.mark.parametrize("name", ["A", "C"])
def test_float32_cuts_agree_closely(matepel_dirs, name):
    cfg, _ = mm.load_plain(matepel_dirs[name])
    reqs = scenarios.make_requests([120], cfg["vocab"], seed=3)
    runner = make_runner(matepel_dirs[name], dtype=torch.float32, device="cuda", num_pages=64, page_size=8)
    a = _replay(runner, scenarios.whole(reqs))["r0"]
    b = _replay(runner, scenarios.portions(reqs))["r0"]
    c = _replay(runner, scenarios.tail_decode(reqs))["r0"]
    assert rel_err(a, b) < 2e-5 and rel_err(a, c) < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_batch_of_unequal_requests_equals_each_alone(matepel_dirs, name, dtype):
    cfg, _ = mm.load_plain(matepel_dirs[name])
    reqs = scenarios.make_requests([5, 70, 2, 33], cfg["vocab"], seed=5)
    runner = make_runner(matepel_dirs[name], dtype=dtype, device="cuda", num_pages=64, page_size=8)
    alone = _replay(runner, scenarios.whole(reqs))
    lg = runner.step([StepEntry(r, t, list(range(len(t)))) for r, t in reqs.items()])
    at = 0
    for r, t in reqs.items():
        if dtype == torch.float32:
            assert rel_err(lg[at:at + len(t)], alone[r]) < 2e-5
        else:
            assert _close(lg[at:at + len(t)], alone[r], dtype)
        at += len(t)


def test_greedy_generation_through_the_engine(matepel_dirs):
    """Engine.generate (scheduler, portions, decode graphs, device sampler) against greedy decoding with the oracle."""
    from neurogrid_b200 import Engine
    cfg, w = mm.load_plain(matepel_dirs["C"])
    prompts = list(scenarios.make_requests([12, 30, 5], cfg["vocab"], seed=9).values())
    eng = Engine(matepel_dirs["C"], dtype="float32", max_seq_len=128, page_size=8, max_requests=2,
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
def test_trace_replay_program(matepel_dirs, tmp_path, dtype):
    folder = matepel_dirs["A" if dtype == "float32" else "C"]
    cfg, w = mm.load_plain(folder)
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
