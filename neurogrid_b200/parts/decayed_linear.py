"""Linear attention whose float32 state decays by one number per head and token: lightning attention (a fixed decay,
activated projections) and the mLSTM (exponential gates with a running maximum and a normaliser)."""
from __future__ import annotations

import torch

from ..cache.manager import SlotNeed
from ..csrc import ops
from ..weights.decl import TensorDecl
from .registry import register


class _DecayedLinear:
    """What the two mixers share: q, k, v and gate projections stacked into one product when bound, the recurrence, the
    heads' norm and sigmoid gate, the output projection.

    Everything behind the projections (and their silu) is float32 in both compute dtypes.  State per request:
    S [heads, key_dim, value_dim] float32, zero at admission.  float32 steps and steps of short portions walk the tokens
    one by one (a token's arithmetic is then the same however its request is cut); bfloat16 steps with a long portion
    regroup the sums chunk by chunk on the tensor cores, with float32 operands as three bfloat16 terms."""

    graph_safe = True      # launches depend on device data and on launch-time constants only
    CHUNKED_MIN_ROWS = 32  # a bfloat16 step whose longest portion has this many tokens runs the chunk-by-chunk kernels

    def __init__(self, spec, *, dtype, device):
        self.spec, self.dtype, self.device = spec, dtype, device
        self.w_in = self.w_o = self.norm = None

    def tensors(self):
        s, n = self.spec, self.spec.names
        qk, vg = s.n_heads * s.key_dim, s.n_heads * s.value_dim
        return {n["q"]: TensorDecl((qk, s.hidden)), n["k"]: TensorDecl((qk, s.hidden)), n["v"]: TensorDecl((vg, s.hidden)),
                n["gate"]: TensorDecl((vg, s.hidden)), n["o"]: TensorDecl((s.hidden, vg)),
                n["norm"]: TensorDecl((vg,), "norm")}

    def bind(self, t):
        n = self.spec.names
        kw = dict(device=self.device, dtype=self.dtype)
        self.w_in = torch.cat([t[n[p]].to(**kw) for p in ("q", "k", "v", "gate")]).contiguous()
        self.w_o = t[n["o"]].to(**kw).contiguous()
        self.norm = t[n["norm"]].to(device=self.device, dtype=torch.float32).contiguous()

    def kernels(self):
        return [("gemm_sm100" if self.dtype == torch.bfloat16 else "gemm_f32", None), ("decayed_linear", None)]

    def scratch_bytes_per_row(self):
        s = self.spec
        per_row = 4 * s.n_heads * s.value_dim
        if self.dtype == torch.bfloat16:
            per_row += 4 * s.n_heads * ((s.key_dim * s.value_dim + s.key_dim + 2) // ops.DECAYED_CHUNK + 5)
        return per_row

    # a caller that ends two mixers with ONE product calls ``core`` and multiplies itself
    def inner_width(self):
        return self.spec.n_heads * self.spec.value_dim

    def out_weight(self):
        return self.w_o, None

    def drop_out_weight(self):
        """The caller keeps a stacked copy of the output matrix and will not call ``forward``."""
        self.w_o = None

    def _chunk_scratch(self, ctx, n):
        """float32 scratch for the chunk-by-chunk kernels, or None: the step walks its tokens."""
        s = self.spec
        if self.dtype != torch.bfloat16 or ctx.max_q < self.CHUNKED_MIN_ROWS or \
                not ops.decayed_linear_chunked_takes(s.key_dim, s.value_dim):
            return None
        need = ops.decayed_linear_scratch(n, ctx.n_entries, s.n_heads, s.key_dim, s.value_dim)
        bound = ops.decayed_linear_scratch(ctx.ws.max_rows, ctx.ws.max_rows // self.CHUNKED_MIN_ROWS + 64, s.n_heads, s.key_dim,
                                           s.value_dim)
        # (scratch whose bound follows from the layer's sizes is named after them: a layer of other sizes has its own)
        return ctx.ws.flat(f"dl_chunks_{s.n_heads}x{s.key_dim}x{s.value_dim}", need, torch.float32, reserve=max(need, bound))

    def forward(self, x, ctx, cache, out_name="mixer_out"):
        o = ctx.ws.buf("dl_out", x.shape[0], self.inner_width(), self.dtype)
        self.core(x, ctx, cache, o)
        return ops.linear_to_residual(o, self.w_o, None, ctx.ws, out_name, residual=ctx.residual)


@register("mixer", "lightning_attention")
class LightningAttention(_DecayedLinear):
    """q, k, v = silu of their projections -> per head S <- decay S + k v^T, o = S^T q -> one RMS norm over all heads
    together with a weight, times sigmoid(gate) -> output projection."""

    def __init__(self, spec, *, dtype, device):
        super().__init__(spec, dtype=dtype, device=device)
        self.decay = ops.decay_powers(spec.decay, device)

    def cache_need(self):
        s = self.spec
        return SlotNeed((s.n_heads, s.key_dim, s.value_dim))

    def core(self, x, ctx, cache, out, out_scale=1.0):
        """out[N, n_heads * value_dim] (may be a block of columns of a wider buffer): the normed, gated heads times
        ``out_scale``."""
        s = self.spec
        n = x.shape[0]
        p = ctx.ws.buf("dl_in", n, self.w_in.shape[0], self.dtype)
        ops.linear(x, self.w_in, None, p)
        raw = ctx.ws.buf("dl_raw", n, s.n_heads * s.value_dim, torch.float32)
        ops.lightning(p, self.decay, self.norm, cache.state, raw, out, ctx.cu_q, ctx.ctx_before, ctx.slots, ctx.row_entry,
                      ctx.n_entries, s.n_heads, s.key_dim, s.value_dim, s.eps, out_scale, scratch=self._chunk_scratch(ctx, n),
                      max_q=ctx.max_q)


@register("mixer", "mlstm")
class MLSTM(_DecayedLinear):
    """q, k, v projections and, per head, log input and forget gates (their preactivations a float32 product) -> the
    matrix memory with its normaliser and running maximum -> each head's o over its root mean square, times a weight and
    sigmoid(gate) -> output projection.  State per request: S, and (n, m) once for every slice of value columns that a
    block of the token-by-token kernel takes; the mixer declares the two needs and is handed the two views."""

    def __init__(self, spec, *, dtype, device):
        super().__init__(spec, dtype=dtype, device=device)
        self.w_gates = self.b_gates = None

    def tensors(self):
        s, n = self.spec, self.spec.names
        return {**super().tensors(), n["input_gate"]: TensorDecl((s.n_heads, s.hidden)),
                n["input_bias"]: TensorDecl((s.n_heads,), "bias"), n["forget_gate"]: TensorDecl((s.n_heads, s.hidden)),
                n["forget_bias"]: TensorDecl((s.n_heads,), "bias")}

    def bind(self, t):
        super().bind(t)
        n = self.spec.names
        self.w_gates = torch.cat([t[n[p]].to(device=self.device, dtype=self.dtype) for p in ("input_gate", "forget_gate")]).contiguous()
        self.b_gates = torch.cat([t[n[p]].to(device=self.device, dtype=torch.float32) for p in ("input_bias", "forget_bias")]).contiguous()

    def cache_need(self):
        s = self.spec
        return (SlotNeed((s.n_heads, s.key_dim, s.value_dim)),
                SlotNeed((s.n_heads, ops.decayed_linear_slices(s.value_dim), s.key_dim + 1)))

    def core(self, x, ctx, cache, out, out_scale=1.0):
        """out[N, n_heads * value_dim] (may be a block of columns of a wider buffer): the normed, gated heads times
        ``out_scale``."""
        s = self.spec
        n = x.shape[0]
        state, nm = cache
        p = ctx.ws.buf("dl_in", n, self.w_in.shape[0], self.dtype)
        ops.linear(x, self.w_in, None, p)
        gates = ops.linear_f32(x, self.w_gates, ctx.ws, f"dl_gates_{s.n_heads}")
        raw = ctx.ws.buf("dl_raw", n, s.n_heads * s.value_dim, torch.float32)
        ops.mlstm(p, gates, self.b_gates, s.gate_cap, self.norm, state.state, nm.state, raw, out, ctx.cu_q, ctx.ctx_before,
                  ctx.slots, ctx.row_entry, ctx.n_entries, s.n_heads, s.key_dim, s.value_dim, s.eps, out_scale,
                  scratch=self._chunk_scratch(ctx, n), max_q=ctx.max_q)
