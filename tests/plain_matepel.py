"""A plain, slow statement of the Matepel decoder: float64, whole sequences, one function per mechanism.

Shares no code with the package.  ``cfg`` is the dictionary of config.json, ``w`` maps tensor names to float64
tensors; a sequence is a list of token ids, positions count from 0.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_div(x, eps):
    """x over its root mean square along the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms_div(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ lightning attention
def decayed_sum(q, k, v, decay, state=None):
    """Per head S <- decay_h S + k_t v_t^T, o_t = S^T q_t.  q, k [T,H,d], v [T,H,dv] -> (o [T,H,dv], S [H,d,dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if state is None else state.clone()
    lam = torch.as_tensor(decay, dtype=F64)[:, None, None]
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = lam * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def lightning(h, w, pre, m, eps, state=None):
    """(output [T, width], state after the last token)."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[pre + "q"].T).view(T, H, d)
    k = silu(h @ w[pre + "k"].T).view(T, H, d)
    v = silu(h @ w[pre + "v"].T).view(T, H, dv)
    o, S = decayed_sum(q, k, v, m["decay"], state)
    o = rms_norm(o.reshape(T, H * dv), w[pre + "norm"], eps)           # one norm over all heads together
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, S


# ------------------------------------------------------------------------------------------------ the parallel mixer's left side
def scaled_frequencies(rot):
    """(frequency of every rotated pair, factor on its cosine and sine): base^(-2i/dims), with ``scaling`` blended
    towards the frequency over ``factor`` where a pair turns too seldom within ``original`` positions."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    at = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, d]: coordinates i and i + dims/2 (i < dims/2) of every head are turned by position * f_i; cosine and
    sine carry the scaling's factor."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f, mag = scaled_frequencies(rot)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = (mag * torch.cos(ang))[:, None, :], (mag * torch.sin(ang))[:, None, :]
    a, b = x[..., :half], x[..., half:2 * half]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., 2 * half:]], -1)


def shared_kv_attention(h, w, pre, m):
    """Grouped-query causal attention whose values are the unrotated keys; the softmax's denominator holds one more 1."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).view(T, H, d)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).view(T, G, d)
    v = k
    q, k = rotate(q, pos, m.get("rot")), rotate(k, pos, m.get("rot"))
    out = torch.zeros(T, H, d, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * m["scale"]
        s = s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf)
        top = s.max(-1, keepdim=True).values.clamp_min(0.0)            # the extra term's score is 0
        e = torch.exp(s - top)
        out[:, hd] = (e @ v[:, g]) / (torch.exp(-top) + e.sum(-1, keepdim=True))
    return out.reshape(T, H * d) @ w[pre + "o"].T + w[pre + "o.b"]


# ------------------------------------------------------------------------------------------------ the parallel mixer's right side
def log_gates(h, w, pre, cap):
    """(log input gate, log forget gate) [T, heads]: soft-capped preactivations, the forget gate through log sigmoid."""
    soft = lambda z: cap * torch.tanh(z / cap)
    i = soft(h @ w[pre + "i"].T + w[pre + "i.b"])
    f = torch.nn.functional.logsigmoid(soft(h @ w[pre + "f"].T + w[pre + "f.b"]))
    return i, f


def matrix_memory(q, k, v, i, f, state=None):
    """The exponentially gated memory with its stabiliser: q, k [T,H,d], v [T,H,dv], i, f [T,H] ->
    (o [T,H,dv], (S [H,d,dv], n [H,d], m [H]))."""
    T, H, d = q.shape
    if state is None:
        S, n, m = torch.zeros(H, d, v.shape[-1], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    else:
        S, n, m = (s.clone() for s in state)
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o, (S, n, m)


def mlstm(h, w, pre, m, eps, state=None):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).view(T, H, d)
    v = (h @ w[pre + "v"].T).view(T, H, dv)
    i, f = log_gates(h, w, pre, m["gate_cap"])
    o, state = matrix_memory(q, k, v, i, f, state)
    o = rms_div(o, eps).reshape(T, H * dv) * w[pre + "norm"]           # a norm per head, a weight per coordinate of all heads
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, state


def parallel_mixer(h, w, pre, m, eps):
    left = shared_kv_attention(h, w, pre + "left.", m["left"])
    right, _ = mlstm(h, w, pre + "right.", m["right"], eps)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_ff(h, w, pre, mlp):
    lim = mlp["limit"]
    g = (h @ w[pre + "gate"].T).clamp(max=lim)
    u = (h @ w[pre + "up"].T).clamp(-lim, lim)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


# ------------------------------------------------------------------------------------------------ the model
def connect(xs, y, mix, out_w):
    """Every copy anew from all old ones and the sublayer's output."""
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out_w[t] * y for t in range(n)]


def forward(cfg, w, tokens, *, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the stream, summed over its copies, after every layer)."""
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = rms_norm(w["embed"][torch.as_tensor(tokens)], w["embed.norm"], eps)
    n_streams = cfg.get("streams")
    xs = [x.clone() for _ in range(n_streams or 1)]
    one = torch.ones(1, dtype=F64)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer.get("mlp") is not None else (1,):
            hc = {k: w[f"{pre}hc{q}.{k}"] for k in ("in", "out", "mix")} if n_streams else {"in": one, "out": one, "mix": one[None]}
            u = sum(hc["in"][s] * xs[s] for s in range(len(xs)))
            hn = rms_norm(u, w[f"{pre}norm{q}"], eps)
            if q == 2:
                y = clamped_ff(hn, w, pre + "mlp.", layer["mlp"])
            elif layer["type"] == "lightning":
                y, _ = lightning(hn, w, pre + "mix.", m, eps)
            else:
                y = parallel_mixer(hn, w, pre + "mix.", m, eps)
            xs = connect(xs, y, hc["mix"], mult * hc["out"])
        after.append(sum(xs))
    logits = rms_norm(sum(xs), w["final.norm"], eps) @ w["head"].T
    return (logits, after) if return_layers else logits
