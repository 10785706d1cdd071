"""A plain, slow statement of the Pepulix decoder: float64, whole sequences, one function per mechanism.

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


def causal(T):
    return torch.ones(T, T).tril().bool()


# ------------------------------------------------------------------------------------------------ rotations
def pair_frequencies(rot):
    """(one frequency per rotated pair, factor on cosines and sines): base^(-2i/dims); with ``scaling`` the pairs that turn
    less than ``slow`` times within ``original`` positions take the frequency over ``factor``, those that turn more than
    ``fast`` times keep theirs, the ones between are blended linearly in their index."""
    dims, base = rot["dims"], rot["base"]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64), 1.0

    def index_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(index_of(sc["fast"])), 0)
    last = min(math.ceil(index_of(sc["slow"])), dims - 1)
    f = []
    for i in range(dims // 2):
        plain = base ** (-2.0 * i / dims)
        share = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        f.append(share * plain / sc["factor"] + (1.0 - share) * plain)
    return torch.tensor(f, dtype=F64), 1.0 + 0.1 * math.log(sc["factor"])


def rotate(x, rot, interleaved):
    """x [T, heads, d], row t at position t: the first rot.dims coordinates in pairs (2i, 2i+1) or (i, i + dims/2)."""
    if not rot or not rot["dims"]:
        return x
    n = rot["dims"]
    f, mag = pair_frequencies(rot)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * f
    c, s = (mag * torch.cos(ang))[:, None], (mag * torch.sin(ang))[:, None]
    out = x.clone()
    first = slice(0, n, 2) if interleaved else slice(0, n // 2)
    second = slice(1, n, 2) if interleaved else slice(n // 2, n)
    a, b = x[..., first], x[..., second]
    out[..., first], out[..., second] = a * c - b * s, b * c + a * s
    return out


# ------------------------------------------------------------------------------------------------ sigmoid attention
def sigmoid_weights(q, k, scale, bias):
    """One head: weight of key j for query i, sigmoid(scale q_i . k_j + bias) for j <= i, else 0."""
    return torch.sigmoid(scale * (q @ k.T) + bias).masked_fill(~causal(q.shape[0]), 0.0)


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, pre, m, eps, v_first=None):
    """(output [T, width], this layer's values as cached [T, G, vdim]).  ``v_first``: the cached values of the first layer
    that mixes (None: this layer does not mix, or is that first one)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).view(T, H, d)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).view(T, G, d)
    v = (h @ w[pre + "v"].T + w[pre + "v.b"]).view(T, G, dv)
    q, k = (rms_div(rotate(x, m.get("rot"), False), eps) for x in (q, k))
    v = rms_div(v, eps)
    if v_first is not None:
        v = mix_values(v, v_first, w[pre + "vmix"])
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = sigmoid_weights(q[:, hd], k[:, g], m["scale"], w[pre + "pb"][hd]) @ v[:, g]
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    return (out * gate[:, :, None]).reshape(T, H * dv) @ w[pre + "o"].T, v


# ------------------------------------------------------------------------------------------------ latent attention
def latent_attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m.get("rot_dim", 0), m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).view(T, H, d + r)
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :rank], w[pre + "dkv.norm"], eps)
    k = (c @ w[pre + "uk"].T).view(T, H, d)
    v = (c @ w[pre + "uv"].T).view(T, H, dv)
    q_rot = rotate(q[:, :, d:], m.get("rot"), True)
    k_rot = rotate(down[:, None, rank:], m.get("rot"), True)[:, 0]
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        s = (q[:, hd, :d] @ k[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]
        out[:, hd] = torch.softmax(s.masked_fill(~causal(T), -math.inf), -1) @ v[:, hd]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------ matrix memory
def log_gates(h, w, pre, cap):
    """(log input gate, log forget gate) [T, heads]."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return (soft(h @ w[pre + "i"].T + w[pre + "i.b"]),
            torch.nn.functional.logsigmoid(soft(h @ w[pre + "f"].T + w[pre + "f.b"])))


def matrix_memory(q, k, v, i, f):
    """q, k [T,H,d], v [T,H,dv], log gates i, f [T,H] -> o [T,H,dv]; memory, normaliser and running maximum start at 0."""
    T, H, d = q.shape
    S, n, top = torch.zeros(H, d, v.shape[-1], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, add = torch.exp(f[t] + top - new)[:, None], torch.exp(i[t] - new)[:, None]
        S = keep[..., None] * S + (add * k[t])[:, :, None] * v[t][:, None, :]
        n = keep * n + add * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o


def mlstm(h, w, pre, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).view(T, H, d)
    v = (h @ w[pre + "v"].T).view(T, H, dv)
    o = rms_div(matrix_memory(q, k, v, *log_gates(h, w, pre, m["gate_cap"])), eps)
    return (o.reshape(T, H * dv) * w[pre + "norm"] * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h, w, pre):
    act = silu(h @ w[pre + "gate"].T + w[pre + "gate.b"]) * (h @ w[pre + "up"].T + w[pre + "up.b"])
    return act @ w[pre + "down"].T + w[pre + "down.b"]


def routing_weights(h, w, pre, router):
    """[T, experts + identity] routing weights, zero for what is not chosen."""
    s = torch.softmax(h @ w[pre + "router"].T, -1)
    chosen = torch.topk(s + w[pre + "correction"], router["top"], -1).indices
    mask = torch.zeros_like(s).scatter_(-1, chosen, 1.0)
    return s * mask / ((s * mask).sum(-1, keepdim=True) + 1e-20)


def expert_ff(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def moe_ff(h, w, pre, mlp):
    r = mlp["router"]
    weights = routing_weights(h, w, pre, r)
    y = weights[:, r["experts"]:].sum(-1, keepdim=True) * h           # identity experts: the input itself
    for e in range(r["experts"]):
        y = y + weights[:, e:e + 1] * expert_ff(h, w, f"{pre}e{e}.")
    return y


# ------------------------------------------------------------------------------------------------ the model
def connect(xs, y, mix, out_w):
    """Every copy anew from all old ones and the sublayer's output."""
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out_w[t] * y for t in range(n)]


def forward(cfg, w, tokens, *, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the stream, summed over its copies, after every layer)."""
    eps, n_streams = cfg["norm"]["eps"], cfg.get("streams")
    x = w["embed"][torch.as_tensor(tokens)]
    xs = [x.clone() for _ in range(n_streams or 1)]
    one = torch.ones(1, dtype=F64)
    after, v_first = [], None
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer.get("mlp") is not None else (1,):
            hc = {k: w[f"{pre}hc{q}.{k}"] for k in ("in", "out", "mix")} if n_streams else {"in": one, "out": one, "mix": one[None]}
            u = sum(hc["in"][s] * xs[s] for s in range(len(xs)))
            hn = rms_norm(u, w[f"{pre}norm{q}"], eps)
            if q == 2:
                mlp = layer["mlp"]
                y = dense_ff(hn, w, pre + "mlp.") if mlp["kind"] == "dense" else moe_ff(hn, w, pre + "mlp.", mlp)
            elif layer["type"] == "attention":
                mixes = bool(m.get("v_mix"))
                y, v = attention(hn, w, pre + "mix.", m, eps, v_first if mixes else None)
                if mixes and v_first is None:
                    v_first = v
            elif layer["type"] == "latent_attention":
                y = latent_attention(hn, w, pre + "mix.", m, eps)
            else:
                y = mlstm(hn, w, pre + "mix.", m, eps)
            xs = connect(xs, y, hc["mix"], hc["out"])
        after.append(sum(xs))
    logits = rms_norm(sum(xs), w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    logits = cap * torch.tanh(logits / cap) if cap else logits
    return (logits, after) if return_layers else logits
