"""Tiny Pepulix configurations and weights for the tests.

The weights are drawn so that the mechanisms show in the logits: attention scores reach from far below to far above the
sigmoid's bend, so a few keys weigh nearly one and most nearly nothing; values are mixed by shares well inside (0, 1); the
recurrent gates range from forgetful to nearly none and from shut to wide open; the copies of the stream are mixed by
matrices far from the identity; the corrections change which experts are chosen, and identity experts are chosen often."""
from __future__ import annotations

import json
import os

import torch

from matepel_models import load_plain  # noqa: F401  (the tests read model folders through it)
from neurogrid_b200.config import config_from_dict
from neurogrid_b200.models import declare_tensors
from neurogrid_b200.weights import write_file


def _attention(heads, kv, dim, vdim, scale, mlp, rot=None, v_mix=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp, base=1000.0, scaling=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot_dim"], m["rot"] = rot_dim, {"base": base, "dims": rot_dim}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def _ff(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, identity, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}}


# A: three copies of the stream, every option, sizes different wherever two could be equal; the layer that the others' values
# are mixed with is not the first attention
PEPU_A = {
    "architecture": "Pepulix", "vocab": 131, "width": 60, "streams": 3, "norm": {"eps": 2e-6}, "logit_softcap": 9.0,
    "layers": [
        _attention(2, 1, 9, 7, 0.8, _ff(36), v_mix=False),
        _attention(4, 2, 20, 12, 0.4, _moe(6, 3, 3, 20), (1000.0, 16), True),
        _mlstm(3, 8, 10, 3.0, _ff(40)),
        _latent(3, 12, 8, 10, 28, 20, 0.35, _moe(5, 2, 1, 16), 1000.0, (6.0, 64, 8.0, 0.5)),
        _attention(6, 2, 14, 12, 0.5, None, (50.0, 4), True),
        _latent(2, 6, 4, 14, 18, 33, 0.5, None, 30.0),
        _attention(2, 2, 16, 12, 0.6, _moe(4, 0, 4, 24), (200.0, 16), True),
    ],
}

# B: values that could be equal are, or are 1, and what can be left out is; B0: plain residual sums
PEPU_B = {
    "architecture": "Pepulix", "vocab": 61, "width": 40, "streams": 1, "norm": {"eps": 1e-5},
    "layers": [
        _attention(1, 1, 8, 8, 0.7, _ff(24), None, True),
        _latent(1, 8, 0, 8, 8, 8, 0.4, _moe(1, 1, 1, 8)),
        _mlstm(1, 8, 8, 1.0, None),
        _attention(2, 1, 6, 8, 0.9, _moe(2, 1, 2, 8), (10000.0, 6), True),
        _latent(2, 2, 2, 2, 4, 4, 1.0, _moe(3, 0, 1, 8), 10000.0, (1.0, 128, 4.0, 1.0)),
    ],
}
PEPU_B0 = {**{k: v for k, v in PEPU_B.items() if k != "streams"}, "vocab": 67, "logit_softcap": 25.0}

# C: head sizes that every tensor-core kernel takes: KV groups of four and of three heads, latents of 32 and of 64 padded
# columns with at most and with more than eight heads, recurrent heads that run chunk by chunk
PEPU_C = {
    "architecture": "Pepulix", "vocab": 90, "width": 72, "streams": 2, "norm": {"eps": 1e-6}, "logit_softcap": 20.0,
    "layers": [
        _mlstm(3, 48, 32, 6.0, _ff(56)),
        _attention(4, 1, 32, 48, 0.3, _moe(8, 3, 3, 16), (10000.0, 24), True),
        _latent(5, 16, 16, 24, 40, 40, 0.3, _ff(64), 10000.0, (8.0, 512, 16.0, 1.0)),
        _attention(6, 2, 64, 16, 0.2, None, (500.0, 64)),
        _latent(12, 8, 8, 8, 16, 24, 0.45, _moe(4, 2, 2, 24), 100.0, (3.0, 100, 10.0, 1.0)),
        _attention(3, 1, 16, 48, 0.5, _moe(5, 1, 2, 16), None, True),
        _mlstm(2, 16, 64, 12.0, None),
    ],
}

# D: a width that is no multiple of eight, five copies, more query heads of a key/value head than a tile has rows, more latent
# heads than the latent cores take, a cached row wider than any of them, recurrent heads of odd sizes
PEPU_D = {
    "architecture": "Pepulix", "vocab": 70, "width": 50, "streams": 5, "norm": {"eps": 1e-5}, "logit_softcap": 12.0,
    "layers": [
        _attention(34, 2, 7, 5, 0.9, _ff(30), (10.0, 4), True),
        _latent(66, 3, 2, 4, 11, 30, 0.7, None, 10.0, (4.0, 40, 6.0, 0.25)),
        _mlstm(1, 17, 45, 2.0, _moe(3, 5, 4, 7)),
        _latent(2, 5, 6, 3, 9, 520, 0.6, _ff(10), 20.0),
        _attention(4, 2, 30, 5, 0.35, None, None, True),
    ],
}

CONFIGS = {"A": (PEPU_A, 61), "B": (PEPU_B, 62), "B0": (PEPU_B0, 63), "C": (PEPU_C, 64), "D": (PEPU_D, 65)}
PAGE_SIZE = {"A": 8, "B": 16, "B0": 4, "C": 8, "D": 8}


def draw_weights(config: dict, seed: int, calm: bool = False):
    """name -> bfloat16 tensor for every tensor the configuration declares.  ``calm``: the routers hardly look at the token
    and the corrections decide, so that no choice is close (for comparisons in bfloat16)."""
    decls = declare_tensors(config_from_dict(config).model_spec())
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(decls):
        d = decls[name]
        parts = name.split(".")
        leaf = parts[-1]
        rnd = lambda *s: torch.randn(*s, generator=g)
        if len(parts) > 1 and parts[1] in ("hc1", "hc2"):
            n = d.shape[0]
            if leaf == "in":
                t = 1.0 / n + 0.3 * rnd(d.shape)
            elif leaf == "out":
                t = 1.0 + 0.4 * rnd(d.shape)
            else:                                           # mixes the copies; columns sum to about one
                t = 0.6 * torch.eye(n) + 0.4 / n + 0.15 * rnd(d.shape)
        elif leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * rnd(d.shape)
        elif leaf == "vmix":
            t = 0.25 + 0.5 * torch.rand(d.shape, generator=g)
        elif leaf == "pb":
            t = -2.0 + 1.5 * rnd(d.shape)
        elif leaf == "correction":                          # of the scores' size: the choice is not the largest scores'
            t = 1.0 / d.shape[0] * rnd(d.shape)
            if calm:
                t = torch.linspace(0.0, 0.5, d.shape[0])[torch.randperm(d.shape[0], generator=g)]
        elif name.endswith("mix.f.b"):                      # from forgetful to nearly no decay
            t = torch.linspace(-1.5, 5.0, d.shape[0])[torch.randperm(d.shape[0], generator=g)] + 0.3 * rnd(d.shape)
        elif leaf == "b":
            t = 0.7 * rnd(d.shape)
        elif name == "embed":
            t = 0.45 * rnd(d.shape)
        else:
            gain = {"i": 2.5, "f": 1.5, "gate": 1.5, "up": 1.5, "uq": 1.6, "router": 0.01 if calm else 1.5}.get(leaf, 1.0)
            t = gain * rnd(d.shape) / d.shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(config: dict, seed: int, folder: str, weights=None, calm: bool = False) -> str:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_file(os.path.join(folder, "model.safetensors"), weights or draw_weights(config, seed, calm))
    return folder
