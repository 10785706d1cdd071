"""Tiny Matepel configurations and weights for the tests.

The weights are drawn so that the mechanisms show in the logits: projections keep activations of order one, the matrices
behind attention scores and their biases are larger (a peaked softmax whose scores reach both sides of the sink's 0), the
recurrent gates range from forgetful to nearly none and from shut to wide open (so that the running maximum moves and
both branches of the denominator are met), the clamps of the feed-forward bite, the copies of the stream are mixed by
matrices far from the identity."""
from __future__ import annotations

import json
import os

import torch

from neurogrid_b200.config import config_from_dict
from neurogrid_b200.models import declare_tensors
from neurogrid_b200.weights import write_file


def _lightning(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def _left(heads, kv, dim, scale, rot=None, scaling=None):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if rot:
        d["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling:
            d["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return d


def _right(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _parallel(left, right, mlp, scales=None):
    m = {"left": left, "right": right}
    if scales:
        m["left_scale"], m["right_scale"] = scales
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def _ff(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


# A: three copies of the stream, both layer kinds with and without a feed-forward, grouped heads, sizes different
# wherever two could be equal, a rescaled partial rotation all of whose branches are met
MATE_A = {
    "architecture": "Matepel", "vocab": 133, "width": 56, "streams": 3, "residual_mult": 0.7, "norm": {"eps": 2e-6},
    "layers": [
        _lightning(3, 8, 10, [0.3, 0.9, 0.995], _ff(40, 0.9)),
        _parallel(_left(4, 2, 20, 0.3, (1000.0, 16), (6.0, 64, 8.0, 0.5)), _right(2, 12, 6, 3.0), _ff(36, 1.3), (0.8, 1.25)),
        _lightning(2, 14, 40, [0.5, 1.0]),
        _parallel(_left(6, 3, 12, 0.4, (50.0, 4), (2.0, 300, 20.0, 2.0)), _right(5, 24, 36, 9.0), None, (1.4, 0.6)),
    ],
}

# B: values that could be equal are, or are 1, and what can be left out is: one copy of the stream, one head, no rotation
# and a rotation of the whole head, a scaling by 1, no scales; B0: plain residual sums
MATE_B = {
    "architecture": "Matepel", "vocab": 61, "width": 40, "streams": 1, "norm": {"eps": 1e-5},
    "layers": [
        _parallel(_left(1, 1, 8, 0.35), _right(1, 8, 8, 1.0), _ff(24, 2.0)),
        _lightning(1, 8, 8, [0.0], None),
        _parallel(_left(2, 2, 6, 0.5, (10000.0, 6), (1.0, 128, 4.0, 1.0)), _right(2, 5, 7, 15.0), None),
        _lightning(2, 5, 33, [0.99, 0.2], _ff(16, 0.5)),
    ],
}
MATE_B0 = {**{k: v for k, v in MATE_B.items() if k != "streams"}, "vocab": 67, "residual_mult": 0.5}

# C: head sizes that every tensor-core kernel takes: a KV group of four heads, recurrent heads that run chunk by chunk with
# value slices of 16, 32 and 64 columns, layers of different sizes
MATE_C = {
    "architecture": "Matepel", "vocab": 90, "width": 72, "streams": 2, "residual_mult": 1.3, "norm": {"eps": 1e-6},
    "layers": [
        _lightning(2, 32, 128, [0.97, 0.6], None),
        _parallel(_left(4, 1, 32, 0.25, (10000.0, 24), (8.0, 512, 16.0, 1.0)), _right(3, 48, 32, 6.0), _ff(56, 1.1), (0.9, 1.15)),
        _lightning(4, 16, 16, [0.999, 0.99, 0.8, 0.1], _ff(32, 3.0)),
        _parallel(_left(6, 2, 48, 0.2, (500.0, 48), (3.0, 100, 10.0, 1.0)), _right(2, 16, 64, 12.0), None, (1.1, 0.7)),
    ],
}

# D: a width that is no multiple of eight, five copies, more query heads of a key/value head than a tile has rows, recurrent
# heads wider than a block's slice by an odd number, an odd key size
MATE_D = {
    "architecture": "Matepel", "vocab": 70, "width": 50, "streams": 5, "residual_mult": 0.9, "norm": {"eps": 1e-5},
    "layers": [
        _parallel(_left(34, 2, 7, 0.35, (10.0, 4), (4.0, 40, 6.0, 0.25)), _right(1, 17, 45, 2.0), _ff(30, 1.0), (1.0, 0.5)),
        _lightning(3, 33, 70, [0.95, 0.7, 0.9999], None),
    ],
}

CONFIGS = {"A": (MATE_A, 51), "B": (MATE_B, 52), "B0": (MATE_B0, 53), "C": (MATE_C, 54), "D": (MATE_D, 55)}
PAGE_SIZE = {"A": 8, "B": 16, "B0": 4, "C": 8, "D": 8}


def draw_weights(config: dict, seed: int):
    """name -> bfloat16 tensor for every tensor the configuration declares."""
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
        elif name.endswith("right.f.b"):                    # from forgetful to nearly no decay
            t = torch.linspace(-1.5, 5.0, d.shape[0])[torch.randperm(d.shape[0], generator=g)] + 0.3 * rnd(d.shape)
        elif name.endswith("right.i.b"):
            t = 1.0 * rnd(d.shape)
        elif leaf == "b":
            t = 0.7 * rnd(d.shape)
        elif name == "embed":
            t = 0.6 * rnd(d.shape)
        else:
            gain = {"head": 2.0, "i": 2.5, "f": 1.5, "gate": 1.5, "up": 1.5}.get(leaf, 1.0)
            if ".left." in name and leaf in ("q", "k"):
                gain = 1.6
            t = gain * rnd(d.shape) / d.shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(config: dict, seed: int, folder: str, weights=None) -> str:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_file(os.path.join(folder, "model.safetensors"), weights or draw_weights(config, seed))
    return folder


def load_plain(folder: str):
    """(config mapping, name -> float64 tensor) of a model folder."""
    from neurogrid_b200.weights.safetensors_io import MappedFiles, read_header
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    files = MappedFiles()
    w = {k: files.read(e).double() for k, e in read_header(os.path.join(folder, "model.safetensors")).items()}
    files.close()
    return cfg, w
