"""Typed configuration of the Matepel decoder, read from its own ``config.json`` keys.

Matepel is a pre-norm decoder (RMS norms with plain weights) whose layers are listed one by one in ``layers``; the
embedding passes an RMS norm of its own.  With ``streams`` the residual stream is that many copies tied by
hyper-connections (every sublayer reads a weighted sum of the copies and writes, times ``residual_mult``, into all of
them through a mixing matrix), and the final norm reads their sum; without it a layer adds residual_mult times its
sublayers' outputs to one stream.

* ``type`` ``lightning``: linear attention with a fixed decay per head (``decay``) on silu-activated projections; one RMS
  norm over all heads together, a sigmoid gate.
* ``type`` ``parallel``: two mixers side by side on the same normed input, result left_scale * left + right_scale *
  right.  ``mixer.left``: grouped-query causal softmax attention without a v projection (the values are the keys as
  projected, before rotation), biases on q, k and the output projection, a partial rotation in pairs (i, i + dims/2)
  whose frequencies may be rescaled by index (``rot.scaling``), and one more 1 in the softmax's denominator.
  ``mixer.right``: the matrix memory of xLSTM, a recurrence with exponential gates soft-capped by ``gate_cap``; heads over
  their root mean square, a weight, a sigmoid gate.

The feed-forward (``mlp``, or null for none) is dense: down(g sigmoid(1.702 g) (u + 1)) with g = min(gate x, limit),
u = clamp(up x, -limit, limit).

Keys: ``architecture``, ``vocab``, ``width``, ``streams``, ``residual_mult``, ``norm.eps``, ``layers[i].type``,
``layers[i].mixer.{heads, dim, vdim, decay}``, ``layers[i].mixer.{left_scale, right_scale}``, ``layers[i].mixer.left.{heads,
kv_heads, dim, vdim, scale, rot.{base, dims, scaling.{factor, original, fast, slow}}}``, ``layers[i].mixer.right.{heads,
dim, vdim, gate_cap}``, ``layers[i].mlp.{kind, ff, limit}``.  Tensor names: ``embed``, ``embed.norm``, ``l<i>.norm1``,
``l<i>.norm2``, ``l<i>.hc1.{in, out, mix}``, ``l<i>.hc2.{in, out, mix}``, ``l<i>.mix.{q, k, v, g, o, norm}``,
``l<i>.mix.left.{q, q.b, k, k.b, o, o.b}``, ``l<i>.mix.right.{q, k, v, g, o, norm, i, i.b, f, f.b}``, ``l<i>.mlp.{gate, up,
down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .dodilix import MAX_STREAMS, _rot
from .lfm2 import ConfigError
from .metanex import _need
from .specs import (LayerSpec, LightningSpec, MLSTMSpec, MappedAttentionSpec, ModelSpec, NoPositionSpec, RMSNormSpec, RopeSpec,
                    ScheduleEntry, SideBySideSpec, SwiGLUSpec)

LAYER_TYPES = ("lightning", "parallel")
GLU_ALPHA = 1.702           # the clamped activation's sigmoid(alpha g)
MAX_KEY_DIM = 512           # what the recurrent kernels take
MAX_HEAD_DIM = 256          # ... and the attention kernels, whose values are as wide as the keys


def _yarn(m: Mapping[str, Any], path: str) -> Optional[Tuple[float, float, float, float]]:
    """(factor, original, fast, slow) of a rotation's ``scaling``, or None."""
    sc = (m.get("rot") or {}).get("scaling")
    if sc is None:
        return None
    return tuple(_need(sc, path + "rot.scaling.", key, float) for key in ("factor", "original", "fast", "slow"))


@dataclass(frozen=True)
class MatepelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    streams: int                                  # 0: one stream and plain residual sums
    layers: Tuple[Mapping[str, Any], ...]
    raw: Mapping[str, Any]

    architecture = "Matepel"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MatepelConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks required key 'layers' (a list of layer descriptions)")
        for i, layer in enumerate(layers):
            path = f"layers[{i}]."
            t = _need(layer, path, "type", str)
            if t not in LAYER_TYPES:
                raise ConfigError(f"{path}type = {t!r}; allowed: {', '.join(LAYER_TYPES)}")
            m, mp = layer.get("mixer"), path + "mixer."
            if not isinstance(m, Mapping):
                raise ConfigError(f"config.json lacks required key {path}mixer")
            if t == "lightning":
                for key in ("heads", "dim", "vdim"):
                    _need(m, mp, key, int)
                decay = m.get("decay")
                if not isinstance(decay, (list, tuple)) or len(decay) != m["heads"] \
                        or not all(isinstance(v, (int, float)) and not isinstance(v, bool) and 0 <= v <= 1 for v in decay):
                    raise ConfigError(f"{mp}decay must list {m['heads']} numbers between 0 and 1, one per head")
                if m["dim"] > MAX_KEY_DIM:
                    raise ConfigError(f"{mp}dim = {m['dim']}; at most {MAX_KEY_DIM}")
            else:
                left, lp = m.get("left"), mp + "left."
                for key in ("heads", "kv_heads", "dim"):
                    _need(left, lp, key, int)
                if left["heads"] % left["kv_heads"]:
                    raise ConfigError(f"{lp}heads = {left['heads']} is not a multiple of kv_heads = {left['kv_heads']}")
                if left.get("vdim") is not None and _need(left, lp, "vdim", int) != left["dim"]:
                    raise ConfigError(f"{lp}vdim = {left['vdim']} must equal dim = {left['dim']}: the values are the keys")
                if left["dim"] > MAX_HEAD_DIM:
                    raise ConfigError(f"{lp}dim = {left['dim']}; at most {MAX_HEAD_DIM}")
                _need(left, lp, "scale", float)
                rot = _rot(left, lp, left["dim"])
                if _yarn(left, lp) is not None and rot and rot[0] == 1.0:
                    raise ConfigError(f"{lp}rot.base = 1 cannot be rescaled")
                right, rp = m.get("right"), mp + "right."
                for key in ("heads", "dim", "vdim"):
                    _need(right, rp, key, int)
                if right["dim"] > MAX_KEY_DIM:
                    raise ConfigError(f"{rp}dim = {right['dim']}; at most {MAX_KEY_DIM}")
                _need(right, rp, "gate_cap", float)
                for key in ("left_scale", "right_scale"):
                    if m.get(key) is not None:
                        _need(m, mp, key, float, positive=False)
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{path}mlp.kind = {mlp.get('kind')!r}; allowed: dense")
                _need(mlp, path + "mlp.", "ff", int)
                _need(mlp, path + "mlp.", "limit", float)
        streams = 0
        if d.get("streams") is not None:
            streams = _need(d, "", "streams", int)
            if streams > MAX_STREAMS:
                raise ConfigError(f"streams = {streams}; at most {MAX_STREAMS}")
        mult = _need(d, "", "residual_mult", float, positive=False) if d.get("residual_mult") is not None else 1.0
        cfg = cls(vocab=_need(d, "", "vocab", int), width=_need(d, "", "width", int),
                  norm_eps=_need(d.get("norm"), "norm.", "eps", float), residual_mult=mult, streams=streams,
                  layers=tuple(layers), raw=dict(d))
        if not (math.isfinite(cfg.norm_eps) and math.isfinite(mult)):
            raise ConfigError("norm.eps and residual_mult must be finite")
        return cfg

    def to_dict(self) -> dict:
        return dict(self.raw)

    # ------------------------------------------------------------------ the model, as data
    def _mixer_spec(self, i: int, layer: Mapping[str, Any]):
        D, m = self.width, layer["mixer"]
        if layer["type"] == "lightning":
            return LightningSpec(hidden=D, n_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"],
                                 decay=tuple(float(v) for v in m["decay"]), eps=self.norm_eps)
        l, r, lp = m["left"], m["right"], f"layers[{i}].mixer.left."
        rot = _rot(l, lp, l["dim"])
        head = l["dim"] + l["dim"] % 2                       # (a rotation of an odd head's first coordinates leaves the last)
        position = RopeSpec(head, rot[0], "half", rotary_dims=rot[1], yarn=_yarn(l, lp)) if rot else NoPositionSpec()
        left = MappedAttentionSpec(hidden=D, n_heads=l["heads"], n_kv_heads=l["kv_heads"], key_dim=l["dim"], value_dim=l["dim"],
                                   position=position, softmax_scale=float(l["scale"]), n_maps=1, eps=self.norm_eps, bias=True,
                                   unit_sink=True, shared_kv=True)
        right = MLSTMSpec(hidden=D, n_heads=r["heads"], key_dim=r["dim"], value_dim=r["vdim"], gate_cap=float(r["gate_cap"]),
                          eps=self.norm_eps)
        return SideBySideSpec(hidden=D, left=left, right=right, eps=self.norm_eps, combine="weighted",
                              left_scale=float(m.get("left_scale", 1.0)), right_scale=float(m.get("right_scale", 1.0)))

    def model_spec(self) -> ModelSpec:
        D = self.width
        norm = RMSNormSpec(D, self.norm_eps, tensor="")
        options = dict(streams=self.streams or 1, residual_mult=self.residual_mult, plain=not self.streams)
        specs = []
        for i, layer in enumerate(self.layers):
            mlp = layer.get("mlp")
            ffn = None if mlp is None else SwiGLUSpec(D, mlp["ff"], names=dict(gate="gate", up="up", down="down"), weight_suffix="",
                                                      activation="clamped_glu", limit=float(mlp["limit"]), glu_alpha=GLU_ALPHA)
            names = dict(mixer="mix", ffn="mlp", mixer_norm="norm1", ffn_norm="norm2", mixer_hc="hc1", ffn_hc="hc2")
            specs.append(LayerSpec(mixer=self._mixer_spec(i, layer), ffn=ffn, mixer_norm=norm,
                                   ffn_norm=norm if ffn is not None else None, prefix=f"l{i}.", names=names, block="hyper",
                                   options=options))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden=D, layers=tuple(specs),
                         schedule=tuple(ScheduleEntry(i, i) for i in range(len(specs))), final_norm=norm, tie_head=False,
                         max_positions=0, embed_name="embed", final_norm_name="final.norm", head_name="head",
                         streams=self.streams or 1, embed_norm=norm, embed_norm_name="embed.norm")
