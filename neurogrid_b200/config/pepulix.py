"""Typed configuration of the Pepulix decoder, read from its own ``config.json`` keys.

Pepulix is a pre-norm decoder (RMS norms with plain weights) whose layers are listed one by one in ``layers``.  With
``streams`` the residual stream is that many copies tied by hyper-connections (every sublayer reads a weighted sum of the
copies and writes into all of them through a mixing matrix), and the final norm reads their sum; without it a layer adds
its sublayers' outputs to one stream.  The head is the embedding table; logits are soft-capped by ``logit_softcap``.

* ``type`` ``attention``: grouped-query causal attention without softmax: a key weighs sigmoid(score + a number per head),
  not normalised.  Biases on q, k and v; a partial rotation in pairs (i, i + dims/2), then q and k over their root mean
  square per head; values over theirs; with ``v_mix`` the values are blended with those of the first such layer; a
  sigmoid gate per head.
* ``type`` ``latent_attention``: causal softmax attention whose queries pass a normed latent (``q_rank``) and whose keys and
  values are expanded from a normed latent (``kv_rank``) per token; q and k also have ``rot_dim`` rotated coordinates (pairs
  (2i, 2i+1), frequencies rescaled by index with ``rot.scaling``), the key's shared by all heads; no gate.
* ``type`` ``mlstm``: the matrix memory of xLSTM, a recurrence with exponential gates soft-capped by ``gate_cap``; heads over
  their root mean square, a weight, a sigmoid gate.

The feed-forward (``mlp``, or null for none) is ``dense`` (down(silu(gate x) * up x), biases on all three) or ``moe``: softmax
scores over all of ``router.experts`` experts and ``router.identity`` identity experts behind them (their output is their
input), the ``router.top`` largest by score plus a stored correction, weighted by their scores over the scores' sum.

Keys: ``architecture``, ``vocab``, ``width``, ``streams``, ``norm.eps``, ``logit_softcap``, ``layers[i].type``,
``layers[i].mixer.{heads, kv_heads, dim, vdim, scale, v_mix, rot.{base, dims}}``, ``layers[i].mixer.{heads, dim, rot_dim,
vdim, q_rank, kv_rank, scale, rot.{base, dims, scaling.{factor, original, fast, slow}}}``, ``layers[i].mixer.{heads, dim,
vdim, gate_cap}``, ``layers[i].mlp.{kind, ff}`` or ``layers[i].mlp.{kind, router.{experts, identity, top}, expert.ff}``.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.{in, out, mix}``, ``l<i>.hc2.{in, out, mix}``,
``l<i>.mix.{q, q.b, k, k.b, v, v.b, vmix, pb, g, o}``, ``l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o}``,
``l<i>.mix.{q, k, v, g, o, norm, i, i.b, f, f.b}``, ``l<i>.mlp.{gate, gate.b, up, up.b, down, down.b}`` or
``l<i>.mlp.{router, correction, e<j>.{gate, up, down}}``, ``final.norm``.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .dodilix import MAX_STREAMS, _rot
from .lfm2 import ConfigError
from .matepel import MAX_KEY_DIM, _yarn
from .metanex import _need
from .specs import (LatentAttentionSpec, LayerSpec, MappedAttentionSpec, MLSTMSpec, ModelSpec, MoESpec, NoPositionSpec,
                    RMSNormSpec, RopeSpec, ScheduleEntry, SwiGLUSpec)

LAYER_TYPES = ("attention", "latent_attention", "mlstm")
MAX_VALUE_DIM = 256         # what the attention kernels take
MAX_LATENT = 768            # ... a cached row of the latent attention, its rotated part included
MAX_TOP = 32                # experts a token uses


def _at_most(m: Mapping[str, Any], path: str, key: str, most: int) -> None:
    if m[key] > most:
        raise ConfigError(f"{path}{key} = {m[key]}; at most {most}")


def _check_attention(m: Mapping[str, Any], mp: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _need(m, mp, key, int)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{mp}heads = {m['heads']} is not a multiple of kv_heads = {m['kv_heads']}")
    _at_most(m, mp, "dim", MAX_KEY_DIM)
    _at_most(m, mp, "vdim", MAX_VALUE_DIM)
    _need(m, mp, "scale", float)
    _rot(m, mp, m["dim"])
    if (m.get("rot") or {}).get("scaling") is not None:
        raise ConfigError(f"{mp}rot.scaling: this layer type's rotation is not rescaled")
    if not isinstance(m.get("v_mix", False), bool):
        raise ConfigError(f"{mp}v_mix must be true or false, got {m['v_mix']!r}")


def _check_latent(m: Mapping[str, Any], mp: str) -> None:
    for key in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
        _need(m, mp, key, int)
    _need(m, mp, "scale", float)
    rot_dim = _rot_dim(m, mp)
    rot = _rot(m, mp, rot_dim)
    if _yarn(m, mp) is not None and rot and rot[0] == 1.0:
        raise ConfigError(f"{mp}rot.base = 1 cannot be rescaled")
    if m["kv_rank"] + rot_dim > MAX_LATENT:
        raise ConfigError(f"{mp}kv_rank + rot_dim = {m['kv_rank'] + rot_dim}; at most {MAX_LATENT}")


def _rot_dim(m: Mapping[str, Any], mp: str) -> int:
    rot_dim = _need(m, mp, "rot_dim", int, positive=False) if m.get("rot_dim") is not None else 0
    if rot_dim < 0 or rot_dim % 2:
        raise ConfigError(f"{mp}rot_dim = {rot_dim} must be even and not negative")
    return rot_dim


def _check_mlp(mlp: Mapping[str, Any], mp: str) -> None:
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        _need(mlp, mp, "ff", int)
    elif kind == "moe":
        r, rp = mlp.get("router"), mp + "router."
        routed = _need(r, rp, "experts", int)
        if r.get("identity") is not None:
            if _need(r, rp, "identity", int, positive=False) < 0:
                raise ConfigError(f"{rp}identity = {r['identity']} must not be negative")
            routed += r["identity"]
        if _need(r, rp, "top", int) > min(routed, MAX_TOP):
            raise ConfigError(f"{rp}top = {r['top']}; at most {min(routed, MAX_TOP)} of {routed} experts")
        _need(mlp.get("expert"), mp + "expert.", "ff", int)
    else:
        raise ConfigError(f"{mp}kind = {kind!r}; allowed: dense, moe")


@dataclass(frozen=True)
class PepulixConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    streams: int                                  # 0: one stream and plain residual sums
    layers: Tuple[Mapping[str, Any], ...]
    raw: Mapping[str, Any]

    architecture = "Pepulix"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "PepulixConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks required key 'layers' (a list of layer descriptions)")
        mixing = None                             # the first layer whose values the others blend in
        for i, layer in enumerate(layers):
            path = f"layers[{i}]."
            t = _need(layer, path, "type", str)
            if t not in LAYER_TYPES:
                raise ConfigError(f"{path}type = {t!r}; allowed: {', '.join(LAYER_TYPES)}")
            m, mp = layer.get("mixer"), path + "mixer."
            if not isinstance(m, Mapping):
                raise ConfigError(f"config.json lacks required key {path}mixer")
            if t == "attention":
                _check_attention(m, mp)
                if m.get("v_mix"):
                    values = (m["kv_heads"], m["vdim"])
                    if mixing is not None and values != mixing[1]:
                        raise ConfigError(f"{mp}v_mix: (kv_heads, vdim) = {values} differs from layers[{mixing[0]}]'s {mixing[1]}")
                    mixing = mixing or (i, values)
            elif t == "latent_attention":
                _check_latent(m, mp)
            else:
                for key in ("heads", "dim", "vdim"):
                    _need(m, mp, key, int)
                _at_most(m, mp, "dim", MAX_KEY_DIM)
                _need(m, mp, "gate_cap", float)
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], path + "mlp.")
        streams = 0
        if d.get("streams") is not None:
            streams = _need(d, "", "streams", int)
            if streams > MAX_STREAMS:
                raise ConfigError(f"streams = {streams}; at most {MAX_STREAMS}")
        cfg = cls(vocab=_need(d, "", "vocab", int), width=_need(d, "", "width", int),
                  norm_eps=_need(d.get("norm"), "norm.", "eps", float),
                  logit_softcap=_need(d, "", "logit_softcap", float) if d.get("logit_softcap") is not None else None,
                  streams=streams, layers=tuple(layers), raw=dict(d))
        if not math.isfinite(cfg.norm_eps):
            raise ConfigError("norm.eps must be finite")
        return cfg

    def to_dict(self) -> dict:
        return dict(self.raw)

    # ------------------------------------------------------------------ the model, as data
    def _mixer_spec(self, i: int, layer: Mapping[str, Any]):
        D, m, mp = self.width, layer["mixer"], f"layers[{i}].mixer."
        if layer["type"] == "mlstm":
            return MLSTMSpec(hidden=D, n_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"], gate_cap=float(m["gate_cap"]),
                             eps=self.norm_eps)
        if layer["type"] == "latent_attention":
            rot_dim = _rot_dim(m, mp)
            rot = _rot(m, mp, rot_dim)
            position = RopeSpec(rot_dim, rot[0] if rot else 1.0, "adjacent", rotary_dims=rot[1] if rot else 0,
                                yarn=_yarn(m, mp) if rot else None) if rot_dim else None
            return LatentAttentionSpec(hidden=D, n_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"], q_rank=m["q_rank"],
                                       kv_rank=m["kv_rank"], softmax_scale=float(m["scale"]), eps=self.norm_eps, window=None,
                                       rope_dim=rot_dim, position=position, gate="none")
        rot = _rot(m, mp, m["dim"])
        head = m["dim"] + m["dim"] % 2                       # (a rotation of an odd head's first coordinates leaves the last)
        position = RopeSpec(head, rot[0], "half", rotary_dims=rot[1]) if rot else NoPositionSpec()
        first = next((j for j, l in enumerate(self.layers) if l["type"] == "attention" and l["mixer"].get("v_mix")), None)
        mix = None if not m.get("v_mix") else "source" if i == first else "mix"
        return MappedAttentionSpec(hidden=D, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                                   position=position, softmax_scale=float(m["scale"]), n_maps=1, qk_norm=True, norm_weight=False,
                                   eps=self.norm_eps, bias=True, o_bias=False, weights="sigmoid", score_bias=True,
                                   value_norm=True, value_mix=mix, head_gate=True)

    def _ffn_spec(self, layer: Mapping[str, Any]):
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        if mlp.get("kind", "dense") == "dense":
            return SwiGLUSpec(self.width, mlp["ff"], names=dict(gate="gate", up="up", down="down"), weight_suffix="", bias=True)
        r = mlp["router"]
        return MoESpec(hidden=self.width, n_experts=r["experts"], top_k=r["top"], expert_ff=mlp["expert"]["ff"],
                       scoring="softmax_all", correction=True, identity=int(r.get("identity") or 0))

    def model_spec(self) -> ModelSpec:
        D = self.width
        norm = RMSNormSpec(D, self.norm_eps, tensor="")
        options = dict(streams=self.streams or 1, plain=not self.streams)
        names = dict(mixer="mix", ffn="mlp", mixer_norm="norm1", ffn_norm="norm2", mixer_hc="hc1", ffn_hc="hc2")
        specs = []
        for i, layer in enumerate(self.layers):
            ffn = self._ffn_spec(layer)
            specs.append(LayerSpec(mixer=self._mixer_spec(i, layer), ffn=ffn, mixer_norm=norm,
                                   ffn_norm=norm if ffn is not None else None, prefix=f"l{i}.", names=names, block="hyper",
                                   options=options))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden=D, layers=tuple(specs),
                         schedule=tuple(ScheduleEntry(i, i) for i in range(len(specs))), final_norm=norm, tie_head=True,
                         max_positions=0, embed_name="embed", final_norm_name="final.norm",
                         logit_softcap=self.logit_softcap, streams=self.streams or 1)
