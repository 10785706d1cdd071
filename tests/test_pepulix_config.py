"""Pepulix on the CPU: configuration keys and errors, the model as data, declared tensors, cache needs, the oracle's own
properties, and the engine's host side with every launcher replaced by its plain statement."""
import copy
import math
import tempfile

import pytest
import torch

import kernel_refs
import pepulix_models as pm
import plain_pepulix as plain
import scenarios
from helpers import make_runner, rel_err
from neurogrid_b200.cache.manager import PagedNeed, SlotNeed
from neurogrid_b200.config import config_from_dict
from neurogrid_b200.config.lfm2 import ConfigError
from neurogrid_b200.config.specs import LatentAttentionSpec, MappedAttentionSpec, MoESpec, RopeSpec
from neurogrid_b200.engine import StepEntry
from neurogrid_b200.models import declare_tensors
from neurogrid_b200.models.decoder import Decoder
from neurogrid_b200.parts.position import Rope

F64 = torch.float64


def test_spec_of_every_option():
    spec = config_from_dict(pm.PEPU_A).model_spec()
    assert spec.architecture == "Pepulix" and spec.streams == 3 and spec.tie_head and spec.logit_softcap == 9.0
    assert [l.block for l in spec.layers] == ["hyper"] * 7
    assert all(l.options == dict(streams=3, plain=False) for l in spec.layers)
    assert [(e.layer, e.cache, e.writes) for e in spec.schedule] == [(i, i, True) for i in range(7)]
    assert [getattr(l.mixer, "value_mix", None) for l in spec.layers] == [None, "source", None, None, "mix", None, "mix"]
    a = spec.layers[1].mixer
    assert (a.weights, a.score_bias, a.value_norm, a.head_gate, a.out_gate, a.bias, a.o_bias) == \
        ("sigmoid", True, True, True, False, True, False)
    assert (a.qk_norm, a.norm_weight, a.eps, a.softmax_scale, a.window, a.chunk) == (True, False, 2e-6, 0.4, None, None)
    assert (a.position.pairing, a.position.rotary_dims, a.position.theta, a.position.yarn) == ("half", 16, 1000.0, None)
    assert spec.layers[0].mixer.position.kind == "none"
    m = spec.layers[2].mixer
    assert (m.kind, m.n_heads, m.key_dim, m.value_dim, m.gate_cap) == ("mlstm", 3, 8, 10, 3.0)
    l = spec.layers[3].mixer
    assert (l.kind, l.gate, l.rope_dim, l.q_rank, l.kv_rank, l.window) == ("latent_attention", "none", 8, 28, 20, None)
    assert (l.position.pairing, l.position.rotary_dims, l.position.yarn) == ("adjacent", 8, (6.0, 64.0, 8.0, 0.5))
    assert spec.layers[5].mixer.position.yarn is None
    f = spec.layers[0].ffn
    assert (f.kind, f.activation, f.bias, f.intermediate) == ("swiglu", "silu", True, 36)
    r = spec.layers[1].ffn
    assert (r.kind, r.scoring, r.correction, r.n_experts, r.identity, r.top_k, r.expert_ff, r.shared_ff, r.n_groups) == \
        ("moe", "softmax_all", True, 6, 3, 3, 20, 0, 1)
    assert spec.layers[4].ffn is None and spec.layers[6].ffn.identity == 0
    b = config_from_dict(pm.PEPU_B).model_spec()
    assert b.logit_softcap is None and b.layers[1].mixer.rope_dim == 0 and b.layers[1].mixer.position is None
    plain_spec = config_from_dict(pm.PEPU_B0).model_spec()
    assert plain_spec.streams == 1 and all(l.options == dict(streams=1, plain=True) for l in plain_spec.layers)


def test_declared_tensors():
    names = declare_tensors(config_from_dict(pm.PEPU_A).model_spec())
    for n, shape in {"embed": (131, 60), "final.norm": (60,), "l0.hc1.mix": (3, 3), "l0.hc2.in": (3,), "l0.mix.q": (18, 60),
                     "l0.mix.q.b": (18,), "l0.mix.v.b": (7,), "l0.mix.pb": (2,), "l0.mix.g": (2, 60), "l0.mix.o": (60, 14),
                     "l0.mlp.gate.b": (36,), "l0.mlp.down.b": (60,), "l1.mix.vmix": (), "l4.mix.vmix": (), "l1.mix.k.b": (40,),
                     "l1.mlp.router": (9, 60), "l1.mlp.correction": (9,), "l1.mlp.e5.down": (60, 20), "l2.mix.norm": (30,),
                     "l2.mix.i": (3, 60), "l2.mix.f.b": (3,), "l3.mix.dq": (28, 60), "l3.mix.dq.norm": (28,),
                     "l3.mix.uq": (60, 28), "l3.mix.dkv": (28, 60), "l3.mix.dkv.norm": (20,), "l3.mix.uk": (36, 20),
                     "l3.mix.uv": (30, 20), "l3.mix.o": (60, 30)}.items():
        assert names[n].shape == shape, n
    absent = ("head", "l0.mix.vmix", "l0.mix.o.b", "l1.mlp.e6.", "l1.mlp.e0.gate.b", "l3.mix.g", "l4.norm2", "l4.hc2", "l1.mlp.shared")
    assert not any(n.startswith(absent) for n in names)
    assert not any(".hc" in n for n in declare_tensors(config_from_dict(pm.PEPU_B0).model_spec()))


def _broken(path, value):
    cfg = copy.deepcopy(pm.PEPU_A)
    node = cfg
    for k in path[:-1]:
        node = node[k]
    if value is None:
        node.pop(path[-1])
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "conv", "type"),
    (("layers", 0, "mixer", "heads"), 3, None),
    (("layers", 1, "mixer", "heads"), 5, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), None, "vdim"),
    (("layers", 1, "mixer", "vdim"), 300, "vdim"),
    (("layers", 1, "mixer", "dim"), 513, "dim"),
    (("layers", 1, "mixer", "scale"), None, "scale"),
    (("layers", 1, "mixer", "v_mix"), 1, "v_mix"),
    (("layers", 1, "mixer", "rot", "dims"), 22, "rot.dims"),
    (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}, "rot.scaling"),
    (("layers", 4, "mixer", "vdim"), 24, "v_mix"),
    (("layers", 1, "mlp", "router", "top"), 10, "top"),
    (("layers", 1, "mlp", "router", "identity"), -1, "identity"),
    (("layers", 1, "mlp", "expert"), None, "expert"),
    (("layers", 1, "mlp", "kind"), "sparse", "kind"),
    (("layers", 0, "mlp", "ff"), None, "ff"),
    (("layers", 2, "mixer", "gate_cap"), None, "gate_cap"),
    (("layers", 2, "mixer", "dim"), 600, "dim"),
    (("layers", 3, "mixer", "kv_rank"), None, "kv_rank"),
    (("layers", 3, "mixer", "kv_rank"), 800, "kv_rank"),
    (("layers", 3, "mixer", "rot_dim"), 7, "rot_dim"),
    (("layers", 3, "mixer", "rot", "dims"), 10, "rot.dims"),
    (("layers", 3, "mixer", "rot", "scaling", "slow"), None, "rot.scaling.slow"),
    (("layers", 3, "mixer", "rot", "base"), 1.0, "rot.base"),
    (("streams",), 40, "streams"),
    (("logit_softcap",), -1.0, "logit_softcap"),
    (("norm",), None, "norm.eps"),
])
def test_config_errors_name_the_key(path, value, word):
    if word is None:                                         # three query heads on one key/value head are fine
        config_from_dict(_broken(path, value))
        return
    with pytest.raises(ConfigError) as e:
        config_from_dict(_broken(path, value))
    assert word in str(e.value)


def test_cache_needs():
    spec = config_from_dict(pm.PEPU_A).model_spec()
    needs = Decoder(spec, dtype=torch.float32, device="cpu").cache_needs()
    assert needs[1] == PagedNeed(2, 20, None, True, v_heads=2, v_dim=12, keep_first=0)
    assert needs[2] == (SlotNeed((3, 8, 10)), SlotNeed((3, 1, 9)))
    assert needs[3] == PagedNeed(1, 32, None, values=False)                   # 20 latent + 8 rotated columns, in sixteens
    assert needs[5] == PagedNeed(1, 48, None, values=False)                   # 33 + 4
    half = Decoder(spec, dtype=torch.bfloat16, device="cpu").cache_needs()
    assert half[5] == PagedNeed(1, 64, None, values=False)                    # in steps the tensor-core core takes


def test_specs_refuse_what_no_kernel_does():
    kw = dict(hidden=8, n_heads=2, n_kv_heads=1, key_dim=4, value_dim=4, softmax_scale=1.0, position=RopeSpec(4, 100.0))
    for bad in (dict(weights="tanh"), dict(score_bias=True), dict(weights="sigmoid", sink=True), dict(weights="sigmoid", unit_sink=True),
                dict(weights="sigmoid", n_maps=2), dict(value_mix="first"), dict(value_norm=True, shared_kv=True),
                dict(head_gate=True, out_gate=True)):
        with pytest.raises(ValueError):
            MappedAttentionSpec(**kw, **bad)
    moe = dict(hidden=8, n_experts=2, expert_ff=4)
    with pytest.raises(ValueError):
        MoESpec(**moe, top_k=1, identity=2)                                    # softmax over the chosen: no identity experts
    with pytest.raises(ValueError):
        MoESpec(**moe, top_k=5, identity=2, scoring="softmax_all")
    with pytest.raises(ValueError):
        LatentAttentionSpec(8, 1, 4, 4, 4, 700, 1.0, 1e-5, rope_dim=70, position=RopeSpec(70, 10.0))
    with pytest.raises(ValueError):
        LatentAttentionSpec(8, 1, 4, 4, 4, 4, 1.0, 1e-5, gate="row")


@pytest.mark.parametrize("rot", [
    dict(base=1000.0, dims=8, scaling=dict(factor=6.0, original=64, fast=8.0, slow=0.5)),         # all three branches
    dict(base=10000.0, dims=24, scaling=dict(factor=8.0, original=512, fast=16.0, slow=1.0)),
    dict(base=10.0, dims=4, scaling=dict(factor=4.0, original=4, fast=6.0, slow=5.0)),            # both edges at the start
    dict(base=100.0, dims=32, scaling=dict(factor=3.0, original=100000, fast=2.0, slow=1.0)),     # nothing is divided
    dict(base=1e6, dims=64, scaling=dict(factor=1.0, original=1536, fast=40.0, slow=2.0)),
    dict(base=30.0, dims=10),
])
def test_frequencies(rot):
    sc = rot.get("scaling")
    part = Rope(RopeSpec(rot["dims"], rot["base"], "adjacent", rotary_dims=rot["dims"],
                         yarn=(sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None), device="cpu").kernel_args()
    f, mag = plain.pair_frequencies(rot)
    assert torch.allclose(part.inv_freq.double(), f, rtol=1e-6, atol=0) and abs(part.magnitude - mag) < 1e-12


LENS = {"A": [1, 9, 40, 67, 23], "B": [3, 50, 30], "B0": [2, 41], "C": [2, 17, 90, 33], "D": [1, 30, 12]}


@pytest.mark.parametrize("name", ["A", "B", "B0", "C", "D"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
def test_engine_host_side_against_plain(pepulix_dirs, monkeypatch, name, cut):
    """The step function, cache manager and parts on the CPU, every launcher replaced by its plain statement: the states,
    pages, slots and mixed values reach the right layer of the right request however the work is cut."""
    kernel_refs.install(monkeypatch)
    cfg, w = pm.load_plain(pepulix_dirs[name])
    reqs = scenarios.make_requests(LENS[name], cfg["vocab"], seed=17)
    ps = pm.PAGE_SIZE[name]
    cap = 128 if cut == "mixed" else 256
    runner = make_runner(pepulix_dirs[name], dtype=torch.float32, device="cpu", page_size=ps, num_pages=cap // ps,
                         max_requests=4, max_seq_len=cap)
    steps = {"whole": scenarios.whole, "tail_decode": lambda r: scenarios.tail_decode(r, 12), "portions": scenarios.portions,
             "mixed": lambda r: scenarios.mixed(r, cap, round_to=ps)}[cut](reqs)
    got = []
    for s in steps:
        got.append(runner.step([StepEntry(e["id"], e["tokens"], e["want"]) for e in s["entries"]]).clone())
        for r in s["end"]:
            runner.finish(r)
        runner.cache.check()
    got = scenarios.collect(steps, lambda i: got[i])
    for r, t in reqs.items():
        assert rel_err(got[r], plain.forward(cfg, w, t)) < 2e-5, (r, len(t))
    assert all(f == cap // ps for f in runner.cache.pages_free()) and runner.cache.slots_free() == 4


def test_oracle_is_causal_and_its_mechanisms_bite():
    cfg, w = pm.load_plain(pm.write_model(pm.PEPU_A, 5, tempfile.mkdtemp()))
    toks = scenarios.make_requests([48], cfg["vocab"], seed=2)["r0"]
    a = plain.forward(cfg, w, toks)
    assert rel_err(a[:30], plain.forward(cfg, w, toks[:30])) < 1e-12
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    assert rel_err(plain.forward(cfg, w, other)[40:], a[40:]) > 1e-4         # the first token still shows

    def changed(edit):
        c2, w2 = copy.deepcopy(cfg), dict(w)
        edit(c2, w2)
        return rel_err(plain.forward(c2, w2, toks), a)

    def scale(name, f):
        return lambda c, ww: ww.__setitem__(name, ww[name] * f)

    mixer = lambda c, i: c["layers"][i]["mixer"]
    for i in (1, 4, 6):
        assert changed(scale(f"l{i}.mix.pb", 0.9)) > 1e-4, i
        assert changed(scale(f"l{i}.mix.g", 0.0)) > 1e-3, i
        assert changed(lambda c, ww: mixer(c, i).__setitem__("scale", mixer(c, i)["scale"] * 0.9)) > 1e-4, i
        for b in ("q.b", "k.b", "v.b"):
            assert changed(scale(f"l{i}.mix.{b}", 0.0)) > 1e-4, (i, b)
    assert changed(scale("l4.mix.vmix", 0.9)) > 1e-4 and changed(scale("l6.mix.vmix", 0.9)) > 1e-4
    assert changed(scale("l1.mix.vmix", 0.0)) == 0.0                          # the first layer's own share is not used
    assert changed(lambda c, ww: mixer(c, 4).__setitem__("v_mix", False)) > 1e-3
    assert changed(lambda c, ww: mixer(c, 1)["rot"].__setitem__("dims", 12)) > 1e-4
    assert changed(lambda c, ww: mixer(c, 3)["rot"].pop("scaling")) > 1e-5
    assert changed(lambda c, ww: mixer(c, 3)["rot"]["scaling"].__setitem__("factor", 3.0)) > 1e-5
    assert changed(scale("l3.mix.dq.norm", 0.8)) > 1e-5 and changed(scale("l3.mix.dkv.norm", 0.8)) > 1e-5
    assert changed(scale("l2.mix.i.b", 0.5)) > 1e-4 and changed(scale("l2.mix.f.b", 0.5)) > 1e-4
    assert changed(lambda c, ww: mixer(c, 2).__setitem__("gate_cap", 2.0)) > 1e-4
    for b in ("gate.b", "up.b", "down.b"):
        assert changed(scale(f"l2.mlp.{b}", 0.0)) > 1e-4, b
    assert changed(scale("l1.mlp.correction", 0.0)) > 1e-4
    assert changed(lambda c, ww: ww.__setitem__("l1.mlp.router", torch.cat([ww["l1.mlp.router"][3:], ww["l1.mlp.router"][:3]]))) > 1e-3
    assert changed(scale("l1.hc2.mix", 0.9)) > 1e-4 and changed(lambda c, ww: c.__setitem__("logit_softcap", 8.0)) > 1e-3


def test_sigmoid_weights_and_mixed_values_of_the_oracle():
    """Weights are no softmax: two equal keys weigh twice one, and a key far below the bend nothing."""
    q = torch.tensor([[0.0, 0.0], [1.0, 0.0], [1.0, 0.0]], dtype=F64)
    k = torch.tensor([[1.0, 0.0], [1.0, 0.0], [-50.0, 0.0]], dtype=F64)
    w = plain.sigmoid_weights(q, k, 2.0, -1.0)
    s = torch.sigmoid(torch.tensor(1.0, dtype=F64))
    assert torch.allclose(w[0], torch.sigmoid(torch.tensor([-1.0, -math.inf, -math.inf], dtype=F64)))
    assert torch.allclose(w[2], torch.stack([s, s, torch.zeros((), dtype=F64)]), atol=1e-12)
    assert torch.equal(plain.mix_values(torch.ones(2, dtype=F64), 3 * torch.ones(2, dtype=F64), 0.25), torch.full((2,), 1.5, dtype=F64))
