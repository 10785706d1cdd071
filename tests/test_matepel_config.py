"""Matepel on the CPU: configuration keys and errors, the model as data, declared tensors, cache needs, the oracle's own
properties, and the engine's host side with every launcher replaced by its plain statement."""
import copy
import math
import tempfile

import pytest
import torch

import kernel_refs
import matepel_models as mm
import plain_matepel as plain
import scenarios
from helpers import make_runner, rel_err
from neurogrid_b200.cache.manager import PagedNeed, SlotNeed
from neurogrid_b200.config import config_from_dict
from neurogrid_b200.config.lfm2 import ConfigError
from neurogrid_b200.config.specs import MappedAttentionSpec, RopeSpec
from neurogrid_b200.engine import StepEntry
from neurogrid_b200.models import declare_tensors
from neurogrid_b200.models.decoder import Decoder
from neurogrid_b200.parts.position import Rope


def test_spec_of_every_option():
    spec = config_from_dict(mm.MATE_A).model_spec()
    assert spec.architecture == "Matepel" and spec.streams == 3 and spec.embed_norm.eps == 2e-6
    assert [l.block for l in spec.layers] == ["hyper"] * 4
    assert all(l.options == dict(streams=3, residual_mult=0.7, plain=False) for l in spec.layers)
    assert [(e.layer, e.cache, e.writes) for e in spec.schedule] == [(i, i, True) for i in range(4)]
    light, par = spec.layers[0].mixer, spec.layers[1].mixer
    assert (light.kind, light.n_heads, light.key_dim, light.value_dim, light.decay) == \
        ("lightning_attention", 3, 8, 10, (0.3, 0.9, 0.995))
    assert par.kind == "side_by_side" and par.combine == "weighted" and (par.left_scale, par.right_scale) == (0.8, 1.25)
    left, right = par.left, par.right
    assert (left.shared_kv, left.unit_sink, left.sink, left.bias, left.window, left.chunk) == (True, True, False, True, None, None)
    assert (left.position.pairing, left.position.rotary_dims, left.position.theta, left.position.yarn) == \
        ("half", 16, 1000.0, (6.0, 64.0, 8.0, 0.5))
    assert (right.kind, right.gate_cap, right.key_dim, right.value_dim) == ("mlstm", 3.0, 12, 6)
    ff = spec.layers[0].ffn
    assert (ff.activation, ff.limit, ff.glu_alpha, ff.intermediate) == ("clamped_glu", 0.9, 1.702, 40)
    assert spec.layers[2].ffn is None and spec.layers[3].ffn is None
    b = config_from_dict(mm.MATE_B).model_spec()
    assert b.layers[0].mixer.left.position.kind == "none" and b.layers[0].options["residual_mult"] == 1.0
    assert (b.layers[0].mixer.left_scale, b.layers[0].mixer.right_scale) == (1.0, 1.0)
    plain_spec = config_from_dict(mm.MATE_B0).model_spec()
    assert plain_spec.streams == 1 and all(l.options == dict(streams=1, residual_mult=0.5, plain=True) for l in plain_spec.layers)


def test_declared_tensors():
    names = declare_tensors(config_from_dict(mm.MATE_A).model_spec())
    for n, shape in {"embed": (133, 56), "embed.norm": (56,), "head": (133, 56), "final.norm": (56,), "l0.hc1.mix": (3, 3),
                     "l0.hc2.in": (3,), "l0.mix.q": (24, 56), "l0.mix.v": (30, 56), "l0.mix.g": (30, 56), "l0.mix.o": (56, 30),
                     "l0.mix.norm": (30,), "l0.mlp.gate": (40, 56), "l1.mix.left.q": (80, 56), "l1.mix.left.q.b": (80,),
                     "l1.mix.left.k": (40, 56), "l1.mix.left.k.b": (40,), "l1.mix.left.o": (56, 80), "l1.mix.left.o.b": (56,),
                     "l1.mix.right.i": (2, 56), "l1.mix.right.i.b": (2,), "l1.mix.right.f": (2, 56), "l1.mix.right.f.b": (2,),
                     "l1.mix.right.norm": (12,), "l1.mix.right.v": (12, 56), "l1.mlp.down": (56, 36), "l1.norm2": (56,),
                     "l3.mix.right.norm": (180,)}.items():
        assert names[n].shape == shape, n
    assert not any(n.startswith(("l2.hc2", "l2.norm2", "l2.mlp", "l1.mix.left.v", "l1.mix.left.sink")) for n in names)
    assert not any(".hc" in n for n in declare_tensors(config_from_dict(mm.MATE_B0).model_spec()))


def _broken(path, value):
    cfg = copy.deepcopy(mm.MATE_A)
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
    (("layers", 0, "mixer", "decay"), [0.5, 0.5], "decay"),
    (("layers", 0, "mixer", "decay"), [0.5, 0.5, 1.5], "decay"),
    (("layers", 0, "mixer", "vdim"), None, "vdim"),
    (("layers", 0, "mixer", "dim"), 1024, "dim"),
    (("layers", 0, "mlp", "limit"), None, "limit"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"),
    (("layers", 1, "mixer", "left", "heads"), 5, "kv_heads"),
    (("layers", 1, "mixer", "left", "vdim"), 16, "vdim"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 22, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "scaling", "slow"), None, "rot.scaling.slow"),
    (("layers", 1, "mixer", "left", "rot", "base"), 1.0, "rot.base"),
    (("layers", 1, "mixer", "left", "scale"), None, "scale"),
    (("layers", 1, "mixer", "right", "gate_cap"), None, "gate_cap"),
    (("streams",), 40, "streams"),
    (("norm",), None, "norm.eps"),
])
def test_config_errors_name_the_key(path, value, word):
    with pytest.raises(ConfigError) as e:
        config_from_dict(_broken(path, value))
    assert word in str(e.value)


def test_cache_needs():
    needs = Decoder(config_from_dict(mm.MATE_A).model_spec(), dtype=torch.float32, device="cpu").cache_needs()
    assert set(needs) == {0, 1, 2, 3}
    assert needs[0] == SlotNeed((3, 8, 10)) and needs[2] == SlotNeed((2, 14, 40))
    paged, state, nm = needs[3]
    assert paged == PagedNeed(3, 12, None, True, v_heads=3, v_dim=12)
    assert state == SlotNeed((5, 24, 36)) and nm == SlotNeed((5, 2, 25))       # 36 value columns: two slices, each with n and m


def test_specs_refuse_what_no_kernel_does():
    kw = dict(hidden=8, n_heads=2, n_kv_heads=1, key_dim=4, value_dim=4, softmax_scale=1.0)
    rope = RopeSpec(4, 100.0, "half", yarn=(2.0, 64.0, 8.0, 1.0))
    with pytest.raises(ValueError):
        MappedAttentionSpec(position=rope, qk_norm=True, norm_weight=False, **kw)      # that norm assumes lengths stay
    with pytest.raises(ValueError):
        MappedAttentionSpec(position=rope, sink=True, unit_sink=True, **kw)
    with pytest.raises(ValueError):
        MappedAttentionSpec(position=rope, shared_kv=True, **{**kw, "value_dim": 6})
    with pytest.raises(ValueError):
        RopeSpec(4, 100.0, "half", yarn=(2.0, 64.0, 8.0, 1.0), freq_scaling=(2.0, 1.0, 4.0, 64.0))


@pytest.mark.parametrize("rot", [
    dict(base=1000.0, dims=16, scaling=dict(factor=6.0, original=64, fast=8.0, slow=0.5)),        # all three branches
    dict(base=10000.0, dims=24, scaling=dict(factor=8.0, original=512, fast=16.0, slow=1.0)),
    dict(base=50.0, dims=4, scaling=dict(factor=2.0, original=300, fast=20.0, slow=2.0)),
    dict(base=10.0, dims=4, scaling=dict(factor=4.0, original=4, fast=6.0, slow=5.0)),            # both edges at the start
    dict(base=100.0, dims=32, scaling=dict(factor=3.0, original=100000, fast=2.0, slow=1.0)),     # nothing is divided
    dict(base=1e6, dims=64, scaling=dict(factor=1.0, original=1536, fast=40.0, slow=2.0)),
])
def test_rescaled_frequencies(rot):
    sc = rot["scaling"]
    part = Rope(RopeSpec(rot["dims"], rot["base"], "half", rotary_dims=rot["dims"],
                         yarn=(sc["factor"], sc["original"], sc["fast"], sc["slow"])), device="cpu").kernel_args()
    f, mag = plain.scaled_frequencies(rot)
    assert torch.allclose(part.inv_freq.double(), f, rtol=1e-6, atol=0)
    assert abs(part.magnitude - mag) < 1e-12 and abs(mag - (0.1 * math.log(sc["factor"]) + 1)) < 1e-12


LENS = {"A": [1, 9, 40, 67, 23], "B": [3, 50, 30], "B0": [2, 41], "C": [2, 17, 90, 33], "D": [1, 30, 12]}


@pytest.mark.parametrize("name", ["A", "B", "B0", "C", "D"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed"])
def test_engine_host_side_against_plain(matepel_dirs, monkeypatch, name, cut):
    """The step function, cache manager and parts on the CPU, every launcher replaced by its plain statement: the
    states, pages and slots reach the right layer of the right request however the work is cut."""
    kernel_refs.install(monkeypatch)
    cfg, w = mm.load_plain(matepel_dirs[name])
    reqs = scenarios.make_requests(LENS[name], cfg["vocab"], seed=17)
    ps = mm.PAGE_SIZE[name]
    cap = 128 if cut == "mixed" else 256
    runner = make_runner(matepel_dirs[name], dtype=torch.float32, device="cpu", page_size=ps, num_pages=cap // ps,
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
    cfg, w = mm.load_plain(mm.write_model(mm.MATE_A, 5, tempfile.mkdtemp()))
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

    left = lambda c, i=1: c["layers"][i]["mixer"]["left"]
    assert changed(lambda c, ww: c.__setitem__("residual_mult", 0.75)) > 1e-3
    assert changed(scale("embed.norm", 0.9)) > 1e-4
    assert changed(lambda c, ww: c["layers"][0]["mixer"].__setitem__("decay", [0.3, 0.9, 0.99])) > 1e-4
    assert changed(scale("l2.mix.g", 0.0)) > 1e-3
    assert changed(lambda c, ww: ww.__setitem__("l0.mix.norm", ww["l0.mix.norm"].flip(0))) > 1e-3
    assert changed(lambda c, ww: left(c)["rot"].__setitem__("dims", 12)) > 1e-4
    assert changed(lambda c, ww: left(c)["rot"].pop("scaling")) > 1e-4
    assert changed(lambda c, ww: left(c)["rot"]["scaling"].__setitem__("factor", 3.0)) > 1e-4
    assert changed(lambda c, ww: left(c)["rot"]["scaling"].__setitem__("slow", 1.0)) > 1e-5
    assert changed(scale("l1.mix.left.q.b", 0.0)) > 1e-3
    assert changed(scale("l1.mix.left.k.b", 0.0)) > 1e-3
    assert changed(scale("l1.mix.left.o.b", 0.0)) > 1e-3
    assert changed(lambda c, ww: c["layers"][1]["mixer"].__setitem__("left_scale", 0.85)) > 1e-4
    assert changed(lambda c, ww: c["layers"][1]["mixer"]["right"].__setitem__("gate_cap", 2.0)) > 1e-4
    assert changed(scale("l1.mix.right.i.b", 0.5)) > 1e-4
    assert changed(scale("l1.mix.right.f.b", 0.5)) > 1e-4
    assert changed(lambda c, ww: c["layers"][1]["mlp"].__setitem__("limit", 1.1)) > 1e-4
    assert changed(scale("l1.hc2.mix", 0.9)) > 1e-4


def test_matrix_memory_branches():
    """The oracle's memory: the running maximum starts at 0 and both sides of the denominator's maximum are met."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v = r(12, 1, 4), r(12, 1, 4), r(12, 1, 3)
    low = torch.full((12, 1), -6.0, dtype=torch.float64)
    o, (S, n, m) = plain.matrix_memory(q, k, v, low, torch.full((12, 1), -0.01, dtype=torch.float64))
    assert abs(float(m) + 0.12) < 1e-12                        # no input gate reaches the decaying start
    want = math.exp(-6) * (k[0] * q[0]).sum() * v[0, 0]        # the normaliser is far below exp(-m): divided by that
    assert torch.allclose(o[0, 0], want / (math.exp(0.01) * math.exp(-0.01) + 1e-6) , rtol=2e-2)
    high = torch.full((12, 1), 4.0, dtype=torch.float64)
    o, (_, _, m) = plain.matrix_memory(q, k, v, high, torch.full((12, 1), -0.5, dtype=torch.float64))
    assert float(m) == 4.0 and torch.allclose(o[0, 0], v[0, 0] * torch.sign((k[0] * q[0]).sum()), rtol=1e-3)
