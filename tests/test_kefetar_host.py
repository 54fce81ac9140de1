"""Kefetar without a GPU: the configuration's checks, what the builder makes of a configuration (parts, tensor names and
shapes, cache needs, which layer leads the blended values), the library's pieces that need no kernel (the divided frequency
table, a gain without dimensions, convolution weights laid out over padded heads), and the plain implementation's mechanisms
against restatements of their own definitions."""
import copy
import math

import numpy as np
import pytest
import torch

from tinyllama_c_b200.config import ConfigError, config_from_dict
from tinyllama_c_b200.config.base import lookup_architecture
from tinyllama_c_b200.parts.base import ChunkRequest, KVRequest, PartSpec, StateRequest
from tinyllama_c_b200.parts.position import RotaryNeox
from tinyllama_c_b200.weights.loader import WeightError, check_tensors, random_tensors

import configs
from plain import kefetar_plain as plain


def build(cfg: dict):
    c = config_from_dict(cfg)
    return lookup_architecture(c.architecture)[1](c)


def test_builder_names_shapes_and_cache_needs():
    m = build(configs.KEFETAR_A)
    got = {s.name: tuple(s.shape) for s in m.weight_specs()}
    assert got["embed"] == (150, 52) and got["head"] == (150, 52) and got["final.norm"] == ()
    # attention: heads of 24 and values of 16, two taps on every channel of q, k and v, a gate of the values' size, no share
    assert got["l0.norm1"] == () and got["l0.norm2"] == () and got["l0.canon1"] == (52, 3) and got["l0.canon2"] == (52, 3)
    assert got["l0.mix.q"] == (96, 52) and got["l0.mix.k"] == (48, 52) and got["l0.mix.v"] == (32, 52) and got["l0.mix.g"] == (64, 52)
    assert got["l0.mix.q.conv"] == (96, 2) and got["l0.mix.k.conv"] == (48, 2) and got["l0.mix.v.conv"] == (32, 2)
    assert got["l0.mix.o"] == (52, 64) and "l0.mix.vmix" not in got
    assert got["l0.mlp.up"] == (44, 52) and got["l0.mlp.down"] == (52, 44) and got["l0.mlp.act"] == (4,) and "l0.mlp.gate" not in got
    # retention, no feed-forward
    assert got["l1.mix.q"] == (36, 52) and got["l1.mix.v"] == (60, 52) and got["l1.mix.g"] == (60, 52) and got["l1.mix.o"] == (52, 60)
    assert "l1.norm2" not in got and "l1.canon2" not in got and not any(n.startswith("l1.mlp") for n in got)
    # the first of the layers that blend has no share of its own to take, the later ones do
    assert "l2.mix.vmix" not in got and got["l3.mix.vmix"] == () and got["l5.mix.vmix"] == ()
    reqs = m.cache_requests()
    assert reqs[0] == [StateRequest("canon1", (2, 52)), KVRequest("kv", 2, 24), StateRequest("kv.conv", (1, 8 * 24)), StateRequest("canon2", (2, 52))]
    assert reqs[1] == [StateRequest("canon1", (2, 52)), StateRequest("retention", (3, 20, 12))]
    assert reqs[3] == [StateRequest("canon1", (2, 52)), KVRequest("kv", 1, 32)]            # one tap keeps nothing
    assert reqs[4] == [StateRequest("canon1", (2, 52)), StateRequest("retention", (2, 6, 10)), StateRequest("canon2", (2, 52))]
    assert m.layers[2].mixers[0].v_mix == dict(group="v", first=True) and m.layers[3].mixers[0].v_mix == dict(group="v", name="vmix")
    assert m.layers[0].mixers[0].v_mix is None and m.layers[0].mixers[0].softcap == 4.0 and m.layers[2].mixers[0].softcap == 0.0
    assert all(isinstance(r, ChunkRequest) for r in m.layers[1].step_requests())


def test_one_tap_in_front_of_a_sublayer_keeps_nothing():
    cfg = copy.deepcopy(configs.KEFETAR_A)
    cfg["canon"]["taps"] = 1
    assert build(cfg).cache_requests()[1] == [StateRequest("retention", (3, 20, 12))]


def test_what_is_stored_although_nothing_reads_it_is_no_fault():
    m = build(configs.KEFETAR_A)
    tensors = random_tensors(m, 1)
    assert tensors["l0.norm1"].shape == () and tensors["l3.mix.vmix"].shape == ()
    check_tensors(m, dict(tensors, **{"l2.mix.vmix": torch.tensor(0.5), "l0.mix.vmix": torch.tensor(0.5), "l1.norm2": torch.tensor(1.0)}))
    with pytest.raises(WeightError, match="l1.mix.vmix"):
        check_tensors(m, dict(tensors, **{"l1.mix.vmix": torch.tensor(0.5)}))
    with pytest.raises(WeightError, match="l3.mix.vmix"):
        check_tensors(m, {k: v for k, v in tensors.items() if k != "l3.mix.vmix"})


@pytest.mark.parametrize("edit,text", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"].update(v_mix="yes"), "v_mix"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=33), "blended"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=0.9), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(heads=0), "heads"),
    (lambda c: c["layers"][1].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(width=0), "width"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_faults_are_named(edit, text):
    cfg = copy.deepcopy(configs.KEFETAR_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(cfg)


# ---- pieces of the library that need no kernel --------------------------------------------------------------------------------
def test_frequencies_divided_by_a_constant():
    for base, dims, factor in ((10000.0, 24, 2.5), (500.0, 2, 8.0), (1e6, 128, 1.0)):
        part = RotaryNeox(dims + 4, base, dims, dict(kind="linear", factor=factor))
        part.bind({}, torch.float32, "cpu")
        want = plain.frequencies(dict(base=base, dims=dims, scaling=dict(factor=factor)))
        assert np.allclose(part.inv_freq.numpy(), want, rtol=1e-7) and part.amplitude == 1.0
        assert math.isclose(float(part.inv_freq[0]), 1.0 / factor, rel_tol=1e-7)
    with pytest.raises(ValueError, match="scaling"):
        RotaryNeox(8, 100.0, 8, dict(kind="linear"))


def test_a_gain_without_dimensions_serves_every_coordinate():
    norm = PartSpec("norm", "rmsnorm", dict(width=6, eps=1e-5, weight_name="g", one_gain=True)).build()
    norm.bind({"g": torch.tensor(1.5, dtype=torch.bfloat16)}, torch.float32, "cpu")
    assert torch.equal(norm.weight, torch.full((6,), 1.5)) and norm.weight.is_contiguous()


def test_convolution_weights_follow_the_padded_heads():
    m = build(configs.KEFETAR_A)
    tensors = random_tensors(m, 2)
    att = m.layers[3].mixers[0]                      # six query heads of 20 and one key head, values of 32: heads of 32 columns
    att.bind({k: v.float() for k, v in tensors.items()}, torch.float32, "cpu")
    assert att.conv_w.shape == (1, 8 * 32)
    w = att.conv_w.t().reshape(8, 32, 1)
    assert torch.equal(w[:6, :20].reshape(-1, 1), tensors["l3.mix.q.conv"].float()) and not w[:7, 20:].any()
    assert torch.equal(w[7], tensors["l3.mix.v.conv"].float()) and math.isclose(att.mix_share, float(tensors["l3.mix.vmix"]))


def test_faults_of_a_mixer_are_named():
    att = dict(hidden=8, n_heads=2, n_kv_heads=1, head_dim=4, prefix="", position=PartSpec("position", "none", dict(head_dim=4)))
    make = lambda **kw: PartSpec("mixer", "attention", dict(att, **kw)).build()
    for kw in (dict(conv_taps=18), dict(v_mix=dict(group="v", first=True)), dict(conv_taps=2, v_mix=dict(group="v")),
               dict(conv_taps=2, v_mix=dict(first=True)), dict(conv_taps=2, values="keys")):
        with pytest.raises(ValueError, match="attention"):
            make(**kw)
    with pytest.raises(ValueError, match="decays"):
        PartSpec("mixer", "retention", dict(hidden=8, n_heads=2, key_dim=4, v_dim=4, decay=[0.5], eps=1e-5, position=att["position"],
                                            names={n: n for n in "qkvgo"})).build()
    with pytest.raises(ValueError, match="polynomial"):
        PartSpec("feed_forward", "mlp", dict(hidden=8, intermediate=4, names=dict(up="u", down="d"), act="polynorm")).build()


# ---- the plain mechanisms against their definitions --------------------------------------------------------------------------------
def test_plain_convolution_and_sublayer_input():
    u = np.array([[1.0], [10.0], [100.0]])
    w = np.array([[2.0, 3.0]])                         # newest tap last
    assert np.allclose(plain.causal_conv(u, w)[:, 0], [3.0, 32.0, 320.0])
    x = np.array([[3.0, 4.0], [0.0, 0.0]])
    h = x / math.sqrt(12.5 + 0.5) * 2.0
    h[1] = 0.0
    got = plain.sublayer_input(x, np.array(2.0), np.array([[1.0, 0.0], [0.0, 5.0]]), 0.5)
    assert np.allclose(got[0], [h[0, 0], 6 * h[0, 1]]) and np.allclose(got[1], [h[0, 0], 0.0])


def test_plain_retention_against_its_unrolled_sum():
    g = np.random.default_rng(1)
    q, k, v = g.standard_normal((5, 3)), g.standard_normal((5, 3)), g.standard_normal((5, 2))
    a = 0.7
    want = np.array([sum(a ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)) for t in range(5)])
    assert np.allclose(plain.retention_scan(q, k, v, a), want)


def test_plain_rotation_pairs_and_capped_scores():
    x = np.arange(8, dtype=np.float64).reshape(1, 1, 8)
    f = np.array([0.5, 0.25])
    a = np.float32(3) * f.astype(np.float32)
    h = plain.rotate_halves(x, [3], f)[0, 0]
    assert np.allclose(h[0], 0 * math.cos(a[0]) - 2 * math.sin(a[0])) and np.allclose(h[3], 3 * math.cos(a[1]) + 1 * math.sin(a[1]))
    assert np.array_equal(h[4:], x[0, 0, 4:])
    q, k, v = np.ones((2, 1)), np.array([[1000.0], [0.0]]), np.array([[1.0], [0.0]])
    assert np.allclose(plain.attend(q, k, v, 1.0, 2.0)[1, 0], math.exp(2) / (1 + math.exp(2))) and plain.attend(q, k, v, 1.0, None)[1, 0] > 0.999
    assert np.allclose(plain.mix_values(np.array([2.0]), np.array([6.0]), 0.25), [3.0])


def test_plain_polynomial_over_normed_powers():
    z = np.array([[1.0, -2.0]])
    got = plain.polynorm(z, (0.5, 2.0, -1.0, 0.25), 0.0)
    n1, n2, n3 = math.sqrt(2.5), math.sqrt((1 + 16) / 2), math.sqrt((1 + 64) / 2)
    assert np.allclose(got[0], [0.5 * 1 / n1 + 2 * 1 / n2 - 1 / n3 + 0.25, 0.5 * -2 / n1 + 2 * 4 / n2 + 8 / n3 + 0.25])
