"""Fobatar without a GPU: the configuration's checks, what the builder makes of a configuration (parts, tensor names and shapes,
integer tables, cache needs, run order), the library's pieces that need no kernel (pages of chunks that are over, weights over
padded heads, a norm's multiplier, a table's checks, which layers may leave the next one's input), and the plain
implementation's mechanisms against restatements of their own definitions."""
import copy
import math

import numpy as np
import pytest
import torch

from tinyllama_c_b200.cache import Cache
from tinyllama_c_b200.config import ConfigError, config_from_dict
from tinyllama_c_b200.config.base import lookup_architecture
from tinyllama_c_b200.parts.base import KVRequest, LayerRun, PartSpec, StateRequest
from tinyllama_c_b200.parts.position import RotaryInterleaved
from tinyllama_c_b200.weights.loader import WeightError, check_tensors, load_model, random_tensors, write_random_model

import configs
from plain import fobatar_plain as plain


def build(cfg: dict):
    c = config_from_dict(cfg)
    return lookup_architecture(c.architecture)[1](c)


def test_builder_names_shapes_and_cache_needs():
    m = build(configs.FOBATAR_A)
    specs = {s.name: s for s in m.weight_specs()}
    got = {n: tuple(s.shape) for n, s in specs.items()}
    assert got["embed"] == (150, 52) and got["final.norm"] == (52,) and "head" not in got and m.head_name is None
    assert m.embed_scale == 0.8
    # attention: four query heads of 24 on two key heads, values of 16, two taps on every channel, whole-projection norms, a gate row a head
    assert all(got[f"l0.{n}"] == (52,) for n in ("norm1", "norm1b", "norm2", "norm2b"))
    assert got["l0.mix.q"] == (96, 52) and got["l0.mix.k"] == (48, 52) and got["l0.mix.v"] == (32, 52) and got["l0.mix.o"] == (52, 64)
    assert got["l0.mix.q.conv"] == (96, 2) and got["l0.mix.k.conv"] == (48, 2) and got["l0.mix.v.conv"] == (32, 2)
    assert got["l0.mix.q.norm"] == (96,) and got["l0.mix.k.norm"] == (48,) and got["l0.mix.g"] == (4, 52)
    # experts by a table of integers, a shared expert without a gate
    assert got["l0.mlp.table"] == (150, 2) and specs["l0.mlp.table"].below == 4 and "l0.mlp.router" not in got
    assert got["l0.mlp.e3.gate"] == (20, 52) and got["l0.mlp.e0.down"] == (52, 20) and "l0.mlp.e4.gate" not in got
    assert got["l0.mlp.shared.up"] == (12, 52) and "l0.mlp.shared.sg" not in got and "l2.mlp.shared.up" not in got
    # latent attention without a feed-forward
    assert got["l1.mix.q"] == (48, 52) and got["l1.mix.dkv"] == (26, 52) and got["l1.mix.dkv.norm"] == (20,)
    assert got["l1.mix.uk"] == (30, 20) and got["l1.mix.uv"] == (42, 20) and got["l1.mix.g"] == (3, 52) and got["l1.mix.o"] == (52, 42)
    assert got["l1.norm1b"] == (52,) and "l1.norm2" not in got and "l1.norm2b" not in got and not any(n.startswith("l1.mlp") for n in got)
    reqs = m.cache_requests()
    assert reqs[0] == [KVRequest("kv", 2, 24, chunk=5), StateRequest("kv.conv", (1, 8 * 24))]
    assert reqs[1] == [KVRequest("latent", 1, 26, values=False)] and reqs[2] == reqs[4] == reqs[0]
    assert reqs[6] == [KVRequest("kv", 1, 32, chunk=70), StateRequest("kv.conv", (3, 8 * 32))]
    assert reqs[7] == [KVRequest("kv", 2, 16)]                         # one tap keeps nothing
    assert m.layers[2].mixers[0].sink and m.layers[2].mixers[0].chunk == 70 and m.layers[3].mixers[0].chunk == 0


def test_run_order_of_a_repeated_range():
    run = lambda i, again=False: LayerRun(i, add_embedding=again)
    assert build(configs.FOBATAR_A).schedule == [run(0), run(1), run(0, True), run(1), run(0, True), run(1), run(2), run(3), run(4)]
    assert build(configs.FOBATAR_B).schedule == [run(0), run(1), run(2), run(1, True), run(2), run(3), run(4)]
    cfg = copy.deepcopy(configs.FOBATAR_B)
    del cfg["loop"]
    assert build(cfg).schedule == [run(i) for i in range(5)]


def test_a_folder_with_an_integer_table_round_trips_and_is_checked(tmp_path):
    d = write_random_model(dict(configs.FOBATAR_B), str(tmp_path / "m"), seed=3)
    m = load_model(d, "float32", "cpu")
    table = m.layers[1].ffn.table
    assert table.dtype == torch.int32 and tuple(table.shape) == (97, 3) and int(table.max()) < 8 and int(table.min()) >= 0
    assert all(len(set(r.tolist())) == 3 for r in table)
    tensors = random_tensors(build(configs.FOBATAR_B), 3)
    assert torch.equal(tensors["l1.mlp.table"], table)
    other = build(configs.FOBATAR_B)
    with pytest.raises(WeightError, match="l1.mlp.table"):
        check_tensors(other, dict(tensors, **{"l1.mlp.table": tensors["l1.mlp.table"].float()}))
    with pytest.raises(WeightError, match="l1.mix.g"):
        check_tensors(other, dict(tensors, **{"l1.mix.g": tensors["l1.mix.g"].to(torch.int32)}))
    bad = tensors["l1.mlp.table"].clone()
    bad[5, 1] = 8
    with pytest.raises(ValueError, match="l1.mlp.table"):
        other.bind(dict(tensors, **{"l1.mlp.table": bad}), torch.float32, "cpu")
    # norms of a feed-forward that is not there may be stored all the same
    check_tensors(other, dict(tensors, **{"l2.norm2": torch.ones(64), "l2.norm2b": torch.ones(64)}))


@pytest.mark.parametrize("edit,text", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rot"),
    (lambda c: c["layers"][1]["mixer"].update(heads=0), "heads"),
    (lambda c: c["layers"][1].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=-1.0), "limit"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.update(residual_mult="half"), "residual_mult"),
    (lambda c: c.update(embedding=dict(scale=None)), "embedding"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(width=0), "width"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_faults_are_named(edit, text):
    cfg = copy.deepcopy(configs.FOBATAR_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(cfg)


# ---- pieces of the library that need no kernel ------------------------------------------------------------------------------------
def test_pages_of_chunks_that_are_over_are_given_back():
    """Chunks of 100 positions in pages of 64: a page goes when every later query's chunk begins behind it, not earlier."""
    c = Cache({0: [KVRequest("kv", 1, 4, chunk=100)], 1: [KVRequest("kv", 1, 4)], 2: [KVRequest("kv", 1, 4, chunk=100)]},
              max_tokens=64 * 8, max_seqs=2, dtype=torch.float32, device="cpu")
    assert len(c.kv_groups) == 2
    chunked, whole = c.kv_groups
    s = c.acquire()
    held = lambda: [i for i, p in enumerate(chunked.pages_of[s]) if p >= 0]
    c.reserve(s, 99)
    c.commit(s, 99)
    assert held() == [0, 1]                       # the next query, at 99, sees 0 .. 99
    c.reserve(s, 1)
    c.commit(s, 1)
    assert held() == [1]                          # at 100 a new chunk begins, inside page 1
    c.reserve(s, 99)
    c.commit(s, 99)
    assert held() == [1, 2, 3]
    c.reserve(s, 102)
    c.commit(s, 102)
    assert held() == [4] and whole.pool.n_held == 5   # the next query, at 301, sees 300 and 301
    c.check()
    c.release(s)
    assert chunked.pool.n_held == 0
    c.check()


def test_weights_over_padded_heads_and_a_norms_multiplier():
    m = build(configs.FOBATAR_A)
    tensors = random_tensors(m, 2)
    att = m.layers[2].mixers[0]                      # six query heads of 20 and one key head, values of 32: heads of 32 columns
    att.bind({k: v.float() for k, v in tensors.items()}, torch.float32, "cpu")
    q, k = att.q_norm_w.reshape(6, 32), att.k_norm_w.reshape(1, 32)
    assert torch.equal(q[:, :20].reshape(-1), tensors["l2.mix.q.norm"].float()) and not q[:, 20:].any() and not k[:, 20:].any()
    assert att.conv_w.shape == (4, 8 * 32)
    # the gate: a row per head behind the projections, filled up to a multiple of 8
    assert att.g_off == 8 * 32 and att.qkv.out_features == 8 * 32 + 8
    assert torch.equal(att.qkv.weight[att.g_off:att.g_off + 6], tensors["l2.mix.g"].float()) and not att.qkv.weight[att.g_off + 6:].any()
    out = m.layers[2].mixer_out_norm
    out.bind({k: v for k, v in tensors.items()}, torch.float32, "cpu")
    assert torch.allclose(out.weight, tensors["l2.norm1b"].float() * 0.6)


def test_frequencies_along_a_ramp():
    for base, dims, sc in ((500.0, 20, dict(factor=2.0, original=100, fast=16.0, slow=1.0)), (100.0, 8, dict(factor=4.0, original=64, fast=8.0, slow=2.0))):
        part = RotaryInterleaved(dims + 4, base, dims, dict(sc, kind="ramp"))
        part.bind({}, torch.float32, "cpu")
        want, grow = plain.frequencies(dict(base=base, dims=dims, scaling=sc))
        assert np.allclose(part.inv_freq.numpy(), want, rtol=1e-6) and math.isclose(part.amplitude, grow)
        f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
        assert (want <= f * (1 + 1e-12)).all() and (want >= f / sc["factor"] * (1 - 1e-12)).all() and math.isclose(want[0], 1.0)


def test_which_layers_leave_the_next_ones_input():
    m = build(configs.FOBATAR_B)
    assert all(layer.entry is layer.mixer_norm for layer in m.layers)      # plain RMS norms in front of every mixer
    assert build(configs.KEFETAR_A).layers[0].entry is None                # a norm that keeps rows must see the step itself


def test_faults_of_parts_are_named():
    att = dict(hidden=8, n_heads=2, n_kv_heads=1, head_dim=4, prefix="", position=PartSpec("position", "none", dict(head_dim=4)),
               names={k: k for k in "qkvgo"})
    for kw in (dict(chunk=4, window=3), dict(gate="silu", gate_per="head"), dict(gate="sigmoid", gate_per="row")):
        with pytest.raises(ValueError, match="attention"):
            PartSpec("mixer", "attention", dict(att, **kw)).build()
    moe = dict(hidden=8, n_experts=4, top=2, expert_ff=8, expert_names={k: "e{e}." + k for k in ("gate", "up", "down")})
    for kw in (dict(router_name=None), dict(router_name="r", table_name="t", vocab=5), dict(router_name=None, table_name="t"),
               dict(router_name=None, table_name="t", vocab=5, router_bias_name="b"), dict(router_name="r", shared_gate_name="sg")):
        with pytest.raises(ValueError, match="moe"):
            PartSpec("feed_forward", "moe", dict(moe, **kw)).build()


# ---- the plain mechanisms against their definitions ------------------------------------------------------------------------------------
def test_plain_chunks_sink_and_gate():
    seen = [[j for j in range(7) if plain.visible(i, j, 3)] for i in range(7)]
    assert seen == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    q, k, v = np.ones((2, 1)), np.array([[2.0], [0.5]]), np.array([[1.0], [10.0]])
    e = math.exp(2.0), math.exp(0.5)
    assert np.allclose(plain.attend(q, k, v, 1.0, None, sink=True)[1, 0], (e[0] + 10 * e[1]) / (1 + e[0] + e[1]))
    assert np.allclose(plain.attend(q, k, v, 1.0, 1, sink=True)[1, 0], 10 * e[1] / (1 + e[1]))
    assert np.allclose(plain.attend(q, k, v, 1.0)[0, 0], 1.0)
    out = plain.head_gate(np.ones((1, 2, 3)), np.array([[1.0, 2.0]]), np.array([[0.0, 0.0], [1.0, -1.0]]))
    assert np.allclose(out[0, 0], 0.5) and np.allclose(out[0, 1], 1 / (1 + math.exp(1.0)))


def test_plain_rotation_of_neighbours_grows_what_it_turns():
    x = np.arange(6, dtype=np.float64).reshape(1, 1, 6)
    f = np.array([0.5, 0.25])
    a = np.float32(3) * f.astype(np.float32)
    h = plain.rotate_neighbours(x, [3], f, 1.5)[0, 0]
    assert np.allclose(h[2], 1.5 * (2 * math.cos(a[1]) - 3 * math.sin(a[1]))) and np.allclose(h[1], 1.5 * (1 * math.cos(a[0]) + 0 * math.sin(a[0])))
    assert np.array_equal(h[4:], x[0, 0, 4:])


def test_plain_experts_of_a_table():
    assert np.isclose(plain.clamped_swish(np.array(5.0), np.array(-9.0), 2.0), 2.0 / (1 + math.exp(-1.702 * 2.0)) * (-2.0 + 1.0))
    assert np.isclose(plain.clamped_swish(np.array(-5.0), np.array(0.5), 2.0), -5.0 / (1 + math.exp(1.702 * 5.0)) * 1.5)
    g = np.random.default_rng(1)
    W = {f"e{e}.{n}": g.standard_normal(s) for e in range(3) for n, s in (("gate", (4, 2)), ("up", (4, 2)), ("down", (2, 4)))}
    W.update({f"shared.{n}": g.standard_normal(s) for n, s in (("gate", (4, 2)), ("up", (4, 2)), ("down", (2, 4)))})
    W["table"] = np.array([[0, 2], [1, 0]])
    h = g.standard_normal((2, 2))
    mlp = dict(router=dict(experts=3, top=2), expert=dict(ff=4, limit=1.0), shared=dict(ff=4, limit=0.3))
    got = plain.table_moe(h, [1, 0], W, "", mlp)
    want = 0.5 * (plain.expert(h[0], W, "e1.", 1.0) + plain.expert(h[0], W, "e0.", 1.0)) + plain.expert(h[0], W, "shared.", 0.3)
    assert np.allclose(got[0], want)
    want = 0.5 * (plain.expert(h[1], W, "e0.", 1.0) + plain.expert(h[1], W, "e2.", 1.0)) + plain.expert(h[1], W, "shared.", 0.3)
    assert np.allclose(got[1], want)
