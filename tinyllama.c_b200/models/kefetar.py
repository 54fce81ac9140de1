"""Kefetar: per layer a mixer and then an optional dense feed-forward, each reading

    c(n(x))_t,    n(x) = x / sqrt(mean(x^2) + eps) * g (one number g),    c(h)_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j)

(a norm with a single gain, then the normed row plus a short causal convolution of the normed rows, weights of its own per
sublayer), and added to the stream one after the other.  Two kinds of mixer.  'retention': linear attention with one fixed
decay per head, rotated queries and keys, the heads' results normed without a weight and gated by silu(W_g h).
'attention': grouped-query attention whose projected q, k and v first pass a short causal convolution per channel, a
split-half rotation with frequencies divided by a constant, scores capped by tanh, an output gate sigmoid(W_g h), and, where
the layer says so, values blended with those of the first such layer of the same token, v <- (1 - lam) v + lam v_first.
The feed-forward is W_down act(W_up h) with act a polynomial over normed powers, a N(z) + b N(z^2) + c N(z^3) + e.  The final
norm has a single gain too; the head is a matrix of its own.  This file only turns a KefetarConfig into data: one
LayerSpec per layer and the tensor names ('l<i>.' + norm1, norm2, canon1, canon2, mix.*, mlp.*; 'embed'; 'final.norm'; 'head').
"""
from __future__ import annotations

from typing import List, Optional

from ..config.base import register_architecture
from ..config.kefetar import KefetarConfig
from ..parts.base import LayerSpec, PartSpec
from .model import Model


def _input(cfg: KefetarConfig, i: int, sublayer: int) -> PartSpec:
    """What sublayer 1 (the mixer) or 2 (the feed-forward) of layer i reads."""
    return PartSpec("norm", "rmsnorm_conv", dict(width=cfg.width, eps=cfg.eps, weight_name=f"l{i}.norm{sublayer}", one_gain=True,
                                                 conv_name=f"l{i}.canon{sublayer}", taps=cfg.taps, cache_key=f"canon{sublayer}"))


def _position(m: dict) -> PartSpec:
    rot = m["rot"]
    if rot["dims"] == 0:
        return PartSpec("position", "none", dict(head_dim=m["dim"]))
    scaling = dict(kind="linear", factor=rot["scaling"]["factor"]) if rot.get("scaling") is not None else None
    return PartSpec("position", "rope_neox", dict(head_dim=m["dim"], theta=rot["base"], rope_dim=rot["dims"], scaling=scaling))


def _mixer(cfg: KefetarConfig, i: int) -> PartSpec:
    layer, p = cfg.layers[i], f"l{i}.mix."
    m = layer["mixer"]
    if layer["type"] == "retention":
        return PartSpec("mixer", "retention", dict(hidden=cfg.width, n_heads=m["heads"], key_dim=m["dim"], v_dim=m["vdim"], decay=m["decay"],
                                                   eps=cfg.eps, position=_position(m), names={n: p + n for n in ("q", "k", "v", "g", "o")}))
    v_mix = None
    if m.get("v_mix"):
        v_mix = dict(group="v", first=True) if i == cfg.first_mixed else dict(group="v", name="vmix")
    return PartSpec("mixer", "attention", dict(
        hidden=cfg.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"], prefix=p, position=_position(m),
        scale=m["scale"], softcap=m.get("softcap") or 0.0, gate="sigmoid", conv_taps=m["conv"], v_mix=v_mix,
        names=dict(q="q", k="k", v="v", g="g", o="o")))


def _feed_forward(cfg: KefetarConfig, i: int) -> Optional[PartSpec]:
    mlp, p = cfg.layers[i].get("mlp"), f"l{i}.mlp."
    if mlp is None:
        return None
    return PartSpec("feed_forward", "mlp", dict(hidden=cfg.width, intermediate=mlp["ff"], act="polynorm", act_eps=cfg.eps,
                                                names=dict(up=p + "up", down=p + "down", act=p + "act")))


def layer_specs(cfg: KefetarConfig) -> List[LayerSpec]:
    specs = []
    for i in range(len(cfg.layers)):
        ffn = _feed_forward(cfg, i)
        specs.append(LayerSpec(_input(cfg, i, 1), (_mixer(cfg, i),), _input(cfg, i, 2) if ffn is not None else None, ffn))
    return specs


def build(cfg: KefetarConfig) -> Model:
    # what a folder may hold although nothing reads it: the share of a layer whose values are not blended (the first of
    # those that are among them), the norm and convolution in front of a feed-forward that is not there
    unused = []
    for i, layer in enumerate(cfg.layers):
        if layer["type"] == "attention" and (not layer["mixer"].get("v_mix") or i == cfg.first_mixed):
            unused.append(f"l{i}.mix.vmix")
        if layer.get("mlp") is None:
            unused += [f"l{i}.norm2", f"l{i}.canon2"]
    final = PartSpec("norm", "rmsnorm", dict(width=cfg.width, eps=cfg.eps, weight_name="final.norm", one_gain=True))
    return Model(cfg, layer_specs(cfg), None, final, embed_name="embed", head_name="head", vocab=cfg.vocab, hidden=cfg.width,
                 unused_tensors=unused)


register_architecture("Kefetar", KefetarConfig, build)
