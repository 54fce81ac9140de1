"""Fobatar: every sublayer stands between two RMS norms and enters the stream times a constant m,

    x <- x + m n1b(mixer(n1(x)));   x <- x + m n2b(ff(n2(x)))

with two kinds of mixer.  'attention': grouped-query attention whose projected q, k and v pass a short causal convolution per
channel, whose whole query and key projections are RMS-normed, a rotation of neighbouring pairs with frequencies blended along
a ramp over the pair index and enlarged cosines and sines, keys of the query's own chunk of positions only, a sink of score 0,
and an output gate of one sigmoid per head.  'latent_attention': all heads attend over one normed low-rank row per token and a
rotated key part that they share, without a sink, with the same kind of rotation and gate.  The feed-forward is a mixture of
experts without a router: a stored table gives every token id its experts, each weighted 1 / top, beside a shared expert;
experts multiply a clamped swish of the gate by the clamped up-projection plus one.  A range of layers may repeat: every
pass has caches of its own, and every pass but the first begins with the embedding output added to the stream.  The head is
the embedding table without its scale.  This file only turns a FobatarConfig into data: one LayerSpec per layer, the run
order, and the tensor names ('l<i>.' + norm1, norm1b, norm2, norm2b, mix.*, mlp.*; 'embed'; 'final.norm').
"""
from __future__ import annotations

from typing import List, Optional

from ..config.base import register_architecture
from ..config.fobatar import FobatarConfig
from ..parts.base import LayerRun, LayerSpec, PartSpec
from .model import Model

SWISH_ALPHA = 1.702        # inside the sigmoid of the experts' clamped swish


def _norm(cfg: FobatarConfig, name: str, scale: float = 1.0) -> PartSpec:
    return PartSpec("norm", "rmsnorm", dict(width=cfg.width, eps=cfg.eps, weight_name=name, scale=scale))


def _position(rot: dict, dim: int) -> PartSpec:
    if rot["dims"] == 0:
        return PartSpec("position", "none", dict(head_dim=dim))
    scaling = dict(rot["scaling"], kind="ramp") if rot.get("scaling") is not None else None
    return PartSpec("position", "rope_interleaved", dict(head_dim=dim, theta=rot["base"], rope_dim=rot["dims"], scaling=scaling))


def _mixer(cfg: FobatarConfig, i: int) -> PartSpec:
    layer, p = cfg.layers[i], f"l{i}.mix."
    m = layer["mixer"]
    if layer["type"] == "attention":
        return PartSpec("mixer", "attention", dict(
            hidden=cfg.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"], prefix=p,
            position=_position(m["rot"], m["dim"]), scale=m["scale"], conv_taps=m["conv"],
            names={k: k for k in ("q", "k", "v", "g", "o")}, whole_norm=dict(q="q.norm", k="k.norm", eps=cfg.eps), sink=True,
            chunk=(m.get("mask") or {}).get("size"), gate="sigmoid", gate_per="head"))
    names = {k: p + k for k in ("q", "dkv", "uk", "uv", "g", "o")}
    return PartSpec("mixer", "latent_attention", dict(
        hidden=cfg.width, n_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], kv_rank=m["kv_rank"],
        scale=m["scale"], eps=cfg.eps, position=_position(m["rot"], m["rot_dim"]), names=dict(names, dkv_norm=p + "dkv.norm")))


def _feed_forward(cfg: FobatarConfig, i: int) -> Optional[PartSpec]:
    mlp, p = cfg.layers[i].get("mlp"), f"l{i}.mlp."
    if mlp is None:
        return None
    router, expert, shared = mlp["router"], mlp["expert"], mlp.get("shared")
    shared_part = None if shared is None else PartSpec("feed_forward", "swiglu", dict(
        hidden=cfg.width, intermediate=shared["ff"], prefix=p + "shared.", names=dict(gate="gate", up="up", down="down"),
        act="swish_clamped", limit=shared["limit"], alpha=SWISH_ALPHA))
    return PartSpec("feed_forward", "moe", dict(
        hidden=cfg.width, n_experts=router["experts"], top=router["top"], expert_ff=expert["ff"], router_name=None,
        table_name=p + "table", vocab=cfg.vocab, expert_names={k: p + "e{e}." + k for k in ("gate", "up", "down")},
        weight_on="output", act="swish_clamped", limit=expert["limit"], alpha=SWISH_ALPHA, shared=shared_part))


def layer_specs(cfg: FobatarConfig) -> List[LayerSpec]:
    specs, m = [], float(cfg.residual_mult)
    for i in range(len(cfg.layers)):
        ffn = _feed_forward(cfg, i)
        specs.append(LayerSpec(_norm(cfg, f"l{i}.norm1"), (_mixer(cfg, i),), _norm(cfg, f"l{i}.norm2") if ffn is not None else None, ffn,
                               mixer_out_norm=_norm(cfg, f"l{i}.norm1b", m),
                               ffn_out_norm=_norm(cfg, f"l{i}.norm2b", m) if ffn is not None else None))
    return specs


def run_order(cfg: FobatarConfig) -> List[LayerRun]:
    """The layers in the order they run: the repeated range `times` times in a row, every entry with a cache of its own; every
    pass but the first begins with the embedding output added to the stream."""
    n, loop = len(cfg.layers), cfg.loop
    if loop is None:
        return [LayerRun(i) for i in range(n)]
    order = [LayerRun(i) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [LayerRun(i, add_embedding=t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [LayerRun(i) for i in range(loop["stop"], n)]


def build(cfg: FobatarConfig) -> Model:
    # a layer without a feed-forward has no use for the feed-forward's norms, stored or not
    unused = [f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.get("mlp") is None for n in ("norm2", "norm2b")]
    return Model(cfg, layer_specs(cfg), run_order(cfg), _norm(cfg, "final.norm"), embed_name="embed", head_name=None,
                 vocab=cfg.vocab, hidden=cfg.width, embed_scale=cfg.embed_scale, unused_tensors=unused)


register_architecture("Fobatar", FobatarConfig, build)
