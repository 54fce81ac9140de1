"""Fobatar configuration: a list of layers, each a mixer and an optional feed-forward of experts that a table of token ids
chooses, every sublayer between two norms, and a range of layers that repeats.

config.json names the architecture in 'architecture' and gives 'vocab', 'width', 'embedding' ({'scale'}), 'norm' ({'eps'}),
'residual_mult', 'layers' (one object per layer with 'type' (the mixer), 'mixer' (its sizes and constants) and 'mlp' (the
feed-forward, or null)) and optionally 'loop' ({'start', 'stop', 'times'}: layers start .. stop - 1 run `times` times in a row).

  attention mixer:         heads, kv_heads, dim, vdim, conv (taps), scale, rot, mask {size}
  latent_attention mixer:  heads, dim, rot_dim, vdim, kv_rank, scale, rot
  rot:                     {base, dims, scaling {factor, original, fast, slow}}
  mlp kind 'moe':          router {experts, top}, expert {ff, limit}, and optionally shared {ff, limit}

'rot.scaling' and 'mask' may be absent (plain frequencies; every earlier key is seen).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig


def _int(v: Any, least: int = 1) -> bool:
    return isinstance(v, int) and not isinstance(v, bool) and v >= least


def _num(v: Any) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


MIXER_SIZES = {"attention": ("heads", "kv_heads", "dim", "vdim", "conv"),
               "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank")}


@dataclass(frozen=True)
class FobatarConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm: Dict[str, Any]
    embedding: Dict[str, Any] = field(default_factory=lambda: {"scale": 1.0})
    residual_mult: float = 1.0
    loop: Optional[Dict[str, Any]] = None
    initializer_range: float = 0.02

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": dict(self.embedding),
               "norm": dict(self.norm), "residual_mult": self.residual_mult, "layers": [dict(l) for l in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        return out

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def embed_scale(self) -> float:
        return float(self.embedding["scale"])

    def validate(self) -> None:
        bad = []
        for k in ("vocab", "width"):
            if not _int(getattr(self, k)):
                bad.append(f"'{k}' must be a positive integer, got {getattr(self, k)!r}")
        if not (isinstance(self.norm, dict) and _num(self.norm.get("eps")) and self.norm["eps"] > 0):
            bad.append("'norm' must be an object with a positive 'eps'")
        if not (isinstance(self.embedding, dict) and _num(self.embedding.get("scale"))):
            bad.append("'embedding' must be an object with a number 'scale'")
        if not _num(self.residual_mult):
            bad.append(f"'residual_mult' must be a number, got {self.residual_mult!r}")
        if not (isinstance(self.layers, (list, tuple)) and len(self.layers) > 0):
            bad.append("'layers' must be a non-empty list")
            raise ConfigError("config.json: " + "; ".join(bad))
        object.__setattr__(self, "layers", tuple(self.layers))
        n = len(self.layers)
        if self.loop is not None:
            lp = self.loop
            if not (isinstance(lp, dict) and _int(lp.get("start"), 0) and _int(lp.get("stop"), 0) and _int(lp.get("times"))
                    and lp["start"] < lp["stop"] <= n):
                bad.append(f"'loop' must give 0 <= start < stop <= {n} and times >= 1, got {lp!r}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                bad.append(f"{where} must be an object with a 'mixer' object")
                continue
            self._check_mixer(f"{where}.mixer", layer.get("type"), layer["mixer"], bad)
            if layer.get("mlp") is not None:
                self._check_mlp(f"{where}.mlp", layer["mlp"], bad)
        if bad:
            raise ConfigError("config.json: " + "; ".join(bad))

    @staticmethod
    def _check_mixer(where: str, kind: Any, m: Dict[str, Any], bad: list) -> None:
        if kind not in MIXER_SIZES:
            bad.append(f"{where}: the layer's 'type' must be one of {sorted(MIXER_SIZES)}, got {kind!r}")
            return
        for k in MIXER_SIZES[kind]:
            if not _int(m.get(k)):
                bad.append(f"{where}.{k} must be a positive integer, got {m.get(k)!r}")
        if not _num(m.get("scale")):
            bad.append(f"{where}.scale must be a number")
        turned = m.get("dim") if kind == "attention" else m.get("rot_dim")     # how many values of a head may turn
        rot = m.get("rot")
        if not (isinstance(rot, dict) and _num(rot.get("base")) and rot["base"] > 1 and _int(rot.get("dims"), 0)
                and rot["dims"] % 2 == 0 and _int(turned) and rot["dims"] <= turned):
            bad.append(f"{where}.rot must give a 'base' above 1 and an even 'dims' of at most {turned!r}")
        elif rot.get("scaling") is not None:
            sc = rot["scaling"]
            keys = ("factor", "original", "fast", "slow")
            if not (isinstance(sc, dict) and all(_num(sc.get(k)) and sc[k] > 0 for k in keys)):
                bad.append(f"{where}.rot.scaling must give positive numbers {', '.join(keys)}")
        if kind != "attention":
            return
        if _int(m.get("heads")) and _int(m.get("kv_heads")) and m["heads"] % m["kv_heads"]:
            bad.append(f"{where}.heads must be a multiple of kv_heads")
        if m.get("mask") is not None and not (isinstance(m["mask"], dict) and _int(m["mask"].get("size"))):
            bad.append(f"{where}.mask must give a positive integer 'size'")

    @staticmethod
    def _check_mlp(where: str, mlp: Any, bad: list) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
            bad.append(f"{where} must be null or an object of kind 'moe'")
            return
        router = mlp.get("router")
        if not (isinstance(router, dict) and _int(router.get("experts")) and _int(router.get("top")) and router["top"] <= router["experts"]):
            bad.append(f"{where}.router must give 'experts' and a 'top' of at most that many")
        for key in ("expert", "shared"):
            part = mlp.get(key)
            if key == "shared" and part is None:
                continue
            if not (isinstance(part, dict) and _int(part.get("ff")) and _num(part.get("limit")) and part["limit"] > 0):
                bad.append(f"{where}.{key} must give a positive integer 'ff' and a positive 'limit'")
