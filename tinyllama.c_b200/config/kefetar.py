"""Kefetar configuration: a list of layers, each a mixer and an optional dense feed-forward, every one of them behind an RMS
norm with a single gain and a short convolution over time.

config.json names the architecture in 'architecture' and gives 'vocab', 'width', 'norm' ({'eps'}), 'canon' ({'taps'}: of the
convolution in front of every sublayer) and 'layers' (one object per layer with 'type' (the mixer), 'mixer' (its sizes and
constants) and 'mlp' (the feed-forward, or null)).

  retention mixer:   heads, dim, vdim, decay (one number per head), rot {base, dims}
  attention mixer:   heads, kv_heads, dim, vdim, conv (taps), scale, and optionally softcap (capped scores), v_mix (whether
                     the values are blended with those of the first such layer), rot {base, dims, scaling {factor}}
  mlp kind 'dense':  ff

'rot.scaling' may be absent (plain frequencies); 'rot.dims' may be 0 (nothing is rotated).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig


def _int(v: Any, least: int = 1) -> bool:
    return isinstance(v, int) and not isinstance(v, bool) and v >= least


def _num(v: Any) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


@dataclass(frozen=True)
class KefetarConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm: Dict[str, Any]
    canon: Dict[str, Any]
    initializer_range: float = 0.02

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": dict(self.norm),
                "canon": dict(self.canon), "layers": [dict(l) for l in self.layers]}

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def taps(self) -> int:
        return int(self.canon["taps"])

    @property
    def first_mixed(self) -> Optional[int]:
        """The first layer whose values later ones are blended with."""
        return next((i for i, l in enumerate(self.layers) if l["type"] == "attention" and l["mixer"].get("v_mix")), None)

    def validate(self) -> None:
        bad = []
        for k in ("vocab", "width"):
            if not _int(getattr(self, k)):
                bad.append(f"'{k}' must be a positive integer, got {getattr(self, k)!r}")
        if not (isinstance(self.norm, dict) and _num(self.norm.get("eps")) and self.norm["eps"] > 0):
            bad.append("'norm' must be an object with a positive 'eps'")
        if not (isinstance(self.canon, dict) and _int(self.canon.get("taps"))):
            bad.append("'canon' must be an object with a positive integer 'taps'")
        if not (isinstance(self.layers, (list, tuple)) and len(self.layers) > 0):
            bad.append("'layers' must be a non-empty list")
            raise ConfigError("config.json: " + "; ".join(bad))
        object.__setattr__(self, "layers", tuple(self.layers))
        shared = None                                    # size of the values that are blended: one for all layers that do
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                bad.append(f"{where} must be an object with a 'mixer' object")
                continue
            m, kind = layer["mixer"], layer.get("type")
            if kind not in ("retention", "attention"):
                bad.append(f"{where}.type must be 'retention' or 'attention', got {kind!r}")
                continue
            for k in ("heads", "dim", "vdim") + (("kv_heads", "conv") if kind == "attention" else ()):
                if not _int(m.get(k)):
                    bad.append(f"{where}.mixer.{k} must be a positive integer, got {m.get(k)!r}")
            rot = m.get("rot")
            if not (isinstance(rot, dict) and _num(rot.get("base")) and rot["base"] > 0 and _int(rot.get("dims"), 0)
                    and rot["dims"] % 2 == 0 and _int(m.get("dim")) and rot["dims"] <= m["dim"]):
                bad.append(f"{where}.mixer.rot must give a positive 'base' and an even 'dims' of at most dim")
            elif rot.get("scaling") is not None:
                sc = rot["scaling"]
                if not (isinstance(sc, dict) and _num(sc.get("factor")) and sc["factor"] > 0):
                    bad.append(f"{where}.mixer.rot.scaling must give a positive 'factor'")
            if kind == "retention":
                d = m.get("decay")
                if not (isinstance(d, (list, tuple)) and all(_num(a) for a in d) and _int(m.get("heads")) and len(d) == m["heads"]):
                    bad.append(f"{where}.mixer.decay must list one number per head")
            else:
                if _int(m.get("heads")) and _int(m.get("kv_heads")) and m["heads"] % m["kv_heads"]:
                    bad.append(f"{where}.mixer.heads must be a multiple of kv_heads")
                if not _num(m.get("scale")):
                    bad.append(f"{where}.mixer.scale must be a number")
                if m.get("softcap") is not None and not (_num(m["softcap"]) and m["softcap"] > 0):
                    bad.append(f"{where}.mixer.softcap must be a positive number where it is given")
                if m.get("v_mix") is not None and not isinstance(m["v_mix"], bool):
                    bad.append(f"{where}.mixer.v_mix must be true or false")
                elif m.get("v_mix") and _int(m.get("kv_heads")) and _int(m.get("vdim")):
                    size = (m["kv_heads"], m["vdim"])
                    if shared is not None and size[0] * size[1] != shared[0] * shared[1]:
                        bad.append(f"{where}.mixer: values of {size[0]} heads of {size[1]} cannot be blended with {shared[0]} heads of {shared[1]}")
                    shared = shared or size
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                bad.append(f"{where}.mlp must be null or an object of kind 'dense'")
            elif not _int(mlp.get("ff")):
                bad.append(f"{where}.mlp.ff must be a positive integer")
        if bad:
            raise ConfigError("config.json: " + "; ".join(bad))
