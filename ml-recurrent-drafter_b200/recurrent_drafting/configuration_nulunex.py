"""Configuration of the Nulunex decoder: a list of layers, each with its own mixer (chunked attention or latent attention
over a sliding window) and an optional dense gated feed-forward; a layer may use another layer's weights."""
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Union

from .configuration_common import JsonConfig, rotation

ARCHITECTURE = "Nulunex"
GLU_ALPHA = 1.702  # slope inside the feed-forward's sigmoid


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    rot_base: float
    scale: float
    chunk: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "AttentionConfig":
        c = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), *rotation(d), float(d["scale"]),
                int(d["mask"]["size"]))
        if c.heads % c.kv_heads or c.rot_dims % 2 or c.rot_dims > c.dim or c.chunk < 1 or c.vdim != c.dim:
            raise ValueError(f"inconsistent attention configuration {d}")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                "rot": {"dims": self.rot_dims, "base": self.rot_base}, "scale": self.scale, "mask": {"size": self.chunk}}


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    rot_dims: int
    rot_base: float
    scale: float
    window: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LatentAttentionConfig":
        c = cls(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"]), *rotation(d), float(d["scale"]),
                int(d["mask"]["size"]))
        if c.rot_dims % 2 or c.rot_dims > c.rot_dim or c.window < 1:
            raise ValueError(f"inconsistent latent attention configuration {d}")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
                "rot": {"dims": self.rot_dims, "base": self.rot_base}, "scale": self.scale, "mask": {"size": self.window}}


@dataclass(frozen=True)
class GatedFeedForwardConfig:
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "GatedFeedForwardConfig":
        if d["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        return cls(int(d["ff"]), float(d["limit"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "kind": "dense", "limit": self.limit}


MIXERS = {"attention": AttentionConfig, "latent_attention": LatentAttentionConfig}


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: Union[AttentionConfig, LatentAttentionConfig]
    mlp: Optional[GatedFeedForwardConfig]  # None: the layer has none
    weights_of: Optional[int] = None  # index of the layer whose tensors this one uses

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LayerConfig":
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown layer type {d['type']!r}")
        mlp, shared = d.get("mlp"), d.get("weights_of")
        return cls(d["type"], MIXERS[d["type"]].from_dict(d["mixer"]), None if mlp is None else GatedFeedForwardConfig.from_dict(mlp),
                   None if shared is None else int(shared))

    def to_dict(self) -> Dict[str, Any]:
        out = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclass(frozen=True)
class NulunexConfig(JsonConfig):
    vocab_size: int
    hidden_size: int
    layers: List[LayerConfig]
    norm_eps: float

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def owner(self, index: int) -> int:
        """The layer whose tensors layer `index` uses."""
        seen = set()
        while self.layers[index].weights_of is not None:
            seen.add(index)
            index = self.layers[index].weights_of
            if index in seen or not 0 <= index < len(self.layers):
                raise ValueError(f"weights_of of layer {min(seen)} leads to no layer with weights of its own")
        return index

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NulunexConfig":
        c = cls(int(d["vocab"]), int(d["width"]), [LayerConfig.from_dict(x) for x in d["layers"]], float(d["norm"]["eps"]))
        for i, layer in enumerate(c.layers):
            o = c.layers[c.owner(i)]
            if (o.type, o.mixer, o.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ValueError(f"layer {i} uses the weights of a layer it differs from")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "layers": [x.to_dict() for x in self.layers]}
