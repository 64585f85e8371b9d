"""Configuration of the Dilavik decoder: a list of layers, each with its own mixer (sliding-window attention or
matrix-memory recurrence) and an optional dense feed-forward."""
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Union

from .configuration_common import JsonConfig, rotation

ARCHITECTURE = "Dilavik"


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    rot_base: float
    scale: float
    window: int
    keep_first: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "AttentionConfig":
        c = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), *rotation(d), float(d["scale"]),
                int(d["mask"]["size"]), int(d["mask"]["keep_first"]))
        if c.heads % c.kv_heads or c.rot_dims % 2 or c.rot_dims > c.dim or c.window < 1 or c.keep_first < 0:
            raise ValueError(f"inconsistent attention configuration {d}")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                "rot": {"dims": self.rot_dims, "base": self.rot_base}, "scale": self.scale,
                "mask": {"size": self.window, "keep_first": self.keep_first}}


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "MatrixMemoryConfig":
        return cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["gate_cap"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


MIXERS = {"attention": AttentionConfig, "mlstm": MatrixMemoryConfig}


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: Union[AttentionConfig, MatrixMemoryConfig]
    ff: Optional[int]  # width of the dense feed-forward; None: the layer has none

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LayerConfig":
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown layer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        return cls(d["type"], MIXERS[d["type"]].from_dict(d["mixer"]), None if mlp is None else int(mlp["ff"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(),
                "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff}}


@dataclass(frozen=True)
class DilavikConfig(JsonConfig):
    vocab_size: int
    hidden_size: int
    layers: List[LayerConfig]
    embedding_scale: float
    norm_eps: float
    norm_groups: int

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "DilavikConfig":
        c = cls(int(d["vocab"]), int(d["width"]), [LayerConfig.from_dict(x) for x in d["layers"]],
                float(d["embedding"]["scale"]), float(d["norm"]["eps"]), int(d["norm"]["groups"]))
        if c.hidden_size % c.norm_groups:
            raise ValueError(f"{c.norm_groups} norm groups do not divide a width of {c.hidden_size}")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
                "layers": [x.to_dict() for x in self.layers]}
