"""What the configurations share that are read from a nested config.json."""
import json
import os
from typing import Any, Dict, Tuple


class JsonConfig:
    """from_dict / to_dict of a subclass, as a file of a checkpoint directory."""

    @classmethod
    def from_pretrained(cls, path: str):
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def save_pretrained(self, path: str) -> None:
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)


def rotation(d: Dict[str, Any]) -> Tuple[int, float]:
    """(rotated dimensions, base) of a mixer."""
    rot = d.get("rot") or {"dims": 0, "base": 1.0}
    return int(rot["dims"]), float(rot["base"])
