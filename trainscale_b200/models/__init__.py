"""Model classes by architecture name: which class a config.json describes, how it is built and how its weights load.

`EngineCore`, `hub.load_pretrained` and the command lines go through this table; a new design adds one `Architecture`.
"""
from __future__ import annotations

import importlib
from dataclasses import dataclass
from typing import Any, Callable


@dataclass(frozen=True)
class Architecture:
    """`module` is imported when the architecture is first used and defines `PRESETS` (name -> config),
    `build_model(config, dtype, device, seed)` and `load_model(config, state_dict, dtype, device)`, where config is a
    preset name or the dictionary of a config.json."""
    name: str
    module: str
    matches: Callable[[dict[str, Any]], bool]

    def _mod(self):
        return importlib.import_module(self.module)

    @property
    def presets(self) -> dict[str, Any]:
        return self._mod().PRESETS

    def build(self, config, dtype, device=None, seed: int | None = None):
        return self._mod().build_model(config, dtype=dtype, device=device, seed=seed)

    def load(self, config: dict, state_dict: dict, dtype, device=None):
        return self._mod().load_model(config, state_dict, dtype, device)


ARCHITECTURES: list[Architecture] = []


def register_architecture(arch: Architecture) -> Architecture:
    ARCHITECTURES.append(arch)
    return arch


def architecture_of(config: dict[str, Any]) -> Architecture:
    """The architecture of a config.json; the Llama-style decoder reads every HuggingFace-style one."""
    for a in ARCHITECTURES:
        if a.matches(config):
            return a
    raise ValueError(f"no model class for architecture {config.get('architecture')!r}; known: "
                     f"{', '.join(a.name for a in ARCHITECTURES)}")


def is_preset(name: str) -> bool:
    return any(name in a.presets for a in ARCHITECTURES)


def build_preset(name: str, dtype, device=None, seed: int | None = None):
    for a in ARCHITECTURES:
        if name in a.presets:
            return a.build(name, dtype, device, seed)
    raise KeyError(name)


register_architecture(Architecture("Mezilix", f"{__name__}.mezilix", lambda c: c.get("architecture") == "Mezilix"))
register_architecture(Architecture("Vibepel", f"{__name__}.vibepel", lambda c: c.get("architecture") == "Vibepel"))
register_architecture(Architecture("Kabulix", f"{__name__}.kabulix", lambda c: c.get("architecture") == "Kabulix"))
register_architecture(Architecture("Lovurax", f"{__name__}.lovurax", lambda c: c.get("architecture") == "Lovurax"))
register_architecture(Architecture("Llama", f"{__name__}.llama", lambda c: "architecture" not in c))
