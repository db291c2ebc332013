"""One registry from an architecture's name to everything needed to serve it.

The reference maps ``hf_config.architectures[0]`` to a module, a model class, a
``parse_config`` and an ``iter_weights`` by name, imported lazily
(python/freetoken/models/register.py:11-143, python/freetoken/engine/config.py:88-92).
Here an :class:`Architecture` holds the typed configuration's reader, the
function that turns it into a :class:`ModelPlan`, and the checkpoint-name rule;
the model itself is always the generic :class:`freetoken_b200.models.Model`
built from the plan.  Adding an architecture is one ``register_architecture``
call; nothing else in the framework changes.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Mapping, Optional, Sequence, Tuple

from .config.model_plan import ModelPlan


@dataclass(frozen=True)
class Architecture:
    name: str
    read_config: Callable[[Mapping[str, Any]], Any]   # config.json dict -> typed config
    build_plan: Callable[[Any], ModelPlan]
    config_to_dict: Callable[[Any], Dict[str, Any]]
    rename_tensor: Callable[[str], Optional[str]] = lambda name: name
    # ``(config.json dict, {checkpoint tensor name: shape}) -> dict`` for a design some of whose sizes
    # only the checkpoint's tensor shapes state; called with the file headers of a model folder
    # before ``read_config``
    sizes_from_tensors: Optional[Callable[[Mapping[str, Any], Mapping[str, Tuple[int, ...]]], Mapping[str, Any]]] = None


_ARCHITECTURES: Dict[str, Architecture] = {}


def register_architecture(arch: Architecture, aliases: Sequence[str] = ()) -> Architecture:
    for name in (arch.name, *aliases):
        _ARCHITECTURES[name] = arch
    return arch


def get_architecture(name: str) -> Architecture:
    _load_builtin()
    try:
        return _ARCHITECTURES[name]
    except KeyError:
        known = ", ".join(sorted(_ARCHITECTURES))
        raise ValueError(f"Model architecture '{name}' is not supported (known: {known})") from None


def known_architectures() -> Tuple[str, ...]:
    _load_builtin()
    return tuple(sorted(_ARCHITECTURES))


def architecture_of(config: Mapping[str, Any]) -> Architecture:
    names = config.get("architectures") or []
    if not names and config.get("architecture"):
        names = [config["architecture"]]          # some designs name themselves in the singular
    if not names:
        raise ValueError("config.json has no 'architectures' entry to choose the model by")
    return get_architecture(names[0])


def read_model_config(folder_or_file: str) -> Tuple[Architecture, Any]:
    """``(architecture, typed config)`` of a model folder (or config.json path)."""
    path = folder_or_file
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        raw = json.load(f)
    arch = architecture_of(raw)
    if arch.sizes_from_tensors is not None and os.path.isdir(folder_or_file):
        from .weights.safetensors_io import Checkpoint
        with Checkpoint(folder_or_file) as ckpt:
            shapes = {}
            for name, entry in ckpt.entries.items():
                model_name = arch.rename_tensor(name)
                if model_name is not None:
                    shapes[model_name] = tuple(entry.shape)
        raw = arch.sizes_from_tensors(raw, shapes)
    return arch, arch.read_config(raw)


_loaded = False


def _load_builtin() -> None:
    global _loaded
    if _loaded:
        return
    _loaded = True
    from .config import minimax_m3 as m3
    register_architecture(
        Architecture(
            name=m3.ARCHITECTURES[0],
            read_config=m3.MiniMaxM3Config.from_dict,
            build_plan=m3.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
            rename_tensor=m3.rename_checkpoint_tensor,
        ),
        aliases=m3.ARCHITECTURES[1:],
    )
    from .config import fazinex
    register_architecture(
        Architecture(
            name=fazinex.ARCHITECTURE,
            read_config=fazinex.FazinexConfig.from_dict,
            build_plan=fazinex.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
        ),
    )
    from .config import nirelix
    register_architecture(
        Architecture(
            name=nirelix.ARCHITECTURE,
            read_config=nirelix.NirelixConfig.from_dict,
            build_plan=nirelix.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
            sizes_from_tensors=nirelix.sizes_from_tensors,
        ),
    )
    from .config import tonapel
    register_architecture(
        Architecture(
            name=tonapel.ARCHITECTURE,
            read_config=tonapel.TonapelConfig.from_dict,
            build_plan=tonapel.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
        ),
    )
    from .config import mezapel
    register_architecture(
        Architecture(
            name=mezapel.ARCHITECTURE,
            read_config=mezapel.MezapelConfig.from_dict,
            build_plan=mezapel.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
        ),
    )
    from .config import dizatar
    register_architecture(
        Architecture(
            name=dizatar.ARCHITECTURE,
            read_config=dizatar.DizatarConfig.from_dict,
            build_plan=dizatar.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
        ),
    )
    from .config import besuzen
    register_architecture(
        Architecture(
            name=besuzen.ARCHITECTURE,
            read_config=besuzen.BesuzenConfig.from_dict,
            build_plan=besuzen.build_plan,
            config_to_dict=lambda cfg: cfg.to_dict(),
            sizes_from_tensors=besuzen.sizes_from_tensors,
        ),
    )
