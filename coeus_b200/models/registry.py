"""Model registry: which architecture a model directory holds, how its ``config.json`` becomes a
configuration, how its tensors become a model, and how a model is written back.

An architecture recognises its own ``config.json``; ``resolve`` asks the registered ones in order
and ``load_dir`` / ``save_dir`` do the file work.  The command line, the server and the trace
runner load every model directory through here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Mapping, Optional

import torch

from ..foundation.error import ProcessingError


@dataclass(frozen=True)
class Architecture:
    name: str
    matches: Callable[[Mapping[str, Any]], bool]                # on the parsed config.json
    load: Callable[..., Any]        # (state, config, device=, training=, dtype=) -> model
    export: Callable[[Any], tuple]  # model -> (state dict, config.json fields)
    owns: Callable[[Any], bool]     # whether a model object is of this architecture


_ARCHITECTURES: List[Architecture] = []


def register(arch: Architecture) -> None:
    if any(a.name == arch.name for a in _ARCHITECTURES):
        raise ProcessingError.invalid_input(f"architecture '{arch.name}' is registered already")
    _ARCHITECTURES.append(arch)


def architectures() -> List[str]:
    _ensure()
    return [a.name for a in _ARCHITECTURES]


def _ensure() -> None:
    if _ARCHITECTURES:
        return
    from ..checkpoint import hf
    from . import hybrid
    for name in hybrid.ARCHITECTURES:
        register(Architecture(
            name, lambda c, name=name: c.get("architecture") == name, hybrid.load_hybrid,
            hybrid.export_hybrid,
            lambda m, name=name: getattr(m.cfg, "architecture", None) == name))
    register(Architecture(
        "gpt2", lambda c: c.get("model_type") == "gpt2", hf.load_hf_gpt2, hf.to_hf_gpt2,
        lambda m: getattr(m.cfg, "pos", None) == "learned"))
    register(Architecture(
        "llama", lambda c: "architecture" not in c, hf.load_hf_llama, hf.to_hf_llama,
        lambda m: hasattr(m.cfg, "num_heads")))


def resolve(config: Mapping[str, Any]) -> Architecture:
    _ensure()
    for a in _ARCHITECTURES:
        if a.matches(config):
            return a
    raise ProcessingError.unsupported(
        f"architecture '{config.get('architecture')}'", f"known: {', '.join(architectures())}")


def architecture_of(model: Any) -> Architecture:
    _ensure()
    for a in _ARCHITECTURES:
        if a.owns(model):
            return a
    raise ProcessingError.unsupported(f"export of a {type(model).__name__}")


def read_config(path: str) -> Dict[str, Any]:
    import json
    import os
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def load_dir(path: str, device="cuda", training: bool = False,
             dtype: Optional[torch.dtype] = None):
    """A model directory: ``config.json`` plus one ``.safetensors`` file or several (sharded with
    an index).  ``dtype`` is the working precision where the architecture offers a choice."""
    import glob
    import os

    from ..checkpoint.formats import load_safetensors
    config = read_config(path)
    arch = resolve(config)
    files = sorted(glob.glob(os.path.join(path, "*.safetensors")))
    if not files:
        raise ProcessingError.invalid_input(f"no .safetensors file in {path}")
    state: Dict[str, torch.Tensor] = {}
    for fpath in files:
        tensors, _ = load_safetensors(fpath)
        state.update(tensors)
    kw = {} if dtype is None else {"dtype": dtype}
    return arch.load(state, config, device=device, training=training, **kw)


def save_dir(model: Any, path: str) -> None:
    import json
    import os

    from ..checkpoint.formats import save_safetensors
    os.makedirs(path, exist_ok=True)
    state, fields = architecture_of(model).export(model)
    save_safetensors(os.path.join(path, "model.safetensors"), state, {"format": "pt"})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(fields, f, indent=1)
