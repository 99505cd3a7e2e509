"""Model registry: which family a name or a ``config.json`` belongs to, and how to load a model folder.

``family_for_config`` looks at the keys model folders use to name their class (``architecture``, ``architectures``,
``model_type``). ``load_model`` reads a folder (config.json + *.safetensors) through the family's own configuration and
weight loader; ``load_engine`` wraps it in the family's step engine where it has one.
"""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class Family:
    name: str
    module: str                        # package with the configuration class, init_params, forward, generate
    config: str                        # name of the configuration class in it
    aliases: Tuple[str, ...] = ()      # values of architecture / architectures / model_type
    from_dir: Optional[str] = None     # "module:function" (path, dtype, device, family) -> (config, params)
    engine: Optional[str] = None       # step engine class in ``module``

    def mod(self):
        return importlib.import_module(self.module)

    def config_class(self):
        return getattr(self.mod(), self.config)


_BASE = "jax_gpt_b200.models."
_FOLDER = _BASE + "registry:_folder_with_config"
FAMILIES: Dict[str, Family] = {f.name: f for f in (
    Family("gpt2", _BASE + "gpt2", "GPTConfig", ("GPT2LMHeadModel", "gpt2")),
    Family("qwen35", _BASE + "qwen35", "Qwen35Config", ("qwen3_5_moe",)),
    Family("deepseek_v3", _BASE + "deepseek_v3", "DeepSeekV3Config", ("DeepseekV3ForCausalLM", "deepseek_v3")),
    Family("vobunex", _BASE + "vobunex", "VobunexConfig", ("Vobunex",), from_dir=_FOLDER, engine="VobunexEngine"),
    Family("fovudra", _BASE + "fovudra", "FovudraConfig", ("Fovudra",), from_dir=_FOLDER, engine="FovudraEngine"),
    Family("munazen", _BASE + "munazen", "MunazenConfig", ("Munazen",), from_dir=_FOLDER, engine="MunazenEngine"),
    Family("mopalorn", _BASE + "mopalorn", "MopalornConfig", ("Mopalorn",), from_dir=_FOLDER, engine="MopalornEngine"),
)}


def family_for_config(config: dict) -> Family:
    names = [config.get("architecture"), config.get("model_type"), *(config.get("architectures") or [])]
    for f in FAMILIES.values():
        if any(n is not None and (n == f.name or n in f.aliases) for n in names):
            return f
    raise KeyError(f"no model family for {[n for n in names if n]} (known: {sorted(FAMILIES)})")


def family_for_dir(path: str) -> Family:
    with open(os.path.join(path, "config.json")) as fh:
        return family_for_config(json.load(fh))


def load_model(path: str, dtype=torch.bfloat16, device="cuda") -> Tuple[Family, Any, dict]:
    """(family, config, parameters) of a model folder."""
    f = family_for_dir(path)
    if f.from_dir is None:
        raise NotImplementedError(f"family {f.name!r} loads through its own scripts, not from a config.json folder")
    mod, fn = f.from_dir.split(":")
    config, params = getattr(importlib.import_module(mod), fn)(path, dtype, device, f)
    return f, config, params


def load_engine(path: str, dtype=torch.bfloat16, device="cuda", **kw):
    """The family's step engine over a model folder; ``kw`` goes to the engine (cache size, graphs)."""
    f, config, params = load_model(path, dtype, device)
    if f.engine is None:
        raise NotImplementedError(f"family {f.name!r} has no step engine")
    return getattr(f.mod(), f.engine)(params, config, **kw)


def _folder_with_config(path, dtype, device, family):
    """Folders whose configuration class reads config.json (``from_dir``) and whose module loads tensors by name."""
    from ..utils.safetensors_dir import SafetensorsDir
    config = family.config_class().from_dir(path)
    return config, family.mod().load_from_state_dict(SafetensorsDir(path), config, dtype, device)
