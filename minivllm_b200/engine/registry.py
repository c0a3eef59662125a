"""Model families by the `architecture` entry of a configuration, and model folders (config.json and
model.safetensors) as engine configurations.

A family names its configuration class (`from_dict`), its model class, and whether a folder can be loaded.
Configurations without the entry are Qwen3-shaped, as before there was a choice.
"""
import json
import os
from dataclasses import dataclass

from .dafotar import DafotarConfig, DafotarForCausalLM
from .fozerax import FozeraxConfig, FozeraxForCausalLM
from .qwen3 import Qwen3Config, Qwen3ForCausalLM
from .sipazen import SipazenConfig, SipazenForCausalLM
from .subivik import SubivikConfig, SubivikForCausalLM
from .weights import SafetensorsWeights


@dataclass(frozen=True)
class ModelFamily:
    name: str
    config: type
    model: type
    kernels: str                  # source group of csrc/build.py
    loads_folders: bool = False


FAMILIES = {f.name: f for f in (
    ModelFamily("Qwen3ForCausalLM", Qwen3Config, Qwen3ForCausalLM, "qwen3"),
    ModelFamily("Sipazen", SipazenConfig, SipazenForCausalLM, "sipazen", loads_folders=True),
    ModelFamily("Fozerax", FozeraxConfig, FozeraxForCausalLM, "fozerax", loads_folders=True),
    ModelFamily("Dafotar", DafotarConfig, DafotarForCausalLM, "dafotar", loads_folders=True),
    ModelFamily("Subivik", SubivikConfig, SubivikForCausalLM, "subivik", loads_folders=True),
)}
DEFAULT_FAMILY = "Qwen3ForCausalLM"


def family_of(config):
    name = config.get("architecture", DEFAULT_FAMILY)
    if name not in FAMILIES:
        raise ValueError(f"unknown architecture '{name}' (known: {', '.join(sorted(FAMILIES))})")
    return FAMILIES[name]


def folder_config(path, **engine):
    """Engine configuration of the model in folder `path`; `engine` holds the engine's own entries (dtype, pool
    sizes, limits, ...)."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    if "architecture" not in config:
        raise ValueError(f"{path}/config.json names no architecture")
    if not family_of(config).loads_folders:
        raise ValueError(f"{config['architecture']}: this family's checkpoints cannot be loaded from a folder")
    return {**config, **engine, "model_dir": path}


def build_model(config, model_cfg, tp_rank, tp_size, dtype, device):
    """The model of a configuration: weights from `config['weights']` (a WeightSource), from the folder
    `config['model_dir']`, or seeded."""
    family = family_of(config)
    kw = {}
    if config.get("weights") is not None:
        kw["weights"] = config["weights"]
    elif config.get("model_dir") is not None:
        kw["weights"] = SafetensorsWeights(os.path.join(config["model_dir"], "model.safetensors"), dtype, device)
    return family.model(model_cfg, tp_rank=tp_rank, tp_size=tp_size, dtype=dtype, device=device,
                        seed=config.get("seed", 0), **kw)
