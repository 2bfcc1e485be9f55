"""Model families by the `architecture` entry of a `config.json`: the configuration class, the model description and the
program that serves it. `load_model` reads a folder with `config.json` and `model.safetensors`."""
import json
import os
from dataclasses import dataclass
from importlib import import_module
from typing import Any, Callable, Dict, Optional

__all__ = ["Architecture", "ARCHITECTURES", "register_architecture", "architecture", "load_config", "load_model"]


@dataclass(frozen=True)
class Architecture:
    name: str
    config: Callable[[Dict[str, Any]], Any]   # entries of config.json -> configuration object
    model: Optional[Callable[..., Any]] = None  # (configuration, dtype) -> model description for SequenceGenerator
    dtypes: tuple = ("bfloat16", "float32")


ARCHITECTURES: Dict[str, Architecture] = {}


def register_architecture(arch: Architecture) -> Architecture:
    ARCHITECTURES[arch.name] = arch
    return arch


def architecture(name: str) -> Architecture:
    if name not in ARCHITECTURES:
        raise KeyError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name]


def _decoder(family: str):
    def make(d: Dict[str, Any]):
        cls = import_module(f"{__package__}.decoder").DecoderConfig
        return cls(family=family, **{k: v for k, v in d.items() if k != "architecture"})

    return make


def _served(name: str, module: str) -> Architecture:
    """An architecture whose module (loaded on first use) has a class `<name>`, which describes the model to
    `SequenceGenerator`, and its configuration `<name>Config`."""
    def config(d: Dict[str, Any]):
        return getattr(import_module(f"{__package__}.{module}"), f"{name}Config").from_dict(d)

    def model(cfg, dtype: str = "bfloat16"):
        return getattr(import_module(f"{__package__}.{module}"), name)(cfg, dtype)

    return Architecture(name, config, model)


# trained / generated with DecoderTrainer and DecoderGenerator, which take the configuration object
for _family, _name in (("gptj", "GPT-J"), ("gpt2", "GPT-2"), ("llama", "Llama")):
    register_architecture(Architecture(_name, _decoder(_family)))
for _name, _module in (("Dunelix", "dunelix"), ("Zirunex", "zirunex")):
    register_architecture(_served(_name, _module))


def load_config(folder: str):
    """`(architecture, configuration)` of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        d = json.load(f)
    if "architecture" not in d:
        raise ValueError(f"{folder}/config.json names no architecture")
    arch = architecture(d["architecture"])
    return arch, arch.config(d)


def load_model(folder: str, dtype: str = "bfloat16", **generator_options):
    """A `SequenceGenerator` with the folder's weights loaded."""
    from ..utils.safetensors import read_safetensors
    from .sequence_generator import SequenceGenerator

    arch, cfg = load_config(folder)
    if arch.model is None:
        raise ValueError(f"architecture {arch.name!r} is not served from a checkpoint folder")
    if dtype not in arch.dtypes:
        raise ValueError(f"architecture {arch.name!r} runs in {arch.dtypes}, not in {dtype!r}")
    gen = SequenceGenerator(arch.model(cfg, dtype), **generator_options)
    return gen.load_checkpoint(read_safetensors(os.path.join(folder, "model.safetensors")))
