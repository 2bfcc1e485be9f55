"""Model families: GPT-2, GPT-J and Llama shaped decoders assembled from the add-on layers, their training program
(`DecoderTrainer`) and the int4 tensor-parallel decoding program (`DecoderGenerator`); Dunelix and Zirunex, served from
a checkpoint folder by `SequenceGenerator`; the registry of architectures (`load_model`)."""
from .decoder import DecoderBlock, DecoderConfig, DecoderEmbedding, DecoderHead

__all__ = ["DecoderConfig", "DecoderBlock", "DecoderEmbedding", "DecoderHead", "DecoderTrainer", "PipelineTrainer",
           "DecoderGenerator", "Dunelix", "DunelixConfig", "Zirunex", "ZirunexConfig", "SequenceGenerator", "load_model",
           "load_config", "register_architecture", "ARCHITECTURES"]

_LAZY = {"DecoderTrainer": "trainer", "PipelineTrainer": "pipeline_trainer", "DecoderGenerator": "generator",
         "Dunelix": "dunelix", "DunelixConfig": "dunelix", "Zirunex": "zirunex", "ZirunexConfig": "zirunex",
         "SequenceGenerator": "sequence_generator", "load_model": "registry", "load_config": "registry",
         "register_architecture": "registry", "ARCHITECTURES": "registry"}


def __getattr__(name):
    # the programs import the transforms and the session: loaded on first use
    if name in _LAZY:
        import importlib

        return getattr(importlib.import_module(f"{__name__}.{_LAZY[name]}"), name)
    raise AttributeError(f"module {__name__!r} has no attribute {name!r}")
