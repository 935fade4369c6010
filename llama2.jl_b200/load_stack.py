"""Layer-stack models: a folder with config.json and model.safetensors, and the registry of model sources."""
import json
import os

from .load_gguf import load_gguf_model
from .model import LanguageModel, StackConfig, _DeviceModel

# config.json "architecture" -> configuration class.  The library has its own table of the same names (csrc/stack_config.cpp),
# which knows the designs themselves.
ARCHITECTURES = {"Savozen": StackConfig, "Perezen": StackConfig}


def load_stack_model(path: str, seq_len: int, compute: str = "bfloat16", device: int = -1, stream=None) -> LanguageModel:
    """The model in folder `path`, its weights read and uploaded by the library.  The folder holds no tokenizer: prompts are ids."""
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    name = raw.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unsupported model architecture: {name}")
    config = ARCHITECTURES[name](raw, int(seq_len), compute)
    model = LanguageModel(config, None, None, device=device, stream=stream)
    model._dev = _DeviceModel.from_dir(path, config, device, stream)
    return model


def load_model(path: str, seq_len: int = 512, **kw) -> LanguageModel:
    """Any model this package reads, chosen by what `path` is: a folder with a config.json, or a GGUF file."""
    if os.path.isdir(path):
        return load_stack_model(path, seq_len, **kw)
    return load_gguf_model(path, seq_len=seq_len, **kw)
