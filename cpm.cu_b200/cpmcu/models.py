"""Model registry: which class serves a checkpoint directory, by its config.json."""
import json
import os

from .fabulix import FabulixLLM
from .llm import LLM
from .llm_w4a16_gptq_marlin import W4A16GPTQMarlinLLM
from .tipetar import TipetarLLM

# config.json 'architecture' (or the first of 'architectures') -> class; everything else is Llama-format
ARCHITECTURES = {"Fabulix": FabulixLLM, "Tipetar": TipetarLLM}


def model_class(config):
    """Class for a parsed config.json."""
    names = [config.get("architecture")] + list(config.get("architectures") or [])
    for name in names:
        if name in ARCHITECTURES:
            return ARCHITECTURES[name]
    return W4A16GPTQMarlinLLM if config.get("quantization_config") else LLM


def open_model(path, **kwargs):
    """The model in directory `path`, with storage allocated and weights loaded.  kwargs as for the class."""
    with open(os.path.join(path, "config.json")) as f:
        cls = model_class(json.load(f))
    llm = cls(path, **kwargs)
    llm.init_storage()
    llm.load_from_hf()
    return llm
