"""Model class by ``config.json``: the one loader behind the serving command line and the trace runner."""
from __future__ import annotations

import json
import os

import torch

from .layered_config import LayeredConfig, is_layered


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def load_pretrained(path: str, torch_dtype: torch.dtype, device):
    """The model stored in folder ``path`` (``config.json`` + weights), in ``torch_dtype`` on ``device``."""
    if is_layered(read_config(path)):
        from .layered import LayeredForCausalLM

        return LayeredForCausalLM.from_pretrained(path, torch_dtype=torch_dtype, device=device)
    from .hf import RavenForCausalLM

    return RavenForCausalLM.from_pretrained(path, torch_dtype=torch_dtype).to(device)


def random_model(name: str, torch_dtype: torch.dtype, device, seed: int = 0):
    """A registry shape with random weights."""
    from .. import registry

    if name in registry.layered_configs:
        from .layered import LayeredForCausalLM

        return LayeredForCausalLM(LayeredConfig.from_name(name), torch_dtype, device).init_weights(seed)
    from ..config import ModelConfig
    from .hf import RavenForCausalLM
    from .hf_config import RavenConfig

    torch.manual_seed(seed)
    with torch.device(device):
        model = RavenForCausalLM(RavenConfig.from_model_config(ModelConfig.from_name(name)))
    return model.to(torch_dtype)
