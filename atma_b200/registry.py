"""Which class serves which design: config.json's "architecture" names it.

A registered class has
    kernel_library          "b200" or "decoder": the library its kernels live in
    from_config(config, tensors, dtype, device)
    new_state(max_seqs, num_blocks, block_size, max_positions)   everything its sequences keep on the device
    forward(batch, state)   logits (fp32) of the rows ``batch.logit_rows`` (None if there are none); ``batch`` is an
                            ``engine.StepBatch``
    chunked_prefill         prompts may come in portions
    mixed_batches           decoding sequences and prompt portions may share a step
    graph_decode            a step of decoding sequences only can be captured in a CUDA graph
    vocab
and may have
    max_positions           the longest sequence the design can represent (absent or None: no limit)
    cache_reach             (window, first): later positions see only a sequence's last ``window`` and first ``first``
                            keys, so that pages between them are given back (absent or None: every key stays)
"""

import importlib
import os

import torch

from .checkpoint import read_config, read_safetensors

_MODELS = {"Atma": ("atma_b200.model", "AtmaModel"), "Rizurax": ("atma_b200.rizurax", "RizuraxModel"),
           "Zemivik": ("atma_b200.zemivik", "ZemivikModel")}


def architectures():
    return sorted(_MODELS)


def register_model(architecture, module, name):
    """Add a design: ``name`` in ``module`` (imported when first asked for) serves "architecture": ``architecture``."""
    _MODELS[architecture] = (module, name)


def model_class(config):
    arch = config.get("architecture")
    if arch not in _MODELS:
        raise ValueError(f"unknown architecture {arch!r}; this build serves {', '.join(architectures())}")
    module, name = _MODELS[arch]
    return getattr(importlib.import_module(module), name)


def build_kernels(config):
    """Compile the kernel library the design needs if this checkout does not have it yet."""
    from .build import LIBS, build
    which = model_class(config).kernel_library
    if not os.path.exists(LIBS[which]):
        build(which)


def load_model(folder, dtype=torch.bfloat16, device="cuda"):
    """The model of a folder with config.json and model.safetensors."""
    config = read_config(folder)
    return model_class(config).from_config(config, read_safetensors(os.path.join(folder, "model.safetensors")), dtype, device)
