"""What the models that are assembled from config.json have in common: their weights by name, their per-layer state, and
what the engine asks of a model."""

import torch

from .mixers import RotaryTable


def joint_reach(mixers):
    """What some mixer can still see of a sequence's keys: (window, kept first ones), or None for all of them."""
    reaches = [m.reach for m in mixers]
    if not reaches or any(r is None for r in reaches):
        return None
    return max(r[0] for r in reaches), max(r[1] for r in reaches)


class ConfiguredModel:
    """Subclasses read ``config`` in ``_build`` (weights through ``_w``), list the mixer of every layer run in
    ``self.run_mixers`` and implement ``forward(batch, state, record=None)``."""

    kernel_library = "decoder"
    chunked_prefill = mixed_batches = graph_decode = True
    max_positions = None                   # the longest sequence the design can represent, None = no limit

    def __init__(self, config, tensors, dtype=torch.bfloat16, device="cuda"):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"{config.get('architecture')} runs in float32 or bfloat16, not {dtype}")
        self.config, self.dtype, self.device = config, dtype, torch.device(device)
        # matrix products accumulate in fp32 and are not split with 16-bit partial sums; fp32 means fp32
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        torch.backends.cuda.matmul.allow_tf32 = False
        self.width, self.vocab, self.eps = config["width"], config["vocab"], float(config["norm"]["eps"])
        self._tensors, self._tables, self.run_mixers = tensors, {}, []
        self._build(config)
        del self._tensors

    @classmethod
    def from_config(cls, config, tensors, dtype=torch.bfloat16, device="cuda"):
        return cls(config, tensors, dtype, device)

    def _build(self, config):
        raise NotImplementedError

    def _w(self, name, *shape, dtype=None):
        """Tensor ``name`` on the device in the activation dtype (or ``dtype``); its shape must be ``shape`` if given."""
        if name not in self._tensors:
            raise KeyError(f"the checkpoint has no tensor {name}")
        t = self._tensors[name]
        if shape and tuple(t.shape) != shape:
            raise ValueError(f"tensor {name} is {tuple(t.shape)}, the configuration says {shape}")
        return t.to(self.device, dtype or self.dtype).contiguous()

    def _rotary(self, rot):
        rot = rot or {"dims": 0, "base": 1.0}
        key = repr(sorted((k, repr(v)) for k, v in rot.items()))
        if key not in self._tables:
            self._tables[key] = RotaryTable(rot["dims"], rot["base"], rot.get("scaling"), self.device)
        return self._tables[key]

    @property
    def cache_reach(self):
        return joint_reach(self.run_mixers)

    def new_state(self, max_seqs, num_blocks, block_size=256, max_positions=None):
        """One cache or state per layer run."""
        for t in self._tables.values():
            t.reserve(max_positions or num_blocks * block_size)
        return [m.new_state(max_seqs, num_blocks, block_size) for m in self.run_mixers]
