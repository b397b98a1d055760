"""Token mixers of the configured decoder models.

A mixer sits between a layer's norm and its output projection: it owns its input projection (one matrix for all of its
parts), says how many columns it hands to the output projection (``width``), and keeps its per-sequence state in a
tensor dictionary from ``new_state``.  ``run(h, out, batch, state)`` fills ``out`` (rows, width) for the step's rows:
decoding sequences (one row each, first) and prompt portions take their own kernels.  All constants are arguments, so a
design combines mixers by configuration.
"""

import math

import torch

from . import decoder_ops as ops


def rotary_frequencies(dims, base, scaling=None):
    """Frequencies of the dims/2 channel pairs (float64) and the factor on cos and sin.  ``scaling`` (YaRN): ``factor``,
    ``original`` (context length), ``fast`` and ``slow`` (turns over that context): pairs that turn more often than
    ``fast`` keep their frequency, those below ``slow`` are divided by the factor, with a linear ramp between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq = float(base) ** (-2.0 * i / max(dims, 1))
    if not scaling:
        return freq, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq * (1 - ramp) + freq / factor * ramp, 0.1 * math.log(factor) + 1.0


class RotaryTable:
    """cos and sin of every position and channel pair, fp32 from float64 angles; grown on demand."""

    def __init__(self, dims, base, scaling, device):
        self.dims, self.device = dims, device
        self.freq, self.amplitude = rotary_frequencies(dims, base, scaling)
        self.table = None

    def reserve(self, positions):
        if self.dims == 0 or (self.table is not None and self.table.shape[0] >= positions):
            return
        angle = torch.arange(positions, dtype=torch.float64, device=self.device)[:, None] * self.freq.to(self.device)
        self.table = (torch.stack([torch.cos(angle), torch.sin(angle)], -1) * self.amplitude).float().contiguous()


class SoftmaxAttention:
    """Causal softmax attention over a paged cache, grouped key/value heads, rotary positions on the first
    ``rotary.dims`` channels of every map, one map per head or two (differential: o = a1 - lam * a2, divided by its root
    mean square, times ``out_scale``)."""

    def __init__(self, w_q, w_k, w_v, *, heads, kv_heads, maps, dim, vdim, scale, rotary, lam=0.0, out_scale=1.0, eps=0.0):
        self.w_in = torch.cat([w_q, w_k, w_v]).contiguous()
        self.heads, self.kv_heads, self.maps, self.dim, self.vdim = heads, kv_heads, maps, dim, vdim
        self.scale, self.rotary, self.lam, self.out_scale, self.eps = scale, rotary, lam, out_scale, eps
        self.width = heads * vdim

    def new_state(self, max_seqs, num_blocks, block_size):
        dt, dev = self.w_in.dtype, self.w_in.device
        zeros = lambda n: torch.zeros(num_blocks, block_size, self.kv_heads, n, device=dev, dtype=dt)   # finite: masked keys weigh 0
        return {"k": zeros(self.maps * self.dim), "v": zeros(self.vdim)}

    def run(self, h, out, batch, state):
        z = ops.linear(h, self.w_in)
        q = ops.rotary_store(z, batch.positions, batch.slot_mapping, self.rotary.table, state["k"], state["v"], heads=self.heads,
                             kv_heads=self.kv_heads, maps=self.maps, dim=self.dim, vdim=self.vdim, rot_dims=self.rotary.dims)
        kw = dict(scale=self.scale, lam=self.lam, out_scale=self.out_scale, eps=self.eps)
        for group, call in ((batch.decode, ops.softmax_decode), (batch.prefill, ops.softmax_prefill)):
            if group is not None:
                r = group.rows
                call(q[r], state["k"], state["v"], group, out[r], **kw)


class GatedDelta:
    """The gated delta rule behind short convolutions, with a silu-gated per-head norm (see ``decoder_ops.DeltaWeights``)."""

    def __init__(self, w_q, w_k, w_v, w_gate, w_a, w_b, weights, eps):
        self.w_in = torch.cat([w_q, w_k, w_v, w_gate, w_a, w_b]).contiguous()
        self.weights, self.eps = weights, eps
        self.width = weights.heads * weights.vdim

    def new_state(self, max_seqs, num_blocks, block_size):
        w, dev = self.weights, self.w_in.device
        return {"conv": torch.zeros(max_seqs, w.taps, w.channels, device=dev, dtype=self.w_in.dtype),
                "state": torch.zeros(max_seqs, w.heads, w.dim, w.vdim, device=dev, dtype=torch.float32)}

    def run(self, h, out, batch, state):
        z = ops.linear(h, self.w_in)
        for group, call in ((batch.decode, ops.delta_step), (batch.prefill, ops.delta_prefill)):
            if group is not None:
                r = group.rows
                call(z[r], self.weights, state["conv"], state["state"], group, out[r], self.eps)
