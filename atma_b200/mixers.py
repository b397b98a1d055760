"""Token mixers of the configured decoder models.

A mixer sits between a layer's norm and its output projection: it owns its input projection (one matrix for all of its
parts), says how many columns it hands to the output projection (``width``), and keeps its per-sequence state in a
tensor dictionary from ``new_state``.  ``run(h, out, batch, state, carry)`` fills ``out`` (rows, width) for the step's
rows: decoding sequences (one row each, first) and prompt portions take their own kernels; ``carry`` is a dictionary in
which the layers of one step leave values for later ones.  All constants are arguments, so a design combines mixers by
configuration.
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
    """Causal softmax attention over a paged cache, grouped key/value heads, one map per head or two (differential:
    o = a1 - lam * a2, divided by its root mean square, times ``out_scale``; ``eps`` inside that root).

    Before the scores either ``rotary`` (a RotaryTable: positions on the first ``rotary.dims`` channels of every map) or
    ``norms`` = (q weight, k weight, eps): q and k divided by their root mean square over the whole projection.
    ``window`` and ``keep_first``: position i sees key j <= i if i - j < window (None = every key) or j < keep_first.
    ``sink``: the score of an added key that has no value (None = none).  ``w_gate``: the result is multiplied by
    sigmoid(w_gate h).  ``first_values``: "leave" puts this layer's values into the step's carry, a number lam caches
    (1 - lam) v + lam v_first with the values left there, None does neither."""

    def __init__(self, w_q, w_k, w_v, *, heads, kv_heads, maps, dim, vdim, scale, rotary=None, norms=None, lam=0.0, out_scale=1.0, eps=0.0,
                 window=None, keep_first=0, sink=None, w_gate=None, first_values=None):
        if rotary is not None and (norms is not None or first_values is not None):
            raise ValueError("rotary positions do not combine with projection norms or value mixing")
        self.w_in = torch.cat([w_q, w_k, w_v] + ([] if w_gate is None else [w_gate])).contiguous()
        self.heads, self.kv_heads, self.maps, self.dim, self.vdim = heads, kv_heads, maps, dim, vdim
        self.scale, self.rotary, self.lam, self.out_scale, self.eps = scale, rotary, lam, out_scale, eps
        self.norms = norms if norms is not None else (None, None, 0.0)
        self.window, self.keep_first, self.sink, self.first_values = window, keep_first, sink, first_values
        self.gated = w_gate is not None
        self.width = heads * vdim

    @property
    def reach(self):
        """Which keys a later position can still see: (window, kept first ones); None = all of them."""
        return None if self.window is None else (self.window, self.keep_first)

    def new_state(self, max_seqs, num_blocks, block_size):
        dt, dev = self.w_in.dtype, self.w_in.device
        zeros = lambda n: torch.zeros(num_blocks, block_size, self.kv_heads, n, device=dev, dtype=dt)   # finite: masked keys weigh 0
        return {"k": zeros(self.maps * self.dim), "v": zeros(self.vdim)}

    def _store(self, z, batch, state, carry):
        """K and V of the step's rows into the cache; returns q (rows, heads, maps, dim)."""
        if self.rotary is not None:
            return ops.rotary_store(z, batch.positions, batch.slot_mapping, self.rotary.table, state["k"], state["v"], heads=self.heads,
                                    kv_heads=self.kv_heads, maps=self.maps, dim=self.dim, vdim=self.vdim, rot_dims=self.rotary.dims)
        nq, nk, nv = self.heads * self.maps * self.dim, self.kv_heads * self.maps * self.dim, self.kv_heads * self.vdim
        mix = {}
        if self.first_values == "leave":
            carry["first_values"] = z[:, nq + nk:nq + nk + nv]
        elif self.first_values is not None:
            mix = dict(v_first=carry["first_values"], lam=self.first_values)
        q_weight, k_weight, eps = self.norms
        q = ops.norm_store(z, batch.slot_mapping, state["k"], state["v"], nq, q_weight=q_weight, k_weight=k_weight, eps=eps, **mix)
        return q.view(-1, self.heads, self.maps, self.dim)

    def run(self, h, out, batch, state, carry=None):
        z = ops.linear(h, self.w_in)
        q = self._store(z, batch, state, carry)
        gate = z[:, z.shape[1] - self.width:] if self.gated else None
        kw = dict(scale=self.scale, lam=self.lam, out_scale=self.out_scale, eps=self.eps, window=self.window, keep_first=self.keep_first,
                  sink=self.sink)
        for group, call in ((batch.decode, ops.softmax_decode), (batch.prefill, ops.softmax_prefill)):
            if group is not None:
                r = group.rows
                call(q[r], state["k"], state["v"], group, out[r], gate=None if gate is None else gate[r], **kw)


class GatedDelta:
    """The gated delta rule behind short convolutions, with a silu-gated per-head norm (see ``decoder_ops.DeltaWeights``)."""

    reach = (0, 0)                                        # no keys in the cache

    def __init__(self, w_q, w_k, w_v, w_gate, w_a, w_b, weights, eps):
        self.w_in = torch.cat([w_q, w_k, w_v, w_gate, w_a, w_b]).contiguous()
        self.weights, self.eps = weights, eps
        self.width = weights.heads * weights.vdim

    def new_state(self, max_seqs, num_blocks, block_size):
        w, dev = self.weights, self.w_in.device
        return {"conv": torch.zeros(max_seqs, w.taps, w.channels, device=dev, dtype=self.w_in.dtype),
                "state": torch.zeros(max_seqs, w.heads, w.dim, w.vdim, device=dev, dtype=torch.float32)}

    def run(self, h, out, batch, state, carry=None):
        z = ops.linear(h, self.w_in)
        for group, call in ((batch.decode, ops.delta_step), (batch.prefill, ops.delta_prefill)):
            if group is not None:
                r = group.rows
                call(z[r], self.weights, state["conv"], state["state"], group, out[r], self.eps)
