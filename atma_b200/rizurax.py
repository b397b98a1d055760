"""Rizurax: a decoder-only language model whose layers each hold a token mixer (gated delta rule or differential
attention) and, optionally, a gelu-gated feed-forward, both fed by their own norm of the same residual stream:

    x <- x + mixer(norm1(x)) + ff(norm2(x))

A stretch of layers may run several times in a row with the same weights; every pass has its own cache or state.  The
embedding adds a hashed bigram term.  The residual stream is fp32.

config.json: ``vocab``, ``width``, ``norm.eps``, ``embedding.bigram`` (buckets, mul_prev, mul_cur), ``layers`` (type,
mixer sizes, mlp or null) and ``loop`` (start, stop, times).  Tensors: embed, bigram, l<i>.norm1/2, l<i>.mix.*,
l<i>.mlp.gate/up/down, final.norm, head.

A layer's mixer output and its feed-forward activation lie side by side in one buffer, so that W_o and W_down are one
matrix product whose sum is what the residual stream receives; the add, the next layer's two norms and the conversion
of their results are one launch.
"""

from types import SimpleNamespace

import torch

from . import decoder_ops as ops
from .configured import ConfiguredModel
from .mixers import GatedDelta, SoftmaxAttention

UNIT_EPS = 1e-6                # inside the root of the unit vectors of q and k


def layer_order(config):
    """Layer index of every layer run, looped stretches unrolled."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    if not 0 <= start <= stop <= n or times < 0:
        raise ValueError(f"loop {loop} does not fit {n} layers")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


class RizuraxModel(ConfiguredModel):
    def _build(self, config):
        self.order = layer_order(config)
        self.embed = self._w("embed", self.vocab, self.width)
        big = (config.get("embedding") or {}).get("bigram")
        self.bigram = self._w("bigram", big["buckets"] + 1, self.width) if big else None
        self.bigram_mul = (big["mul_prev"], big["mul_cur"]) if big else (0, 0)
        self.layers = [self._layer(i, e) for i, e in enumerate(config["layers"])]
        self.final_norm, self.head = self._w("final.norm", self.width), self._w("head", self.vocab, self.width)
        self.run_mixers = [self.layers[i].mixer for i in self.order]           # a looped layer has a cache per pass

    # ---- weights ----------------------------------------------------------------------------------------------
    def _layer(self, i, entry):
        p, D, m = f"l{i}.", self.width, entry["mixer"]
        kind = entry["type"]
        if kind == "attention":
            mixer = self._attention(p + "mix.", m)
        elif kind == "delta":
            mixer = self._delta(p + "mix.", m)
        else:
            raise ValueError(f"layer {i}: unknown mixer {kind!r}")
        layer = SimpleNamespace(mixer=mixer, norm1=self._w(p + "norm1", D), norm2=None, w_gate_up=None, ff=0)
        w_out = [self._w(p + "mix.o", D, mixer.width)]
        if entry.get("mlp") is not None:
            if entry["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {entry['mlp']['kind']!r}")
            layer.ff = entry["mlp"]["ff"]
            layer.norm2 = self._w(p + "norm2", D)
            layer.w_gate_up = torch.cat([self._w(p + "mlp.gate", layer.ff, D), self._w(p + "mlp.up", layer.ff, D)]).contiguous()
            w_out.append(self._w(p + "mlp.down", D, layer.ff))
        layer.w_out = torch.cat(w_out, dim=1).contiguous()
        return layer

    def _attention(self, p, m):
        D, H, G, d, e = self.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        diff = float(m["diff"])
        lq1, lk1, lq2, lk2 = (self._w(p + n, d, dtype=torch.float32) for n in ("lq1", "lk1", "lq2", "lk2"))
        lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff)
        return SoftmaxAttention(self._w(p + "q", H * 2 * d, D), self._w(p + "k", G * 2 * d, D), self._w(p + "v", G * e, D), heads=H,
                                kv_heads=G, maps=2, dim=d, vdim=e, scale=float(m["scale"]), rotary=self._rotary(m.get("rot")), lam=lam,
                                out_scale=1.0 - diff, eps=self.eps)

    def _delta(self, p, m):
        D, H, G, d, e, taps = self.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        f32 = torch.float32
        weights = ops.DeltaWeights(self._w(p + "q.conv", G * d, taps), self._w(p + "k.conv", G * d, taps), self._w(p + "v.conv", H * e, taps),
                                   self._w(p + "A_log", H, dtype=f32), self._w(p + "dt_bias", H, dtype=f32), self._w(p + "norm", e), heads=H,
                                   kv_heads=G, dim=d, vdim=e, unit_eps=UNIT_EPS, q_scale=d ** -0.5)
        return GatedDelta(self._w(p + "q", G * d, D), self._w(p + "k", G * d, D), self._w(p + "v", H * e, D), self._w(p + "g", H * e, D),
                          self._w(p + "a", H, D), self._w(p + "b", H, D), weights, self.eps)

    # ---- the step ---------------------------------------------------------------------------------------------
    @torch.no_grad()
    def forward(self, batch, state, record=None):
        """One step: the batch's rows through all layers, caches and states updated; fp32 logits of ``batch.logit_rows``
        (None when empty).  ``record``: a list that receives the residual stream after every layer run."""
        x = ops.embed_bigram(batch.ids, batch.prev, self.embed, self.bigram, *self.bigram_mul)
        runs = [self.layers[i] for i in self.order]
        h1, h2 = ops.residual_norms(x, None, (runs[0].norm1, runs[0].norm2), self.eps) if runs else (None, None)
        y = None
        for r, layer in enumerate(runs):
            act = torch.empty((x.shape[0], layer.mixer.width + layer.ff), device=x.device, dtype=self.dtype)
            layer.mixer.run(h1, act[:, :layer.mixer.width], batch, state[r])
            if layer.ff:
                ops.gelu_gated_linear(h2, layer.w_gate_up, act[:, layer.mixer.width:])
            y = ops.linear(act, layer.w_out)
            if r + 1 < len(runs):
                h1, h2 = ops.residual_norms(x, y, (runs[r + 1].norm1, runs[r + 1].norm2), self.eps)
                if record is not None:
                    record.append(x.clone())
        if record is not None and y is not None:
            record.append(x + y)
        if batch.logit_rows is None:
            return None
        xs, ys = x.index_select(0, batch.logit_rows), None if y is None else y.index_select(0, batch.logit_rows)
        h, = ops.residual_norms(xs, ys, (self.final_norm,), self.eps)
        return ops.linear_f32_out(h, self.head)

    def weight_bytes(self):
        """Bytes of weights one decode step reads (a looped layer's once per pass)."""
        per = [l.mixer.w_in.numel() + l.w_out.numel() + (l.w_gate_up.numel() if l.ff else 0) for l in self.layers]
        return (sum(per[i] for i in self.order) + self.head.numel()) * self.head.element_size()
