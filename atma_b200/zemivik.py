"""Zemivik: a decoder-only language model with norms behind its sublayers: attention and feed-forward read the residual
stream itself, and what they add to it is normalised:

    x <- x + norm1(attention(x)),  x <- x + norm2(ff(x))

The stream starts as the norm of the scaled embedding plus a learned position vector.  Attention: grouped heads, q and k
normalised over their whole projections, no rotation, a sliding window with kept first tokens, a sink of score zero in the
softmax, values mixed with those of the first layer that mixes, a sigmoid gate on the result.  Feed-forward: squared relu
with biases.  The residual stream is fp32.

config.json: ``vocab``, ``width``, ``max_positions``, ``norm.eps``, ``embedding.scale`` and ``layers`` (type, ``mixer``:
heads, kv_heads, dim, vdim, scale, ``mask`` (size, keep_first), v_mix; ``mlp``: kind, ff, or null).  Tensors: embed, pos,
embed.norm, l<i>.norm1/2, l<i>.mix.{q,k,v,q.norm,k.norm,vmix,g,o}, l<i>.mlp.{up,up.b,down,down.b}, final.norm, head.

A sublayer's bias, its norm, the residual add and the conversion of the new stream for the next matrix product are one
launch.
"""

from types import SimpleNamespace

import torch

from . import decoder_ops as ops
from .configured import ConfiguredModel
from .mixers import SoftmaxAttention

SINK_SCORE = 0.0


class ZemivikModel(ConfiguredModel):
    def _build(self, config):
        D = self.width
        self.max_positions = config["max_positions"]
        self.embed, self.embed_scale = self._w("embed", self.vocab, D), float(config["embedding"]["scale"])
        self.pos, self.embed_norm = self._w("pos", self.max_positions, D), self._w("embed.norm", D)
        self.mixing = [i for i, e in enumerate(config["layers"]) if e["mixer"].get("v_mix")]
        self.layers = [self._layer(i, e) for i, e in enumerate(config["layers"])]
        self.final_norm, self.head = self._w("final.norm", D), self._w("head", self.vocab, D)
        self.run_mixers = [layer.mixer for layer in self.layers]

    def _layer(self, i, entry):
        p, D = f"l{i}.", self.width
        if entry["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
        layer = SimpleNamespace(mixer=self._attention(i, p + "mix.", entry["mixer"]), norm1=self._w(p + "norm1", D), ff=0)
        layer.w_o = self._w(p + "mix.o", D, layer.mixer.width)
        if entry.get("mlp") is not None:
            if entry["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {entry['mlp']['kind']!r}")
            layer.ff = entry["mlp"]["ff"]
            layer.norm2 = self._w(p + "norm2", D)
            layer.w_up, layer.b_up = self._w(p + "mlp.up", layer.ff, D), self._w(p + "mlp.up.b", layer.ff)
            layer.w_down, layer.b_down = self._w(p + "mlp.down", D, layer.ff), self._w(p + "mlp.down.b", D)
        return layer

    def _attention(self, i, p, m):
        D, H, G, d, e = self.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if H % G:
            raise ValueError(f"layer {i}: {H} query heads over {G} key/value heads")
        mask = m.get("mask") or {}
        first_values = None
        if i in self.mixing:
            first = self.config["layers"][self.mixing[0]]["mixer"]
            if first["kv_heads"] * first["vdim"] != G * e:
                raise ValueError(f"layer {i}: its values differ in width from layer {self.mixing[0]}'s, which it mixes in")
            first_values = "leave" if i == self.mixing[0] else float(self._w(p + "vmix", dtype=torch.float32))
        return SoftmaxAttention(self._w(p + "q", H * d, D), self._w(p + "k", G * d, D), self._w(p + "v", G * e, D), heads=H, kv_heads=G, maps=1,
                                dim=d, vdim=e, scale=float(m["scale"]), norms=(self._w(p + "q.norm", H * d), self._w(p + "k.norm", G * d), self.eps),
                                window=mask.get("size"), keep_first=mask.get("keep_first") or 0, sink=SINK_SCORE, w_gate=self._w(p + "g", H * e, D),
                                first_values=first_values)

    @torch.no_grad()
    def forward(self, batch, state, record=None):
        """One step: the batch's rows through all layers, caches updated; fp32 logits of ``batch.logit_rows`` (None when
        empty).  ``record``: a list that receives the residual stream after every layer."""
        x, h = ops.embed_position_norm(batch.ids, batch.positions, self.embed, self.pos, self.embed_norm, self.eps, self.embed_scale)
        carry, pending = {}, None                              # pending: the last sublayer's result, not yet added to x
        for layer, kept in zip(self.layers, state):
            if pending is not None:
                h = ops.residual_post_norm(x, *pending)
                if record is not None:
                    record.append(x.clone())
            o = torch.empty((x.shape[0], layer.mixer.width), device=x.device, dtype=self.dtype)
            layer.mixer.run(h, o, batch, kept, carry)
            pending = (ops.linear(o, layer.w_o), layer.norm1, self.eps)
            if layer.ff:
                h = ops.residual_post_norm(x, *pending)
                u = ops.squared_relu_linear(h, layer.w_up, layer.b_up)
                pending = (ops.linear(u, layer.w_down), layer.norm2, self.eps, layer.b_down)
        if record is not None and pending is not None:         # once more without the rows' selection
            full = x.clone()
            ops.residual_post_norm(full, *pending)
            record.append(full)
        rows = batch.logit_rows
        if rows is None:
            return None
        if pending is None:
            h, = ops.residual_norms(x.index_select(0, rows), None, (self.final_norm,), self.eps, offset=0.0)
        else:                                                  # the last add and the final norm, of the wanted rows only
            y, *rest = pending
            h = ops.residual_post_norm(x.index_select(0, rows), y.index_select(0, rows), *rest, next_weight=self.final_norm, in_place=False)
        return ops.linear_f32_out(h, self.head)

    def weight_bytes(self):
        """Bytes of weights one decode step reads."""
        per = [l.mixer.w_in.numel() + l.w_o.numel() + (l.w_up.numel() + l.w_down.numel() if l.ff else 0) for l in self.layers]
        return (sum(per) + self.head.numel()) * self.head.element_size()
