"""Small configurations and attention cases for the Zemivik tests (CPU tensors; the tests move them)."""

import torch

from oracle import zemivik as Z


def layer(heads, kv_heads, dim, vdim, *, size=9, keep=3, scale=None, v_mix=True, ff=40):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.1 * dim ** -0.5, "v_mix": v_mix,
                      "mask": {"size": size, "keep_first": keep}}}


def config(layers, *, vocab=97, width=80, eps=3e-6, scale=3.0, max_positions=700):
    return {"architecture": "Zemivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions,
            "embedding": {"scale": scale}, "layers": layers}


CONFIGS = {
    # every layer with sizes, a window and a constant of its own; layers that do not mix before, between and after those that do;
    # one without feed-forward
    "mixed": config([layer(6, 2, 12, 20, size=17, keep=5, v_mix=False, ff=56), layer(4, 2, 24, 12, size=33, keep=0), layer(2, 1, 16, 24, size=1, keep=1, ff=None),
                     layer(3, 3, 8, 8, size=64, keep=2, scale=0.7, ff=24), layer(4, 1, 20, 16, size=5, keep=40, v_mix=False)]),
    # one head, widths that are no multiple of a vector, kept tokens of which there are more than a short prompt has
    "odd": config([layer(1, 1, 5, 7, size=12, keep=70, ff=13), layer(3, 1, 6, 7, size=3, keep=0, ff=9), layer(7, 7, 3, 1, size=100, keep=1, ff=21, scale=1.9)],
                  vocab=61, width=45, scale=0.5, max_positions=421),
    # head sizes that the tensor-core kernels serve when the weights are 16-bit: pairs of heads that share keys, pairs that do not,
    # an odd last head; windows around a page, a tile and far more than the prompt
    "wide": config([layer(4, 2, 64, 128, size=128, keep=4, ff=256), layer(3, 3, 128, 64, size=100, keep=130, v_mix=False, ff=128),
                    layer(6, 2, 64, 128, size=20, keep=0, ff=None), layer(4, 4, 128, 64, size=5000, keep=3, ff=160)], vocab=160, width=192),
    # one layer that sees nothing but the first tokens, one that sees everything
    "ends": config([layer(2, 2, 16, 16, size=0, keep=6, ff=None), layer(2, 1, 16, 32, size=10 ** 9, keep=0, v_mix=False, ff=None)], width=48, scale=1.0),
}


def attention_case(shape, dtype, lengths, starts, block_size, window, keep, sink, seed, spike=True):
    """Random q, k, v of a step's rows with their whole history in a shuffled paged cache and the oracle's output.  With
    ``spike`` many rows look hard at one key: one that is just inside or just outside the window, the last kept one or the
    one after it, the first, or their own, so that a single key's absence or presence decides the row."""
    H, G, dim, vdim = shape
    total, g = sum(lengths), torch.Generator().manual_seed(seed)
    ctx = [s + n for s, n in zip(starts, lengths)]
    pages = [-(-c // block_size) for c in ctx]
    nb = sum(pages) + 3
    perm = torch.randperm(nb, generator=g).tolist()
    tables, at = [], 0
    for p in pages:
        tables.append(perm[at:at + p] + [0] * (max(pages) - p))
        at += p
    kc, vc = torch.randn(nb, block_size, G, dim, generator=g) * 50, torch.randn(nb, block_size, G, vdim, generator=g) * 50     # stale rows
    q, z = torch.randn(total, H, dim, generator=g), torch.randn(total, H * vdim, generator=g) * 2
    scale, head_of = 1.2 * dim ** -0.5, [h // (H // G) for h in range(H)]
    outs, r0 = [], 0
    for s, n in enumerate(lengths):
        k, v = torch.randn(ctx[s], G, dim, generator=g), torch.randn(ctx[s], G, vdim, generator=g)
        if spike:
            for i in range(n):
                pos = starts[s] + i
                target = [pos - window + 1, pos - window, keep - 1, keep, 0, pos, None][i % 7 if n > 1 else (s + seed) % 7]
                if target is not None and 0 <= target <= pos:
                    q[r0 + i] = k[target, head_of] * 3.0
        q, k, v, z = (t.to(dtype).float() for t in (q, k, v, z))
        idx = torch.arange(ctx[s])
        rows = torch.tensor(tables[s])[idx // block_size] * block_size + idx % block_size
        kc.view(-1, G, dim)[rows], vc.view(-1, G, vdim)[rows] = k, v
        see = Z.visible_fast(ctx[s], window, keep)[starts[s]:]
        o = torch.zeros(n, H, vdim, dtype=torch.float64)
        for h in range(H):
            sc = q[r0:r0 + n, h].double() @ k[:, head_of[h]].double().T * scale
            o[:, h] = Z.sink_softmax(sc, see, sink) @ v[:, head_of[h]].double()
        outs.append(Z.gate(o.reshape(n, H * vdim), z[r0:r0 + n].double()))
        r0 += n
    kw = dict(scale=scale, window=window, keep_first=keep, sink=sink)
    return q.to(dtype).view(total, H, 1, dim).cuda(), kc.to(dtype).cuda(), vc.to(dtype).cuda(), z.to(dtype).cuda(), tables, torch.cat(outs), kw
