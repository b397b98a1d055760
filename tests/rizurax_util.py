"""Small configurations, weights and row groups for the Rizurax tests (CPU tensors; the tests move them)."""

import torch

from atma_b200.engine import TILE_ROWS, RowGroup

YARN = {"factor": 6.0, "original": 512, "fast": 24.0, "slow": 1.5}


def attention(heads, kv_heads, dim, vdim, *, rot=8, base=900.0, scaling=YARN, scale=None, diff=0.3, ff=40):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale or 1.3 * dim ** -0.5,
                      "rot": {"dims": rot, "base": base, **({"scaling": scaling} if scaling else {})}}}


def delta(heads, kv_heads, dim, vdim, *, conv=3, ff=40):
    return {"type": "delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, *, vocab=97, width=80, loop=None, eps=3e-6, bigram=(53, 11, 5)):
    cfg = {"architecture": "Rizurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "embedding": {"bigram": None if bigram is None else {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


CONFIGS = {
    # grouped heads, all sizes different, a loop in the middle, two layers without feed-forward, another base per layer
    "mixed": config([attention(6, 2, 12, 20, rot=8, ff=56), delta(6, 3, 20, 12, conv=5), attention(2, 1, 24, 8, rot=24, base=30.0, scaling=None, ff=None),
                     delta(2, 2, 8, 36, conv=2, ff=None)], loop=(1, 3, 3)),
    # a single head, one tap, the loop over everything, widths that are no multiple of a vector
    "odd": config([delta(1, 1, 5, 7, conv=1, ff=13), attention(3, 3, 6, 10, rot=2, diff=0.8, ff=9), delta(3, 1, 33, 65, conv=4, ff=21)], vocab=61,
                  width=45, loop=(0, 3, 2), bigram=(17, 3, 29)),
    # head sizes that the tensor-core kernels serve when the weights are 16-bit
    "wide": config([delta(4, 2, 128, 128, conv=4, ff=256), attention(4, 2, 64, 128, rot=32, base=5000.0, ff=192), attention(2, 2, 128, 64, rot=64, ff=128),
                    delta(2, 1, 128, 256, conv=3, ff=None)], vocab=160, width=192, bigram=(71, 13, 7)),
    # no loop, no bigram, no feed-forward anywhere
    "bare": config([attention(2, 2, 16, 16, ff=None), delta(2, 1, 16, 24, ff=None)], width=48, bigram=None),
}


def group(lengths, starts, slots, tables, device="cuda", decode=False, first_row=0):
    """A RowGroup from host lists; ``tables``: block table rows."""
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    t_seq = [s for s, n in enumerate(lengths) for _ in range(-(-n // TILE_ROWS))]
    t_row = [r for n in lengths for r in range(0, n, TILE_ROWS)]
    return RowGroup(slice(first_row, first_row + cu[-1]), len(lengths), max(lengths), cu[-1], i32(cu), i32(starts),
                    torch.tensor(slots, dtype=torch.int64, device=device), i32(tables),
                    None if decode else i32([s for s, n in enumerate(lengths) for _ in range(n)]), None if decode else i32(t_seq),
                    None if decode else i32(t_row), tuple(lengths), tuple(slots))


def prompt(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def logit_error(got, want):
    """Root mean square over the vocabulary of the difference without its mean, relative to the logits' spread; per row."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()
