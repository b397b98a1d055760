"""Plain CPU restatement of the Zemivik decoder, one function per mechanism.  TEST INFRASTRUCTURE ONLY.

Whole sequences from their first token, no cache, no chunks, no shared code with the product path: what the tests compare
the kernels and the engine with.  Ordinary torch tensors (fp32 or fp64) in and out, written the way the equations read.
``w`` maps tensor names to tensors, ``cfg`` is the parsed config.json.
"""

import torch


def rms(x, eps):
    """x over its root mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def embed(tokens, w, scale, eps):
    rows = torch.tensor(tokens)
    s = w["embed"][rows] * scale + w["pos"][: len(tokens)]
    return rms(s, eps) * w["embed.norm"]


def visible(n, size, keep_first):
    """(n, n) bool: row i sees column j."""
    see = torch.zeros(n, n, dtype=torch.bool)
    for i in range(n):
        for j in range(i + 1):
            see[i, j] = i - j < size or j < keep_first
    return see


def visible_fast(n, size, keep_first):
    """The same without loops, for long sequences."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def sink_softmax(scores, see, sink=0.0):
    """Weights of the visible scores over exp(sink) + the sum of their exponentials; last axis."""
    s = scores.masked_fill(~see, float("-inf"))
    top = s.amax(-1, keepdim=True).clamp_min(sink)
    e = torch.exp(s - top)
    return e / (torch.exp(sink - top) + e.sum(-1, keepdim=True))


def attend(q, k, v, scale, see, sink=0.0):
    """q (T, H, d), k (T, G, d), v (T, G, e) -> (T, H, e); query head h uses key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[2], dtype=v.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = sink_softmax(q[:, h] @ k[:, g].T * scale, see, sink) @ v[:, g]
    return out


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def gate(o, z):
    return o * torch.sigmoid(z)


def attention_mixer(h, w, p, m, eps, v_first):
    """Returns the mixer's result and the values of the first layer that mixes (None before it)."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = h @ w[p + "v"].T
    if m["v_mix"]:
        if v_first is None:
            v_first = v
        else:
            v = mix_values(v, v_first, w[p + "vmix"])
    see = visible_fast(T, m["mask"]["size"], m["mask"]["keep_first"])
    o = attend(q, k, v.view(T, G, e), m["scale"], see).reshape(T, H * e)
    return gate(o, h @ w[p + "g"].T) @ w[p + "o"].T, v_first


def feed_forward(h, w, p):
    return torch.relu(h @ w[p + "up"].T + w[p + "up.b"]) ** 2 @ w[p + "down"].T + w[p + "down.b"]


def forward(cfg, w, tokens, dtype=torch.float64):
    """Logits (T, vocab) of one sequence and the residual stream after every layer (layers, T, width)."""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x, v_first, runs = embed(tokens, w, cfg["embedding"]["scale"], eps), None, []
    for i, e in enumerate(cfg["layers"]):
        p = f"l{i}."
        o, v_first = attention_mixer(x, w, p + "mix.", e["mixer"], eps, v_first)
        x = x + rms(o, eps) * w[p + "norm1"]
        if e["mlp"] is not None:
            x = x + rms(feed_forward(x, w, p + "mlp."), eps) * w[p + "norm2"]
        runs.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(runs)


def random_weights(cfg, seed):
    """Weights in the design's names and shapes, bf16-representable, as float32."""
    g = torch.Generator().manual_seed(seed)
    D, w = cfg["width"], {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (torch.randn(shape, generator=g) * std + mean).bfloat16().float()

    put("embed", cfg["vocab"], D, std=0.3)
    put("pos", cfg["max_positions"], D, std=0.6)
    put("embed.norm", D, std=0.2, mean=1.0)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(p + "norm1", D, std=0.2, mean=0.8), put(p + "norm2", D, std=0.2, mean=0.8)
        put(p + "mix.q", H * d, D), put(p + "mix.k", G * d, D), put(p + "mix.v", G * vd, D)
        put(p + "mix.q.norm", H * d, std=0.3, mean=1.2), put(p + "mix.k.norm", G * d, std=0.3, mean=1.2)
        put(p + "mix.vmix", std=0.2, mean=0.4)
        put(p + "mix.g", H * vd, D), put(p + "mix.o", D, H * vd)
        if e["mlp"] is not None:
            ff = e["mlp"]["ff"]
            put(p + "mlp.up", ff, D), put(p + "mlp.up.b", ff, std=0.3)
            put(p + "mlp.down", D, ff), put(p + "mlp.down.b", D, std=0.3)
    put("final.norm", D, std=0.2, mean=1.0)
    put("head", cfg["vocab"], D)
    return w
