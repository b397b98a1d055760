"""Plain CPU restatement of the Rizurax decoder, one function per mechanism.  TEST INFRASTRUCTURE ONLY.

Whole sequences from their first token, no cache, no chunks, no shared code with the product path: what
the tests compare the kernels and the engine with.  Every function takes and returns ordinary torch tensors (fp32 or fp64); loops run
over tokens and heads exactly as the equations are written.  ``w`` is a mapping from tensor names to tensors, ``cfg``
the parsed config.json.
"""

import math

import torch


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm_centered(x, weight, eps):
    """x / sqrt(mean x^2 + eps) * (1 + weight)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1 + weight)


def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """Row of the bigram table for every token of a sequence; the first token has the row after the last bucket."""
    rows = []
    for t, cur in enumerate(tokens):
        rows.append(buckets if t == 0 else (tokens[t - 1] * mul_prev + cur * mul_cur) % buckets)
    return rows


def embed(tokens, w, bigram):
    x = w["embed"][torch.tensor(tokens)]
    if bigram is None:
        return x
    return x + w["bigram"][torch.tensor(bigram_rows(tokens, bigram["mul_prev"], bigram["mul_cur"], bigram["buckets"]))]


def causal_conv_silu(x, taps):
    """x (T, C), taps (C, K), the last tap on the current token; zeros before the start; then silu."""
    T, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                out[t] += x[src] * taps[:, j]
    return out / (1 + torch.exp(-out))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp_min(0)


def delta_rule(q, k, v, g, beta, state=None):
    """q, k (T, H, K); v (T, H, V); g (decay factor), beta (T, H).  Returns o (T, H, V) and the last state (H, K, V)."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=v.dtype) if state is None else state.clone()
    o = torch.zeros_like(v)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def delta_mixer(h, w, p, mix, eps):
    T = h.shape[0]
    H, G, K, V = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    conv = {n: causal_conv_silu(h @ w[f"{p}{n}"].T, w[f"{p}{n}.conv"]) for n in ("q", "k", "v")}
    q = unit(conv["q"].view(T, G, K)) * K ** -0.5
    k = unit(conv["k"].view(T, G, K))
    head_of = [i // (H // G) for i in range(H)]
    v = conv["v"].view(T, H, V)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_rule(q[:, head_of], k[:, head_of], v, g, beta)
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * w[p + "norm"]
    gate = (h @ w[p + "g"].T).view(T, H, V)
    o = o * gate * torch.sigmoid(gate)
    return o.reshape(T, H * V) @ w[p + "o"].T


def rotary_frequencies(rot):
    """(frequencies of the pairs, factor on cos and sin); float64."""
    n = rot["dims"]
    i = torch.arange(n // 2, dtype=torch.float64)
    f = rot["base"] ** (-2 * i / n)
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0

    def turn_dim(t):
        return n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(rot["base"]))

    lo = max(math.floor(turn_dim(sc["fast"])), 0)
    hi = min(math.ceil(turn_dim(sc["slow"])), n - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot, first_position=0):
    """x (T, heads, dim): neighbouring pairs of the first rot.dims channels are turned by position * frequency."""
    f, m = rotary_frequencies(rot)
    T, n = x.shape[0], rot["dims"]
    a = (torch.arange(first_position, first_position + T, dtype=torch.float64)[:, None] * f).to(torch.float64)
    c, s = (m * torch.cos(a)).to(x.dtype)[:, None], (m * torch.sin(a)).to(x.dtype)[:, None]
    out = x.clone()
    out[..., 0:n:2] = x[..., 0:n:2] * c - x[..., 1:n:2] * s
    out[..., 1:n:2] = x[..., 1:n:2] * c + x[..., 0:n:2] * s
    return out


def causal_softmax_attention(q, k, v, scale):
    """q (T, H, d), k (T, H, d), v (T, H, e) -> (T, H, e)."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, -1), v)


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_combine(a1, a2, lam, diff, eps):
    o = a1 - lam * a2
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * (1 - diff)


def attention_mixer(h, w, p, mix, eps):
    T = h.shape[0]
    H, G, d, e = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rotate((h @ w[p + "q"].T).view(T, H * 2, d), mix["rot"]).view(T, H, 2, d)
    k = rotate((h @ w[p + "k"].T).view(T, G * 2, d), mix["rot"]).view(T, G, 2, d)
    v = (h @ w[p + "v"].T).view(T, G, e)
    head_of = [i // (H // G) for i in range(H)]
    k, v = k[:, head_of], v[:, head_of]
    a1 = causal_softmax_attention(q[:, :, 0], k[:, :, 0], v, mix["scale"])
    a2 = causal_softmax_attention(q[:, :, 1], k[:, :, 1], v, mix["scale"])
    lam = differential_lambda(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), mix["diff"])
    return differential_combine(a1, a2, lam, mix["diff"], eps).reshape(T, H * e) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer(x, w, i, entry, eps):
    p = f"l{i}."
    mixer = {"delta": delta_mixer, "attention": attention_mixer}[entry["type"]]
    out = x + mixer(rms_norm_centered(x, w[p + "norm1"], eps), w, p + "mix.", entry["mixer"], eps)
    if entry["mlp"] is not None:
        out = out + feed_forward(rms_norm_centered(x, w[p + "norm2"], eps), w, p + "mlp.")
    return out


def layer_order(cfg):
    """Indices of the layers in the order they run; the looped ones appear once per pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, w, tokens, dtype=torch.float64):
    """Logits (T, vocab) of one sequence and the residual stream after every layer run (runs, T, width)."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w, cfg["embedding"].get("bigram"))
    runs = []
    for i in layer_order(cfg):
        x = layer(x, w, i, cfg["layers"][i], eps)
        runs.append(x)
    return rms_norm_centered(x, w["final.norm"], eps) @ w["head"].T, torch.stack(runs)


def random_weights(cfg, seed, scale=1.0):
    """Weights in the design's names and shapes, bf16-representable, as float32."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = (shape[-1] ** -0.5 if std is None else std) * scale
        w[name] = (torch.randn(*shape, generator=g) * std + mean).bfloat16().float()

    put("embed", V, D, std=1.0)
    if cfg["embedding"].get("bigram"):
        put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, D, std=0.7)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        put(p + "norm1", D, std=0.2)
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if e["type"] == "delta":
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * vd)):
                put(p + "mix." + n, rows, D)
                put(p + f"mix.{n}.conv", rows, m["conv"], std=0.5)
            put(p + "mix.b", H, D)
            put(p + "mix.a", H, D)
            put(p + "mix.A_log", H, std=0.5, mean=-1.0)
            put(p + "mix.dt_bias", H, std=0.5, mean=-2.0)
            put(p + "mix.norm", vd, std=0.2, mean=1.0)
            put(p + "mix.g", H * vd, D)
            put(p + "mix.o", D, H * vd)
        else:
            for n, rows in (("q", H * 2 * d), ("k", G * 2 * d), ("v", G * vd)):
                put(p + "mix." + n, rows, D)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + "mix." + n, d, std=0.3)
            put(p + "mix.o", D, H * vd)
        if e["mlp"] is not None:
            put(p + "norm2", D, std=0.2)
            ff = e["mlp"]["ff"]
            put(p + "mlp.gate", ff, D)
            put(p + "mlp.up", ff, D)
            put(p + "mlp.down", D, ff)
    put("final.norm", D, std=0.2)
    put("head", V, D)
    return w
