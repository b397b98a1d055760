"""``python bench.py --zemivik``: prefill and decode throughput of Zemivik at a few layer sizes beside the framework's
closest other models at the same width, depth, feed-forward size and vocabulary - Rizurax with attention layers only, and
``AtmaModel`` - and every kernel of the design beside the like kernel of those models, each with its own roofline.  Random
weights, synthetic tokens, bf16, one GPU.  Timing as in ``bench_decoder``."""

import torch

from bench_decoder import BS, VOCAB, atma_leg, batch_of, dev_ms, model_leg, rizurax_leg, roof

WINDOW, KEEP = 1024, 4


def config(width, layers, max_positions):
    """Every fourth layer sees everything, the others a window; per-layer feed-forward of 12 * width^2 weights."""
    H = width // 128
    layer = lambda size: {"type": "attention", "mlp": {"kind": "dense", "ff": 6 * width},
                          "mixer": {"heads": H, "kv_heads": max(2, H // 4), "dim": 128, "vdim": 128, "scale": 0.1, "v_mix": True,
                                    "mask": {"size": size, "keep_first": KEEP}}}
    return {"architecture": "Zemivik", "vocab": VOCAB, "width": width, "max_positions": max_positions, "norm": {"eps": 1e-6},
            "embedding": {"scale": 4.0}, "layers": [layer(max_positions if i % 4 == 3 else WINDOW) for i in range(layers)]}


def weights(cfg, seed, device):
    """Random weights in the design's names, drawn on the device."""
    g = torch.Generator(device=device).manual_seed(seed)
    D, w = cfg["width"], {}

    def put(name, *shape, std=None, mean=0.0):
        w[name] = (torch.randn(shape, device=device, generator=g) * (shape[-1] ** -0.5 if std is None else std) + mean).bfloat16()
    put("embed", cfg["vocab"], D, std=0.3), put("pos", cfg["max_positions"], D, std=0.5), put("embed.norm", D, std=0.1, mean=1.0)
    for i, e in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", e["mixer"], e["mlp"]["ff"]
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(p + "norm1", D, std=0.1, mean=1.0), put(p + "norm2", D, std=0.1, mean=1.0)
        put(p + "mix.q", H * d, D), put(p + "mix.k", G * d, D), put(p + "mix.v", G * vd, D), put(p + "mix.g", H * vd, D), put(p + "mix.o", D, H * vd)
        put(p + "mix.q.norm", H * d, std=0.1, mean=1.0), put(p + "mix.k.norm", G * d, std=0.1, mean=1.0), put(p + "mix.vmix", std=0.1, mean=0.3)
        put(p + "mlp.up", ff, D), put(p + "mlp.up.b", ff, std=0.1), put(p + "mlp.down", D, ff), put(p + "mlp.down.b", D, std=0.1)
    put("final.norm", D, std=0.1, mean=1.0), put("head", cfg["vocab"], D)
    return w


def seen_keys(T, window, keep):
    """Sum over the positions of a sequence of the keys they see."""
    i = torch.arange(T, dtype=torch.float64) + 1
    near = i.clamp_max(window)
    return float((near + (i - near).clamp_max(keep)).sum())


def kernel_legs(peaks, device, only=None):
    """{name: {"zemivik": roofline, "like": [kernel, roofline]}}"""
    import atma_b200 as ab
    from atma_b200 import decoder_ops as ops
    from atma_b200.layer import PackedMaps
    H, G, DK = 8, 2, 128
    g = torch.Generator(device=device).manual_seed(1)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g, dtype=torch.bfloat16)
    out = {}

    def want(name):
        return only is None or only == name

    P = {n: torch.full((H,), v, device=device) for n, v in (("null_base", 2.0), ("null_slope_raw", 0.5), ("len_gain_raw", -1.0), ("mag_beta_raw", -1.5))}
    P["v_null"] = torch.zeros(H, DK, device=device)
    if want("softmax_prefill"):
        for T, window in ((32768, None), (65536, WINDOW)):
            b, nb = batch_of(device, 1, T)
            q, kc, vc, gate, o = rnd(T, H, 1, DK), rnd(nb, BS, G, DK), rnd(nb, BS, G, DK), rnd(T, H * DK), rnd(T, H * DK)
            ms = dev_ms(lambda: ops.softmax_prefill(q, kc, vc, b.prefill, o, scale=0.09, window=window, keep_first=KEEP if window else 0, sink=0.0, gate=gate), 5)
            pq, pk = rnd(1, T, H, DK), rnd(2, 1, T, G, DK)
            n = torch.arange(1, T + 1, dtype=torch.float32, device=device)
            lk = dev_ms(lambda: ab.polar_attention_fwd(pq.transpose(1, 2), pk[0].transpose(1, 2), pk[1].transpose(1, 2), n, window=window, **P), 5)
            fl = lambda keep: 4.0 * DK * H * seen_keys(T, window or T, keep)
            out["softmax_prefill" + ("_window" if window else "")] = {
                "shape": f"T={T}, {H}/{G} heads of {DK}" + (f", window {window}" if window else ""), "zemivik": roof(ms, peaks, flops=fl(KEEP)),
                "like": ["polar_prefill", roof(lk, peaks, flops=fl(0))]}
            del q, kc, vc, gate, o, pq, pk
    if want("softmax_decode"):
        for B, ctx, window in ((64, 16384, None), (64, 16384, WINDOW), (256, 4096, WINDOW)):
            b, nb = batch_of(device, B, ctx, True)
            q, gate, o = rnd(B, H, 1, DK), rnd(B, H * DK), rnd(B, H * DK)
            caches = [(rnd(nb, BS, G, DK), rnd(nb, BS, G, DK)) for _ in range(2 if window else 1)]     # windows: rotating, beyond L2
            it = iter(range(10 ** 9))
            pick = lambda: caches[next(it) % len(caches)]
            ms = dev_ms(lambda: ops.softmax_decode(q, *pick(), b.decode, o, scale=0.09, window=window, keep_first=KEEP if window else 0, sink=0.0, gate=gate), 20)
            cl, pq, pg = torch.full((B,), ctx, dtype=torch.int32, device=device), rnd(B, H, DK), rnd(B, H, DK)
            lk = dev_ms(lambda: ab.polar_attention_decode(pq, *pick(), b.decode.block_tables, cl, window=window, gate=pg, **P), 20)
            nbytes = B * (min(ctx, window + KEEP) if window else ctx) * G * 2 * DK * 2.0
            out[f"softmax_decode_{B}" + ("_window" if window else "")] = {
                "shape": f"{B} x {ctx}, {H}/{G} heads of {DK}" + (f", window {window}" if window else ""), "zemivik": roof(ms, peaks, nbytes),
                "like": ["polar_decode", roof(lk, peaks, nbytes)]}
            del caches
    if want("rows"):
        n, D = 65536, 2048
        b, nb = batch_of(device, 8, n // 8)
        z, first = rnd(n, (2 * H + 2 * G) * DK), rnd(n, G * DK)
        kc, vc, wq, wk = rnd(nb, BS, G, DK), rnd(nb, BS, G, DK), rnd(H * DK), rnd(G * DK)
        ms = dev_ms(lambda: ops.norm_store(z, b.slot_mapping, kc, vc, H * DK, q_weight=wq, k_weight=wk, eps=1e-6, v_first=first, lam=0.3))
        maps = PackedMaps([n // 8] * 8, list(range(8)), device)
        qg, kk, vv = rnd(n, H, 2 * DK), rnd(n, G, DK), rnd(n, G, DK)
        ws, st = [rnd(C, 4) for C in (H * DK, G * DK, G * DK)], [torch.zeros(8, C, 3, dtype=torch.bfloat16, device=device) for C in (H * DK, G * DK, G * DK)]
        fk, fv, sm = rnd(n, G, DK), rnd(n, G, DK), torch.arange(n, device=device)
        lk = dev_ms(lambda: ab.qkv_prep_prefill(qg, kk, vv, *ws, *st, maps.token_seq_starts, maps.token_seq_ends, maps.token_seq_slots, fk, fv, sm))
        out["norm_store"] = {"shape": f"{n} rows, {H}/{G} heads of {DK}", "zemivik": roof(ms, peaks, n * (2 * H + 5 * G) * DK * 2.0),
                             "like": ["qkv_prep_prefill", roof(lk, peaks, n * (2 * H + 5 * G) * DK * 2.0)]}
        del z, first, qg, kk, vv
        x, y, w, bias = torch.randn(n, D, device=device), rnd(n, D), rnd(D), rnd(D)
        like = ["residual_norms (two norms)", roof(dev_ms(lambda: ops.residual_norms(x, y, (w, bias), 1e-6)), peaks, n * D * 14.0)]
        ms = dev_ms(lambda: ops.residual_post_norm(x, y, w, 1e-6, bias))
        out["residual_post_norm"] = {"shape": f"{n} x {D}, fp32 residual", "zemivik": roof(ms, peaks, n * D * 12.0), "like": like}
        ms = dev_ms(lambda: ops.residual_post_norm(x, y, w, 1e-6, bias, next_weight=w))
        out["residual_post_norm_next"] = {"shape": f"{n} x {D}, and the next norm", "zemivik": roof(ms, peaks, n * D * 12.0), "like": like}
        ids, pos = (torch.randint(0, VOCAB, (n,), device=device, dtype=torch.int32) for _ in range(2))
        e, pt = rnd(VOCAB, D), rnd(VOCAB, D)
        ms = dev_ms(lambda: ops.embed_position_norm(ids, pos, e, pt, w, 1e-6, 3.0))
        lk = dev_ms(lambda: ops.embed_bigram(ids, pos, e, pt, 101, 7))
        out["embed_position_norm"] = {"shape": f"{n} x {D}", "zemivik": roof(ms, peaks, n * D * 10.0), "like": ["embed_bigram", roof(lk, peaks, n * D * 8.0)]}
        del x, y, e, pt
        zf, bf = rnd(n // 2, 4 * D), rnd(4 * D)
        ms = dev_ms(lambda: ops.bias_squared_relu(zf, bf, zf))
        gu = rnd(n // 2, 4 * D)
        lk = dev_ms(lambda: ab.squared_relu_gate(gu[:, :2 * D], gu[:, 2 * D:]))
        out["bias_squared_relu"] = {"shape": f"{n // 2} x {4 * D}", "zemivik": roof(ms, peaks, 2.0 * zf.numel() * 2),
                                    "like": ["squared_relu_gate", roof(lk, peaks, 1.5 * gu.numel() * 2)]}
        del zf, gu
        nd = 8                                               # a decode step's rows: launch-bound, in us
        b, nb = batch_of(device, nd, BS, True)
        z, first = rnd(nd, (2 * H + 2 * G) * DK), rnd(nd, G * DK)
        kc, vc = rnd(nb, BS, G, DK), rnd(nb, BS, G, DK)
        x, y = torch.randn(nd, D, device=device), rnd(nd, D)
        out["decode_rows_us"] = {"norm_store": 1e3 * dev_ms(lambda: ops.norm_store(z, b.slot_mapping, kc, vc, H * DK, q_weight=wq, k_weight=wk, eps=1e-6, v_first=first, lam=0.3), 50),
                                 "residual_post_norm": 1e3 * dev_ms(lambda: ops.residual_post_norm(x, y, w, 1e-6, bias), 50),
                                 "residual_norms": 1e3 * dev_ms(lambda: ops.residual_norms(x, y, (w, bias), 1e-6), 50)}
    if want("linear"):
        D, ff, copies = 2048, 12288, 8
        wf, bf, xs = [rnd(ff, D) * D ** -0.5 for _ in range(copies)], rnd(ff), rnd(8, D)
        it = iter(range(10 ** 9))
        ms = dev_ms(lambda: ops.squared_relu_linear(xs, wf[next(it) % copies], bf), 24)
        lk = dev_ms(lambda: ab.decode_linear(xs, wf[next(it) % copies], None, gated=True), 24)
        out["squared_relu_linear"] = {"shape": f"8 x {D} -> {ff}", "zemivik": roof(ms, peaks, 2.0 * ff * D), "like": ["decode_linear gated", roof(lk, peaks, 2.0 * ff * D)]}
    for e in out.values():                                     # how much farther from its roofline than the like kernel
        if "like" in e:
            e["distance_ratio"] = e["like"][1]["frac"] / e["zemivik"]["frac"]
    return out


def run(peaks, device, only=None):
    res = {"kernels": kernel_legs(peaks, device, only)}
    if only is None or only == "models":
        prompts, decodes, layers = [(4, 4096), (1, 32768)], [(8, 8192), (64, 8192)], 8
        for width in (1024, 2048, 4096):
            cfg = config(width, layers, 32768)
            res[f"width_{width}"] = {"layers": layers, "zemivik": model_leg(cfg, weights(cfg, 5, device), prompts, decodes, device),
                                     "rizurax": rizurax_leg(width, layers, prompts, decodes, device, 1),
                                     "atma": atma_leg(width, layers, prompts, decodes, device)}
    from atma_b200 import decoder_ops
    res["device_status"] = decoder_ops.device_status()
    return res
