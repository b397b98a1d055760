"""``python bench.py --rizurax``: prefill and decode throughput of Rizurax at a few layer sizes beside the framework's
closest other model (``AtmaModel``) at the same width, depth, feed-forward and vocabulary, and every kernel of the design
beside the like kernel of that model, each with its own roofline.  Random weights, synthetic tokens, bf16, one GPU.

Kernel times are CUDA events around back-to-back launches (the queue is filled behind a sleep kernel, so host time is not
in them) over inputs larger than L2."""

import torch
import torch.nn.functional as F

VOCAB = 32768
BS = 256


def dev_ms(fn, iters=10, warm=3):
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda._sleep(40_000_000)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def roof(ms, peaks, nbytes=None, flops=None):
    if flops is not None:
        v, peak, unit, bound = flops / (ms * 1e-3) / 1e12, peaks["tf_burst"], "TFLOP/s", "tensor"
    else:
        v, peak, unit, bound = nbytes / (ms * 1e-3) / 1e9, peaks["hbm"], "GB/s", "hbm"
    return {"ms": ms, "bound": bound, "achieved": v, "unit": unit, "frac": v / peak}


# ---- whole models ------------------------------------------------------------------------------------------------------
def rizurax_config(width, layers, attention_every=None):
    """``attention_every`` n: every n-th layer is attention (default: the third of four)."""
    H = width // 128
    G = max(2, H // 4)
    rot = {"dims": 32, "base": 500000.0, "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}
    mlp = {"kind": "dense", "ff": 4 * width}
    delta = {"type": "delta", "mlp": mlp, "mixer": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": H, "kv_heads": G, "dim": 64, "vdim": 128, "diff": 0.4, "scale": 0.125, "rot": rot}}
    return {"architecture": "Rizurax", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, 
            "layers": [att if (i % 4 == 2 if attention_every is None else i % attention_every == 0) else delta for i in range(layers)],
            "embedding": {"bigram": {"buckets": 4093, "mul_prev": 101, "mul_cur": 7}}}


def rizurax_weights(cfg, seed, device):
    """Random weights in the design's names, drawn on the device."""
    g = torch.Generator(device=device).manual_seed(seed)
    D, w = cfg["width"], {}

    def put(name, *shape, std=None, mean=0.0):
        w[name] = (torch.randn(*shape, device=device, generator=g) * (shape[-1] ** -0.5 if std is None else std) + mean).bfloat16()
    put("embed", cfg["vocab"], D, std=1.0)
    put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, D, std=0.5)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        H, G, d, vd, ff = m["heads"], m["kv_heads"], m["dim"], m["vdim"], e["mlp"]["ff"]
        put(p + "norm1", D, std=0.1), put(p + "norm2", D, std=0.1)
        if e["type"] == "delta":
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * vd)):
                put(p + "mix." + n, rows, D), put(p + f"mix.{n}.conv", rows, m["conv"], std=0.5)
            put(p + "mix.a", H, D), put(p + "mix.b", H, D), put(p + "mix.g", H * vd, D)
            put(p + "mix.A_log", H, std=0.5, mean=-1.0), put(p + "mix.dt_bias", H, std=0.5, mean=-2.0), put(p + "mix.norm", vd, std=0.1, mean=1.0)
        else:
            put(p + "mix.q", H * 2 * d, D), put(p + "mix.k", G * 2 * d, D), put(p + "mix.v", G * vd, D)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + "mix." + n, d, std=0.2)
        put(p + "mix.o", D, H * vd)
        put(p + "mlp.gate", ff, D), put(p + "mlp.up", ff, D), put(p + "mlp.down", D, ff)
    put("final.norm", D, std=0.1), put("head", cfg["vocab"], D)
    return w


def rizurax_leg(width, layers, prompts, decodes, device, attention_every=None):
    cfg = rizurax_config(width, layers, attention_every)
    return model_leg(cfg, rizurax_weights(cfg, 5, device), prompts, decodes, device)


def model_leg(cfg, weights, prompts, decodes, device):
    """Prompt and captured decode steps of a configured model through the engine's step builder."""
    from atma_b200.engine import CacheManager, ModelRunner, Sequence, _CapturedStep
    from atma_b200.registry import model_class
    n_par = sum(t.numel() for t in weights.values())
    model = model_class(cfg).from_config(cfg, weights, torch.bfloat16, device)
    weights.clear()
    out = {"parameters": n_par, "prefill": {}, "decode": {}}
    g = torch.Generator().manual_seed(6)

    def runner(n_seqs, per_seq):
        pages = -(-per_seq // BS)
        cache = CacheManager(n_seqs * pages, BS, n_seqs, pages)
        state = model.new_state(n_seqs, n_seqs * pages, BS, pages * BS)
        return cache, ModelRunner(model, cache, state), state

    for n, T in prompts:
        cache, run, state = runner(n, T)
        seqs = [Sequence(i, torch.randint(0, VOCAB, (T,), generator=g).tolist()) for i in range(n)]
        for s in seqs:
            cache.admit(s), cache.extend(s, T)
        batch = run.build([(s, T) for s in seqs], [T * (i + 1) - 1 for i in range(n)])
        ms = dev_ms(lambda: model.forward(batch, state), 3, 2)
        out["prefill"][f"{n}x{T}"] = {"ms": ms, "tok_s": n * T / (ms * 1e-3)}
        del cache, run, state, batch
    for n, ctx in decodes:
        cache, run, state = runner(n, ctx)
        seqs = [Sequence(i, [0] * ctx) for i in range(n)]
        for s in seqs:
            cache.admit(s), cache.extend(s, ctx)
            s.done = ctx - 1
        batch = run.build([(s, 1) for s in seqs], range(n), pad_decode_to=n)
        step = _CapturedStep(model, state, batch)
        step.run(batch)
        ms = dev_ms(step.graph.replay, 20, 3)
        out["decode"][f"{n}x{ctx}"] = {"ms_per_step": ms, "tok_s": n / (ms * 1e-3)}
        del cache, run, state, batch, step
    del model
    torch.cuda.empty_cache()
    return out


def atma_leg(width, layers, prompts, decodes, device):
    from atma_b200.layer import PackedMaps
    from atma_b200.model import AtmaModel, CapturedDecode, random_state_dict
    kw = dict(layers=layers, hidden=width, head_dim=128, num_kv_heads=max(2, width // 128 // 4))
    sd = random_state_dict(vocab=VOCAB, seed=5, device=device, **kw)
    n_par = sum(t.numel() for t in sd.values())
    model = AtmaModel(sd, device=device, **kw)
    del sd
    out = {"parameters": n_par, "prefill": {}, "decode": {}}
    g = torch.Generator().manual_seed(6)
    for n, T in prompts:
        state = model.new_state(n, n * T // BS, BS)
        ids = torch.randint(0, VOCAB, (n * T,), generator=g).to(device)
        maps, sm = PackedMaps([T] * n, list(range(n)), device), torch.arange(n * T, device=device)
        last = torch.arange(1, n + 1, device=device) * T - 1
        ms = dev_ms(lambda: model.logits(model.prefill(ids, [T] * n, list(range(n)), state, sm, maps=maps)[last]), 3, 2)
        out["prefill"][f"{n}x{T}"] = {"ms": ms, "tok_s": n * T / (ms * 1e-3)}
        del state
    for n, ctx in decodes:
        pages = ctx // BS
        state = model.new_state(n, n * pages, BS)
        cap = CapturedDecode(model, state, batch=n, max_blocks=pages)
        bt = torch.randperm(n * pages, generator=g).int().view(n, pages).to(device)
        cap.block_tables.copy_(bt)
        cap.context_lens.fill_(ctx)
        cap.slot_mapping.copy_((bt[:, -1].long() * BS + BS - 1).int())
        cap.capture()
        ms = dev_ms(cap.replay, 20, 3)
        out["decode"][f"{n}x{ctx}"] = {"ms_per_step": ms, "tok_s": n / (ms * 1e-3)}
        del state, cap
    del model
    torch.cuda.empty_cache()
    return out


# ---- kernels -----------------------------------------------------------------------------------------------------------
def batch_of(device, n, T, decode=False):
    """A step of n sequences in a shuffled cache: their whole prompts, or the last of T tokens; and the cache's pages."""
    from types import SimpleNamespace
    from atma_b200.engine import CacheManager, ModelRunner, Sequence
    host = SimpleNamespace(chunked_prefill=True, graph_decode=False, device=device)        # what ModelRunner asks of a model
    pages = -(-T // BS)
    cache = CacheManager(n * pages, BS, n, pages)
    perm = torch.randperm(n * pages, generator=torch.Generator().manual_seed(2)).tolist()
    cache.free_pages.clear(), cache.free_pages.extend(perm)
    seqs = [Sequence(i, [0] * T) for i in range(n)]
    for s in seqs:
        cache.admit(s), cache.extend(s, T)
        s.done = T - 1 if decode else 0
    return ModelRunner(host, cache, None, False).build([(s, 1 if decode else T) for s in seqs], []), n * pages


def kernel_legs(peaks, device, only=None):
    """{name: {"rizurax": roofline, "like": [kernel, roofline]}}"""
    from functools import partial
    import atma_b200 as ab
    from atma_b200 import decoder_ops as ops
    from atma_b200.layer import PackedMaps
    H, G, DK = 8, 2, 128
    g = torch.Generator(device=device).manual_seed(1)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g, dtype=torch.bfloat16)
    out, step_of = {}, partial(batch_of, device)

    def want(name):
        return only is None or only == name

    P = {n: torch.full((H,), v, device=device) for n, v in (("null_base", 2.0), ("null_slope_raw", 0.5), ("len_gain_raw", -1.0), ("mag_beta_raw", -1.5))}
    P["v_null"] = torch.zeros(H, DK, device=device)
    if want("softmax_prefill"):
        T = 32768
        b, nb = step_of(1, T)
        q, kc, vc, o = rnd(T, H, 2, 64), rnd(nb, BS, G, 128), rnd(nb, BS, G, 128), rnd(T, H * 128)
        ms = dev_ms(lambda: ops.softmax_prefill(q, kc, vc, b.prefill, o, scale=0.125, lam=0.3, out_scale=0.6, eps=1e-6), 5)
        fl = 2.0 * (2 * 64 + 2 * 128) * H * T * (T + 1) / 2
        pq, pk = rnd(1, T, H, DK), rnd(2, 1, T, G, DK)
        n = torch.arange(1, T + 1, dtype=torch.float32, device=device)
        lk = dev_ms(lambda: ab.polar_attention_fwd(pq.transpose(1, 2), pk[0].transpose(1, 2), pk[1].transpose(1, 2), n, **P), 5)
        out["softmax_prefill"] = {"shape": f"T={T}, {H}/{G} heads, two maps of 64, vdim 128", "rizurax": roof(ms, peaks, flops=fl),
                                  "like": ["polar_prefill", roof(lk, peaks, flops=4.0 * DK * H * T * (T + 1) / 2)]}
    if want("softmax_decode"):
        B, ctx = 64, 16384
        b, nb = step_of(B, ctx, True)
        q, kc, vc, o = rnd(B, H, 2, 64), rnd(nb, BS, G, 128), rnd(nb, BS, G, 128), rnd(B, H * 128)
        ms = dev_ms(lambda: ops.softmax_decode(q, kc, vc, b.decode, o, scale=0.125, lam=0.3, out_scale=0.6, eps=1e-6))
        nbytes = B * ctx * G * 256 * 2.0
        cl, pq = torch.full((B,), ctx, dtype=torch.int32, device=device), rnd(B, H, DK)
        lk = dev_ms(lambda: ab.polar_attention_decode(pq, kc, vc, b.decode.block_tables, cl, **P))
        out["softmax_decode"] = {"shape": f"{B} x {ctx}, {H}/{G} heads", "rizurax": roof(ms, peaks, nbytes), "like": ["polar_decode", roof(lk, peaks, nbytes)]}
        del kc, vc
    if want("delta_scan"):
        B, T = 8, 16384
        b, _ = step_of(B, T)
        n = B * T
        ch = 2 * H * DK + H * DK
        z = rnd(n, ch + H * DK + 2 * H)
        w = ops.DeltaWeights(*(rnd(H * DK, 4) * 0.4 for _ in range(3)), torch.full((H,), -1.0, device=device), torch.full((H,), -1.0, device=device),
                             rnd(DK), heads=H, kv_heads=H, dim=DK, vdim=DK, unit_eps=1e-6, q_scale=DK ** -0.5)
        conv, state = torch.zeros(B, 4, ch, device=device, dtype=torch.bfloat16), torch.zeros(B, H, DK, DK, device=device)
        parts = ops.DeltaParts(z, w, conv, state, b.prefill)
        ms_p = dev_ms(parts.prepare)
        ms_s = dev_ms(parts.scan, 5)
        o = rnd(n, H * DK)
        ms_n = dev_ms(lambda: ops.head_norm_silu_gate(parts.o, w.norm, z[:, ch:ch + H * DK], o, 1e-6))
        q, k, v = F.normalize(rnd(B, T, H, DK), dim=-1), F.normalize(rnd(B, T, H, DK), dim=-1), rnd(B, T, H, DK)
        beta, gl = torch.sigmoid(rnd(B, T, H).float()), -F.softplus(rnd(B, T, H).float())
        lk = dev_ms(lambda: ab.chunk_gated_delta_rule(q=q, k=k, v=v, g=gl, beta=beta, scale=1.0, output_final_state=True,
                                                      use_qk_l2norm_in_kernel=True), 5)
        nb_s = 4.0 * n * H * DK * 2 + 2.0 * n * H * 4 + B * H * DK * DK * 4.0
        out["delta_scan"] = {"shape": f"{B} x {T}, {H} heads of 128", "rizurax": roof(ms_s, peaks, nb_s), "like": ["chunk_gated_delta_rule", roof(lk, peaks, nb_s)]}
        nb_p = 2.0 * n * ch * 2
        tot = 65536
        maps = PackedMaps([tot // 8] * 8, list(range(8)), device)
        qg, kk, vv = rnd(tot, H, 2 * DK), rnd(tot, G, DK), rnd(tot, G, DK)
        ws = [rnd(C, 4) for C in (H * DK, G * DK, G * DK)]
        st = [torch.zeros(8, C, 3, dtype=torch.bfloat16, device=device) for C in (H * DK, G * DK, G * DK)]
        kc, vc, sm = rnd(tot, G, DK), rnd(tot, G, DK), torch.arange(tot, device=device)
        lp = dev_ms(lambda: ab.qkv_prep_prefill(qg, kk, vv, *ws, *st, maps.token_seq_starts, maps.token_seq_ends, maps.token_seq_slots, kc, vc, sm))
        like_p = roof(lp, peaks, tot * (2 * H + 5 * G) * DK * 2.0)
        out["delta_prepare"] = {"shape": f"{n} rows of {ch} channels, 4 taps", "rizurax": roof(ms_p, peaks, nb_p), "like": ["qkv_prep_prefill", like_p]}
        gt = rnd(tot, H * DK)
        ln = dev_ms(lambda: ab.rms_sigmoid_gate(v.view(-1, H, DK)[:tot], gt))
        out["head_norm_silu_gate"] = {"shape": f"{n} x {H} x 128", "rizurax": roof(ms_n, peaks, 3.0 * n * H * DK * 2),
                                      "like": ["rms_sigmoid_gate", roof(ln, peaks, 3.0 * tot * H * DK * 2)]}
        del z, parts, q, k, v
        b2, nb = step_of(8, tot // 8)
        z = rnd(tot, (H + G) * 128 + G * 128)
        kc2, vc2 = rnd(nb, BS, G, 128), rnd(nb, BS, G, 128)
        table = torch.zeros(tot, 16, 2, device=device)
        ms_r = dev_ms(lambda: ops.rotary_store(z, b2.positions, b2.slot_mapping, table, kc2, vc2, heads=H, kv_heads=G, maps=2, dim=64, vdim=128, rot_dims=32))
        out["rotary_store"] = {"shape": f"{tot} rows, {H}/{G} heads", "rizurax": roof(ms_r, peaks, 2.0 * z.numel() * 2), "like": ["qkv_prep_prefill", like_p]}
    if want("delta_step"):
        for B in (64, 256):
            ch = 3 * H * DK
            z = rnd(B, ch + H * DK + 2 * H)
            w = ops.DeltaWeights(*(rnd(H * DK, 4) * 0.4 for _ in range(3)), torch.full((H,), -1.0, device=device), torch.full((H,), -1.0, device=device),
                                 rnd(DK), heads=H, kv_heads=H, dim=DK, vdim=DK, unit_eps=1e-6, q_scale=DK ** -0.5)
            b, _ = step_of(B, 64, True)
            conv = torch.zeros(B, 4, ch, device=device, dtype=torch.bfloat16)
            states = [torch.zeros(B, H, DK, DK, device=device) for _ in range(4)]                # the tables rotate: 4 x B x 0.5 MB
            o = rnd(B, H * DK)
            it = iter(range(10 ** 9))
            ms = dev_ms(lambda: ops.delta_step(z, w, conv, states[next(it) % 4], b.decode, o, 1e-6), 20)
            nbytes = 2.0 * B * H * DK * DK * 4
            q, k, v, lgt, gate = rnd(B, H, DK), rnd(B, H, DK), rnd(B, H, DK), rnd(B, 2 * H), rnd(B, H * DK)
            sl = torch.arange(B, device=device)
            lk = dev_ms(lambda: ab.gated_delta_decode_step_fused(q, k, v, states[next(it) % 4], sl, gate_logits=(lgt[:, :H], lgt[:, H:]), gate=gate), 20)
            out[f"delta_step_{B}"] = {"shape": f"{B} sequences, {H} heads", "rizurax": roof(ms, peaks, nbytes), "like": ["gated_delta_decode_step_fused", roof(lk, peaks, nbytes)]}
    if want("rows"):
        n, D = 65536, 2048
        x, y, w1, w2 = torch.randn(n, D, device=device), rnd(n, D), rnd(D), rnd(D)
        ms = dev_ms(lambda: ops.residual_norms(x, y, (w1, w2), 1e-6))
        xb = rnd(n, D)
        lk = dev_ms(lambda: ab.add_rms_norm(xb, y, w1))
        out["residual_norms"] = {"shape": f"{n} x {D}, fp32 residual, two norms", "rizurax": roof(ms, peaks, n * D * (8.0 + 2 + 4)),
                                 "like": ["add_rms_norm", roof(lk, peaks, n * D * 8.0)]}
        gu, o = rnd(n // 2, 4 * D), rnd(n // 2, 2 * D)
        ms = dev_ms(lambda: ops.gelu_gate(gu[:, :2 * D], gu[:, 2 * D:], o))
        lk = dev_ms(lambda: ab.squared_relu_gate(gu[:, :2 * D], gu[:, 2 * D:]))
        out["gelu_gate"] = {"shape": f"{n // 2} x {2 * D}", "rizurax": roof(ms, peaks, 3.0 * o.numel() * 2), "like": ["squared_relu_gate", roof(lk, peaks, 3.0 * o.numel() * 2)]}
        ids, prev = torch.randint(0, VOCAB, (n,), device=device, dtype=torch.int32), torch.randint(0, VOCAB, (n,), device=device, dtype=torch.int32)
        e, bg = rnd(VOCAB, D), rnd(4094, D)
        ms = dev_ms(lambda: ops.embed_bigram(ids, prev, e, bg, 101, 7))
        lk = dev_ms(lambda: e[ids.long()])
        out["embed_bigram"] = {"shape": f"{n} x {D}", "rizurax": roof(ms, peaks, n * D * 8.0), "like": ["embedding gather (torch)", roof(lk, peaks, n * D * 4.0)]}
        del x, y, gu
    if want("linear"):
        D, Fh, copies = 2048, 8192, 6
        wf = [rnd(2 * Fh, D) * D ** -0.5 for _ in range(copies)]
        xs, o = rnd(8, D), rnd(8, Fh)
        it = iter(range(10 ** 9))
        ms = dev_ms(lambda: ops.gelu_gated_linear(xs, wf[next(it) % copies], o), 24)
        lk = dev_ms(lambda: ab.decode_linear(xs, wf[next(it) % copies], None, gated=True), 24)
        out["gelu_gated_linear"] = {"shape": f"8 x {D} -> {Fh}", "rizurax": roof(ms, peaks, 2.0 * 2 * Fh * D), "like": ["decode_linear gated", roof(lk, peaks, 2.0 * 2 * Fh * D)]}
    for e in out.values():                                     # how much farther from its roofline than the like kernel
        e["distance_ratio"] = e["like"][1]["frac"] / e["rizurax"]["frac"]
    return out


def run(peaks, device, only=None):
    res = {"kernels": kernel_legs(peaks, device, only)}
    if only is None:
        prompts, decodes, layers = [(4, 4096), (1, 32768)], [(8, 8192), (64, 8192)], 8
        for width in (1024, 2048, 4096):
            res[f"width_{width}"] = {"layers": layers, "rizurax": rizurax_leg(width, layers, prompts, decodes, device),
                                     "atma": atma_leg(width, layers, prompts, decodes, device)}
    from atma_b200 import decoder_ops
    res["device_status"] = decoder_ops.device_status()
    return res
