"""GPU: every mechanism of the Zemivik decoder against the plain oracle, then the whole model through the engine - prompts,
portions, decoding, unequal batches, reused pages and slots, pages that are given back, generation."""

import pytest
import torch

from oracle import zemivik as Z
from tests.conftest import max_abs, max_rel
from tests.gpu_util import rand
from tests.rizurax_util import group, logit_error, prompt
from tests.zemivik_util import CONFIGS, attention_case, config, layer

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
EVERY = 10 ** 9


def ops():
    from atma_b200 import decoder_ops
    return decoder_ops


@pytest.fixture(autouse=True, scope="module")
def no_expired_waits():
    yield
    assert ops().device_status() == 0


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ---- row operations ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [1, 45, 80, 1028, 4096, 9000])
def test_embedding_with_positions_and_norm(dtype, D):
    V, P = 501, 97
    e, p, w = rand((V, D), 1, dtype), rand((P, D), 2, dtype), rand((D,), 3, dtype)
    ids, pos = [5, 500, 0, 5, 3], [0, 96, 1, 40, 95]
    for table in (p, None):
        s = e[ids].double() * 2.5 + (0 if table is None else p[pos].double())
        x, h = ops().embed_position_norm(_i32(ids), _i32(pos), e.cuda(), None if table is None else table.cuda(), w.cuda(), 1e-4, 2.5, 0.5)
        want = Z.rms(s, 1e-4) * (0.5 + w.double())
        assert x.dtype == F32 and h.dtype == dtype and max_rel(x, want) < 1e-6 and max_rel(h, want) < (1e-6 if dtype == F32 else 5e-3)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [1, 45, 80, 192, 1028, 4096, 9000])
@pytest.mark.parametrize("bias", [True, False])
def test_residual_with_the_norm_behind_the_sublayer(dtype, D, bias):
    x, y = rand((5, D), 1, scale=3.0), rand((5, D), 2, dtype)
    y[3] *= 1e-3                                                         # eps decides
    b, w, wn = (rand((D,), s, dtype, 0.5) for s in (3, 4, 5))
    if bias:
        b[:] = (b.float() * 1e-3).to(dtype)
    t = y.double() + (b.double() if bias else 0)
    want = x.double() + Z.rms(t, 1e-5) * (1 + w.double())
    tol = 1e-6 if dtype == F32 else 5e-3
    for nw in (None, wn):
        for in_place in (True, False):
            g = x.cuda()
            h = ops().residual_post_norm(g, y.cuda(), w.cuda(), 1e-5, b.cuda() if bias else None, None if nw is None else nw.cuda(), 1.0, in_place)
            assert max_rel(g, want) < 1e-6 if in_place else torch.equal(g.cpu(), x)
            assert h.dtype == dtype and max_rel(h, want if nw is None else Z.rms(want, 1e-5) * (1 + nw.double())) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 13), (7, 40), (3, 1024), (70, 2056)])
def test_bias_and_squared_relu(dtype, rows, width):
    z, b = rand((rows, width + 16), 1, dtype), rand((width,), 2, dtype)
    want = torch.relu(z[:, 8:8 + width].double() + b.double()) ** 2
    out = torch.zeros(rows, width + 8, dtype=dtype, device="cuda")
    ops().bias_squared_relu(z.cuda()[:, 8:8 + width], b.cuda(), out[:, :width])
    assert max_rel(out[:, :width], want) < (1e-6 if dtype == F32 else 6e-3) and out[:, width:].abs().max() == 0
    g = z.cuda()
    v = g[:, 8:8 + width]
    ops().bias_squared_relu(v, None, v)
    assert max_rel(v, torch.relu(z[:, 8:8 + width].double()) ** 2) < (1e-6 if dtype == F32 else 6e-3)
    assert torch.equal(g[:, :8].cpu(), z[:, :8]) and torch.equal(g[:, 8 + width:].cpu(), z[:, 8 + width:])


@pytest.mark.parametrize("rows,n,k", [(1, 48, 96), (16, 128, 256), (9, 80, 64), (40, 128, 256), (3, 42, 45)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_squared_relu_linear(dtype, rows, n, k):
    x, w, b = rand((rows, k), 1, dtype), rand((n, k), 2, dtype, k ** -0.5), rand((n,), 3, dtype)
    want = torch.relu(x.double() @ w.double().T + b.double()) ** 2
    assert max_rel(ops().squared_relu_linear(x.cuda(), w.cuda(), b.cuda()), want) < (3e-6 if dtype == F32 else 1.2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,dim,vdim,extra", [(4, 2, 64, 128, 512), (3, 3, 6, 10, 30), (2, 1, 9, 7, 1), (32, 8, 128, 128, 0), (1, 1, 1, 1, 0), (16, 4, 72, 24, 8)])
def test_projection_norms_value_mixing_and_cache_write(dtype, H, G, dim, vdim, extra):
    n, slots, nq, nk, nv = 6, 40, H * dim, G * dim, G * vdim
    z, first = rand((n, nq + nk + nv + extra), 1, dtype), rand((n, nv + 8), 2, dtype)
    z[1] *= 1e-3                                                        # eps decides
    z[2, :nq] *= 1e2                                                    # q and k have norms of their own
    wq, wk = rand((nq,), 3, dtype), rand((nk,), 4, dtype)
    sm = [3, 39, -1, 0, 7, 21]
    want_q, want_k = Z.rms(z[:, :nq].double(), 1e-5) * wq.double(), Z.rms(z[:, nq:nq + nk].double(), 1e-5) * wk.double()
    v = z[:, nq + nk:nq + nk + nv].double()
    tol = 2e-6 if dtype == F32 else 6e-3
    fc = first.cuda()[:, :nv]
    for norm, mix in ((True, None), (True, fc), (False, fc), (False, None)):
        kc, vc = torch.zeros(slots, 1, G, dim, dtype=dtype, device="cuda"), torch.zeros(slots, 1, G, vdim, dtype=dtype, device="cuda")
        kw = dict(q_weight=wq.cuda(), k_weight=wk.cuda(), eps=1e-5) if norm else {}
        q = ops().norm_store(z.cuda(), torch.tensor(sm, device="cuda"), kc, vc, nq, v_first=mix, lam=0.3, **kw)
        wv = v if mix is None else Z.mix_values(v, first[:, :nv].double(), 0.3)
        stored = torch.zeros(slots, dtype=torch.bool)
        for r in range(n):
            a, b = (want_q[r], want_k[r]) if norm else (z[r, :nq], z[r, nq:nq + nk])
            assert max_rel(q[r], a) < tol
            if sm[r] >= 0:
                stored[sm[r]] = True
                assert max_rel(kc[sm[r]].reshape(-1), b) < tol and max_rel(vc[sm[r]].reshape(-1), wv[r]) < tol
        assert kc[~stored].abs().max() == 0 and vc[~stored].abs().max() == 0


# ---- softmax attention: windows, kept first keys, sink, gate -------------------------------------------------------------------
SHAPES = [(4, 2, 64, 128), (3, 3, 64, 64), (4, 1, 128, 128), (5, 5, 128, 64), (6, 2, 12, 20), (2, 1, 33, 65), (16, 2, 64, 128), (2, 1, 40, 256), (1, 1, 64, 64)]
MASKS = [(40, 3), (1, 0), (128, 130), (129, 1), (300, 0), (EVERY, 0), (17, 300)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("lengths,starts,block_size", [((130, 3, 257), (0, 500, 127), 128), ((2, 40, 129), (255, 0, 600), 256), ((45, 17), (3, 90), 16)])
def test_windowed_prompt_rows(dtype, shape, window, keep, lengths, starts, block_size):
    H, G, dim, vdim = shape
    q, kc, vc, z, tables, want, kw = attention_case(shape, dtype, lengths, starts, block_size, window, keep, 0.0, 3)
    gr = group(list(lengths), list(starts), list(range(len(lengths))), tables)
    out = torch.zeros(q.shape[0], H * vdim + 8, dtype=dtype, device="cuda")
    ops().softmax_prefill(q, kc, vc, gr, out[:, :H * vdim], gate=z, **kw)
    assert max_rel(out[:, :H * vdim], want) < (2e-5 if dtype == F32 else 1.5e-2) and out[:, H * vdim:].abs().max() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("contexts,block_size,splits", [((1, 64, 700, 129, 41, 40), 64, None), ((256, 257, 3), 128, 5), ((33, 1500), 16, 3), ((1023, 511), 256, 1)])
def test_windowed_single_rows(dtype, shape, window, keep, contexts, block_size, splits):
    H, G, dim, vdim = shape
    n = len(contexts)
    for seed in (5, 6, 7, 8):                                            # which key each row looks hard at
        q, kc, vc, z, tables, want, kw = attention_case(shape, dtype, [1] * n, [c - 1 for c in contexts], block_size, window, keep, 0.0, seed)
        gr = group([1] * n + [1], [c - 1 for c in contexts] + [-1], list(range(n)) + [-1], tables + [[0] * len(tables[0])], decode=True)
        q, z = (torch.cat([t, torch.full_like(t[:1], float("nan"))]) for t in (q, z))      # a padded sequence: zeros, nothing read
        out = torch.full((n + 1, H * vdim), 9.0, dtype=dtype, device="cuda")
        ops().softmax_decode(q, kc, vc, gr, out, n_splits=splits, gate=z, **kw)
        assert max_rel(out[:n], want) < (2e-5 if dtype == F32 else 1.5e-2)
        assert out[n].abs().max() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(4, 2, 64, 128), (6, 2, 12, 20)])
@pytest.mark.parametrize("sink", [None, -3.0, 0.0, 4.5, 40.0])
def test_sink(dtype, shape, sink):
    """Sinks of other scores than zero, and none; scores far below and above them."""
    H, G, dim, vdim = shape
    for seed, far in ((1, -60.0), (2, 0.0), (3, 60.0)):
        n, g = 70, torch.Generator().manual_seed(seed)
        q, k, v = (torch.randn(n, h, c, generator=g).to(dtype).float() for h, c in ((H, dim), (G, dim), (G, vdim)))
        q[..., 0], k[..., 0] = 1.0, far / dim ** -0.5                    # every score is moved by ``far``
        q, k, v = (t.to(dtype) for t in (q, k, v))
        s = float("-inf") if sink is None else sink
        want = torch.cat([torch.stack([Z.sink_softmax(q[i:i + 1, h].double() @ k[:, h // (H // G)].double().T * dim ** -0.5,
                                                      torch.arange(n)[None] <= i, torch.tensor(s, dtype=torch.float64))[0]
                                       @ v[:, h // (H // G)].double() for h in range(H)]).reshape(1, -1) for i in range(n)])
        kc, vc = torch.zeros(1, 128, G, dim, dtype=dtype, device="cuda"), torch.zeros(1, 128, G, vdim, dtype=dtype, device="cuda")
        kc[0, :n], vc[0, :n] = k.cuda(), v.cuda()
        out, one = torch.empty(n, H * vdim, dtype=dtype, device="cuda"), torch.empty(2, H * vdim, dtype=dtype, device="cuda")
        ops().softmax_prefill(q.cuda()[:, :, None].contiguous(), kc, vc, group([n], [0], [0], [[0]]), out, scale=dim ** -0.5, sink=sink)
        tol = 2e-5 if dtype == F32 else 1.5e-2
        assert max_rel(out, want) < tol
        for splits in (1, 2):
            ops().softmax_decode(q.cuda()[[5, 69], :, None].contiguous(), kc, vc, group([1, 1], [5, 69], [0, 1], [[0], [0]], decode=True), one,
                                 scale=dim ** -0.5, sink=sink, n_splits=splits)
            assert max_rel(one, want[[5, 69]]) < tol


def test_which_kernel_serves_which_shape():
    import ctypes
    from atma_b200 import _lib
    lib = _lib.load_decoder()
    for dim, vdim, dt, want in [(64, 128, 1, 1), (128, 64, 1, 1), (64, 128, 0, 0), (12, 20, 1, 0)]:
        a = _lib.SoftmaxArgs(H=4, G=2, maps=1, dim=dim, vdim=vdim, dtype=dt, block_size=256, num_blocks=4, max_blocks=4)
        assert lib.atma_softmax_prefill_path(ctypes.byref(a)) == want and lib.atma_softmax_decode_path(ctypes.byref(a)) == want


# ---- the whole model through the engine ----------------------------------------------------------------------------------------
_models, _oracle = {}, {}


def model(name, dtype):
    if (name, dtype) not in _models:
        from atma_b200.zemivik import ZemivikModel
        cfg = CONFIGS[name]
        w = Z.random_weights(cfg, 7)
        _models[name, dtype] = (cfg, w, ZemivikModel(cfg, w, dtype))
    return _models[name, dtype]


def oracle(name, tokens):
    key = (name, tuple(tokens))
    if key not in _oracle:
        _oracle[key] = Z.forward(CONFIGS[name], Z.random_weights(CONFIGS[name], 7), tokens)
    return _oracle[key]


def engine(m, **kw):
    from atma_b200.engine import Engine
    return Engine(m, **{"max_tokens": 1200, "max_seqs": 6, "block_size": 128, **kw})


TOL = {F32: 5e-5, BF16: 0.08}


def close(got, want, dtype):
    e = logit_error(got, want)
    assert e.max() < TOL[dtype] and e.median() < TOL[dtype] / 3, (float(e.median()), float(e.max()), int(e.argmax()))


def run_cuts(e, name, tokens, cuts):
    got, at = [], 0
    for n in cuts:
        got.append(e.feed([(name, tokens[at:at + n], list(range(n)))]))
        at += n
    assert at == len(tokens)
    e.release(name)
    return torch.cat(got)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(name, dtype):
    cfg, w, m = model(name, dtype)
    t = prompt(300, cfg["vocab"], 1)
    want, runs = oracle(name, t)
    e = engine(m, graphs=False)
    rec, plain = [], m.forward
    m.forward = lambda b, s: plain(b, s, rec)
    try:
        got = run_cuts(e, "a", t, [300])
    finally:
        del m.forward
    assert len(rec) == len(runs)
    for i, (a, b) in enumerate(zip(rec, runs)):
        assert max_rel(a, b) < (2e-5 if dtype == F32 else 0.04), i
    close(got, want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [(1,) * 60, (200, 1, 1, 1, 97), (2,) * 20 + (110, 150), (63, 2, 64, 21, 3, 147), (127, 1, 2, 20), (5, 1, 9, 1, 1, 60, 73, 150),
                                  (3,) * 100])
def test_portions_and_single_tokens(name, dtype, cuts):
    cfg, w, m = model(name, dtype)
    t = prompt(300, cfg["vocab"], 1)
    close(run_cuts(engine(m), "a", t[:sum(cuts)], cuts), oracle(name, t)[0][:sum(cuts)], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("block_size", [16, 128])
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_unequal_batches_with_reused_pages_and_slots(name, dtype, block_size):
    cfg, w, m = model(name, dtype)
    ts = {c: prompt(n, cfg["vocab"], 40 + n) for c, n in zip("abcdefg", (1, 70, 150, 33, 5, 129, 140))}
    e = engine(m, max_seqs=4, max_tokens=500, block_size=block_size, graphs=False)
    at, got = {c: 0 for c in ts}, {c: [] for c in ts}

    def step(**portions):
        entries = [(c, ts[c][at[c]:at[c] + n], list(range(n))) for c, n in portions.items()]
        out, r = e.feed(entries), 0
        for c, n in portions.items():
            got[c].append(out[r:r + n])
            r, at[c] = r + n, at[c] + n
            if at[c] == len(ts[c]):
                e.release(c)
    step(a=1, b=64, c=3, d=16)
    step(b=2, c=61, d=1, e=4)
    step(b=1, c=1, d=1, e=1)
    step(b=3, c=64, d=15, f=128)                       # d and e have left their pages and slots
    step(c=21, f=1, g=2)
    step(g=130)
    step(g=1)
    step(g=7)
    assert all(at[c] == len(ts[c]) for c in ts)
    for c in ts:
        close(torch.cat(got[c]), oracle(name, ts[c])[0], dtype)
    assert len(e.cache.free_slots) == 4 and len(e.cache.free_pages) == e.cache.num_blocks


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name,block_size", [("mixed", 16), ("odd", 8), ("wide", 128)])
def test_long_decoding(dtype, graphs, name, block_size):
    cfg, w, m = model(name, dtype)
    t = prompt(420, cfg["vocab"], 3)
    close(run_cuts(engine(m, block_size=block_size, graphs=graphs), "a", t, [100] + [1] * 320), oracle(name, t)[0], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("graphs", [False, True])
def test_long_sequences_hold_few_pages(dtype, graphs):
    """Two long sequences in turns in a cache that could not hold either whole: the pages behind the window are given
    back, taken by the other, and the first tokens stay."""
    cfg = config([layer(2, 2, 64, 64, size=50, keep=3, ff=48), layer(4, 2, 16, 32, size=30, keep=20, v_mix=False)], width=64)
    w = Z.random_weights(cfg, 11)
    from atma_b200.zemivik import ZemivikModel
    e = engine(ZemivikModel(cfg, w, dtype), max_tokens=256, max_model_len=700, max_seqs=2, block_size=16, graphs=graphs)
    ts = [prompt(690, cfg["vocab"], s) for s in (1, 2)]
    at, got = [0, 0], [[], []]
    for step in range(1200):
        i = step % 2
        n = min(1 if step % 7 else 40, 690 - at[i])
        if n:
            got[i].append(e.feed([(i, ts[i][at[i]:at[i] + n], list(range(n)))]))
            at[i] += n
    assert at == [690, 690] and e.cache.num_blocks < 2 * 690 // 16
    for i in (0, 1):
        assert sum(p >= 0 for p in e.fed[i].pages) <= 2 + (50 + 40) // 16 + 2
        close(torch.cat(got[i]), Z.forward(cfg, w, ts[i])[0], dtype)
        e.release(i)
    assert sorted(e.cache.free_pages) == list(range(e.cache.num_blocks))


def standing_out(size, keep, dim, vdim, n_keep_key):
    """One layer whose last tokens look hard at one token each: the weights read a marked channel pair of the embedding."""
    cfg = config([layer(2, 1, dim, vdim, size=size, keep=keep, scale=0.5, ff=None)], width=64, vocab=90, scale=1.0, max_positions=900)
    w = Z.random_weights(cfg, 9)
    w["pos"] *= 0.05
    for i in range(6):                                                   # token 80 + i asks for token 70 + i through channel i
        w["embed"][80 + i].zero_(), w["embed"][70 + i].zero_()
        w["embed"][70 + i, i], w["embed"][80 + i, 8 + i] = 2.0, 2.0
        w["embed"][70 + i, 20:], w["embed"][80 + i, 20:] = (0.2 * torch.randn(44, generator=torch.Generator().manual_seed(s + i)).bfloat16().float() for s in (1, 50))
    w["embed"][:70, :16] = 0
    wk, wq = torch.randn(dim, 64, generator=torch.Generator().manual_seed(3)) * 0.05, torch.randn(2 * dim, 64, generator=torch.Generator().manual_seed(4)) * 0.05
    for i in range(6):
        wk[i], wq[i], wq[dim + i] = 0, 0, 0
        wk[i, i] = wq[i, 8 + i] = wq[dim + i, 8 + i] = 3.0
    w["l0.mix.k"], w["l0.mix.q"] = wk.bfloat16().float(), wq.bfloat16().float()
    w["l0.mix.q.norm"].fill_(1.5), w["l0.mix.k.norm"].fill_(1.5)
    return cfg, w


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim,vdim", [(64, 64), (24, 20)])
@pytest.mark.parametrize("size,keep,block_size", [(130, 2, 128), (40, 5, 16), (256, 1, 256)])
def test_keys_at_the_edges_stand_out(dtype, dim, vdim, size, keep, block_size):
    """A token asks for one exactly inside the window, one exactly outside, the last kept one, the one after it, and ones at
    a page's border; changing a token that is seen changes the answer, changing one that is not seen does not."""
    from atma_b200.zemivik import ZemivikModel
    cfg, w = standing_out(size, keep, dim, vdim, keep)
    m = ZemivikModel(cfg, w, dtype)
    n = 700
    t = prompt(n, 60, 4)
    # (asked for, asking): positions
    page = 512
    pairs = [(page - 1, page + 20, True), (page, page + 22, True), (600 - size + 1, 600, True), (645 - size, 645, False), (keep - 1, 650, True), (keep, 660, False)]
    for i, (key, asker, _) in enumerate(pairs):
        t[key], t[asker] = 70 + i, 80 + i
    want = Z.forward(cfg, w, t)[0]
    for cuts in ((n,), (500,) + (1,) * 200, (531, 2, 66, 2, 38, 2, 8, 2, 9, 40)):
        close(run_cuts(engine(m, block_size=block_size), "a", t, cuts), want, dtype)
    for i, (key, asker, seen) in enumerate(pairs):
        t2 = list(t)
        t2[key] = 33
        other = Z.forward(cfg, w, t2)[0]
        moved = float(logit_error(other[asker:asker + 1], want[asker:asker + 1])[0])
        assert moved > 2 * TOL[BF16] if seen else moved < 1e-9, (i, moved)
        if seen:
            close(run_cuts(engine(m, block_size=block_size), "b", t2, (asker - 1, 1, 1, n - asker - 1)), other, dtype)


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation_follows_the_oracle(name):
    from atma_b200.engine import SamplingParams
    cfg, w, m = model(name, F32)
    prompts = [prompt(n, cfg["vocab"], 60 + n) for n in (1, 37, 130, 2, 64, 11)]
    e = engine(m, max_seqs=4, block_size=16, max_tokens=600, max_model_len=160, max_step_tokens=50)
    out = e.generate(prompts, SamplingParams(max_new_tokens=12))
    for p, o in zip(prompts, out):
        assert len(o) == 12
        logits = Z.forward(cfg, w, p + o[:-1])[0][len(p) - 1:]
        top = logits.topk(2, -1).values
        clear = (top[:, 0] - top[:, 1]) > 1e-3                            # ties aside
        assert (logits.argmax(-1)[clear] == torch.tensor(o)[clear]).all() and clear.float().mean() > 0.8
    assert e.generate(prompts, SamplingParams(max_new_tokens=12)) == out   # pages and slots in another order
    assert e.cache.promised == 0 and len(e.cache.free_pages) == e.cache.num_blocks


def test_the_longest_sequence():
    cfg, w, m = model("odd", F32)
    t = prompt(cfg["max_positions"], cfg["vocab"], 2)
    e = engine(m)
    close(run_cuts(e, "a", t, [400] + [1] * 21), oracle("odd", t)[0], F32)
    with pytest.raises(ValueError, match="longest"):
        e.feed([("b", t + [1], [])])
    with pytest.raises(ValueError, match="longest"):
        e.add_request(t)


def test_saved_folder_command_line_and_replay(tmp_path, capsys, monkeypatch):
    import io
    import json
    import numpy as np
    from atma_b200 import checkpoint, generate, replay
    from atma_b200.engine import SamplingParams
    cfg, w, m = model("mixed", BF16)
    checkpoint.write_model(tmp_path / "m", cfg, {n: t.bfloat16() for n, t in w.items()})
    p = prompt(20, cfg["vocab"], 5)
    want = engine(m).generate([p], SamplingParams(max_new_tokens=5))[0]
    generate.main(["--model", str(tmp_path / "m"), "--prompt", ",".join(map(str, p)), "--max-new-tokens", "5", "--max-tokens", "600"])
    assert capsys.readouterr().out.strip() == ",".join(map(str, want))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:15], "want": [14, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[15:17], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": p[17:], "want": [2]}], "end": ["a"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    (tmp_path / "o").mkdir()
    assert replay.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "64"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2"]
    got = np.concatenate([np.fromfile(tmp_path / "o" / f, "<f4") for f in ("0.f32", "2.f32")]).reshape(3, -1)
    close(torch.tensor(got), Z.forward(cfg, w, p)[0][[14, 2, 19]], F32)
