"""GPU: every mechanism of the Rizurax decoder against the plain oracle, then the whole model through the engine -
prompts, portions, decoding, unequal batches, reused pages and slots, generation."""

import pytest
import torch

from oracle import rizurax as R
from tests.conftest import max_abs, max_rel
from tests.gpu_util import rand
from tests.rizurax_util import CONFIGS, YARN, attention, config, delta, group, logit_error, prompt

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16


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
def test_embedding_with_bigram(dtype):
    V, D, buckets, mp, mc = 70001, 52, 211, 104729, 99991                # products beyond 32 bits
    e, b = rand((V, D), 1, dtype), rand((buckets + 1, D), 2, dtype)
    ids = [5, 70000, 69999, 0, 5, 3]
    prev = [-1, 70000, 69999, 70000, 0, -1]
    want = torch.stack([e[i].float() + b[buckets if p < 0 else (p * mp + i * mc) % buckets].float() for i, p in zip(ids, prev)])
    got = ops().embed_bigram(_i32(ids), _i32(prev), e.cuda(), b.cuda(), mp, mc)
    assert torch.equal(got.cpu(), want)
    assert torch.equal(ops().embed_bigram(_i32(ids), _i32(prev), e.cuda()).cpu(), e[ids].float())


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [1, 45, 80, 192, 1028, 4096, 8192, 9001])
def test_residual_add_and_two_norms(dtype, D):
    x, y = rand((5, D), 1, scale=3.0), rand((5, D), 2, dtype)
    x[3] *= 1e-4                                                         # eps decides
    y[3] = 0
    w1, w2 = rand((D,), 3, dtype, 0.3), rand((D,), 4, dtype, 0.3)
    s = x + y.float()
    g = x.cuda()
    h1, h2 = ops().residual_norms(g, y.cuda(), (w1.cuda(), w2.cuda()), 1e-5)
    tol = 1e-6 if dtype == F32 else 5e-3
    assert torch.equal(g.cpu(), s)
    for h, w in ((h1, w1), (h2, w2)):
        assert h.dtype == dtype and max_rel(h, R.rms_norm_centered(s.double(), w.double(), 1e-5)) < tol
    g = x.cuda()
    h, none = ops().residual_norms(g, None, (w2.cuda(), None), 1e-5)
    assert none is None and torch.equal(g.cpu(), x) and max_rel(h, R.rms_norm_centered(x.double(), w2.double(), 1e-5)) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 13), (7, 40), (3, 1024)])
def test_gelu_gate(dtype, rows, width):
    gu = rand((rows, 2 * width), 1, dtype, 2.0)
    out = torch.zeros(rows, width + 8, dtype=dtype, device="cuda")
    g = gu.cuda()
    ops().gelu_gate(g[:, :width], g[:, width:], out[:, 8:])
    want = R.gelu_tanh(gu[:, :width].double()) * gu[:, width:].double()
    assert max_rel(out[:, 8:], want) < (1e-6 if dtype == F32 else 6e-3) and out[:, :8].abs().max() == 0


@pytest.mark.parametrize("rows,n,k", [(1, 64, 96), (16, 128, 256), (9, 96, 64), (40, 128, 256), (3, 42, 45)])
def test_gelu_gated_linear_and_linear(rows, n, k):
    x, w = rand((rows, k), 1, BF16), rand((n, k), 2, BF16, k ** -0.5)
    out = torch.empty(rows, n // 2, dtype=BF16, device="cuda")
    ops().gelu_gated_linear(x.cuda(), w.cuda(), out)
    z = x.double() @ w.double().T
    assert max_rel(out, R.gelu_tanh(z[:, :n // 2]) * z[:, n // 2:]) < 1e-2
    assert max_rel(ops().linear(x.cuda(), w.cuda()), z) < 6e-3
    assert max_rel(ops().linear_f32_out(x.cuda(), w.cuda()), z) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,V", [(3, 7), (1, 65), (4, 128), (2, 256), (5, 40)])
def test_head_norm_with_silu_gate(dtype, H, V):
    o, w, z = rand((6, H, V), 1, dtype, 0.02), rand((V,), 2, dtype), rand((6, H * V + 16), 3, dtype, 2.0)
    out = torch.zeros(6, H * V + 24, dtype=dtype, device="cuda")
    ops().head_norm_silu_gate(o.cuda(), w.cuda(), z.cuda()[:, 8:8 + H * V], out[:, 16:16 + H * V], 1e-4)
    od, gd = o.double(), z[:, 8:8 + H * V].double().view(6, H, V)
    want = od / torch.sqrt((od * od).mean(-1, keepdim=True) + 1e-4) * w.double() * gd * torch.sigmoid(gd)
    assert max_rel(out[:, 16:16 + H * V], want.reshape(6, -1)) < (2e-6 if dtype == F32 else 6e-3)
    assert out[:, :16].abs().max() == 0 and out[:, 16 + H * V:].abs().max() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,maps,dim,vdim,rot", [(4, 2, 2, 64, 128, 32), (3, 3, 2, 6, 10, 2), (2, 1, 1, 9, 7, 8), (2, 2, 2, 24, 8, 24), (1, 1, 2, 16, 16, 0)])
def test_rotary_and_cache_write(dtype, H, G, maps, dim, vdim, rot):
    from atma_b200.mixers import RotaryTable
    spec = {"dims": rot, "base": 700.0, "scaling": YARN}
    table = RotaryTable(rot, 700.0, YARN, torch.device("cuda")) if rot else None
    if rot:
        table.reserve(5000)
    n, slots = 6, 40
    z = rand((n, (H + G) * maps * dim + G * vdim), 1, dtype)
    pos, sm = [0, 1, 4999, 17, 300, 2], [3, 39, -1, 0, 7, 21]
    kc = torch.zeros(slots, 1, G, maps * dim, dtype=dtype, device="cuda")
    vc = torch.zeros(slots, 1, G, vdim, dtype=dtype, device="cuda")
    q = ops().rotary_store(z.cuda(), _i32(pos), torch.tensor(sm, device="cuda"), table.table if rot else None, kc, vc, heads=H, kv_heads=G, maps=maps,
                           dim=dim, vdim=vdim, rot_dims=rot)
    turn = (lambda t, p: R.rotate(t[None], spec, p)[0]) if rot else (lambda t, p: t)
    nq, nk = H * maps * dim, G * maps * dim
    tol = 3e-6 if dtype == F32 else 6e-3
    stored = torch.zeros(slots, dtype=torch.bool)
    for r in range(n):
        want_q = turn(z[r, :nq].double().view(H * maps, dim), pos[r])
        assert max_abs(q[r].view(H * maps, dim), want_q) < tol * 4
        if sm[r] >= 0:
            stored[sm[r]] = True
            assert max_abs(kc[sm[r], 0].view(G * maps, dim), turn(z[r, nq:nq + nk].double().view(G * maps, dim), pos[r])) < tol * 4
            assert torch.equal(vc[sm[r], 0].cpu().reshape(-1), z[r, nq + nk:])
    assert kc[~stored].abs().max() == 0 and vc[~stored].abs().max() == 0


# ---- softmax attention -----------------------------------------------------------------------------------------------------
ATT_SHAPES = [(4, 2, 2, 64, 128), (2, 2, 2, 64, 64), (4, 1, 2, 128, 128), (2, 2, 2, 128, 64), (4, 4, 1, 64, 128), (6, 2, 2, 12, 20), (3, 3, 2, 6, 10),
              (2, 1, 1, 33, 65), (8, 2, 2, 64, 128), (12, 1, 2, 64, 128), (2, 1, 2, 40, 256)]


def _attention_case(shape, dtype, lengths, starts, block_size, seed, spike=True):
    """Random q, k, v of a step's rows with their whole history in a shuffled paged cache, some (query, key) pairs scaled
    so that one far key takes most of the weight, and the oracle's output."""
    H, G, maps, dim, vdim = shape
    total, n_seqs = sum(lengths), len(lengths)
    g = torch.Generator().manual_seed(seed)
    ctx = [s + n for s, n in zip(starts, lengths)]
    pages = [-(-c // block_size) for c in ctx]
    perm = torch.randperm(sum(pages) + 3, generator=g).tolist()
    tables, at = [], 0
    for p in pages:
        tables.append(perm[at:at + p] + [0] * (max(pages) - p))
        at += p
    nb = sum(pages) + 3
    kc, vc = torch.randn(nb, block_size, G, maps * dim, generator=g) * 50, torch.randn(nb, block_size, G, vdim, generator=g) * 50   # stale rows
    q = torch.randn(total, H, maps, dim, generator=g)
    scale, lam, out_scale, eps = 1.2 * dim ** -0.5, 0.37, 0.6, 1e-5
    outs, r0 = [], 0
    head_of = [h // (H // G) for h in range(H)]
    for s in range(n_seqs):
        k, v = torch.randn(ctx[s], G, maps, dim, generator=g), torch.randn(ctx[s], G, vdim, generator=g)
        if spike:                                   # row i looks hard at one key: the first, one next to a page border, its own ...
            for i in range(0, lengths[s], 3):
                pos = starts[s] + i
                target = [0, min(block_size, pos), max(0, min(block_size - 1, pos)), pos, pos // 2][(i // 3) % 5]
                for m in range(maps):
                    q[r0 + i, :, m] = k[target, head_of, m] * (2.5 if m == 0 else 1.5)
        q, k, v = q.to(dtype).float(), k.to(dtype).float(), v.to(dtype).float()
        idx = torch.arange(ctx[s])
        rows = torch.tensor(tables[s])[idx // block_size] * block_size + idx % block_size
        kc.view(-1, G, maps * dim)[rows] = k.view(ctx[s], G, -1)
        vc.view(-1, G, vdim)[rows] = v
        a = []
        for m in range(maps):
            sc = torch.einsum("ihd,jhd->hij", q[r0:r0 + lengths[s], :, m].double(), k[:, head_of, m].double()) * scale
            vis = idx[None, :] <= (starts[s] + torch.arange(lengths[s]))[:, None]
            a.append(torch.einsum("hij,jhe->ihe", torch.softmax(sc.masked_fill(~vis, float("-inf")), -1), v[:, head_of].double()))
        outs.append(R.differential_combine(a[0], a[1], lam, 1 - out_scale, eps) if maps == 2 else a[0])
        r0 += lengths[s]
    want = torch.cat(outs).reshape(total, H * vdim)
    kw = dict(scale=scale, lam=lam, out_scale=out_scale, eps=eps)
    return q.to(dtype).cuda(), kc.to(dtype).cuda(), vc.to(dtype).cuda(), tables, want, kw


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", ATT_SHAPES)
@pytest.mark.parametrize("lengths,starts,block_size", [((130, 3, 257), (0, 500, 127), 128), ((2, 40, 129), (255, 0, 256), 256), ((45, 17), (3, 0), 16)])
def test_softmax_prompt_rows(dtype, shape, lengths, starts, block_size):
    H, G, maps, dim, vdim = shape
    q, kc, vc, tables, want, kw = _attention_case(shape, dtype, lengths, starts, block_size, 3)
    gr = group(list(lengths), list(starts), list(range(len(lengths))), tables)
    out = torch.zeros(q.shape[0], H * vdim + 8, dtype=dtype, device="cuda")
    ops().softmax_prefill(q, kc, vc, gr, out[:, :H * vdim], **kw)
    assert max_rel(out[:, :H * vdim], want) < (2e-5 if dtype == F32 else 2.5e-2) and out[:, H * vdim:].abs().max() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", ATT_SHAPES)
@pytest.mark.parametrize("contexts,block_size,splits", [((1, 64, 700, 129), 64, None), ((256, 257, 3), 128, 5), ((33, 1500), 16, 3), ((1023, 511), 256, 1)])
def test_softmax_single_rows(dtype, shape, contexts, block_size, splits):
    H, G, maps, dim, vdim = shape
    n = len(contexts)
    q, kc, vc, tables, want, kw = _attention_case(shape, dtype, [1] * n, [c - 1 for c in contexts], block_size, 5)
    gr = group([1] * n + [1], [c - 1 for c in contexts] + [-1], list(range(n)) + [-1], tables + [[0] * len(tables[0])], decode=True)
    q = torch.cat([q, torch.full_like(q[:1], float("nan"))])                       # a padded sequence: zeros, nothing read
    out = torch.full((n + 1, H * vdim), 9.0, dtype=dtype, device="cuda")
    ops().softmax_decode(q, kc, vc, gr, out, n_splits=splits, **kw)
    assert max_rel(out[:n], want) < (2e-5 if dtype == F32 else 2.5e-2)
    assert out[n].abs().max() == 0


def test_which_kernel_serves_which_shape():
    import ctypes
    from atma_b200 import _lib
    lib = _lib.load_decoder()
    for H, G, maps, dim, vdim, dt, bs, want in [(4, 2, 2, 64, 128, 1, 256, 1), (4, 2, 2, 64, 128, 0, 256, 0), (4, 2, 2, 12, 20, 1, 256, 0)]:
        a = _lib.SoftmaxArgs(H=H, G=G, maps=maps, dim=dim, vdim=vdim, dtype=dt, block_size=bs, num_blocks=4, max_blocks=4)
        assert lib.atma_softmax_prefill_path(ctypes.byref(a)) == want and lib.atma_softmax_decode_path(ctypes.byref(a)) == want
    for H, G, dim, vdim, dt, want in [(4, 2, 128, 128, 1, 1), (4, 2, 128, 128, 0, 0), (4, 2, 64, 32, 1, 0)]:
        a = _lib.DeltaArgs(H=H, G=G, dim=dim, vdim=vdim, dtype=dt)
        assert lib.atma_delta_scan_path(ctypes.byref(a)) == want


# ---- gated delta rule --------------------------------------------------------------------------------------------------------
DELTA_SHAPES = [(4, 2, 128, 128, 4), (2, 2, 128, 256, 3), (3, 1, 33, 65, 2), (1, 1, 5, 7, 1), (6, 3, 20, 12, 5), (2, 1, 256, 40, 4), (4, 4, 64, 32, 7)]


def _delta_case(shape, dtype, T, seed, decay_shift=0.0):
    H, G, K, V, taps = shape
    ch = 2 * G * K + H * V
    z = rand((T, ch + H * V + 2 * H), seed, dtype, 1.5)
    conv = [rand((n, taps), seed + i, dtype, 0.6) for i, n in enumerate((G * K, G * K, H * V), 1)]
    A_log, dt = rand((H,), seed + 5) * 0.7 - 1, rand((H,), seed + 6) - 2 + decay_shift
    norm = (1 + rand((V,), seed + 7, scale=0.3)).to(dtype)
    w = ops().DeltaWeights(*(c.cuda() for c in conv), A_log.cuda(), dt.cuda(), norm.cuda(), heads=H, kv_heads=G, dim=K, vdim=V, unit_eps=1e-6,
                           q_scale=K ** -0.5)
    zd = z.double()
    cut = [0, G * K, 2 * G * K, ch, ch + H * V, ch + H * V + H, ch + H * V + 2 * H]
    zq, zk, zv, zg, za, zb = (zd[:, a:b] for a, b in zip(cut, cut[1:]))
    head_of = [h // (H // G) for h in range(H)]
    rnd = (lambda t: t.to(dtype).double())
    q, k, v = (rnd(R.causal_conv_silu(x, c.double())) for x, c in zip((zq, zk, zv), conv))
    q, k = R.unit(q.view(T, G, K)) * K ** -0.5, R.unit(k.view(T, G, K))
    g = torch.exp(-torch.exp(A_log.double()) * R.softplus(za + dt.double()))
    o, S = R.delta_rule(q[:, head_of], k[:, head_of], v.view(T, H, V), g, torch.sigmoid(zb))
    eps = 1e-5
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * norm.double()
    gate = zg.reshape(T, H, V)
    return z.cuda(), w, (o * gate * torch.sigmoid(gate)).reshape(T, H * V), S, eps


def _delta_tables(w, slots, dtype):
    """Tables whose rows hold what earlier sequences left."""
    conv = torch.full((slots, w.taps, w.channels), 77.0, dtype=dtype, device="cuda")
    state = torch.full((slots, w.heads, w.dim, w.vdim), 33.0, device="cuda")
    return conv, state


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("cuts", [(150,), (64, 86), (2, 2, 3, 1, 63, 65, 2, 12), (1, 1, 1, 147), (127, 1, 1, 1, 20)])
def test_delta_in_portions(dtype, shape, cuts):
    """One sequence in portions (single tokens through the step kernel) against the whole recurrence."""
    T = sum(cuts)
    z, w, want, S, eps = _delta_case(shape, dtype, T, 11)
    conv, state = _delta_tables(w, 3, dtype)
    out, at = torch.empty(T, w.heads * w.vdim, dtype=dtype, device="cuda"), 0
    for n in cuts:
        gr = group([n], [at], [1], [[0]], decode=n == 1)
        (ops().delta_step if n == 1 else ops().delta_prefill)(z[at:at + n], w, conv, state, gr, out[at:at + n], eps)
        at += n
    assert max_rel(out, want) < (3e-5 if dtype == F32 else 2e-2)
    assert max_rel(state[1], S) < (1e-5 if dtype == F32 else 2e-4)                  # the state is fp32-accurate in both
    assert (state[0] == 33).all() and (state[2] == 33).all() and (conv[0] == 77).all() and (conv[2] == 77).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", DELTA_SHAPES[:3])
def test_delta_packed_sequences(dtype, shape):
    """Unequal sequences side by side, fresh and continued, prompts and single tokens, against each alone."""
    lens, first = [3, 65, 128, 200, 64], [0, 70, 0, 1, 64]
    cases = [_delta_case(shape, dtype, f + n + 1, 20 + i, decay_shift=i - 2.0) for i, (n, f) in enumerate(zip(lens, first))]
    w = cases[0][1]
    conv, state = _delta_tables(w, 8, dtype)
    slots = [6, 0, 3, 7, 2]
    for i, c in enumerate(cases):
        c[1].conv, c[1].norm = w.conv, w.norm                                       # one layer's weights for all of them
    def reference(i):
        T = first[i] + lens[i] + 1
        out = torch.empty(T, w.heads * w.vdim, dtype=F32, device="cuda")
        w32 = ops().DeltaWeights(*(t.float() for t in w.conv), w.A_log, w.dt_bias, w.norm.float(), heads=w.heads, kv_heads=w.kv_heads, dim=w.dim,
                                 vdim=w.vdim, unit_eps=1e-6, q_scale=w.q_scale)
        c, s = _delta_tables(w32, 1, F32)
        ops().delta_prefill(cases[i][0].float(), w32, c, s, group([T], [0], [0], [[0]]), out, cases[i][4])
        return out, s[0]
    outs = []
    for i in range(5):                                                              # the continued ones' first parts, alone
        if first[i]:
            ops().delta_prefill(cases[i][0][:first[i]], w, conv, state, group([first[i]], [0], [slots[i]], [[0]]),
                                torch.empty(first[i], w.heads * w.vdim, dtype=dtype, device="cuda"), cases[i][4])
    z = torch.cat([cases[i][0][first[i]:first[i] + lens[i]] for i in range(5)])
    out = torch.empty(z.shape[0], w.heads * w.vdim, dtype=dtype, device="cuda")
    ops().delta_prefill(z, w, conv, state, group(lens, first, slots, [[0]] * 5), out, cases[0][4])
    zs = torch.cat([cases[i][0][-1:] for i in range(5)] + [torch.full_like(z[:1], float("nan"))])
    last = torch.empty(6, w.heads * w.vdim, dtype=dtype, device="cuda")
    ops().delta_step(zs, w, conv, state, group([1] * 6, [f + n for f, n in zip(first, lens)] + [-1], slots + [-1], [[0]] * 6, decode=True), last,
                     cases[0][4])
    at = 0
    for i in range(5):
        ref, S = reference(i)
        got = torch.cat([out[at:at + lens[i]], last[i:i + 1]])
        assert max_rel(got, ref[first[i]:]) < (1e-4 if dtype == F32 else 2e-2), i
        assert max_rel(state[slots[i]], S) < (1e-4 if dtype == F32 else 1.5e-2), i   # bf16: the convolutions' outputs are rounded
        at += lens[i]
    assert last[5].abs().max() == 0


@pytest.mark.parametrize("shift", [-6.0, 3.0, 8.0])
def test_delta_with_slow_and_fast_decay(shift):
    """Decays near one over hundreds of tokens, and decays so strong that a chunk's factors underflow."""
    z, w, want, S, eps = _delta_case((2, 1, 128, 128, 4), BF16, 400, 31, decay_shift=shift)
    conv, state = _delta_tables(w, 1, BF16)
    out = torch.empty(400, 256, dtype=BF16, device="cuda")
    ops().delta_prefill(z, w, conv, state, group([400], [0], [0], [[0]]), out, eps)
    assert torch.isfinite(out).all() and max_rel(out, want) < 2e-2 and max_rel(state[0], S) < 5e-4


# ---- the whole model through the engine ----------------------------------------------------------------------------------------
_cache = {}


def model(name, dtype, **kw):
    key = (name, dtype)
    if key not in _cache:
        from atma_b200.rizurax import RizuraxModel
        cfg = CONFIGS[name]
        w = R.random_weights(cfg, 7)
        _cache[key] = (cfg, w, RizuraxModel(cfg, w, dtype))
    return _cache[key]


def engine(m, **kw):
    from atma_b200.engine import Engine
    kw = {"max_tokens": 1200, "max_seqs": 6, "block_size": 128, **kw}
    return Engine(m, **kw)


_oracle = {}


def oracle_logits(name, tokens):
    key = (name, tuple(tokens))
    if key not in _oracle:
        cfg = CONFIGS[name]
        _oracle[key] = R.forward(cfg, R.random_weights(cfg, 7), tokens)
    return _oracle[key]


TOL = {F32: 1.2e-4, BF16: 0.12}
MED = {F32: 2e-5, BF16: 0.04}


def close(got, want, dtype):
    e = logit_error(got, want)
    few = e.sort().values[: max(1, int(e.numel() * 0.9))].max()          # 16-bit rounding now and then meets a small norm
    assert e.median() < MED[dtype] and few < TOL[dtype] and e.max() < TOL[dtype] * (4 if dtype == BF16 else 1), (float(e.median()), float(e.max()), int(e.argmax()))


def run_cuts(e, name, tokens, cuts, release=True):
    got, at = [], 0
    for n in cuts:
        got.append(e.feed([(name, tokens[at:at + n], list(range(n)))]))
        at += n
    assert at == len(tokens)
    if release:
        e.release(name)
    return torch.cat(got)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(name, dtype):
    cfg, w, m = model(name, dtype)
    t = prompt(150, cfg["vocab"], 1)
    want, runs = oracle_logits(name, t)
    e = engine(m, graphs=False)
    rec, plain = [], m.forward
    m.forward = lambda b, s: plain(b, s, rec)
    try:
        got = run_cuts(e, "a", t, [150])
    finally:
        del m.forward
    assert len(rec) == len(runs)
    for i, (a, b) in enumerate(zip(rec, runs)):
        assert max_rel(a, b) < (1e-4 if dtype == F32 else 0.1), i
    close(got, want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [(1,) * 40, (100, 1, 1, 1, 47), (2,) * 20 + (110,), (63, 2, 64, 21), (127, 1, 2, 20), (5, 1, 9, 1, 1, 60, 73)])
def test_portions_and_single_tokens(name, dtype, cuts):
    cfg, w, m = model(name, dtype)
    t = prompt(150, cfg["vocab"], 1)[:sum(cuts)]
    want = oracle_logits(name, prompt(150, cfg["vocab"], 1))[0][:len(t)]
    close(run_cuts(engine(m), "a", t, cuts), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("block_size", [16, 128])
@pytest.mark.parametrize("name", ["mixed", "wide"])
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
        close(torch.cat(got[c]), oracle_logits(name, ts[c])[0], dtype)
    assert len(e.cache.free_slots) == 4 and len(e.cache.free_pages) == e.cache.num_blocks


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("graphs", [False, True])
def test_long_decoding(dtype, graphs):
    cfg, w, m = model("mixed", dtype)
    t = prompt(420, cfg["vocab"], 3)
    e = engine(m, block_size=16, graphs=graphs)
    close(run_cuts(e, "a", t, [100] + [1] * 320), oracle_logits("mixed", t)[0], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_far_keys_stand_out(dtype):
    """Weights that make single far keys stand out: the last tokens of a prompt ask for the last token of a page, the first
    one of the next and the very first token; the answer has to change when the far token does."""
    from atma_b200.rizurax import RizuraxModel
    cfg = config([attention(4, 2, 16, 24, rot=4, base=1e4, scaling=YARN, ff=48)], width=64, bigram=None)
    w = R.random_weights(cfg, 9)
    w["l0.norm1"].zero_()
    w["l0.mix.k"] = (w["l0.mix.k"] * 2).bfloat16().float()
    # a query is the key of the channels moved by one: token 93 + i asks for token 90 + i
    w["l0.mix.q"] = w["l0.mix.k"].view(2, 32, 64).repeat_interleave(2, 0).reshape(128, 64).roll(-1, 1)
    for i in range(3):
        w["embed"][93 + i] = w["embed"][90 + i].roll(-1)
    m = RizuraxModel(cfg, w, dtype)
    t = prompt(260, 40, 4)
    t[127], t[128], t[0] = 90, 91, 92                                    # last and first of a page, and the very first
    t += [93, 94, 95, 7]
    want = R.forward(cfg, w, t)[0]
    got = run_cuts(engine(m), "a", t, [259, 1, 1, 1, 1, 1])
    close(got, want, dtype)
    for far, asker in ((127, 260), (128, 261), (0, 262)):
        t2 = list(t)
        t2[far] = 33
        other = R.forward(cfg, w, t2)[0]
        assert logit_error(other[asker:asker + 1], want[asker:asker + 1])[0] > 2 * TOL[BF16]
        close(run_cuts(engine(m), "b", t2, [250, 14]), other, dtype)


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation_follows_the_oracle(name):
    from atma_b200.engine import SamplingParams
    cfg, w, m = model(name, F32)
    prompts = [prompt(n, cfg["vocab"], 60 + n) for n in (1, 37, 130, 2, 64, 11)]
    e = engine(m, max_seqs=4, block_size=16, max_tokens=600, max_model_len=160, max_step_tokens=50)
    out = e.generate(prompts, SamplingParams(max_new_tokens=12))
    for p, o in zip(prompts, out):
        assert len(o) == 12
        logits = R.forward(cfg, w, p + o[:-1])[0][len(p) - 1:]
        top = logits.topk(2, -1).values
        clear = (top[:, 0] - top[:, 1]) > 1e-3                            # ties aside
        assert (logits.argmax(-1)[clear] == torch.tensor(o)[clear]).all() and clear.float().mean() > 0.8
    assert e.generate(prompts, SamplingParams(max_new_tokens=12)) == out   # pages and slots in another order


def test_saved_folder_command_line_and_replay(tmp_path, capsys, monkeypatch):
    import io
    import json
    import numpy as np
    from atma_b200 import checkpoint, generate, replay
    cfg, w, m = model("mixed", BF16)
    checkpoint.write_model(tmp_path / "m", cfg, {n: t.bfloat16() for n, t in w.items()})
    p = prompt(20, cfg["vocab"], 5)
    from atma_b200.engine import SamplingParams
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
    close(torch.tensor(got), R.forward(cfg, w, p)[0][[14, 2, 19]], F32)
    assert not (tmp_path / "o" / "1.f32").exists()


def test_the_older_model_generates_through_the_same_engine():
    from atma_b200.engine import SamplingParams
    from atma_b200.model import AtmaModel, random_state_dict
    kw = dict(layers=4, hidden=256, head_dim=64, num_kv_heads=2)
    sd = random_state_dict(**kw, vocab=128, seed=1, device="cuda", dtype=F32)
    m = AtmaModel.from_config({"architecture": "Atma", **kw}, sd, F32)
    prompts = [prompt(n, 128, 70 + n) for n in (1, 40, 9)]
    e = engine(m, max_seqs=3, max_tokens=400, block_size=16)
    out = e.generate(prompts, SamplingParams(max_new_tokens=8))
    st = m.new_state(1, 8, 16)
    for p, o in zip(prompts, out):                                            # each alone, its whole text as one prompt
        ids = torch.tensor(p + o[:-1], device="cuda")
        h = m.prefill(ids, [len(ids)], [0], st, torch.arange(len(ids)))
        logits = m.logits(h)[len(p) - 1:].float()
        top = logits.topk(2, -1).values
        clear = ((top[:, 0] - top[:, 1]) > 1e-3).cpu()
        assert (logits.argmax(-1).cpu()[clear] == torch.tensor(o)[clear]).all() and clear.float().mean() > 0.7
