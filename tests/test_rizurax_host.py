"""CPU: the Rizurax oracle against itself, configuration and checkpoint handling, and the engine's host side (pages,
slots, scheduling, step building, sampling) with a stand-in model."""

import math

import pytest
import torch

from atma_b200 import checkpoint, registry
from atma_b200.engine import CacheManager, Engine, OutOfCache, SamplingParams, Scheduler, Sequence, sample
from oracle import rizurax as R
from tests.rizurax_util import CONFIGS, YARN, prompt


# ---- the oracle's pieces -----------------------------------------------------------------------------------------------
def test_delta_rule_continues_from_its_state_and_reads_after_the_write():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (4, 4, 3))
    dec, beta = torch.rand(9, 2, generator=g, dtype=torch.float64), torch.rand(9, 2, generator=g, dtype=torch.float64)
    o, S = R.delta_rule(q, k, v, dec, beta)
    oa, Sa = R.delta_rule(q[:5], k[:5], v[:5], dec[:5], beta[:5])
    ob, Sb = R.delta_rule(q[5:], k[5:], v[5:], dec[5:], beta[5:], Sa)
    assert torch.allclose(torch.cat([oa, ob]), o) and torch.allclose(Sb, S)
    assert torch.allclose(o[0], beta[0][:, None] * v[0] * (q[0] * k[0]).sum(-1, keepdim=True))


def test_bigram_rows_and_causal_conv():
    assert R.bigram_rows([4, 0, 9], 11, 5, 53) == [53, (4 * 11) % 53, 45]
    x = torch.randn(6, 3, dtype=torch.float64)
    taps = torch.randn(3, 4, dtype=torch.float64)
    y = R.causal_conv_silu(x, taps)
    z = (x[3] * taps[:, 3] + x[2] * taps[:, 2] + x[1] * taps[:, 1] + x[0] * taps[:, 0])
    assert torch.allclose(y[3], z * torch.sigmoid(z))
    x2 = x.clone()
    x2[4:] = 7
    assert torch.equal(R.causal_conv_silu(x2, taps)[:4], y[:4])


def test_rotation_depends_on_the_distance_only_and_leaves_the_rest():
    rot = {"dims": 6, "base": 50.0, "scaling": YARN}
    _, m = R.rotary_frequencies(rot)
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 10, generator=g, dtype=torch.float64), torch.randn(1, 1, 10, generator=g, dtype=torch.float64)
    dots = [(R.rotate(q, rot, p + 5)[..., :6] * R.rotate(k, rot, p)[..., :6]).sum() for p in (0, 3, 40)]
    assert max(dots) - min(dots) < 1e-10
    assert torch.equal(R.rotate(q, rot, 9)[..., 6:], q[..., 6:])
    assert math.isclose(float(R.rotate(q, rot, 9)[..., :6].norm()), m * float(q[..., :6].norm()), rel_tol=1e-12)


@pytest.mark.parametrize("rot", [{"dims": 16, "base": 900.0}, {"dims": 16, "base": 900.0, "scaling": YARN}, {"dims": 2, "base": 30.0, "scaling": YARN},
                                 {"dims": 64, "base": 5e5, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}}])
def test_product_frequencies_match_the_oracle(rot):
    from atma_b200.mixers import rotary_frequencies
    f, m = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    fo, mo = R.rotary_frequencies(rot)
    assert torch.allclose(f, fo, rtol=1e-13) and m == mo


def test_layer_order():
    from atma_b200.rizurax import layer_order
    for cfg in CONFIGS.values():
        assert layer_order(cfg) == R.layer_order(cfg)
    assert layer_order(CONFIGS["mixed"]) == [0, 1, 2, 1, 2, 1, 2, 3]
    with pytest.raises(ValueError):
        layer_order({"layers": [1, 2], "loop": {"start": 1, "stop": 3, "times": 2}})


# ---- folders -----------------------------------------------------------------------------------------------------------
def test_checkpoint_round_trip_and_registry(tmp_path):
    cfg = CONFIGS["odd"]
    w = {n: t.bfloat16() for n, t in R.random_weights(cfg, 3).items()}
    w["table"] = torch.arange(7, dtype=torch.int32)
    checkpoint.write_model(tmp_path, cfg, w)
    back = checkpoint.read_safetensors(tmp_path / "model.safetensors")
    assert back.keys() == w.keys() and all(torch.equal(back[n], w[n]) and back[n].dtype == w[n].dtype for n in w)
    assert registry.model_class(checkpoint.read_config(tmp_path)).__name__ == "RizuraxModel"
    assert registry.model_class({"architecture": "Atma"}).__name__ == "AtmaModel"
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.model_class({"architecture": "Nothing"})
    (tmp_path / "model.safetensors").write_bytes((10 ** 9).to_bytes(8, "little"))
    with pytest.raises(ValueError):
        checkpoint.read_safetensors(tmp_path / "model.safetensors")


def test_model_refuses_wrong_shapes_and_unknown_parts():
    from atma_b200.rizurax import RizuraxModel
    cfg = CONFIGS["bare"]
    w = R.random_weights(cfg, 5)
    RizuraxModel(cfg, w, torch.float32, "cpu")
    with pytest.raises(ValueError, match="l0.norm1"):
        RizuraxModel(cfg, {**w, "l0.norm1": torch.zeros(3)}, torch.float32, "cpu")
    with pytest.raises(KeyError):
        RizuraxModel(cfg, {n: t for n, t in w.items() if n != "head"}, torch.float32, "cpu")
    with pytest.raises(ValueError, match="mixer"):
        RizuraxModel({**cfg, "layers": [{**cfg["layers"][0], "type": "other"}]}, w, torch.float32, "cpu")
    with pytest.raises(ValueError):
        RizuraxModel(cfg, w, torch.float16, "cpu")


# ---- the engine's host side --------------------------------------------------------------------------------------------
def test_pages_and_slots_are_promised_taken_and_given_back():
    c = CacheManager(num_blocks=6, block_size=4, max_seqs=2, max_blocks_per_seq=4)
    a, b, d = (Sequence(n, []) for n in "abd")
    assert c.admit(a, 16) and c.admit(b, 8) and not c.admit(d, 1)          # no slot left
    c.extend(a, 5)
    assert len(a.pages) == 2 and c.promised == 4
    c.extend(b, 8)
    with pytest.raises(OutOfCache):
        c.extend(b, 9)                                                     # the rest is promised to a
    c.extend(a, 16)
    with pytest.raises(OutOfCache):
        c.extend(a, 17)
    c.release(a)
    assert c.admit(d, 16) and d.slot == 0 and c.promised == 4
    c.release(d), c.release(b)
    assert len(c.free_pages) == 6 and len(c.free_slots) == 2 and c.promised == 0
    with pytest.raises(ValueError):
        c.admit(a, 17)


class StandIn:
    """A model on the CPU whose next token is a function of the whole history: it keeps (token, previous token, position)
    in the pages and a running sum in the slots, checks every index it gets, and mixes both into its logits."""
    chunked_prefill = mixed_batches = True
    graph_decode = False
    device = torch.device("cpu")
    vocab = 89

    def new_state(self, max_seqs, num_blocks, block_size, max_positions=None):
        self.bs = block_size
        self.batches = []
        return {"cache": torch.full((num_blocks * block_size, 2), -5), "sum": torch.full((max_seqs,), 10 ** 6)}

    @classmethod
    def next_token(cls, history):
        total = 0
        for t in history:
            total = (total * 3 + t) % 1009
        return (total + 7 * history[0] + 5 * history[-1] + len(history)) % cls.vocab

    def forward(self, b, state):
        self.batches.append((0 if b.decode is None else b.decode.n_seqs, () if b.prefill is None else b.prefill.lengths))
        n = b.ids.numel()
        logits = torch.zeros(n, self.vocab)
        for g in (b.decode, b.prefill):
            if g is None:
                continue
            for s in range(g.n_seqs):
                lo, hi = int(g.cu_rows[s]), int(g.cu_rows[s + 1])
                slot, start = int(g.slots[s]), int(g.start_pos[s])
                for i in range(lo, hi):
                    r, pos = g.rows.start + i, start + i - lo
                    assert int(b.positions[r]) == pos and (g.row_seq is None or int(g.row_seq[i]) == s)
                    row = int(g.block_tables[s, pos // self.bs]) * self.bs + pos % self.bs
                    assert int(b.slot_mapping[r]) == row
                    state["cache"][row] = torch.tensor([int(b.ids[r]), pos])
                    hist = []
                    for p in range(pos + 1):
                        rec = state["cache"][int(g.block_tables[s, p // self.bs]) * self.bs + p % self.bs].tolist()
                        assert rec[1] == p
                        hist.append(rec[0])
                    assert int(b.prev[r]) == (hist[-2] if pos else -1)
                    before = 0 if pos == 0 else int(state["sum"][slot])
                    state["sum"][slot] = (before * 3 + hist[-1]) % 1009
                    tok = (int(state["sum"][slot]) + 7 * hist[0] + 5 * hist[-1] + len(hist)) % self.vocab
                    logits[r, tok] = 1.0
        if b.prefill is not None:
            tiles = sorted(zip(b.prefill.tile_seq.tolist(), b.prefill.tile_row.tolist()))
            assert tiles == [(s, r) for s, k in enumerate(b.prefill.lengths) for r in range(0, k, 128)]
        return None if b.logit_rows is None else logits[b.logit_rows]


class WholePrompts(StandIn):
    chunked_prefill = mixed_batches = False


def expected(prompt_tokens, n):
    h = list(prompt_tokens)
    for _ in range(n):
        h.append(StandIn.next_token(h))
    return h[len(prompt_tokens):]


@pytest.mark.parametrize("model", [StandIn, WholePrompts])
@pytest.mark.parametrize("budget", [3, 17, 1000])
def test_generation_is_the_same_however_it_is_scheduled(model, budget):
    prompts = [prompt(n, StandIn.vocab, 10 + n) for n in (1, 2, 5, 9, 30, 131, 1, 4, 17)]
    e = Engine(model(), max_tokens=640, max_seqs=4, block_size=4, max_model_len=160, max_step_tokens=budget)
    out = e.generate(prompts, SamplingParams(max_new_tokens=6))
    assert out == [expected(p, 6) for p in prompts]
    assert len(e.cache.free_pages) == e.cache.num_blocks and len(e.cache.free_slots) == 4 and e.cache.promised == 0
    batches = e.model.batches
    if model.chunked_prefill:
        assert all(d + sum(p) <= budget for d, p in batches)
        if budget == 17:
            assert any(d and p for d, p in batches)
    else:
        assert not any(d and p for d, p in batches)


def test_stop_ids_and_request_checks():
    p = prompt(4, StandIn.vocab, 1)
    want = expected(p, 8)
    e = Engine(StandIn(), max_tokens=64, max_seqs=2, block_size=4)
    assert e.generate([p], SamplingParams(max_new_tokens=8, stop_ids=(want[2],))) == [want[:want.index(want[2]) + 1]]
    for bad in ([], [StandIn.vocab], [-1]):
        with pytest.raises(ValueError):
            e.add_request(bad)
    with pytest.raises(ValueError):
        e.add_request(p, SamplingParams(max_new_tokens=100))


def test_fed_sequences_in_any_order_and_with_any_places():
    e = Engine(StandIn(), max_tokens=256, max_seqs=3, block_size=4)
    ta, tb, tc = prompt(20, 89, 1), prompt(30, 89, 2), prompt(9, 89, 3)
    got = e.feed([("a", ta[:7], [6, 0]), ("b", tb[:1], [0]), ("c", tc[:5], [])])
    assert got.argmax(-1).tolist() == [StandIn.next_token(ta[:7]), StandIn.next_token(ta[:1]), StandIn.next_token(tb[:1])]
    got = e.feed([("b", tb[1:4], [2]), ("a", ta[7:8], [0]), ("c", tc[5:9], [3])])
    assert got.argmax(-1).tolist() == [StandIn.next_token(h) for h in (tb[:4], ta[:8], tc)]
    assert e.feed([("a", ta[8:11], [])]) is None
    e.release("a"), e.release("c")
    got = e.feed([("d", tc, [8]), ("b", tb[4:5], [0])])                     # pages and slots used again
    assert got.argmax(-1).tolist() == [StandIn.next_token(tc), StandIn.next_token(tb[:5])]


def test_sampling():
    g = torch.Generator().manual_seed(0)
    logits = torch.randn(3, 50, generator=g)
    top = logits.argmax(-1).tolist()
    seqs = [Sequence(0, [], SamplingParams()), Sequence(1, [], SamplingParams(temperature=1.0, top_k=1, seed=1)),
            Sequence(2, [], SamplingParams(temperature=0.7, top_p=1e-6, seed=2))]
    assert sample(logits, seqs) == top
    s = Sequence(3, [], SamplingParams(temperature=1.5, top_k=5, seed=3))
    allowed = set(logits[0].topk(5).indices.tolist())
    drawn = [sample(logits[:1], [s])[0] for _ in range(60)]
    assert set(drawn) <= allowed and len(set(drawn)) > 1
    s2 = Sequence(3, [], SamplingParams(temperature=1.5, top_k=5, seed=3))
    assert [sample(logits[:1], [s2])[0] for _ in range(60)] == drawn


def test_scheduler_needs_room_for_one_sequence():
    c = CacheManager(1, 4, 2, 4)
    s = Scheduler(c, 100, True, True)
    s.add(Sequence(1, [1, 2, 3], SamplingParams(max_new_tokens=5), 3))
    with pytest.raises(OutOfCache):
        s.schedule()


def test_decoder_library_exports_its_header():
    import ctypes
    import os
    import re
    import subprocess
    import tempfile
    from atma_b200 import _lib
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    if not os.path.exists(_lib.DECODER_LIB_PATH):
        from atma_b200.build import build
        build("decoder")
    lib = _lib.load_decoder()
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(root, "include", "atma_decoder.h")).read(), flags=re.S)
    assert sorted(set(re.findall(r"\b(atma_[a-z0-9_]+)\s*\(", text))) == sorted(_lib.DECODER_SYMBOLS)
    with tempfile.TemporaryDirectory() as d:
        src = os.path.join(d, "s.c")
        open(src, "w").write('#include <stdio.h>\n#include "atma_decoder.h"\nint main(void) { printf("%zu %zu\\n", sizeof(atma_softmax_args), '
                             'sizeof(atma_delta_args)); return 0; }\n')
        subprocess.check_call(["gcc", "-I", os.path.join(root, "include"), src, "-o", os.path.join(d, "s")])
        a, b = map(int, subprocess.check_output([os.path.join(d, "s")]).split())
    assert ctypes.sizeof(_lib.SoftmaxArgs) == a and ctypes.sizeof(_lib.DeltaArgs) == b
    assert lib.atma_softmax_prefill(None, None) == _lib.ATMA_ERR_INVALID and b"null args" in lib.atma_last_error()
    args = _lib.DeltaArgs(dtype=2)
    assert lib.atma_delta_step(ctypes.byref(args), None, None, 0, 1e-6, None) == _lib.ATMA_ERR_INVALID


def test_command_line_arguments():
    from atma_b200.generate import ids, parse_args
    a = parse_args(["--model", "m", "--prompt", "1,2", "--prompt", "3", "--top-k", "4"])
    assert [ids(p) for p in a.prompt] == [[1, 2], [3]] and a.top_k == 4 and a.temperature == 0.0


def test_prefill_attention_register_hand_over_fits_the_launch_pool():
    """What setmaxnreg asks for must add up to no more than the CTA is launched with, or the last request never returns."""
    import os
    import re
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    log = os.path.join(root, "atma_b200", "build", "softmax_prefill_sm100.o.log")
    src = open(os.path.join(root, "atma_b200", "csrc", "softmax_prefill_sm100.cu")).read()
    if not os.path.exists(log):
        pytest.skip("no compiler report (the library was not built in this tree)")
    used = [int(x) for x in re.findall(r"Used (\d+) registers", open(log).read())]
    threads = int(re.search(r"kThreads = (\d+)", src).group(1))
    dec, inc = (int(re.search(rf"setmaxnreg\.{w}\.sync\.aligned\.u32 (\d+);", src).group(1)) for w in ("dec", "inc"))
    assert used and threads % 128 == 0 and all(dec * 128 + inc * (threads - 128) <= n * threads for n in used)
