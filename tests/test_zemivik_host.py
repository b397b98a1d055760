"""CPU: the Zemivik oracle's pieces, configuration and checkpoint handling, and the pages that a model with windows gives
back, with a stand-in model that checks what it reads."""

import pytest
import torch

from atma_b200 import checkpoint, registry
from atma_b200.engine import CacheManager, Engine, OutOfCache, SamplingParams, Sequence
from oracle import zemivik as Z
from tests.rizurax_util import prompt
from tests.zemivik_util import CONFIGS, config, layer


# ---- the oracle's pieces -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size,keep", [(1, 0), (3, 0), (3, 2), (0, 2), (50, 0), (2, 50)])
def test_which_keys_are_seen(size, keep):
    see = Z.visible(20, size, keep)
    assert torch.equal(see, Z.visible_fast(20, size, keep))
    for i in range(20):
        assert see[i].nonzero().flatten().tolist() == sorted(set(range(max(i - size + 1, 0), i + 1)) | set(range(min(keep, i + 1))))


def test_sink_softmax():
    s = torch.tensor([[1.0, -2.0, 700.0], [0.0, 0.0, 0.0], [5.0, 1.0, -800.0]], dtype=torch.float64)
    see = torch.tensor([[1, 1, 0], [1, 1, 1], [0, 0, 1]], dtype=torch.bool)
    p = Z.sink_softmax(s, see)
    e = torch.exp(s[0, :2])
    assert torch.allclose(p[0, :2], e / (1 + e.sum())) and p[0, 2] == 0
    assert torch.allclose(p[1], torch.full((3,), 0.25, dtype=torch.float64)) and p[2].sum() == 0
    assert torch.allclose(Z.sink_softmax(s + 900, torch.ones_like(see)).sum(-1), torch.ones(3, dtype=torch.float64))


def test_attention_of_grouped_heads_without_sink_is_softmax():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(7, h, c, generator=g, dtype=torch.float64) for h, c in ((6, 5), (2, 5), (2, 3)))
    see = Z.visible(7, 100, 0)
    got = Z.attend(q, k, v, 0.7, see, torch.tensor(float("-inf"), dtype=torch.float64))
    for h in range(6):
        w = torch.softmax((q[:, h] @ k[:, h // 3].T * 0.7).masked_fill(~see, float("-inf")), -1)
        assert torch.allclose(got[:, h], w @ v[:, h // 3])


def test_values_are_mixed_with_the_first_layer_that_mixes():
    cfg = CONFIGS["mixed"]
    w = {n: t.double() for n, t in Z.random_weights(cfg, 2).items()}
    h = torch.randn(5, cfg["width"], dtype=torch.float64)
    m = cfg["layers"][1]["mixer"]
    _, first = Z.attention_mixer(h, w, "l1.mix.", m, 1e-6, None)
    assert torch.equal(first, h @ w["l1.mix.v"].T)
    _, none = Z.attention_mixer(h, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-6, None)
    assert none is None
    lam = w["l3.mix.vmix"]
    same = dict(w, **{"l3.mix.v": w["l3.mix.v"] * 0})
    a, kept = Z.attention_mixer(h, w, "l3.mix.", cfg["layers"][3]["mixer"], 1e-6, first)
    b, _ = Z.attention_mixer(h, dict(same, **{"l3.mix.v": (1 - lam) * w["l3.mix.v"] + lam * w["l1.mix.v"]}), "l3.mix.", dict(cfg["layers"][3]["mixer"], v_mix=False),
                             1e-6, None)
    assert kept is first and torch.allclose(a, b)


# ---- configuration ---------------------------------------------------------------------------------------------------------
def test_model_from_a_folder(tmp_path):
    cfg = CONFIGS["mixed"]
    checkpoint.write_model(tmp_path, cfg, {n: t.bfloat16() for n, t in Z.random_weights(cfg, 3).items()})
    m = registry.load_model(tmp_path, torch.float32, "cpu")
    assert type(m).__name__ == "ZemivikModel" and "Zemivik" in registry.architectures()
    lam = [float(checkpoint.read_safetensors(tmp_path / "model.safetensors")[f"l{i}.mix.vmix"]) for i in range(5)]
    assert [x.first_values for x in m.run_mixers] == [None, "leave", lam[2], lam[3], None]
    assert m.cache_reach == (64, 40) and m.max_positions == cfg["max_positions"]
    assert [(x.window, x.keep_first, x.scale) for x in m.run_mixers] == \
        [(e["mixer"]["mask"]["size"], e["mixer"]["mask"]["keep_first"], e["mixer"]["scale"]) for e in cfg["layers"]]


def test_model_refuses_wrong_shapes_and_unknown_parts():
    from atma_b200.zemivik import ZemivikModel
    cfg = config([layer(2, 1, 8, 8), layer(2, 2, 8, 4)], width=16)
    w = Z.random_weights(cfg, 5)
    ZemivikModel(cfg, w, torch.float32, "cpu")
    for name in ("pos", "l0.mix.q.norm", "l1.mlp.up.b"):
        with pytest.raises(ValueError, match=name):
            ZemivikModel(cfg, {**w, name: torch.zeros(3)}, torch.float32, "cpu")
    with pytest.raises(KeyError):
        ZemivikModel(cfg, {n: t for n, t in w.items() if n != "l0.mix.g"}, torch.float32, "cpu")
    with pytest.raises(ValueError, match="mixer"):
        ZemivikModel({**cfg, "layers": [{**cfg["layers"][0], "type": "other"}]}, w, torch.float32, "cpu")
    with pytest.raises(ValueError, match="feed-forward"):
        ZemivikModel({**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "other", "ff": 40}}]}, w, torch.float32, "cpu")
    bad = config([layer(2, 1, 8, 8), layer(2, 2, 8, 8)], width=16)
    with pytest.raises(ValueError, match="differ in width"):
        ZemivikModel(bad, Z.random_weights(bad, 5), torch.float32, "cpu")
    with pytest.raises(ValueError):
        ZemivikModel(cfg, w, torch.float16, "cpu")


def test_joint_reach():
    from types import SimpleNamespace as N
    from atma_b200.configured import joint_reach
    assert joint_reach([N(reach=(5, 9)), N(reach=(7, 1))]) == (7, 9)
    assert joint_reach([N(reach=(5, 9)), N(reach=None)]) is None and joint_reach([]) is None


# ---- pages behind the window -------------------------------------------------------------------------------------------------
def test_pages_out_of_sight_are_given_back():
    c = CacheManager(num_blocks=12, block_size=4, max_seqs=2, max_blocks_per_seq=50, reach=(10, 5), max_portion=6)
    assert c.live_pages(8) == 2 and c.live_pages(200) == 2 + 4 + 1
    a = Sequence("a", [])
    assert c.admit(a, 200) and c.promised == 7
    for done in range(0, 198, 6):
        n = min(6, 200 - done)
        c.extend(a, done + n)
        a.done = done + n
        live = {i for i, p in enumerate(a.pages) if p >= 0}
        needed = {j // 4 for j in range(done + n) if j < 5 or j > done - 10}
        assert needed <= live and len(live) + a.reserved <= 7 and c.promised == a.reserved
        assert sorted(c.free_pages) == sorted(set(range(12)) - {p for p in a.pages if p >= 0}) and len(c.free_pages) >= c.promised
    c.release(a)
    assert sorted(c.free_pages) == list(range(12)) and c.promised == 0 and a.reserved == 0


class Windowed:
    """A model on the CPU whose next token is a function of the tokens a position still sees; every page it reads must hold
    the right token."""
    chunked_prefill = mixed_batches = True
    graph_decode = False
    device = torch.device("cpu")
    vocab = 89
    max_positions = 600

    def __init__(self, window, first):
        self.cache_reach = (window, first)

    def new_state(self, max_seqs, num_blocks, block_size, max_positions=None):
        self.bs = block_size
        return {"cache": torch.full((num_blocks * block_size, 2), -5)}

    def next_token(self, history):
        w, f = self.cache_reach
        seen = [t for j, t in enumerate(history) if j < f or len(history) - 1 - j < w]
        total = 0
        for t in seen:
            total = (total * 3 + t) % 1009
        return (total + len(history)) % self.vocab

    def forward(self, b, state):
        w, f = self.cache_reach
        logits = torch.zeros(b.ids.numel(), self.vocab)
        for r in range(b.ids.numel()):
            state["cache"][int(b.slot_mapping[r])] = torch.tensor([int(b.ids[r]), int(b.positions[r])])
        for g in (b.decode, b.prefill):
            for s in range(0 if g is None else g.n_seqs):
                lo, hi, start = int(g.cu_rows[s]), int(g.cu_rows[s + 1]), int(g.start_pos[s])
                table = g.block_tables[s].tolist()
                for i in range(lo, hi):
                    pos, total = start + i - lo, 0
                    for j in range(pos + 1):
                        if j < f or pos - j < w:
                            assert table[j // self.bs] >= 0
                            tok, at = state["cache"][table[j // self.bs] * self.bs + j % self.bs].tolist()
                            assert at == j
                            total = (total * 3 + tok) % 1009
                    logits[g.rows.start + i, (total + pos + 1) % self.vocab] = 1.0
        return None if b.logit_rows is None else logits[b.logit_rows]


@pytest.mark.parametrize("window,first", [(9, 3), (1, 0), (16, 8), (5, 30)])
@pytest.mark.parametrize("budget", [7, 40])
def test_generation_in_a_cache_smaller_than_the_sequences(window, first, budget):
    m = Windowed(window, first)
    prompts = [prompt(n, m.vocab, 30 + n) for n in (1, 150, 40, 3, 90, 12)]
    e = Engine(m, max_tokens=120, max_model_len=400, max_seqs=3, block_size=4, max_step_tokens=budget)
    out = e.generate(prompts, SamplingParams(max_new_tokens=60))
    for p, o in zip(prompts, out):
        h = list(p)
        for _ in range(60):
            h.append(m.next_token(h))
        assert o == h[len(p):]
    assert sorted(e.cache.free_pages) == list(range(e.cache.num_blocks)) and e.cache.promised == 0 and e.cache.num_blocks * 4 < 210


def test_the_longest_sequence_is_the_position_table():
    e = Engine(Windowed(9, 3), max_tokens=5000, max_seqs=2, block_size=256)
    assert e.max_len == 600
    e.feed([("a", [1] * 600, [])])
    with pytest.raises(ValueError, match="longest"):
        e.feed([("a", [1], [])])
    with pytest.raises(ValueError, match="longest"):
        e.feed([("b", [1] * 601, [])])
    assert "b" not in e.fed
    with pytest.raises(ValueError):
        e.add_request([1] * 590, SamplingParams(max_new_tokens=11))


def test_a_cache_without_room_says_so():
    e = Engine(Windowed(500, 0), max_tokens=40, max_model_len=400, max_seqs=1, block_size=4, max_step_tokens=8)
    with pytest.raises(OutOfCache):
        e.generate([[1] * 100], SamplingParams(max_new_tokens=2))
