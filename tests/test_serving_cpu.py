"""The host side of serving without a GPU: scheduler, pages, sliding-window page release and generation over a model that keeps its
'cache' in NumPy and checks everything it is handed; configurations, rotary tables and the registry."""
import json

import numpy as np
import pytest
import torch

import latent_oracle as oracle
import videdra_oracle as videdra
from tlaloc_b200 import registry
from tlaloc_b200.engine import Engine
from tlaloc_b200.latent_decoder import LatentDecoderConfig
from tlaloc_b200.mixed_decoder import MixedDecoderConfig
from tlaloc_b200.paging import PADDING_PAGE, PagePool, Sequence, stage_ragged
from tlaloc_b200.rotary import Rotation, YarnScaling, pair_tables
from tlaloc_b200.scheduler import Request, Scheduler
from tlaloc_b200.step_model import StepModel


class HistoryModel(StepModel):
    """Writes each token id into its slot and answers with a function of the ids it finds through the block table (the last
    `window` of them): any wrong slot, table, length or page shows in the next token."""

    def __init__(self, rows=16, sequences=4, blocks=12, max_blocks=8, block_size=4, vocab=97, window=None):
        super().__init__(rows, sequences, blocks, max_blocks, block_size, vocab, "cpu")
        self.window = window
        self.slots = np.full((blocks * block_size,), -7, np.int64)
        self.steps = []

    @staticmethod
    def answer(history, vocab, window):
        h = history[-window:] if window else history
        return (sum((i + 1) * (t + 3) for i, t in enumerate(reversed(h))) + 5 * len(history)) % vocab

    def run(self, step, want):
        n = len(step.token_ids)
        assert n <= self.max_tokens and len(step.starts) - 1 <= self.max_sequences
        self.steps.append(np.diff(step.starts).tolist())
        assert len(set(step.slot_mapping.tolist())) == n and step.slot_mapping.min() >= self.block_size  # never the padding page
        self.slots[step.slot_mapping] = step.token_ids
        out = torch.full((len(want), self.vocab), -1.0)
        for k, r in enumerate(want):
            end = int(step.seq_lens[r])
            table = step.block_tables[step.row_tables[r]]
            lo = max(0, end - self.window) if self.window else 0
            seen = [int(self.slots[table[p // self.block_size] * self.block_size + p % self.block_size]) for p in range(lo, end)]
            out[k, self.answer([0] * lo + seen, self.vocab, self.window)] = 1.0
        return out

    def greedy(self, logits):
        return logits.argmax(-1)

    status = 0

    def device_status(self):
        return self.status


class RecurrentModel(HistoryModel):
    """Also keeps a number per state slot that every token changes, and answers with it: a wrong slot, a lost or a repeated token, or a slot
    that does not start over with its next sequence shows in every later token.  Attends to the first `keep` tokens and the window."""

    def __init__(self, states=4, keep=0, **kw):
        super().__init__(sequences=kw.pop("sequences", states), **kw)
        self.num_states, self.keep_first = states, keep
        self.numbers = np.full((states + 1,), 12345, np.int64)

    @staticmethod
    def answer_of(number, seen, vocab):
        return int((number + sum((i + 1) * (t + 3) for i, t in enumerate(seen))) % vocab)

    @staticmethod
    def visible(h, window, keep):
        lo = max(0, len(h) - window) if window else 0
        return h[:min(keep, lo)] + h[lo:]

    def run(self, step, want):
        n = len(step.token_ids)
        assert n <= self.max_tokens and len(step.starts) - 1 <= self.max_sequences
        self.slots[step.slot_mapping] = step.token_ids
        out, numbers = torch.full((len(want), self.vocab), -1.0), []
        for r in range(n):
            s = step.row_states[r]
            assert 1 <= s <= self.num_states
            before = 0 if step.positions[r] == 0 else self.numbers[s]
            self.numbers[s] = (before * 31 + int(step.token_ids[r]) + 1) % 1000003
            numbers.append(int(self.numbers[s]))
        for k, r in enumerate(want):
            end, table = int(step.seq_lens[r]), step.block_tables[step.row_tables[r]]
            lo = max(0, end - self.window) if self.window else 0
            places = [*range(min(self.keep_first, lo)), *range(lo, end)]
            seen = [int(self.slots[table[p // self.block_size] * self.block_size + p % self.block_size]) for p in places]
            out[k, self.answer_of(numbers[r], seen, self.vocab)] = 1.0
        return out


def expected_recurrent(prompt, n, vocab=97, window=None, keep=0):
    h, number = [], 0
    for t in prompt:
        h, number = h + [t], (number * 31 + t + 1) % 1000003
    for _ in range(n):
        t = RecurrentModel.answer_of(number, RecurrentModel.visible(h, window, keep), vocab)
        h, number = h + [t], (number * 31 + t + 1) % 1000003
    return h[len(prompt):]


def expected(prompt, n, vocab=97, window=None, stop=()):
    h = list(prompt)
    for _ in range(n):
        h.append(HistoryModel.answer(h, vocab, window))
        if h[-1] in stop:
            break
    return h[len(prompt):]


@pytest.mark.parametrize("window", [None, 1, 4, 5, 9])
@pytest.mark.parametrize("blocks", [9, 12, 40])
def test_generation_under_page_pressure(window, blocks):
    rng = np.random.default_rng(blocks)
    prompts = [rng.integers(0, 97, size=n).tolist() for n in (1, 3, 17, 4, 9, 20, 2)]
    model = HistoryModel(blocks=blocks, window=window)
    eng = Engine(model)
    assert eng.generate(prompts, 9) == [expected(p, 9, window=window) for p in prompts]
    assert eng.pool.free_count == eng.pool.capacity
    assert max(len(s) for s in model.steps) <= 4 and max(sum(s) for s in model.steps) <= 16


@pytest.mark.parametrize("window,keep", [(None, 0), (5, 0), (4, 1), (6, 9), (1, 4)])
@pytest.mark.parametrize("blocks,states", [(9, 4), (12, 2), (40, 1)])
def test_states_and_kept_tokens_under_pressure(window, keep, blocks, states):
    """Sequences that are sent back lose their state and build it up again; kept first tokens stay in their pages."""
    rng = np.random.default_rng(blocks)
    prompts = [rng.integers(0, 97, size=n).tolist() for n in (1, 3, 17, 4, 9, 20, 2)]
    model = RecurrentModel(states=states, keep=keep, blocks=blocks, window=window)
    eng = Engine(model)
    assert eng.generate(prompts, 9) == [expected_recurrent(p, 9, window=window, keep=keep) for p in prompts]
    assert eng.pool.free_count == eng.pool.capacity and eng.pool._free_states == set(range(1, states + 1))


def test_state_slots_that_run_out_and_come_back():
    eng = Engine(RecurrentModel(states=2, blocks=40))
    for k in "ab":
        eng.feed([(k, [1, 2, 3], [])])
    with pytest.raises(RuntimeError, match="state slot"):
        eng.feed([("c", [4], [])])
    eng.sequences.pop("c")
    eng.close("a")
    got, = eng.feed([("c", [7, 9], [1])])
    assert got.argmax(-1).tolist() == expected_recurrent([7, 9], 1)
    pool = PagePool(4, num_states=1)
    s = pool.take_state()
    assert s == 1 and not pool.has_state and pool.take_state() is None
    pool.give_state(s)
    for bad in (0, 1, 2):
        with pytest.raises(ValueError):
            pool.give_state(bad)


def test_pages_between_kept_tokens_and_window_go_back():
    pool, seq = PagePool(10), Sequence()
    assert seq.reserve(pool, 30, 4)  # eight pages
    pages = list(seq.pages)
    assert seq.drop_before(pool, 21, 4, keep_first=5) == 3  # positions 8 .. 19: two pages stay in front
    assert seq.pages == pages[:2] + [PADDING_PAGE] * 3 + pages[5:] and pool.free_count == 4
    assert seq.drop_before(pool, 21, 4, keep_first=5) == 0 and seq.drop_before(pool, 3, 4, keep_first=5) == 0
    seq.release(pool)
    assert pool.free_count == pool.capacity


def test_prompt_portions_and_decoding_share_a_step():
    model = HistoryModel(rows=8, blocks=40)
    Engine(model).generate([[1, 2], list(range(20))], 6)
    assert any(1 in s and max(s) > 1 for s in model.steps)


def test_stop_tokens_and_length_limits():
    want = expected([5, 6], 12)
    eng = Engine(HistoryModel(blocks=40))
    assert eng.generate([[5, 6]], 12, stop=[want[3]]) == [expected([5, 6], 12, stop=[want[3]])]
    assert eng.generate([[1]], 0) == [[]]
    for bad in ([], list(range(30))):
        with pytest.raises(ValueError):
            eng.generate([bad], 9)


def test_a_sequence_no_pool_can_hold_is_an_error():
    with pytest.raises(RuntimeError):
        Engine(HistoryModel(blocks=3)).generate([list(range(20))], 4)


@pytest.mark.parametrize("cut", [1, 2, 3, 16, 25])
def test_feeding_in_portions(cut):
    """Longer than a step takes; two sequences interleaved; a closed one's pages serve the next."""
    rng = np.random.default_rng(cut)
    eng = Engine(HistoryModel(blocks=16))
    texts = {k: rng.integers(0, 97, size=25).tolist() for k in "ab"}
    for lo in range(0, 25, cut):
        for k, t in texts.items():
            part = t[lo:lo + cut]
            got, = eng.feed([(k, part, list(range(len(part))))])
            assert got.argmax(-1).tolist() == [HistoryModel.answer(t[:lo + i + 1], 97, None) for i in range(len(part))]
    eng.close("a")
    got, = eng.feed([("c", texts["a"], [24])])
    assert got.argmax(-1).tolist() == [HistoryModel.answer(texts["a"], 97, None)]
    with pytest.raises(RuntimeError):
        eng.feed([("d", list(range(25)), [])])


def test_a_wait_that_ran_out_is_an_error():
    model = HistoryModel()
    model.status = 1
    with pytest.raises(RuntimeError):
        Engine(model).feed([("a", [1, 2], [1])])
    with pytest.raises(RuntimeError):
        Engine(model).generate([[1, 2]], 2)


def test_pages_behind_the_window_go_back_once():
    pool, seq = PagePool(10), Sequence()
    assert seq.reserve(pool, 20, 4)
    seq.length = 20
    assert seq.drop_before(pool, 3, 4) == 0
    assert seq.drop_before(pool, 11, 4) == 2 and seq.pages[:2] == [PADDING_PAGE] * 2
    assert seq.drop_before(pool, 12, 4) == 1 and seq.drop_before(pool, 12, 4) == 0
    assert pool.free_count == 9 - 2
    assert seq.reserve(pool, 4, 4) and len(seq.pages) == 6
    seq.release(pool)
    assert pool.free_count == 9


def test_the_oldest_request_keeps_its_pages():
    pool = PagePool(6)
    s = Scheduler(pool, block_size=4, max_tokens=64, max_sequences=4)
    a, b = Request("a", list(range(8)), 20), Request("b", list(range(8)), 20)
    s.add(a)
    s.add(b)
    for r, t in s.plan():
        s.advance(r.seq, len(t))
        r.output.append(1)
    preempted = False
    for _ in range(5):
        work = s.plan()
        assert any(r is a for r, _ in work)
        preempted = preempted or b in s.waiting
        for r, t in work:
            s.advance(r.seq, len(t))
            if r.pending == 0:
                r.output.append(1)
    assert preempted and a.seq.length == 13


def test_ragged_staging():
    pool = PagePool(20)
    a, b = Sequence(), Sequence()
    a.reserve(pool, 6, 4)
    a.length = 5
    b.reserve(pool, 7, 4)
    s = stage_ragged([(b, [7, 8, 9, 10, 11, 12, 13]), (a, [3])], max_blocks=3, block_size=4)
    assert s.token_ids.tolist() == [7, 8, 9, 10, 11, 12, 13, 3] and s.positions.tolist() == [0, 1, 2, 3, 4, 5, 6, 5]
    assert s.starts.tolist() == [0, 7, 8] and s.row_tables.tolist() == [0] * 7 + [1] and s.seq_lens.tolist() == [1, 2, 3, 4, 5, 6, 7, 6]
    assert s.slot_mapping.tolist() == [4 * b.pages[p // 4] + p % 4 for p in range(7)] + [4 * a.pages[1] + 1]
    assert s.block_tables.tolist() == [b.pages + [0], a.pages + [0]]
    for bad in ([], [(a, [])], [(a, [1] * 9)]):
        with pytest.raises(ValueError):
            stage_ragged(bad, max_blocks=3, block_size=4)


# ---------------------------------------------------------------------------------------------- configuration

@pytest.mark.parametrize("rot", [dict(dims=8, base=100.0), dict(dims=16, base=10000.0, scaling=dict(factor=4.0, original=128, fast=8.0, slow=1.0)),
                                 dict(dims=2, base=10.0, scaling=dict(factor=2.0, original=64, fast=32.0, slow=16.0)),
                                 dict(dims=64, base=1e6, scaling=dict(factor=1.0, original=4096, fast=32.0, slow=1.0))])
def test_pair_tables(rot):
    s = rot.get("scaling")
    cos, sin = pair_tables(Rotation(rot["dims"], rot["base"], YarnScaling(s["factor"], s["original"], s["fast"], s["slow"]) if s else None), 500)
    x = torch.zeros((500, rot["dims"]), dtype=torch.float64)
    x[:, 0::2] = 1.0  # each pair (1, 0) turns into (cos, sin)
    want = oracle.rotate(x, torch.arange(500), rot)
    assert np.abs(cos - want[:, 0::2].numpy()).max() <= 1e-6 and np.abs(sin - want[:, 1::2].numpy()).max() <= 1e-6
    with pytest.raises(ValueError):
        Rotation(3, 10.0)


def test_configuration_is_read_whole():
    c = oracle.model(oracle.layer(), oracle.layer(window=0, ff=0, scaling=False, heads=7), oracle.layer(weights_of=0), oracle.layer(weights_of=2))
    cfg = LatentDecoderConfig.from_config(json.loads(json.dumps(c)))
    assert [l.weights for l in cfg.layers] == [0, 1, 0, 0] and cfg.window is None
    assert cfg.layers[1].mlp is None and cfg.layers[1].mixer.window is None and cfg.layers[1].mixer.rot.scaling is None
    assert cfg.layers[0].mixer.heads == 3 and cfg.layers[1].mixer.heads == 7 and cfg.eps == 1e-5
    assert {k: tuple(v.shape) for k, v in oracle.make_weights(c).items()} == cfg.tensor_shapes()
    assert LatentDecoderConfig.from_config(oracle.model(oracle.layer(window=7), oracle.layer(window=30))).window == 30
    borrowed = oracle.model(oracle.layer(weights_of=2), oracle.layer(ff=0), oracle.layer())  # a layer may also use a later one's weights
    assert [l.weights for l in LatentDecoderConfig.from_config(borrowed).layers] == [2, 1, 2]
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="gated"),
                   lambda d: d["layers"][2].update(weights_of=2), lambda d: d["layers"][0].update(weights_of=3),
                   lambda d: d["layers"][0]["mixer"]["rot"].update(dims=64)):
        bad = json.loads(json.dumps(c))
        change(bad)
        with pytest.raises(ValueError):
            LatentDecoderConfig.from_config(bad)


def test_configuration_of_mixed_layers_is_read_whole():
    A, R = videdra.attention_layer, videdra.retention_layer
    c = videdra.model(R(mlp=videdra.dense_mlp(30)), A(mlp=videdra.moe_mlp(), window=12, keep=7), A(kv_from=1, window=40, keep=2), R(mlp=videdra.moe_mlp(shared=0, top=1)))
    cfg = MixedDecoderConfig.from_config(json.loads(json.dumps(c)))
    assert {k: tuple(v.shape) for k, v in videdra.make_weights(c).items()} == cfg.tensor_shapes()
    assert cfg.window == 40 and cfg.keep_first == 7 and cfg.recurrent and cfg.layers[2].mlp is None and cfg.layers[3].mlp.shared_ff is None
    assert cfg.layers[1].mixer.row == 2 * 2 * 32 + 2 * 48 and cfg.layers[2].mixer.kv_from == 1 and cfg.layers[0].mixer.decay == tuple(c["layers"][0]["mixer"]["decay"])
    assert MixedDecoderConfig.from_config(videdra.model(A(window=0), A(window=3))).window is None
    alone = MixedDecoderConfig.from_config(videdra.model(R()))
    assert alone.window == 1 and alone.keep_first == 0
    assert not MixedDecoderConfig.from_config(videdra.model(A())).recurrent
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other"), lambda d: d["layers"][2]["mixer"].update(kv_from=2),
                   lambda d: d["layers"][2]["mixer"].update(kv_from=0), lambda d: d["layers"][2]["mixer"].update(kv_heads=3), lambda d: d["layers"][0]["mixer"]["decay"].pop(),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=64), lambda d: d["layers"][1]["mixer"].update(kv_heads=4),
                   lambda d: d["layers"][1]["mlp"]["router"].update(top=8)):
        bad = json.loads(json.dumps(c))
        change(bad)
        with pytest.raises(ValueError):
            MixedDecoderConfig.from_config(bad)


def test_gate_and_factor_are_interleaved_by_sixteen():
    from tlaloc_b200.ops import interleave_gate

    gate, up = torch.arange(2 * 20 * 3.0).reshape(2, 20, 3) + 1, -torch.arange(2 * 20 * 3.0).reshape(2, 20, 3) - 1
    w = interleave_gate(gate, up)
    assert w.shape == (2, 64, 3) and torch.equal(w[1], interleave_gate(gate[1], up[1]))
    for f in range(20):
        r = f // 16 * 32 + f % 16
        assert torch.equal(w[:, r], gate[:, f]) and torch.equal(w[:, r + 16], up[:, f])
    assert torch.all(w[:, 36:48] == 0) and torch.all(w[:, 52:] == 0)


def test_registry_names(tmp_path):
    assert registry.architecture_of({"architecture": "Marotar"}) == "Marotar" and registry.architecture_of({"architecture": "Videdra"}) == "Videdra"
    assert registry.architecture_of({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    with pytest.raises(ValueError):
        registry.architecture_of({"architecture": "unheard of"})
    c = oracle.model(oracle.layer())
    w = oracle.make_weights(c)
    oracle.save(str(tmp_path), c, w)
    got = registry.read_tensors(str(tmp_path))
    assert set(got) == set(w) and all(np.array_equal(got[k], w[k].numpy()) for k in w)
    assert registry.num_blocks(registry.Sizes(100, 1000, 64, 8), 64) == 16 + 8 + 1


def test_command_line_lists_models(capsys):
    from tlaloc_b200.__main__ import main

    assert main(["models"]) == 0
    out = capsys.readouterr().out
    assert "Marotar bfloat16 float32" in out and "Videdra bfloat16 float32" in out
    assert main(["nothing"]) == 2
