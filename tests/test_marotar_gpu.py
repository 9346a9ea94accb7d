"""The Marotar decoder against a plain f64 implementation of its equations, through the framework's own engine: prompts, portions,
token by token, batches, reused pages, windows, sharing of weights, greedy generation, trace replay, the command line (needs a B200)."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import latent_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16


@pytest.fixture(autouse=True)
def no_wait_runs_out():
    """Every device-side wait is bounded; one that runs out leaves a status word (and a wrong result)."""
    yield
    from tlaloc_b200 import _native

    torch.cuda.synchronize()
    assert _native.lib().tlaloc_b200_device_status() == 0


def build(config, weights, dtype=F32, max_len=512, blocks=64, **kw):
    from tlaloc_b200.engine import Engine
    from tlaloc_b200.latent_decoder import LatentDecoder, LatentDecoderConfig

    cfg = LatentDecoderConfig.from_config(config)
    m = LatentDecoder(cfg, num_blocks=blocks, max_len=max_len, dtype=dtype, **kw)
    m.load_tensors({k: v.numpy() for k, v in weights.items()})
    return Engine(m)


def tokens(n, vocab=131, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rms_error(got, want):
    """Root mean square over the vocabulary of the centred difference, over that of the logits: the worst position."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return float((d.square().mean(-1).sqrt() / want.square().mean().sqrt()).max())


def limit(dtype):
    return 2e-5 if dtype == F32 else 4e-2


CONFIGS = {
    "two layers": oracle.model(oracle.layer(), oracle.layer(heads=5, dim=16, rot_dim=16, vdim=24, q_rank=40, kv_rank=72, window=33, ff=120)),
    "shared weights": oracle.model(oracle.layer(window=9), oracle.layer(window=40, ff=0), oracle.layer(window=9, weights_of=0),
                                   oracle.layer(window=40, ff=0, weights_of=1), oracle.layer(window=9, weights_of=2)),
    "weights of a later layer": oracle.model(oracle.layer(window=12, weights_of=1), oracle.layer(window=12)),
    "no feed-forward, no scaling": oracle.model(oracle.layer(ff=0, scaling=False, window=15), eps=1e-3),
    "part of the key part rotated": oracle.model(oracle.layer(rot_dim=24, rot_dims=16, window=50), oracle.layer(window=0, scaling=False)),
    "one head, one pair": oracle.model(oracle.layer(heads=1, dim=8, rot_dim=2, vdim=8, q_rank=8, kv_rank=8, window=1, ff=8), width=40, vocab=33),
    "odd sizes": oracle.model(oracle.layer(heads=3, dim=10, rot_dim=6, vdim=14, q_rank=18, kv_rank=22, window=30, ff=50), width=44, vocab=57),
    "wide": oracle.model(oracle.layer(heads=20, dim=64, rot_dim=32, vdim=64, q_rank=192, kv_rank=256, window=130, ff=640), width=320, vocab=257),
    "wider latent": oracle.model(oracle.layer(heads=40, dim=32, rot_dim=64, vdim=32, q_rank=128, kv_rank=512, window=70, ff=256), width=128, vocab=140),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompts_and_every_layer(name, dtype):
    config = CONFIGS[name]
    w = oracle.make_weights(config)
    eng = build(config, w, dtype)
    t = tokens(200, config["vocab"])
    want_trace, trace = [], []
    want = oracle.forward(config, w, t, want_trace)
    got, = eng.feed([("a", t, list(range(200)))])
    assert rms_error(got, want) <= limit(dtype)
    # the residual stream after every layer, on a fresh sequence
    from tlaloc_b200.paging import Sequence, stage_ragged

    seq = Sequence()
    seq.reserve(eng.pool, 200, eng.model.block_size)
    eng.model.run(stage_ragged([(seq, t)], max_blocks=eng.model.max_blocks, block_size=eng.model.block_size), [], trace)
    assert len(trace) == len(want_trace)
    for a, b in zip(trace, want_trace):
        assert float((a.cpu().double() - b).abs().max()) <= (1e-4 if dtype == F32 else 0.25) * float(b.abs().max())


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["two layers", "shared weights", "wide", "odd sizes"])
def test_portions_of_every_size_and_token_by_token(name, dtype):
    config = CONFIGS[name]
    w = oracle.make_weights(config, seed=1)
    n = 170
    t = tokens(n, config["vocab"], seed=2)
    want = oracle.forward(config, w, t)
    eng = build(config, w, dtype)
    for cut in (1, 2, 3, 31, 32, 33, 64, 65, 100, n):
        rows = []
        for lo in range(0, n, cut):
            part = t[lo:lo + cut]
            rows.append(eng.feed([(cut, part, list(range(len(part))))])[0])
        assert rms_error(torch.cat(rows), want) <= limit(dtype), cut
        eng.close(cut)
    # portions of changing size, then single tokens
    sizes, lo, rows = [2, 40, 3, 64, 2, 2, 33], 0, []
    for s in sizes + [1] * (n - sum(sizes)):
        rows.append(eng.feed([("x", t[lo:lo + s], list(range(s)))])[0])
        lo += s
    assert rms_error(torch.cat(rows), want) <= limit(dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_batch_of_unequal_requests_equals_each_alone(dtype):
    """Prompts, portions and single tokens of several sequences in one step."""
    config = CONFIGS["two layers"]
    w = oracle.make_weights(config, seed=3)
    eng = build(config, w, dtype)
    prompts = [tokens(n, seed=n) for n in (1, 2, 34, 65, 130)]
    want = [oracle.forward(config, w, p) for p in prompts]
    at, got = [0] * len(prompts), [[] for _ in prompts]
    plan = [(1, 1, 32, 1, 64), (0, 1, 1, 33, 2), (0, 0, 1, 31, 40), (0, 0, 0, 0, 1), (0, 0, 0, 0, 23)]
    for counts in plan:
        from tlaloc_b200.paging import Sequence

        work, want_rows, rows = [], [], 0
        for i, c in enumerate(counts):
            if c:
                seq = eng.sequences.setdefault(i, Sequence())
                assert seq.reserve(eng.pool, c, eng.model.block_size)
                work.append((seq, prompts[i][at[i]:at[i] + c]))
                want_rows += range(rows, rows + c)
                rows += c
        logits = eng._run(work, want_rows).cpu()
        lo = 0
        for i, c in enumerate(counts):
            got[i].append(logits[lo:lo + c])
            lo, at[i] = lo + c, at[i] + c
    for i, p in enumerate(prompts):
        assert at[i] == len(p)
        assert rms_error(torch.cat(got[i]), want[i]) <= limit(dtype), i


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_pages_given_back_are_used_again(dtype):
    """A pool barely larger than one sequence: the second and third sequence live on the pages of the first."""
    config = CONFIGS["shared weights"]
    w = oracle.make_weights(config, seed=4)
    eng = build(config, w, dtype, blocks=5, max_len=256)
    seen = set()
    for k in range(3):
        t = tokens(200 - 37 * k, seed=k)
        got, = eng.feed([(k, t, [len(t) - 1])])
        seen.update(p for p in eng.sequences[k].pages if p)
        assert rms_error(got, oracle.forward(config, w, t)[-1:]) <= limit(dtype)
        eng.close(k)
        assert eng.pool.free_count == eng.pool.capacity
    assert len(seen) <= 4


def peaked(window, dtype_seed=5):
    """One layer whose attention is peaked enough for single keys to matter, nothing else on the way to the logits."""
    config = oracle.model(oracle.layer(window=window, ff=0, heads=4))
    return config, oracle.make_weights(config, seed=dtype_seed, q_gain=3.0)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [2, 63, 64, 65, 130])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion of two", "portion of forty"])
def test_window_edge(window, dtype, how):
    """With one layer, a token just outside the window of the last position cannot move its logits at all; the one just inside
    does, by what the equations say."""
    config, w = peaked(window)
    n = 250
    base = tokens(n, seed=6)
    eng = build(config, w, dtype)

    def last(t):
        cut = {"prompt": n, "decoded": 1, "portion of two": 2, "portion of forty": 40}[how]
        if cut < n:
            eng.feed([("s", t[:n - cut], [])])
        out, = eng.feed([("s", t[n - cut:], [cut - 1])])
        eng.close("s")
        return out

    ref = last(base)
    for distance, inside in ((window - 1, True), (window, False), (window + 1, False)):
        t = list(base)
        moved = 0.0
        for other in range(1, 6):  # the replacement that moves the equations most (or any, outside)
            cand = list(base)
            cand[n - 1 - distance] = (base[n - 1 - distance] + 17 * other) % config["vocab"]
            d = float((oracle.forward(config, w, cand)[-1] - oracle.forward(config, w, base)[-1]).abs().max())
            if d >= moved:
                t, moved = cand, d
        got = float((last(t) - ref).abs().max())
        if inside:
            assert moved > 0 and abs(got - moved) <= 0.02 * moved + (1e-4 if dtype == F32 else 0.1), (distance, got, moved)
        else:
            assert moved == 0 and got == 0, (distance, got)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_first_tokens_and_far_keys(dtype):
    """Attention over everything: the first tokens of a long sequence keep their weight, across many pages."""
    config = oracle.model(oracle.layer(window=0, ff=0, heads=2, scaling=False, base=1e6))
    w = oracle.make_weights(config, seed=7, q_gain=4.0)
    n = 400
    t = tokens(n, seed=8)
    eng = build(config, w, dtype)
    whole, = eng.feed([("a", t, list(range(n)))])
    want = oracle.forward(config, w, t)
    assert rms_error(whole, want) <= 2 * limit(dtype)
    eng.feed([("b", t[:380], [])])
    rows = [eng.feed([("b", [x], [0])])[0] for x in t[380:]]
    assert rms_error(torch.cat(rows), want[380:]) <= 2 * limit(dtype)


def test_long_decoding_through_a_window_gives_old_pages_back():
    config = oracle.model(oracle.layer(window=40), oracle.layer(window=25, heads=2))
    w = oracle.make_weights(config, seed=9)
    eng = build(config, w, F32, blocks=4, max_len=512)  # three pages of 64 for 400 tokens
    t = tokens(400, seed=10)
    want = oracle.forward(config, w, t)
    eng.feed([("a", t[:100], [])])
    rows = [eng.feed([("a", [x], [0])])[0] for x in t[100:]]
    assert rms_error(torch.cat(rows), want[100:]) <= limit(F32)
    assert eng.pool.free_count >= 1


def test_graph_replay_equals_the_eager_step():
    """Batches of three pad to four rows; the third step of a size is captured, later ones replay it."""
    config = CONFIGS["two layers"]
    w = oracle.make_weights(config, seed=11)
    eng = build(config, w, F32)
    seqs = [tokens(60, seed=s) for s in (1, 2, 3)]
    want = [oracle.forward(config, w, s) for s in seqs]
    for i in range(60):
        out = eng.feed([(0, seqs[0][i:i + 1], [0])]) if i < 2 else None
        if out is None:
            from tlaloc_b200.paging import Sequence

            work = []
            for k in range(3):
                seq = eng.sequences.setdefault(k, Sequence())
                j = i if k == 0 else i - 2
                assert seq.reserve(eng.pool, 1, eng.model.block_size)
                work.append((seq, [seqs[k][j]]))
            logits = eng._run(work, [0, 1, 2]).cpu()
            for k in range(3):
                assert rms_error(logits[k:k + 1], want[k][i if k == 0 else i - 2][None]) <= limit(F32)
    assert 4 in eng.model._graphs and 1 not in eng.model._graphs


# ---------------------------------------------------------------------------------------------- generation

def test_greedy_generation_matches_the_plain_implementation():
    """Five requests through the scheduler in f32, with a pool that cannot hold them all at once."""
    config = CONFIGS["shared weights"]
    w = oracle.make_weights(config, seed=12)
    prompts = [tokens(n, seed=n) for n in (3, 70, 20, 1, 130)]
    want = [oracle.greedy(config, w, p, 12) for p in prompts]
    eng = build(config, w, F32, blocks=6, max_len=256, max_tokens=48, max_sequences=4)
    assert eng.generate(prompts, 12) == want
    assert eng.pool.free_count == eng.pool.capacity
    assert eng.generate(prompts[:1], 12, stop=[want[0][4]]) == [want[0][:want[0].index(want[0][4]) + 1]]


def test_command_line_and_trace_replay(tmp_path):
    config = CONFIGS["two layers"]
    w = oracle.make_weights(config, seed=13)
    oracle.save(str(tmp_path), config, w)
    prompt = tokens(40, seed=14)
    run = lambda *a, **kw: subprocess.run([sys.executable, *a], capture_output=True, text=True, cwd=ROOT, timeout=300, **kw)
    r = run("-m", "tlaloc_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "6", "--prompt", ",".join(map(str, prompt)))
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.splitlines()[-1]) == oracle.greedy(config, w, prompt, 6)
    want = oracle.forward(config, w, prompt)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": prompt[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": prompt[33:35], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "q", "tokens": prompt[35:], "want": [4]}], "end": ["q"]}]
    r = run(os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40",
            input="\n".join(json.dumps(s) for s in steps) + "\n")
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"]
    got = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)
    assert rms_error(torch.from_numpy(got), want[[0, 32]]) <= limit(F32)
    got = np.fromfile(tmp_path / "2.f32", "<f4").reshape(1, -1)
    assert rms_error(torch.from_numpy(got), want[[39]]) <= limit(F32)
    assert not (tmp_path / "1.f32").exists()


def test_llama_runs_under_the_same_engine(tmp_path):
    """The int8 Llama decoder behind the registry, engine and scheduler: batched generation equals one request at a time."""
    from tlaloc_b200 import registry
    from tlaloc_b200.engine import Engine

    rng = np.random.default_rng(0)
    d, ffn, vocab = 256, 512, 512
    t = {"model.embed_tokens.weight": rng.standard_normal((vocab, d)) * 0.5, "model.norm.weight": np.ones(d), "lm_head.weight": rng.standard_normal((vocab, d)) * 0.1}
    for l in range(2):
        p = f"model.layers.{l}."
        for name, shape in (("self_attn.q_proj", (d, d)), ("self_attn.k_proj", (128, d)), ("self_attn.v_proj", (128, d)), ("self_attn.o_proj", (d, d)),
                            ("mlp.gate_proj", (ffn, d)), ("mlp.up_proj", (ffn, d)), ("mlp.down_proj", (d, ffn))):
            t[p + name + ".weight"] = rng.standard_normal(shape) * shape[1] ** -0.5
        t[p + "input_layernorm.weight"] = t[p + "post_attention_layernorm.weight"] = np.ones(d)
    config = {"architectures": ["LlamaForCausalLM"], "hidden_size": d, "num_hidden_layers": 2, "num_attention_heads": 4, "num_key_value_heads": 2,
              "intermediate_size": ffn, "vocab_size": vocab, "rms_norm_eps": 1e-5, "rope_theta": 10000.0}
    oracle.save(str(tmp_path), config, {k: torch.from_numpy(np.asarray(v, np.float32)) for k, v in t.items()})
    model = registry.load(str(tmp_path), max_len=128, cache_tokens=512, max_sequences=8)
    prompts = [tokens(n, vocab, seed=n) for n in (5, 23, 40)]
    together = Engine(model).generate(prompts, 10)
    alone = [Engine(model).generate([p], 10)[0] for p in prompts]
    assert together == alone and all(len(o) == 10 for o in together)


def test_a_checkpoint_that_does_not_fit_is_refused(tmp_path):
    config = CONFIGS["two layers"]
    w = oracle.make_weights(config)
    bad = dict(w)
    del bad["l0.mix.uk"]
    with pytest.raises(ValueError, match="l0.mix.uk"):
        build(config, bad)
    bad = dict(w, **{"l1.norm2": torch.zeros(3)})
    with pytest.raises(ValueError, match="l1.norm2"):
        build(config, bad)
