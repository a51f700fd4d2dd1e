"""Vuvolix on the GPU against the plain numpy oracle (tests/vuvolix_oracle.py): every mechanism alone and
together, in fp32 and in bf16; prompts, portions, token-by-token decoding, packed batches; page and
session re-use; window edges with a key that stands out; sizes of all kinds; generation and replay
through the entry points a user calls."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nerva_b200 import generate, registry, synth
from nerva_b200.session import CudaHfDecodeSequenceLoop, CudaHfDecodeSequenceSession, SmokeStatus, sampler_config
from tests import vuvolix_models as M
from tests import vuvolix_oracle as O
from tests.conftest import ROOT

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")


def open_session(cfg, w, context, dtype):
    s = CudaHfDecodeSequenceSession(M.checkpoint(cfg, w), context, compute=dtype)
    assert s.status == SmokeStatus.OK, s.error
    return s


def run_portions(session, tokens, sizes):
    """Logits of every position, the tokens cut into portions of the given sizes (the last repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(session.append(tokens[at:at + n], range(n), reset=at == 0))
        at += n
        i += 1
    return np.concatenate(out)


@pytest.fixture(scope="module")
def full():
    cfg = M.full_config()
    w = M.weights(cfg)
    tokens = M.tokens(cfg, 150)
    return cfg, w, tokens, O.forward(cfg, w, tokens)


def plain(**mixer):
    return M.layer(ff=0, window=1000, rot=0, **mixer)


def scaled(cfg, **values):
    cfg.update(values)
    return cfg


MECHANISMS = {
    "attention only": lambda: M.config([plain()], scale=1.0, cap=0),
    "window": lambda: M.config([M.layer(ff=0, window=10, rot=0)], scale=1.0, cap=0),
    "window of one": lambda: M.config([M.layer(ff=0, window=1, rot=0)], scale=1.0, cap=0),
    "rotation of a part": lambda: M.config([M.layer(ff=0, window=1000, rot=12)], scale=1.0, cap=0),
    "rotation of all": lambda: M.config([M.layer(ff=0, window=1000, rot=32, base=300.0)], scale=1.0, cap=0),
    "scaled rotation": lambda: M.config([M.layer(ff=0, window=1000, rot=32, scaling=M.YARN)], scale=1.0, cap=0),
    "scaled rotation, empty ramp": lambda: M.config(
        [M.layer(ff=0, window=1000, rot=8, scaling={"factor": 2.0, "original": 4096, "fast": 1.0, "slow": 1.0})],
        scale=1.0, cap=0),
    "score scale": lambda: M.config([plain(scale=1.7)], scale=1.0, cap=0),
    "value width": lambda: M.config([plain(vdim=72)], scale=1.0, cap=0),
    "one query head per key": lambda: M.config([plain(kv_heads=4)], scale=1.0, cap=0),
    "many query heads per key": lambda: M.config([plain(heads=20, kv_heads=1, dim=16)], scale=1.0, cap=0),
    "feed-forward": lambda: M.config([M.layer(window=1, rot=0, ff=144)], scale=1.0, cap=0),
    "embedding scale": lambda: M.config([plain()], scale=0.05, cap=0),
    "soft cap": lambda: M.config([plain()], scale=1.0, cap=1.5),
    "loop": lambda: M.config([plain(), M.layer(window=5), plain()], scale=1.0, cap=0, loop=(1, 2, 4)),
    "loop from the first layer to the last": lambda: M.config([M.layer(), M.layer(window=9)], cap=0, loop=(0, 2, 2)),
    "loop of one pass": lambda: M.config([M.layer(), M.layer()], cap=0, loop=(0, 1, 1)),
    "large eps": lambda: scaled(M.config([M.layer()]), norm={"eps": 0.3}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism(built_lib, name, dtype):
    """A prompt in one piece and the same token by token (the decode step), both against the oracle."""
    cfg = MECHANISMS[name]()
    w = M.weights(cfg, seed=len(name))
    tokens = M.tokens(cfg, 45)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 64, dtype)
    assert M.distance(s.append(tokens, range(45), reset=True), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [1]), want) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_after_every_layer_run(built_lib, full, dtype):
    cfg, w, tokens, _ = full
    stages = []
    O.forward(cfg, w, tokens[:70], stages)
    got = open_session(cfg, w, 160, dtype).append_with_stream(tokens[:70], reset=True)
    assert len(stages) == len(got) == 8
    for a, b in zip(got, stages):
        assert M.distance(a, b) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[150], [1], [2], [3], [7, 1, 16, 2], [16], [17, 15], [64, 2, 1, 30], [149, 1], [5, 100]],
                         ids=lambda s: "-".join(map(str, s)))
def test_portions(built_lib, full, sizes, dtype):
    cfg, w, tokens, want = full
    got = run_portions(open_session(cfg, w, 160, dtype), tokens, sizes)
    assert M.worst_position(got, want) < 2 * M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("count", [1, 2, 3, 5])
def test_first_tokens(built_lib, full, count, dtype):
    cfg, w, tokens, want = full
    s = open_session(cfg, w, 32, dtype)
    assert M.worst_position(s.append(tokens[:count], range(count), reset=True), want[:count]) < 2 * M.TOLERANCE[dtype]
    # wanted places in any order, some twice
    places = [count - 1, 0, count - 1]
    assert M.worst_position(s.append(tokens[:count], places, reset=True), want[places]) < 2 * M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_of_several_blocks(built_lib, dtype):
    """More positions than one block step carries, more wanted places than one head launch does."""
    cfg = M.config([M.layer(window=300), M.layer(window=70, heads=6, kv_heads=3)], loop=(0, 1, 2))
    w = M.weights(cfg)
    tokens = M.tokens(cfg, 600)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 640, dtype)
    assert M.worst_position(s.append(tokens, range(600), reset=True), want) < 2 * M.TOLERANCE[dtype]
    assert M.worst_position(run_portions(s, tokens, [290, 40, 2, 1, 267]), want) < 2 * M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 32, 63, 64, 65, 130])
def test_window_edges(built_lib, window, dtype):
    """A key that stands out, just inside, just outside and far outside the window, read from a prompt in
    one piece, from portions that cut between key and query, and decoded; the query sits at page and
    tile borders."""
    cfg, w = M.marked_model(window, rot=16)
    s = open_session(cfg, w, 320, dtype)
    for at in (window + 12, 255, 256):
        for back in sorted({max(window - 1, 1), window, window + 1, at}):
            if back > at:
                continue
            tokens = M.marked_tokens(cfg, at + 1, at - back, at)
            want = O.forward(cfg, w, tokens)[-1:]
            for sizes in ([at + 1], [at, 1], [at - back + 1, max(back - 1, 1), 1], [at - 1, 2]):
                s.append(tokens[:1], reset=True)
                done, got = 0, None
                for n in sizes:
                    n = min(n, at + 1 - done)
                    if n:
                        got = s.append(tokens[done:done + n], [n - 1], reset=done == 0)
                        done += n
                assert done == at + 1
                assert M.distance(got, want) < 3 * M.TOLERANCE[dtype], (at, back, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_away_is_found_without_a_window(built_lib, dtype):
    cfg, w = M.marked_model(0, rot=16)
    s = open_session(cfg, w, 720, dtype)
    for key_at in (0, 15, 16, 63, 64, 255, 256, 400):
        tokens = M.marked_tokens(cfg, 701, key_at, 700)
        want = O.forward(cfg, w, tokens)[-1:]
        assert M.distance(s.append(tokens, [700], reset=True), want) < 3 * M.TOLERANCE[dtype], key_at
        s.append(tokens[:700], reset=True)
        assert M.distance(s.append(tokens[700:], [0]), want) < 3 * M.TOLERANCE[dtype], key_at


SIZES = {
    "odd widths": M.config([M.layer(heads=3, kv_heads=1, dim=22, vdim=18, rot=10, ff=75),
                            M.layer(heads=5, kv_heads=5, dim=13, vdim=29, rot=4, ff=33)], width=100, vocab=211),
    "width one below a multiple": M.config([M.layer(ff=63)], width=127, vocab=67),
    "large heads": M.config([M.layer(heads=2, kv_heads=1, dim=200, vdim=256, rot=64, ff=130)], width=192, vocab=97),
    "values wider than keys": M.config([M.layer(heads=4, kv_heads=4, dim=8, vdim=136, rot=8)], width=64, vocab=50),
    "keys wider than values": M.config([M.layer(heads=4, kv_heads=1, dim=256, vdim=16, rot=256)], width=64, vocab=50),
    "twelve heads a key, wide": M.config([M.layer(heads=12, kv_heads=1, dim=64, vdim=64, ff=520)], width=448, vocab=1000),
    "one of everything": M.config([M.layer(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, ff=1)], width=8, vocab=5),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(built_lib, name, dtype):
    cfg = SIZES[name]
    w = M.weights(cfg)
    tokens = M.tokens(cfg, 90)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 96, dtype)
    assert M.distance(s.append(tokens, range(90), reset=True), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [40, 1, 1, 1, 2, 45]), want) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_random_small_models(built_lib, dtype):
    rng = np.random.default_rng(5)
    for seed in range(6):
        layers = []
        for _ in range(int(rng.integers(1, 5))):
            kv = int(rng.integers(1, 4))
            dim = int(rng.integers(2, 65)) * 2
            layers.append(M.layer(heads=kv * int(rng.integers(1, 5)), kv_heads=kv, dim=dim, vdim=int(rng.integers(1, 100)),
                                  rot=2 * int(rng.integers(0, dim // 2 + 1)), window=int(rng.integers(1, 80)),
                                  base=float(rng.choice([100.0, 10000.0, 1e6])), ff=int(rng.choice([0, 50, 128, 210])),
                                  scaling=M.YARN if rng.random() < 0.5 else None, scale=float(rng.uniform(0.05, 0.6))))
        n = len(layers)
        start = int(rng.integers(0, n))
        loop = (start, int(rng.integers(start + 1, n + 1)), int(rng.integers(1, 4))) if rng.random() < 0.7 else None
        cfg = M.config(layers, width=int(rng.integers(10, 300)), vocab=int(rng.integers(5, 600)), loop=loop)
        w = M.weights(cfg, seed)
        tokens = M.tokens(cfg, 120, seed)
        want = O.forward(cfg, w, tokens)
        s = open_session(cfg, w, 128, dtype)
        assert M.distance(s.append(tokens, range(120), reset=True), want) < 1.5 * M.TOLERANCE[dtype], (seed, cfg)
        assert M.distance(run_portions(s, tokens, [50, 2, 30, 1]), want) < 1.5 * M.TOLERANCE[dtype], (seed, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_results_do_not_depend_on_pages_or_on_what_ran_before(built_lib, full, dtype):
    cfg, w, tokens, _ = full
    s = open_session(cfg, w, 160, dtype)
    first = run_portions(s, tokens, [60, 1, 1, 88])
    other = M.tokens(cfg, 160, seed=9)
    s.append(other, reset=True)                    # every page now holds another request's rows
    s.append(other[:3], reset=True)
    assert np.array_equal(run_portions(s, tokens, [60, 1, 1, 88]), first)
    p = open_session(cfg, w, 160, dtype)
    p.set_kv_block_table(synth.permutation(4, synth.T_PAGE_TABLE, 10))
    assert np.array_equal(run_portions(p, tokens, [60, 1, 1, 88]), first)
    fork = s.fork_shared_weights()
    assert fork.status == SmokeStatus.OK
    tail = other[:20]
    assert np.array_equal(fork.append(tail[:10], range(10), reset=True), s.append(tail[:10], range(10), reset=True))
    s.append(tokens, reset=True)                   # the fork's cache is its own
    t = open_session(cfg, w, 160, dtype)
    t.append(tail[:10], reset=True)
    assert np.array_equal(fork.append(tail[10:], range(10)), t.append(tail[10:], range(10)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_packed_batches_of_unequal_requests(built_lib, full, dtype):
    """batch_advance_one over forks at different positions against the oracle on each fork's own history."""
    cfg, w, tokens, _ = full
    root = open_session(cfg, w, 160, dtype)
    lengths = [1, 2, 25, 26, 70, 130]
    forks, histories = [], []
    for i, n in enumerate(lengths):
        f = root.fork_shared_weights()
        assert f.status == SmokeStatus.OK
        history = tokens[i:i + n]
        f.append(history, reset=True)
        first = CudaHfDecodeSequenceLoop(f).advance(1)  # the token the last given position sampled
        assert first.status == SmokeStatus.OK
        forks.append(f)
        histories.append(list(history) + first.tokens)
    for step in range(6):
        out = CudaHfDecodeSequenceSession.batch_advance_one(forks, target_block_tokens=len(forks))
        assert out.status == SmokeStatus.OK and out.block_tokens == len(forks), out.error
        for f, history, token in zip(forks, histories, out.tokens):
            want = O.forward(cfg, w, history)[-1]
            assert M.distance(f.read_logits(), want) < 3 * M.TOLERANCE[dtype]
            assert want.max() - want[token] < 0.3 * want.std()
            history.append(token)


def test_long_decoding_follows_the_oracle(built_lib, full):
    """Greedy generation in fp32, far past every window: each token is the oracle's choice for its history."""
    cfg, w, tokens, _ = full
    s = open_session(cfg, w, 512, "float32")
    start, loop = CudaHfDecodeSequenceLoop.start(s, tokens[:20])
    assert start.status == SmokeStatus.OK
    out = []
    for n in (1, 7, 200, 92):
        r = loop.advance(n)
        assert r.status == SmokeStatus.OK, r.error
        out += r.tokens
    assert len(out) == 300
    want = O.forward(cfg, w, tokens[:20] + out[:-1])[19:]
    picked = want[np.arange(300), out]
    assert (want.max(axis=1) - picked).max() < 1e-3
    assert M.distance(s.read_logits(), want[-1]) < 5 * M.TOLERANCE["float32"]


def test_given_tokens_after_generated_ones(built_lib, full):
    """append continues a generated sequence (the last sampled token has not been run and is dropped)."""
    cfg, w, tokens, _ = full
    s = open_session(cfg, w, 160, "float32")
    _, loop = CudaHfDecodeSequenceLoop.start(s, tokens[:30])
    out = loop.advance(10).tokens
    got = s.append(tokens[30:50], range(20))
    want = O.forward(cfg, w, tokens[:30] + out[:-1] + tokens[30:50])[39:]
    assert M.worst_position(got, want) < 5 * M.TOLERANCE["float32"]
    again = CudaHfDecodeSequenceLoop(s).advance(5).tokens
    want = O.forward(cfg, w, tokens[:30] + out[:-1] + tokens[30:50] + again[:-1])[-5:]
    assert (want.max(axis=1) - want[np.arange(5), again]).max() < 1e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_from_a_model_folder(built_lib, full, tmp_path, dtype):
    cfg, w, tokens, _ = full
    folder = M.write_folder(tmp_path / "m", cfg, w)
    out = generate.generate(registry.load_model(folder), tokens[:40], 24, compute=dtype)
    want = O.forward(cfg, w, tokens[:40] + out[:-1])[39:]
    slack = 1e-3 if dtype == "float32" else 0.3 * want.std()
    assert len(out) == 24 and (want.max(axis=1) - want[np.arange(24), out]).max() < slack
    run = subprocess.run([sys.executable, "-m", "nerva_b200.generate", "--model", folder, "--dtype", dtype, "--tokens", "24",
                          "--prompt", ",".join(map(str, tokens[:40]))], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [int(t) for t in run.stdout.split(",")] == out


def test_seeded_sampling_repeats(built_lib, full):
    cfg, w, tokens, _ = full
    sampler = sampler_config(temperature=1.0, top_p=0.95, top_k=40, seed=11)
    one = generate.generate(M.checkpoint(cfg, w), tokens[:10], 32, sampler)
    assert one == generate.generate(M.checkpoint(cfg, w), tokens[:10], 32, sampler)
    assert one != generate.generate(M.checkpoint(cfg, w), tokens[:10], 32, sampler_config(1.0, 0.95, 40, 12))


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(built_lib, full, tmp_path, dtype):
    """The replay program: requests that overlap, portions, wanted places, sessions that serve a second request."""
    cfg, w, tokens, want = full
    folder = M.write_folder(tmp_path / "m", cfg, w)
    out = tmp_path / "out"
    out.mkdir()
    cuts = {"a": [30, 1, 1, 60], "b": [2, 2, 41], "c": [92]}
    plan = [["a"], ["a", "b"], ["b"], ["a"], ["b", "a"], ["c"]]
    at, turn, steps, expected = dict.fromkeys(cuts, 0), dict.fromkeys(cuts, 0), [], []
    for n, ids in enumerate(plan):
        entries, end, rows = [], [], []
        for i in ids:
            k = cuts[i][turn[i]]
            places = sorted({0, k - 1})
            entries.append({"id": i, "tokens": tokens[at[i]:at[i] + k], "want": places if n != 3 else []})
            rows += [at[i] + p for p in entries[-1]["want"]]
            at[i] += k
            turn[i] += 1
            if turn[i] == len(cuts[i]):
                end.append(i)
        steps.append(json.dumps({"step": n, "entries": entries, "end": end}))
        expected.append(rows)
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "160"], input="\n".join(steps) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert run.stdout.split("\n")[:len(plan)] == [f"done {n}" for n in range(len(plan))]
    for n, rows in enumerate(expected):
        path = out / f"{n}.f32"
        assert path.exists() == bool(rows)
        if rows:
            got = np.fromfile(path, dtype="<f4").reshape(len(rows), cfg["vocab"])
            assert M.worst_position(got, want[rows]) < 2 * M.TOLERANCE[dtype], n


def test_append_refuses_what_does_not_fit(built_lib, full):
    cfg, w, tokens, want = full
    s = open_session(cfg, w, 32, "bfloat16")
    s.append(tokens[:20], reset=True)
    for bad in (tokens[:13], [cfg["vocab"]]):
        with pytest.raises(RuntimeError):
            s.append(bad)
    assert M.distance(s.append(tokens[20:32], range(12)), want[20:32]) < 2 * M.TOLERANCE["bfloat16"]


def test_append_on_the_dense_models(built_lib, tiny_checkpoint):
    """The same call on a dense model: portions and single tokens end where start ends."""
    ids = synth.prompt_ids(synth.TINY_QWEN3, count=40)
    s = CudaHfDecodeSequenceSession(tiny_checkpoint, 64)
    CudaHfDecodeSequenceLoop.start(s, ids)
    want = s.read_logits()
    s.append(ids[:17], reset=True)
    s.append(ids[17:18])
    got = s.append(ids[18:], [21, 0])
    assert np.abs(got[0] - want).max() < 2e-2
    assert np.abs(s.read_logits() - want).max() < 2e-2
    assert got[1].std() > 0
