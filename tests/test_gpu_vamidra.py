"""Vamidra on the GPU against the plain numpy oracle (tests/vamidra_oracle.py): every mechanism alone and
together, in fp32 and in bf16; prompts, portions, token-by-token decoding, packed batches; page, state and
session re-use; window and kept-position edges with a key that stands out; a state that has to last; sizes
of all kinds; generation and replay through the entry points a user calls."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nerva_b200 import generate, parallel_model, registry, sandwich_model, synth
from nerva_b200.session import CudaHfDecodeSequenceLoop, CudaHfDecodeSequenceSession, SmokeStatus, sampler_config
from tests import vamidra_models as M
from tests import vamidra_oracle as O
from tests import vuvolix_models as V
from tests import vuvolix_oracle as VO
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


def wide(**mixer):
    return M.attention(ff=0, **{"window": 1000, "keep": 0, "cap": 0.0, **mixer})


def alone(**mixer):
    return M.config([M.space(ff=0, **mixer)])


MECHANISMS = {
    "attention only": lambda: M.config([wide()]),
    "window": lambda: M.config([wide(window=10)]),
    "window of one": lambda: M.config([wide(window=1)]),
    "kept positions": lambda: M.config([wide(window=6, keep=4)]),
    "kept positions beyond the window": lambda: M.config([wide(window=3, keep=30)]),
    "one kept position, window of one": lambda: M.config([wide(window=1, keep=1)]),
    "score cap": lambda: M.config([wide(cap=0.8)]),
    "score scale": lambda: M.config([wide(scale=0.9, cap=5.0)]),
    "value width": lambda: M.config([wide(vdim=72)]),
    "one query head per key": lambda: M.config([wide(kv_heads=4)]),
    "many query heads per key": lambda: M.config([wide(heads=20, kv_heads=1, dim=16)]),
    "no window at all": lambda: M.config([wide(window=0)]),
    "state space only": lambda: alone(),
    "one head": lambda: alone(heads=1, groups=1, norm_groups=1),
    "one group": lambda: alone(groups=1),
    "a group per head": lambda: alone(groups=6, norm_groups=6),
    "no convolution": lambda: alone(conv=1),
    "two taps": lambda: alone(conv=2),
    "seven taps": lambda: alone(conv=7),
    "sixteen taps": lambda: alone(conv=16),
    "state of one": lambda: alone(state=1),
    "state of 128": lambda: alone(state=128),
    "state of 200": lambda: alone(heads=2, groups=1, state=200, norm_groups=1),
    "norm in one part": lambda: alone(norm_groups=1),
    "norm in parts of 128": lambda: alone(heads=8, vdim=32, groups=2, norm_groups=2),
    "norm in many parts": lambda: alone(norm_groups=48),
    "feed-forward": lambda: M.config([M.attention(window=1, keep=0, ff=144)]),
    "state space and feed-forward": lambda: M.config([M.space(ff=100)]),
    "no logit scale": lambda: M.config([wide()], logit_scale=1.0),
    "loop": lambda: M.config([wide(), M.space(), wide()], loop=(1, 2, 4)),
    "loop from the first layer to the last": lambda: M.config([M.space(), M.attention(window=9)], loop=(0, 2, 2)),
    "loop of one pass": lambda: M.config([M.attention(), M.space()], loop=(0, 1, 1)),
    "large eps": lambda: M.config([M.attention(), M.space()], eps=0.3),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism(built_lib, name, dtype):
    """A prompt in one piece, the same token by token (the decode step), and in portions of a few tokens."""
    cfg = MECHANISMS[name]()
    w = M.weights(cfg, seed=len(name))
    tokens = M.tokens(cfg, 45)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 64, dtype)
    assert M.distance(s.append(tokens, range(45), reset=True), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [1]), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [2, 5, 3, 9, 17, 2]), want) < M.TOLERANCE[dtype]


@dataclasses.dataclass(frozen=True)
class PlainSandwich(sandwich_model.SandwichConfig):
    """Sandwich blocks with RMS norms, silu and passes that begin with their vector alone."""

    def tensor_shapes(self):
        return {k: v for k, v in super().tensor_shapes().items() if k != "loop.in"}

    def native_model(self, compute):
        return parallel_model.native_model(self, compute, embedding_scale=2.0, logit_softcap=3.0, block=sandwich_model.BLOCK_SANDWICH)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sandwich_blocks_of_another_design(built_lib, monkeypatch, dtype):
    """The other norm, activation and loop entry, rotated and normalised q and k, a scaled embedding, capped logits."""
    cfg = M.config([M.attention(kv_heads=4), M.space(), M.attention(window=9)], loop=(1, 3, 2))
    w = M.weights(cfg)
    parsed = sandwich_model.SandwichConfig.from_json(cfg)
    specs = tuple(dataclasses.replace(s, rotary_dims=16, qk_norm=True) if isinstance(s, parallel_model.ParallelLayer) else s
                  for s in parsed.layer_specs)
    plain = PlainSandwich(**{**{f.name: getattr(parsed, f.name) for f in dataclasses.fields(parsed)}, "layer_specs": specs})
    s = CudaHfDecodeSequenceSession(parallel_model.ParallelCheckpoint(
        plain, {k: synth.f32_to_bf16(v).reshape(v.shape) for k, v in w.items()}), 64, compute=dtype)
    assert s.status == SmokeStatus.OK, s.error

    capped = O.capped_attention

    def rotated(q, k, v, scale, cap, mask):
        at = np.arange(len(q))
        freq, magnitude = VO.rotary_frequencies(16, 10000.0)
        return capped(*(VO.rms_norm(VO.rotate(t, at, freq, magnitude), cfg["norm"]["eps"]) for t in (q, k)), v, scale, cap, mask)

    monkeypatch.setattr(O, "capped_attention", rotated)
    monkeypatch.setattr(O, "layer_norm", lambda x, eps, weight: VO.rms_norm(x, eps, weight))
    monkeypatch.setattr(O, "gelu_tanh", O.silu)
    monkeypatch.setattr(O, "begin_pass", lambda x, first, weights, number: (x + weights["loop.step"][number]).astype(np.float32))
    tokens = M.tokens(cfg, 50)
    want = VO.soft_cap(O.forward({**cfg, "logit_scale": 1.0}, {**w, "embed": 2.0 * w["embed"]}, tokens), 3.0)
    assert M.distance(s.append(tokens, range(50), reset=True), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [1, 1, 20, 3, 1]), want) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_parallel_blocks_with_kept_positions_cap_and_gates(built_lib, monkeypatch, dtype):
    cfg = V.config([V.layer(window=9), V.layer(heads=6, kv_heads=3, window=20, ff=0)])
    parsed = parallel_model.ParallelConfig.from_json(cfg)
    parsed = dataclasses.replace(parsed, layer_specs=tuple(
        dataclasses.replace(s, keep_first=4, score_softcap=1.5, head_gate=True) for s in parsed.layer_specs))
    w = V.weights(cfg)
    rng = np.random.default_rng(3)
    for i, heads in enumerate((4, 6)):
        w[f"l{i}.mix.g"] = M.round_bf16(rng.standard_normal((heads, cfg["width"])) * 0.2)
    s = CudaHfDecodeSequenceSession(parallel_model.ParallelCheckpoint(
        parsed, {k: synth.f32_to_bf16(v).reshape(v.shape) for k, v in w.items()}), 64, compute=dtype)
    assert s.status == SmokeStatus.OK, s.error

    def attention_mixer(h, m, get, eps, positions):
        tokens, heads, groups = len(h), m["heads"], m["kv_heads"]
        freq, magnitude = VO.rotary_frequencies(m["rot"]["dims"], m["rot"]["base"])
        q, k = (VO.rms_norm(VO.rotate(VO.linear(get(n), h).reshape(tokens, c, m["dim"]), positions, freq, magnitude), eps)
                for n, c in (("q", heads), ("k", groups)))
        v = VO.linear(get("v"), h).reshape(tokens, groups, m["vdim"])
        a = O.capped_attention(q, k, v, m["scale"], 1.5, O.visible(positions, positions, m["mask"]["size"], 4))
        return VO.linear(get("o"), O.head_gate(a, get("g"), h).reshape(tokens, heads * m["vdim"]))

    monkeypatch.setattr(VO, "attention_mixer", attention_mixer)
    tokens = M.tokens(cfg, 50)
    want = VO.forward(cfg, w, tokens)
    assert M.distance(s.append(tokens, range(50), reset=True), want) < M.TOLERANCE[dtype]
    assert M.distance(run_portions(s, tokens, [1, 1, 20, 3, 1]), want) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_after_every_layer_run(built_lib, full, dtype):
    cfg, w, tokens, _ = full
    stages = []
    O.forward(cfg, w, tokens[:70], stages)
    got = open_session(cfg, w, 160, dtype).append_with_stream(tokens[:70], reset=True)
    assert len(stages) == len(got) == 11
    for a, b in zip(got, stages):
        assert M.distance(a, b) < M.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[150], [1], [2], [3], [7, 1, 16, 2], [15], [16], [17, 15], [64, 2, 1, 30], [63, 65], [149, 1],
                                   [5, 100]], ids=lambda s: "-".join(map(str, s)))
def test_portions(built_lib, full, sizes, dtype):
    cfg, w, tokens, want = full
    got = run_portions(open_session(cfg, w, 160, dtype), tokens, sizes)
    assert M.worst_position(got, want) < 3 * M.TOLERANCE[dtype]  # the worst of 150 positions behind eleven layer runs


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
    cfg = M.config([M.attention(window=300, keep=5), M.space(heads=2, groups=1, norm_groups=2),
                    M.attention(window=70, heads=6, kv_heads=3)], loop=(0, 2, 2))
    w = M.weights(cfg)
    tokens = M.tokens(cfg, 600)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 640, dtype)
    assert M.worst_position(s.append(tokens, range(600), reset=True), want) < 2 * M.TOLERANCE[dtype]
    assert M.worst_position(run_portions(s, tokens, [257, 40, 2, 1, 300]), want) < 2 * M.TOLERANCE[dtype]


def cut_runs(session, tokens, cuts):
    """The last position's logits, the tokens cut into portions of the given sizes."""
    done, got = 0, None
    for n in cuts:
        n = min(n, len(tokens) - done)
        if n:
            got = session.append(tokens[done:done + n], [n - 1], reset=done == 0)
            done += n
    assert done == len(tokens)
    return got


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(1, 0), (2, 1), (15, 16), (16, 15), (17, 17), (32, 4), (63, 33), (64, 64), (65, 1), (130, 70)])
def test_window_and_kept_position_edges(built_lib, window, keep, dtype):
    """A key that stands out, just inside and just outside the window, the last kept position and the next one, and one
    in between, read from a prompt in one piece, from portions that cut between key and query, and decoded; the
    query sits at page and tile borders."""
    cfg, w = M.marked_model(window, keep)
    s = open_session(cfg, w, 320, dtype)
    for at in (window + keep + 12, 255, 256):
        keys = {at - max(window - 1, 1), at - window, at - window - 1, max(keep - 1, 0), keep, (keep + at - window) // 2, 0}
        for key_at in sorted(k for k in keys if 0 <= k < at):
            tokens = M.marked_tokens(cfg, at + 1, key_at, at)
            want = O.forward(cfg, w, tokens)[-1:]
            for cuts in ([at + 1], [at, 1], [key_at + 1, max(at - key_at - 1, 0), 1], [at - 1, 2], [at - 9, 10]):
                assert M.distance(cut_runs(s, tokens, cuts), want) < 3 * M.TOLERANCE[dtype], (at, key_at, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_away_is_found_without_a_window(built_lib, dtype):
    cfg, w = M.marked_model(0, 0)
    s = open_session(cfg, w, 720, dtype)
    for key_at in (0, 15, 16, 63, 64, 255, 256, 400):
        tokens = M.marked_tokens(cfg, 701, key_at, 700)
        want = O.forward(cfg, w, tokens)[-1:]
        assert M.distance(cut_runs(s, tokens, [701]), want) < 3 * M.TOLERANCE[dtype], key_at
        assert M.distance(cut_runs(s, tokens, [700, 1]), want) < 3 * M.TOLERANCE[dtype], key_at


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mixer", [{}, {"heads": 4, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 2}], ids=["small", "large"])
def test_the_state_lasts(built_lib, mixer, dtype):
    """A token that stands out hundreds of tokens ago shows, wherever it lies in its block, chunk or portion."""
    cfg, w = M.remembering_model(**mixer)
    s = open_session(cfg, w, 420, dtype)
    for key_at in (0, 1, 2, 63, 64, 255, 256, 300):
        tokens = M.tokens(cfg, 400)
        tokens[key_at] = M.KEY
        want = O.forward(cfg, w, tokens)[-1:]
        for cuts in ([400], [399, 1], [key_at + 1, 399 - key_at], [key_at, 2, 1, 400], [256, 1, 15, 16, 112]):
            assert M.distance(cut_runs(s, tokens, cuts), want) < 3 * M.TOLERANCE[dtype], (key_at, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_extreme_steps_and_decays(built_lib, dtype):
    """States that forget at once, hardly ever, and that take steps near zero and large ones, side by side."""
    # one norm group: a head whose output nearly vanishes would have its rounding blown up by a norm of its own
    cfg = M.config([M.space(heads=8, groups=2, norm_groups=1)])
    w = M.weights(cfg)
    w["l0.mix.A_log"][:] = M.round_bf16([-9.0, -9.0, 0.0, 0.0, 3.0, 3.0, 5.0, 5.0])
    w["l0.mix.dt_bias"][:] = M.round_bf16([-12.0, 4.0, -12.0, 30.0, -12.0, 4.0, -7.0, 30.0])
    tokens = M.tokens(cfg, 200)
    want = O.forward(cfg, w, tokens)
    s = open_session(cfg, w, 208, dtype)
    assert M.worst_position(s.append(tokens, range(200), reset=True), want) < 2 * M.TOLERANCE[dtype]
    assert M.worst_position(run_portions(s, tokens, [70, 1, 1, 5, 130]), want) < 2 * M.TOLERANCE[dtype]


SIZES = {
    "odd widths": M.config([M.attention(heads=3, kv_heads=1, dim=22, vdim=18, ff=75),
                            M.space(heads=5, vdim=7, state=11, groups=5, norm_groups=7, ff=33)], width=100, vocab=211, loop=(0, 1, 2)),
    "width one below a multiple": M.config([M.attention(ff=63), M.space(ff=63)], width=127, vocab=67),
    "large heads": M.config([M.attention(heads=2, kv_heads=1, dim=200, vdim=256, ff=130)], width=192, vocab=97),
    "wide state-space heads": M.config([M.space(heads=2, vdim=200, state=64, groups=1, norm_groups=1)], width=96, vocab=97),
    "values wider than keys": M.config([M.attention(heads=4, kv_heads=4, dim=8, vdim=136)], width=64, vocab=50),
    "keys wider than values": M.config([M.attention(heads=4, kv_heads=1, dim=256, vdim=16)], width=64, vocab=50),
    "twelve heads a key, wide": M.config([M.attention(heads=12, kv_heads=1, dim=64, vdim=64, ff=520), M.space(
        heads=16, vdim=64, state=128, groups=4, norm_groups=4, ff=520)], width=448, vocab=1000, loop=(1, 2, 2)),
    "one of everything": M.config([M.attention(heads=1, kv_heads=1, dim=1, vdim=1, ff=1), M.space(
        heads=1, vdim=1, state=1, groups=1, conv=1, norm_groups=1, ff=1)], width=8, vocab=5, loop=(0, 2, 2)),
    "feed-forward too wide for the streaming kernel": M.config([M.attention(ff=20000)], width=64, vocab=50),
    "width too wide for the streaming kernels": M.config([M.attention(heads=1, kv_heads=1, dim=16, vdim=16, ff=0), M.space(
        heads=4, vdim=16, state=8, groups=1, norm_groups=1, ff=24)], width=8260, vocab=40),
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
    for seed in range(8):
        layers = []
        for _ in range(int(rng.integers(1, 5))):
            ff = int(rng.choice([0, 50, 128, 210]))
            if rng.random() < 0.5:
                kv = int(rng.integers(1, 4))
                layers.append(M.attention(heads=kv * int(rng.integers(1, 5)), kv_heads=kv, dim=int(rng.integers(1, 130)),
                                          vdim=int(rng.integers(1, 100)), window=int(rng.integers(1, 80)), ff=ff,
                                          keep=int(rng.choice([0, 1, 5, 40])), cap=float(rng.choice([0.0, 1.0, 50.0])),
                                          scale=float(rng.uniform(0.05, 0.3))))
            else:
                groups, heads, vdim = int(rng.integers(1, 4)), int(rng.integers(1, 4)), int(rng.integers(1, 80))
                heads *= groups
                parts = [g for g in range(1, 17) if heads * vdim % g == 0]
                layers.append(M.space(heads=heads, vdim=vdim, state=int(rng.integers(1, 140)), groups=groups, ff=ff,
                                      conv=int(rng.integers(1, 7)), norm_groups=int(rng.choice(parts))))
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
    s.append(other, reset=True)                    # every page and state now holds another request's
    s.append(other[:3], reset=True)
    assert np.array_equal(run_portions(s, tokens, [60, 1, 1, 88]), first)
    s.append(other[:7], reset=True)
    decoded = run_portions(s, tokens[:20], [1])
    assert np.array_equal(run_portions(s, tokens[:20], [1]), decoded)
    p = open_session(cfg, w, 160, dtype)
    p.set_kv_block_table(synth.permutation(4, synth.T_PAGE_TABLE, 10))
    assert np.array_equal(run_portions(p, tokens, [60, 1, 1, 88]), first)
    fork = s.fork_shared_weights()
    assert fork.status == SmokeStatus.OK
    tail = other[:20]
    assert np.array_equal(fork.append(tail[:10], range(10), reset=True), s.append(tail[:10], range(10), reset=True))
    s.append(tokens, reset=True)                   # the fork's cache and state are its own
    t = open_session(cfg, w, 160, dtype)
    t.append(tail[:10], reset=True)
    assert np.array_equal(fork.append(tail[10:], range(10)), t.append(tail[10:], range(10)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_fork_continues_where_its_parent_stands(built_lib, full, dtype):
    cfg, w, tokens, want = full
    s = open_session(cfg, w, 160, dtype)
    s.append(tokens[:61], reset=True)
    fork = s.fork_shared_weights()
    assert M.worst_position(fork.append(tokens[61:80], range(19)), want[61:80]) < 2 * M.TOLERANCE[dtype]
    assert M.worst_position(s.append(tokens[61:62], [0]), want[61:62]) < 2 * M.TOLERANCE[dtype]


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
    # and each alone from there
    for f, history in zip(forks, histories):
        given = [history[-1], 3]
        want = O.forward(cfg, w, history[:-1] + given)[-2:]
        assert M.worst_position(f.append(given, [0, 1]), want) < 3 * M.TOLERANCE[dtype]


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
