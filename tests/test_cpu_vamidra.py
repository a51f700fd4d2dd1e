"""Vamidra without a GPU: configuration and weight loading, requests the library refuses, and the oracle
itself (that it notices the mistakes the GPU tests are there to find)."""
import copy
import json

import numpy as np
import pytest

from nerva_b200 import ffi, parallel_model, registry, sandwich_model, synth
from nerva_b200.session import CudaHfDecodeSequenceSession, SmokeStatus, weight_blocks
from tests import vamidra_models as M
from tests import vamidra_oracle as O

INVALID_REQUEST = 1  # failure stage


def test_configuration_round_trip_and_layer_runs():
    cfg = M.full_config()
    parsed = sandwich_model.SandwichConfig.from_json(cfg)
    again = sandwich_model.SandwichConfig.from_json(json.loads(sandwich_model.dump_config(parsed)))
    assert again == parsed
    assert parsed.layers == 5 and parsed.layer_runs == 11 == len(O.layer_runs(cfg))
    assert [i for i, _ in O.layer_runs(cfg)] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [t for _, t in O.layer_runs(cfg)] == [None, 0, None, None, 1, None, None, 2, None, None, None]
    shapes = parsed.tensor_shapes()
    assert "l2.mlp.gate" not in shapes and "l2.norm2" not in shapes and "l2.norm1b" in shapes
    assert shapes["loop.in"] == (112, 224) and shapes["loop.step"] == (3, 112)
    assert shapes["l0.mix.in"] == (2 * 144 + 2 * 120 + 6, 112) and shapes["l0.mix.conv"] == (144 + 240, 4)
    assert parsed.head_dim == 40 and parsed.heads == 8
    cfg.pop("loop")
    assert "loop.in" not in sandwich_model.SandwichConfig.from_json(cfg).tensor_shapes()


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0].update(type="linear"),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
])
def test_unknown_kinds_are_refused(edit):
    cfg = M.full_config()
    edit(cfg)
    with pytest.raises(ValueError):
        sandwich_model.SandwichConfig.from_json(cfg)


def test_registry_picks_the_loader_by_architecture(tmp_path):
    cfg = M.full_config()
    w = M.weights(cfg)
    ck = registry.load_model(M.write_folder(tmp_path / "m", cfg, w))
    assert isinstance(ck.config, sandwich_model.SandwichConfig) and ck.config.name == "m"
    at = 0
    for b, (name, shape) in zip(weight_blocks(ck), ck.config.tensor_shapes().items()):
        assert np.array_equal(synth.bf16_to_f32(ck.tensors[name].read()).reshape(w[name].shape), w[name]), name
        assert b.offset_bytes == at and b.bytes == 2 * int(np.prod(shape)), name
        at += b.bytes


def test_missing_and_misshapen_tensors_are_errors():
    cfg = M.full_config()
    w = M.weights(cfg)
    with pytest.raises(ValueError, match="l1.mix.g"):
        M.checkpoint(cfg, {k: v for k, v in w.items() if k != "l1.mix.g"})
    w["l0.mix.conv"] = w["l0.mix.conv"][:, :-1]
    with pytest.raises(ValueError, match="l0.mix.conv"):
        M.checkpoint(cfg, w)


def test_streamed_bytes_count_every_pass():
    cfg = sandwich_model.SandwichConfig.from_json(M.config([M.attention(), M.space()], loop=(1, 2, 3)))
    size = {n: 2 * int(np.prod(s)) for n, s in cfg.tensor_shapes().items() if len(s) == 2}
    first = sum(v for n, v in size.items() if n.startswith("l0."))
    looped = sum(v for n, v in size.items() if n.startswith("l1.")) + size["loop.in"]
    assert cfg.streamed_bytes_per_token() == first + 3 * looped + size["head"]


def _create(cfg, edit):
    ck = M.checkpoint(cfg, M.weights(cfg))
    native = ck.native_model("bfloat16")
    edit(native, native._keep)
    ck.native_model = lambda compute: native
    return CudaHfDecodeSequenceSession(ck, 64)


def test_inconsistent_models_are_refused_before_any_device_call(built_lib):
    for edit in (lambda m, ls: setattr(m, "block", 2),
                 lambda m, ls: setattr(m, "block", 0),
                 lambda m, ls: setattr(m, "norm", 2),
                 lambda m, ls: setattr(m, "activation", 2),
                 lambda m, ls: setattr(m, "loop_input", 0),      # the descriptors do not match any more
                 lambda m, ls: setattr(m, "loop_stop", 6),
                 lambda m, ls: setattr(ls[0], "mixer", 2),
                 lambda m, ls: setattr(ls[0], "state_groups", 4),
                 lambda m, ls: setattr(ls[0], "norm_groups", 5),
                 lambda m, ls: setattr(ls[0], "state_size", 257),
                 lambda m, ls: setattr(ls[0], "conv_taps", 0),
                 lambda m, ls: setattr(ls[0], "conv_taps", 17),
                 lambda m, ls: setattr(ls[1], "head_gate", 0),
                 lambda m, ls: setattr(ls[1], "layer_scale", 1),
                 lambda m, ls: setattr(ls[1], "score_softcap", -1.0),
                 lambda m, ls: setattr(ls[1], "kv_heads", 3)):
        s = _create(M.full_config(), edit)
        assert s.status != SmokeStatus.OK and s.create_result.failure_stage == INVALID_REQUEST


def test_a_parallel_block_model_refuses_what_it_has_no_kernels_for(built_lib):
    from tests import vuvolix_models as V
    cfg = V.config([V.layer()])
    for field, value in (("norm", 1), ("loop_input", 1)):
        ck = V.checkpoint(cfg, V.weights(cfg))
        native = parallel_model.native_model(ck.config, "bfloat16", **{field: value})
        native.loop_times = 1
        native.loop_stop = 1
        ck.native_model = lambda compute, n=native: n
        assert CudaHfDecodeSequenceSession(ck, 64).create_result.failure_stage == INVALID_REQUEST
    assert ffi.structs["NervaB200ParallelLayer"]().mixer == 0  # zeroed fields describe what there was before


# ---- the oracle ----

def test_the_mask_keeps_first_positions_and_stays_causal():
    m = O.visible(np.arange(8), np.arange(8), 3, 2)
    assert m[7].tolist() == [True, True, False, False, False, True, True, True]
    assert m[0].tolist() == [True] + [False] * 7 and m[3].all() == m[3, 4] and m[3, :4].all()
    assert O.visible(np.arange(8), np.arange(8), 3, 0)[7].sum() == 3
    assert O.visible(np.arange(8), np.arange(8), 0, 0)[7].all()


def test_layer_norm_ignores_an_offset():
    x = np.random.default_rng(0).standard_normal((3, 50))
    w = np.linspace(0.5, 2.0, 50)
    assert np.allclose(O.layer_norm(x + 7.0, 1e-5, w), O.layer_norm(x, 1e-5, w), atol=1e-5)
    assert np.allclose((O.layer_norm(x, 0.0, np.ones(50)) ** 2).mean(axis=1), 1.0, atol=1e-5)


def test_grouped_norm_treats_every_part_alone():
    x = np.random.default_rng(0).standard_normal((2, 24))
    y = O.grouped_rms_norm(x, 3, 0.0, np.ones(24))
    assert np.allclose((y.reshape(2, 3, 8) ** 2).mean(axis=2), 1.0, atol=1e-5)
    x[:, 8:16] *= 100.0
    assert np.allclose(O.grouped_rms_norm(x, 3, 0.0, np.ones(24)), y, atol=1e-5)


def test_convolution_meets_the_current_token_with_its_last_column():
    u = np.zeros((6, 1))
    u[2] = 1.0
    assert O.causal_convolution(u, np.array([[1.0, 2.0, 3.0]]), [0.5])[:, 0].tolist() == [0.5, 0.5, 3.5, 2.5, 1.5, 0.5]


def test_recurrence_equals_its_sum_over_earlier_tokens():
    rng = np.random.default_rng(1)
    x, b, c = rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 1, 4)), rng.standard_normal((9, 1, 4))
    step, rate, skip = rng.uniform(0.1, 1.0, (9, 2)), np.array([0.5, 2.0]), np.array([0.3, -1.0])
    y = O.state_space_scan(x.astype(np.float32), b, c, step, rate, skip)
    total = np.cumsum(step, axis=0)
    for h in range(2):
        for t in range(9):
            want = skip[h] * x[t, h] + sum(np.exp(-rate[h] * (total[t, h] - total[s, h])) * step[s, h] * (b[s, 0] @ c[t, 0])
                                           * x[s, h] for s in range(t + 1))
            assert np.allclose(y[t, h], want, atol=1e-5)


def test_the_oracle_is_causal():
    cfg = M.full_config()
    w = M.weights(cfg)
    t = M.tokens(cfg, 50)
    assert np.abs(O.forward(cfg, w, t)[:30] - O.forward(cfg, w, t[:30])).max() < 1e-4


def _masks(c):
    return [l["mixer"]["mask"] for l in c["layers"] if l["type"] == "attention"]


MISTAKES = {
    "window one larger": lambda c, w: [m.update(size=m["size"] + 1) for m in _masks(c)],
    "window one smaller": lambda c, w: [m.update(size=m["size"] - 1) for m in _masks(c)],
    "one kept position more": lambda c, w: [m.update(keep_first=m["keep_first"] + 1) for m in _masks(c)],
    "no kept positions": lambda c, w: [m.update(keep_first=0) for m in _masks(c)],
    "no score cap": lambda c, w: [l["mixer"].update(softcap=0) for l in c["layers"] if l["type"] == "attention"],
    "gates left out": lambda c, w: [w.update({n: 0 * w[n]}) for n in w if n.endswith("mix.g")],
    "one pass less": lambda c, w: c["loop"].update(times=c["loop"]["times"] - 1),
    "pass vectors swapped": lambda c, w: w.update({"loop.step": w["loop.step"][::-1]}),
    "halves of the join swapped": lambda c, w: w.update({"loop.in": np.roll(w["loop.in"], c["width"], axis=1)}),
    "norm behind the mixer left out": lambda c, w: w.update({"l0.norm1b": np.ones_like(w["l0.norm1b"])}),
    "norm behind the feed-forward left out": lambda c, w: w.update({"l0.norm2b": np.ones_like(w["l0.norm2b"])}),
    "convolution reversed": lambda c, w: w.update({"l0.mix.conv": w["l0.mix.conv"][:, ::-1]}),
    "convolution bias left out": lambda c, w: w.update({"l0.mix.conv.b": 0 * w["l0.mix.conv.b"]}),
    "skip left out": lambda c, w: w.update({"l0.mix.D": 0 * w["l0.mix.D"]}),
    "step bias left out": lambda c, w: w.update({"l0.mix.dt_bias": 0 * w["l0.mix.dt_bias"]}),
    "one norm group": lambda c, w: c["layers"][0]["mixer"].update(norm_groups=1),
    "logit scale left out": lambda c, w: c.update(logit_scale=1.0),
}
REPLACED = {
    "rms norm instead of layer norm": ("layer_norm", lambda x, eps, w: O.grouped_rms_norm(x, 1, eps, w)),
    "silu instead of gelu": ("gelu_tanh", lambda z: O.silu(z)),
    "state forgotten": ("state_space_scan", lambda x, b, c, step, rate, skip: (skip[:, None] * x).astype(np.float32)),
}


def _mistaken(change):
    cfg = M.full_config()
    w = M.weights(cfg)
    t = M.tokens(cfg, 90)
    right = O.forward(cfg, w, t)
    cfg2, w2 = copy.deepcopy(cfg), dict(w)
    change(cfg2, w2)
    return M.worst_position(O.forward(cfg2, w2, t), right)


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_mistakes_show_above_the_tolerance(name):
    """Each of these, made in the oracle, moves some position by well more than the GPU tests allow."""
    assert _mistaken(MISTAKES[name]) > 3 * M.TOLERANCE["bfloat16"]


@pytest.mark.parametrize("name", sorted(REPLACED))
def test_replaced_mechanisms_show_above_the_tolerance(name, monkeypatch):
    attribute, other = REPLACED[name]
    assert _mistaken(lambda c, w: monkeypatch.setattr(O, attribute, other)) > 3 * M.TOLERANCE["bfloat16"]


@pytest.mark.parametrize("window,keep", [(1, 0), (2, 3), (16, 1), (17, 16), (50, 20)])
def test_a_marked_key_decides_at_the_edges(window, keep):
    """The marker model: the query sees the key at distance window - 1 and not at distance window, and the last kept
    position but not the next one."""
    cfg, w = M.marked_model(window, keep)
    at = 90

    def last(key_at):
        return O.forward(cfg, w, M.marked_tokens(cfg, at + 1, key_at, at))[-1]

    unseen = last(None)
    assert M.distance(last(at - window), unseen) < 0.2
    assert M.distance(last(keep), unseen) < 0.2
    if window > 1:
        assert M.distance(last(at - window + 1), unseen) > 0.3
    if keep:
        assert M.distance(last(keep - 1), unseen) > 0.3


def test_the_first_token_is_remembered():
    cfg, w = M.remembering_model()
    t = M.tokens(cfg, 300)
    t[0] = M.KEY
    other = [5] + t[1:]
    assert M.distance(O.forward(cfg, w, t)[-1], O.forward(cfg, w, other)[-1]) > 5 * M.TOLERANCE["bfloat16"]
