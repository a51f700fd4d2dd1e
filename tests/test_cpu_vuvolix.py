"""Vuvolix without a GPU: configuration and weight loading, requests the library refuses, and the
oracle itself (that it notices the mistakes the GPU tests are there to find)."""
import copy
import ctypes as C
import json

import numpy as np
import pytest

from nerva_b200 import ffi, parallel_model, registry, safetensors_file, synth
from nerva_b200.session import CudaHfDecodeSequenceSession, SmokeStatus, weight_blocks
from tests import vuvolix_models as M
from tests import vuvolix_oracle as O

INVALID_REQUEST = 1  # failure stage


def test_configuration_round_trip_and_layer_runs():
    cfg = M.full_config()
    parsed = parallel_model.ParallelConfig.from_json(cfg)
    again = parallel_model.ParallelConfig.from_json(json.loads(parallel_model.dump_config(parsed)))
    assert again == parsed
    assert parsed.layers == 4 and parsed.layer_runs == 8 == len(O.layer_runs(cfg))
    assert [i for i, _ in O.layer_runs(cfg)] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [t for _, t in O.layer_runs(cfg)] == [None, 0, None, 1, None, 2, None, None]
    assert parsed.layer_specs[2].intermediate == 0 and "l2.mlp.gate" not in parsed.tensor_shapes()
    assert "l2.ls2" not in parsed.tensor_shapes() and parsed.tensor_shapes()["loop.step"] == (3, 128)


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0].update(type="recurrent"),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
])
def test_unknown_kinds_are_refused(edit):
    cfg = M.full_config()
    edit(cfg)
    with pytest.raises(ValueError):
        parallel_model.ParallelConfig.from_json(cfg)


def test_registry_picks_the_loader_by_architecture(tmp_path):
    cfg = M.full_config()
    w = M.weights(cfg)
    ck = registry.load_model(M.write_folder(tmp_path / "m", cfg, w))
    assert isinstance(ck, parallel_model.ParallelCheckpoint) and ck.config.name == "m"
    for name, t in ck.tensors.items():
        assert np.array_equal(synth.bf16_to_f32(t.read()).reshape(w[name].shape), w[name]), name
    cfg["architecture"] = "Unheard"
    with pytest.raises(ValueError, match="Unheard"):
        registry.load_model(M.write_folder(tmp_path / "u", cfg, w))


def test_weights_become_contiguous_file_ranges(tmp_path):
    cfg = M.full_config()
    ck = registry.load_model(M.write_folder(tmp_path / "m", cfg, M.weights(cfg)))
    blocks = weight_blocks(ck)
    at = 0
    for b, (name, shape) in zip(blocks, ck.config.tensor_shapes().items()):
        assert b.offset_bytes == at and b.bytes == 2 * int(np.prod(shape)), name
        assert b.source_file_len == len(str(tmp_path / "m" / "model.safetensors")) and not b.host_source
        at += b.bytes


def test_missing_and_misshapen_tensors_are_errors(tmp_path):
    cfg = M.full_config()
    w = M.weights(cfg)
    short = {k: v for k, v in w.items() if k != "l1.mix.v"}
    with pytest.raises(ValueError, match="l1.mix.v"):
        M.checkpoint(cfg, short)
    w["l0.ls1"] = w["l0.ls1"][:-1]
    with pytest.raises(ValueError, match="l0.ls1"):
        M.checkpoint(cfg, w)
    path = str(tmp_path / "t.safetensors")
    safetensors_file.write_tensors(path, {"a": np.zeros((3, 5), dtype=np.uint16)})
    with open(path, "r+b") as f:
        f.truncate(40)
    with pytest.raises(ValueError):
        safetensors_file.open_tensors(path)


def _create(cfg, edit=None):
    ck = M.checkpoint(cfg, M.weights(cfg))
    native = ck.native_model("bfloat16")
    if edit is not None:
        edit(native, native._keep)
    ck.native_model = lambda compute: native
    return CudaHfDecodeSequenceSession(ck, 64)


def test_inconsistent_models_are_refused_before_any_device_call(built_lib):
    cfg = M.full_config()
    for edit in (lambda m, ls: setattr(m, "loop_stop", 9),
                 lambda m, ls: setattr(m, "compute", 0),
                 lambda m, ls: setattr(ls[0], "kv_heads", 3),
                 lambda m, ls: setattr(ls[0], "rotary_dims", 15),
                 lambda m, ls: setattr(ls[1], "rotary_dims", 64),
                 lambda m, ls: setattr(ls[1], "qk_dim", 300),
                 lambda m, ls: setattr(ls[2], "intermediate", 64)):  # the descriptors do not match any more
        s = _create(cfg, edit)
        assert s.status != SmokeStatus.OK and s.create_result.failure_stage == INVALID_REQUEST
    r = ffi.CreateResult()
    h = C.c_void_p()
    assert ffi.lib().nerva_b200_session_create_parallel(None, None, C.byref(r), C.byref(h)) == -1


def test_append_checks_its_arguments_first(built_lib):
    fn = ffi.lib().nerva_b200_session_append
    ids = np.zeros(2, dtype=np.uint32)
    assert fn(None, ids.ctypes.data, 2, 0, None, 0, None) == -1


def test_float32_is_refused_for_models_that_have_no_fp32_form(built_lib, tiny_checkpoint):
    with pytest.raises(ValueError, match="bfloat16 only"):
        CudaHfDecodeSequenceSession(tiny_checkpoint, 32, compute="float32")


# ---- the oracle ----

def test_rotation_preserves_length_and_depends_on_distance_only():
    freq, magnitude = O.rotary_frequencies(16, 10000.0)
    assert magnitude == 1.0 and freq[0] == 1.0
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 1, 24)).astype(np.float32)
    dots = []
    for shift in (0, 5, 90):
        a = O.rotate(q, [7 + shift], freq, magnitude)
        b = O.rotate(k, [2 + shift], freq, magnitude)
        assert np.allclose(np.linalg.norm(a), np.linalg.norm(q), rtol=1e-5)
        assert np.array_equal(a[..., 16:], q[..., 16:])
        dots.append(float((a * b).sum()))
    assert np.allclose(dots, dots[0], atol=1e-4)


def test_scaled_frequencies_lie_between_plain_and_divided():
    plain, _ = O.rotary_frequencies(32, 10000.0)
    scaled, magnitude = O.rotary_frequencies(32, 10000.0, {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0})
    assert magnitude == pytest.approx(0.1 * np.log(4.0) + 1.0)
    ratio = scaled / plain
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(0.25) and (np.diff(ratio) <= 1e-6).all()


def test_window_mask_counts_the_query_itself():
    m = O.visible(np.arange(6), np.arange(6), 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5


def test_the_oracle_is_causal():
    cfg = M.full_config()
    w = M.weights(cfg)
    t = M.tokens(cfg, 50)
    assert np.abs(O.forward(cfg, w, t)[:30] - O.forward(cfg, w, t[:30])).max() < 1e-4


MISTAKES = {
    "window one larger": lambda c, w: [l["mixer"]["mask"].update(size=l["mixer"]["mask"]["size"] + 1) for l in c["layers"]],
    "window one smaller": lambda c, w: [l["mixer"]["mask"].update(size=l["mixer"]["mask"]["size"] - 1) for l in c["layers"]],
    "no frequency scaling": lambda c, w: c["layers"][0]["mixer"]["rot"].pop("scaling"),
    "rotation over the whole head": lambda c, w: c["layers"][0]["mixer"]["rot"].update(dims=c["layers"][0]["mixer"]["dim"]),
    "one pass less": lambda c, w: c["loop"].update(times=c["loop"]["times"] - 1),
    "pass vectors swapped": lambda c, w: w.update({"loop.step": w["loop.step"][::-1]}),
    "pass vectors left out": lambda c, w: w.update({"loop.step": w["loop.step"] * 0}),
    "mixer scale left out": lambda c, w: w.update({"l0.ls1": np.ones_like(w["l0.ls1"])}),
    "feed-forward scale left out": lambda c, w: w.update({"l0.ls2": np.ones_like(w["l0.ls2"])}),
    "no soft cap": lambda c, w: c.pop("logit_softcap"),
    "embedding scale left out": lambda c, w: c["embedding"].update(scale=1.0),
}


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_mistakes_show_above_the_tolerance(name):
    """Each of these, made in the oracle, moves some position by well more than the GPU tests allow."""
    cfg = M.full_config()
    w = M.weights(cfg)
    t = M.tokens(cfg, 90)
    right = O.forward(cfg, w, t)
    cfg2, w2 = copy.deepcopy(cfg), dict(w)
    MISTAKES[name](cfg2, w2)
    assert M.worst_position(O.forward(cfg2, w2, t), right) > 3 * M.TOLERANCE["bfloat16"]


@pytest.mark.parametrize("window", [1, 2, 16, 17, 50])
def test_a_marked_key_decides_at_the_window_edge(window):
    """The marker model: the query sees the key at distance window - 1 and not at distance window."""
    cfg, w = M.marked_model(window)
    at = 60

    def last(distance):
        key_at = at - distance
        t = M.marked_tokens(cfg, at + 1, key_at, at) if distance else M.marked_tokens(cfg, at + 1, 3, at)
        return O.forward(cfg, w, t)[-1]

    outside = last(window)
    if window > 1:
        assert M.distance(last(window - 1), outside) > 0.3
        assert M.distance(last(1), last(window - 1)) < 0.3
    assert M.distance(last(window + 3), outside) < 0.2
