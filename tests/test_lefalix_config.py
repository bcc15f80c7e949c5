"""The Lefalix configuration, its tensors, its cache and the plain implementation's functions, without a GPU."""
import copy
import math

import numpy as np
import pytest
import torch

from tests.plain import lefalix_plain as P
from tests.test_gpu_lefalix import CONFIGS, attention, config, delta, moe, pair, part


def read(cfg):
    from gophonic_b200 import registry
    return registry.config_class(registry.architecture_of(cfg)).from_dict(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_registry_reads_a_file_and_declares_its_tensors(name):
    from gophonic_b200.config import LefalixConfig
    from gophonic_b200.weights import declare_model
    cfg = CONFIGS[name]
    c = read(cfg)
    assert isinstance(c, LefalixConfig) and c.to_dict() == {k: v for k, v in cfg.items()} and c.num_layers == len(cfg["layers"])
    want = P.tensor_shapes(cfg)
    got = {d.name: d.shape for d in declare_model(c.model_spec())}
    assert set(got) == set(want)
    for n, shape in got.items():      # the ranks are left to the checkpoint
        assert len(shape) == len(want[n]) and all(a is None or a == b for a, b in zip(shape, want[n])), n
    assert {n.rsplit(".", 1)[-1] for n, s in got.items() if None in s} <= {"a1", "a2", "g1", "g2"}


def test_the_constants_travel_in_the_specs():
    c = read(CONFIGS["mix"])
    spec = c.model_spec()
    assert spec.head.tied_to is None and spec.embedding.scale == 1.0 and spec.head.soft_cap == 0.0
    both, ff = spec.layers[0].mixer, spec.layers[0].feed_forward
    left, right = both.mixers
    assert both.factor == 0.5 and both.eps == 1e-5 and both.prefixes == ("left.", "right.")
    assert left.bias and left.out_bias and left.sink_learned and left.qk_norm_after and not left.qk_norm_weight and not left.gate
    assert (left.window, left.conv_taps, left.position.kind, left.position.scaling.factor) == (33, 3, "rope_pairs", 3.0)
    assert not right.channel_decay and right.gate == "silu" and not right.gate_low_rank and right.unit_eps == 1e-6 and right.conv_taps == 2
    assert ff.score == "softmax" and not ff.renorm and ff.act == "swiglu" and ff.group_rank == "largest" and (ff.groups, ff.keep_groups) == (3, 2)
    other = spec.layers[1].mixer
    assert other.channel_decay and other.gate == "sigmoid" and other.gate_low_rank and other.rank is None and (other.heads, other.kv_heads) == (6, 3)
    assert spec.layers[3].feed_forward.kind == "gelu_ff" and spec.layers[2].feed_forward is None and spec.layers[2].feed_forward_norm is None


def test_repeated_layers_in_the_schedule():
    c = read(CONFIGS["mix"])
    runs = [(e.layer, e.enter is not None) for e in c.schedule()]
    assert runs == P.layer_runs(CONFIGS["mix"]) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    assert all(e.cache_of is None for e in c.schedule())          # every pass keeps its own keys and states
    assert [e.layer for e in c.with_layers(2).schedule()] == [0, 1, 1, 1]
    assert [e.layer for e in c.with_layers(1).schedule()] == [0]
    assert all(e.enter is None for e in read(CONFIGS["odd"]).schedule())


def test_what_a_file_leaves_out():
    c = read(config([pair({"heads": 3, "dim": 8, "vdim": 4, "scale": 1, "mask": None}, {"heads": 2, "dim": 4, "vdim": 6}),
                     delta(mlp=moe(4, 2, 8, None))]))
    left, right = c.model_spec().layers[0].mixer.mixers
    assert (left.kv_heads, left.window, left.conv_taps, left.position.kind) == (3, 0, 0, "none") and (right.kv_heads, right.conv_taps) == (2, 0)
    ff = c.model_spec().layers[1].feed_forward
    assert (ff.groups, ff.keep_groups) == (1, 1)


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].update(heads=7), "heads"),
    (lambda c: c["layers"][1]["mixer"].update(conv=-1), "conv"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=4), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5), "keep"),
    (lambda c: c["layers"][3]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
])
def test_a_wrong_file_is_refused(change, message):
    from gophonic_b200.config import ConfigError
    cfg = copy.deepcopy(CONFIGS["mix"])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        read(cfg)


def test_random_weights_need_the_ranks_and_write_a_model_the_plain_reader_takes(tmp_path):
    from gophonic_b200.weights import write_random_model
    with pytest.raises(ValueError, match="a1"):
        write_random_model(read(CONFIGS["delta"]), seed=1, out_dir=str(tmp_path / "no"))
    cfg = copy.deepcopy(CONFIGS["loop"])
    for L in cfg["layers"]:
        L["mixer"].update(rank=6, gate_rank=9)
    d = write_random_model(read(cfg), seed=1, out_dir=str(tmp_path / "m"))
    back, w = P.read_model(d)
    assert {n: tuple(a.shape) for n, a in w.items()} == P.tensor_shapes(cfg, 6, 9)
    assert np.isfinite(P.forward(back, w, [1, 2, 3])).all()


def _cache(cfg, **kw):
    from gophonic_b200 import parts, registry  # noqa: F401
    from gophonic_b200.cache import Cache
    spec = read(cfg).model_spec()
    reqs = [(registry.part_class("block", spec.layers[e.layer].block).cache_request(spec.layers[e.layer]), e.cache_of) for e in spec.schedule]
    return Cache(reqs, 512, "cpu", torch.float32, **kw)


def test_the_pieces_of_a_mixer_in_the_cache():
    cache = _cache(CONFIGS["mix"], max_slots=3)
    left, right = cache.view(0).parts
    assert left.k.shape[1:] == (2, 64, 16) and left.v.shape[1:] == (2, 64, 24) and left.state.shape == (4, 2 * (4 * 16 + 2 * 16 + 2 * 24))
    matrix, rows = right.parts
    assert matrix.state.shape == (4, 3, 12 * 20) and rows.state.shape == (4, 1 * (2 * 3 * 12 + 3 * 20))
    matrix, rows = cache.view(1).parts
    assert matrix.state.shape == (4, 6, 24 * 8) and rows.state.shape == (4, 1 * (2 * 3 * 24 + 6 * 8))
    # the passes of a repeated layer share nothing
    states = [cache.view(pos).parts[0].state for pos in (1, 3, 5)]
    assert len({s.data_ptr() for s in states}) == 3
    keys = [cache.view(pos).parts[0].k for pos in (2, 4, 6)]
    assert len({k.data_ptr() for k in keys}) == 3
    # taps of one, and no convolution, keep no rows
    odd = _cache(CONFIGS["odd"], max_slots=2)
    assert odd.view(0).parts[0].state is None and odd.view(0).parts[1].parts[1] is None and odd.view(1).parts[1] is None
    assert odd.view(3).parts[1].state.shape[1] == 4 * (2 * 7 * 20 + 7 * 33)
    groups = {tuple(g["shape"]) for g in cache.groups() if g["kind"] == "state"}
    assert (6, 24 * 8) in groups and cache.has_state()


def test_slots_and_marks_of_pieces():
    cache = _cache(CONFIGS["mix"], max_slots=2)
    slot = cache.alloc_slot()
    matrix, rows = cache.view(0).parts[1].parts
    matrix.state[slot] = 3.0
    rows.state[slot] = 4.0
    cache.view(0).parts[0].state[slot] = 5.0
    cache.reserve([(slot, 5)])
    cache.commit([(slot, 5)])
    mark = cache.snapshot(slot)
    matrix.state[slot] = -1.0
    cache.view(0).parts[0].state[slot] = -1.0
    cache.restore(slot, mark)
    assert (matrix.state[slot] == 3.0).all() and (cache.view(0).parts[0].state[slot] == 5.0).all() and cache.length(slot) == 5
    cache.free_slot(slot)
    assert cache.alloc_slot() == slot
    for t in (matrix.state, rows.state, cache.view(0).parts[0].state):
        assert (t[slot] == 0.0).all()
    cache.check()


def test_pieces_read_no_other_runs_cache():
    from gophonic_b200.cache import Cache, CacheError
    from gophonic_b200.parts import PartsRequest, StateRequest
    req = PartsRequest((StateRequest((2, 3)), None, PartsRequest((StateRequest((4,)),))))
    cache = Cache([(req, None), (None, None)], 64, "cpu", torch.float32)
    view = cache.view(0)
    assert view.parts[0].state.shape[1:] == (2, 3) and view.parts[1] is None and view.parts[2].parts[0].state.shape[1:] == (4,)
    with pytest.raises(CacheError, match="pieces"):
        Cache([(req, None), (req, 0)], 64, "cpu", torch.float32)


def test_junctions_go_with_the_blocks_that_take_them():
    from types import SimpleNamespace
    from gophonic_b200.config import AddStartSpec
    from gophonic_b200.parts import AddStart
    n, weights = AddStart(AddStartSpec(hidden=4), "", {}, SimpleNamespace(device="cpu")).over_planes()
    assert n == 1 and weights.tolist() == [1.0, 1.0]


# ---- the plain implementation by hand ----------------------------------------------------------
def test_plain_convolution_reaches_back_and_no_further():
    u = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    w = np.array([[1.0, 0.0, 2.0], [0.0, 3.0, 0.0]])
    assert P.convolution(u, w)[:, 0].tolist() == [2.0, 4.0, 7.0, 10.0, 13.0] and P.convolution(u, w)[:, 1].tolist() == [0.0, 30.0, 60.0, 90.0, 120.0]


def test_plain_delta_rule_writes_what_is_missing():
    k = np.array([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]])
    v = np.array([[[2.0]], [[6.0]], [[5.0]]])
    g = np.array([[[0.5, 0.5]], [[0.5, 1.0]], [[0.5, 1.0]]])
    beta = np.array([[1.0], [0.5], [1.0]])
    o = P.delta_recurrence(k, k, v, g, beta)[:, 0, 0]
    # 2; then the held 1 (decayed) goes half of the way to 6; then a key of its own
    assert np.allclose(o, [2.0, 3.5, 5.0])


def test_plain_window_and_sink():
    q = k = np.zeros((4, 2))
    v = np.eye(4)
    out = P.windowed_attention(q, k, v, 1.0, 2, 0.0)
    assert np.allclose(out[0], [0.5, 0, 0, 0]) and np.allclose(out[3], [0, 0, 1 / 3, 1 / 3])
    assert np.allclose(P.windowed_attention(q, k, v, 1.0, None, -50.0)[3], 0.25)


def test_plain_norm_stands_behind_the_rotation():
    f, mag = P.frequencies(4, 100.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    assert math.isclose(mag, 0.1 * math.log(4.0) + 1.0)
    x = np.random.default_rng(0).standard_normal((5, 1, 8))
    y = P.unit_rms(P.rotate_pairs(x, f, mag), 1e-9)
    assert np.allclose((y * y).mean(-1), 1.0) and not np.allclose(y, P.rotate_pairs(P.unit_rms(x, 1e-9), f, mag))


def test_plain_route_counts_a_group_as_its_largest():
    h = np.eye(1)
    w = {"router": np.array([[3.0], [-9.0], [2.9], [2.8]])}
    index, weight = P.route(h, w, "", {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})
    e = np.exp([3.0, -9.0, 2.9, 2.8])
    assert index.tolist() == [[0, 1]] and np.allclose(weight, [[e[0] / e.sum(), e[1] / e.sum()]])


def test_plain_gelu():
    assert np.allclose(P.gelu(np.array([0.0, 1.0, -1.0])), [0.0, 0.8413447460685429, -0.15865525393145707])
