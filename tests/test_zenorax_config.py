"""The Zenorax configuration without a GPU: reading config.json, the registry, the declared tensors, the constants
the specs carry, what a file may leave out, refusals, random weights, the frequencies of stretched rotations, the
cache's storage (a block's own state beside its mixer's), and the plain model's own mechanisms."""
import copy
import json

import numpy as np
import pytest
import torch

from tests.plain import zenorax_plain as P
from tests.test_gpu_zenorax import CONFIGS, RAMP


def test_the_registry_finds_the_design_by_its_name(tmp_path):
    from gophonic_b200 import registry
    from gophonic_b200.config import ZenoraxConfig
    cfg = CONFIGS["mix"]
    assert registry.architecture_of(cfg) == "Zenorax"
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    read = registry.read_config(str(tmp_path))
    assert isinstance(read, ZenoraxConfig) and read.num_layers == len(cfg["layers"])
    assert read.to_dict() == cfg                                       # nothing lost, nothing added
    assert ZenoraxConfig.from_dict(read.to_dict()) == read
    assert read.with_layers(3).to_dict()["layers"] == cfg["layers"][:3]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    from gophonic_b200.config import ZenoraxConfig
    from gophonic_b200.weights import declare_model
    cfg = CONFIGS[name]
    decls = declare_model(ZenoraxConfig.from_dict(cfg).model_spec())
    assert {d.name: tuple(d.shape) for d in decls if not d.optional} == P.tensor_shapes(cfg)
    assert [d.name for d in decls if d.optional] == ["head"]          # the head is the embedding table


def test_the_spec_carries_the_designs_constants():
    from gophonic_b200.config import LinearStretch, RampStretch, ZenoraxConfig
    spec = ZenoraxConfig.from_dict(CONFIGS["mix"]).model_spec()
    assert spec.head.tied_to == "embed" and spec.head.soft_cap == 20.0 and spec.embedding.scale == 0.7
    assert [l.average for l in spec.layers] == [2, 3, 4, 5, 6, 7] and all(l.block == "sandwich" and l.conv_taps == 4 for l in spec.layers)
    a = spec.layers[0].mixer
    assert a.kind == "gated_attention" and (a.heads, a.kv_heads, a.head_dim, a.value_dim, a.scale) == (4, 2, 16, 16, 0.3)
    assert a.value_from_key and a.sink_learned and not a.qk_norm_weight and a.qk_norm_after and a.qk_norm.eps == 1e-5 and a.window == 0
    assert a.position.kind == "rope" and (a.position.rotary_dim, a.position.theta, a.position.scaling) == (8, 100.0, LinearStretch(2.5))
    h = spec.layers[1].mixer
    assert h.kind == "hgrn2" and (h.heads, h.key_dim, h.value_dim, h.eps) == (2, 24, 40, 1e-5)
    b = spec.layers[2].mixer
    assert b.kind == "latent_attention" and b.gate and (b.heads, b.head_dim, b.rot_dim, b.value_dim, b.q_rank, b.kv_rank) == (2, 24, 16, 8, 24, 48)
    assert b.position.kind == "rope_pairs" and b.position.scaling == RampStretch(**RAMP)
    f = spec.layers[1].feed_forward
    assert f.kind == "moe" and (f.experts, f.top, f.intermediate, f.act, f.groups, f.keep_groups) == (9, 2, 24, "relu2", 3, 1)
    assert (f.score, f.renorm, f.weight_on, f.correction, f.router_bias, f.shared) == ("sigmoid", False, "output", True, False, None)
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None


def test_what_a_file_leaves_out_is_not_there():
    from gophonic_b200.config import ZenoraxConfig
    cfg = ZenoraxConfig.from_dict(CONFIGS["odd"])
    spec = cfg.model_spec()
    bare = spec.layers[0].mixer
    assert (bare.kv_heads, bare.value_dim) == (3, 12) and bare.position.kind == "none"
    assert cfg.logit_softcap is None and spec.head.soft_cap == 0.0
    assert spec.layers[1].mixer.position.kind == "none" and spec.layers[3].mixer.position.scaling is None
    assert (spec.layers[0].feed_forward.groups, spec.layers[0].feed_forward.keep_groups) == (1, 1)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="gla"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=24), "vdim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=4), "can be chosen"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=2), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c["norm"].update(eps=0), "eps"),
])
def test_a_wrong_file_is_refused(change, message):
    from gophonic_b200.config import ConfigError, ZenoraxConfig
    cfg = copy.deepcopy(CONFIGS["mix"])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        ZenoraxConfig.from_dict(cfg)


def test_a_norm_behind_the_rotation_is_built_only_where_the_orders_agree():
    from dataclasses import replace
    from types import SimpleNamespace
    from gophonic_b200.config import RampStretch, ZenoraxConfig
    from gophonic_b200.parts.gated_attention import GatedAttention
    spec = ZenoraxConfig.from_dict(CONFIGS["attention"]).model_spec().layers[0].mixer
    tensors = {d.name: torch.zeros(d.shape) for d in GatedAttention.declare(spec, "")}
    assert sorted(tensors) == ["k", "o", "q", "sink"]                  # no value projection, no norm weights
    rt = SimpleNamespace(device="cpu", act_dtype=torch.float32, is_fp32=True)
    part = GatedAttention(spec, "", tensors, rt)
    assert part.qkv.shape[0] == (4 + 2) * 16 and float(part.q_norm.min()) == 1.0
    longer = replace(spec, position=replace(spec.position, scaling=RampStretch(4.0, 64.0, 8.0, 1.0)))     # a rotation that stretches heads
    with pytest.raises(ValueError, match="length"):
        GatedAttention(longer, "", tensors, rt)
    with pytest.raises(ValueError, match="values"):
        GatedAttention(replace(spec, value_dim=8), "", tensors, rt)


def test_random_weights_write_a_model_the_plain_reader_takes(tmp_path):
    from gophonic_b200.config import ZenoraxConfig
    from gophonic_b200.weights import write_random_model
    cfg = CONFIGS["mix"]
    d = write_random_model(ZenoraxConfig.from_dict(cfg), seed=1, out_dir=str(tmp_path / "m"))
    read, w = P.read_model(d)
    assert {n: tuple(a.shape) for n, a in w.items()} == P.tensor_shapes(cfg)
    assert abs(w["l0.norm1b"] - 1).max() < 0.5 and abs(w["l5.dwa"] - 1).max() < 0.5 and abs(w["l1.mix.lower"]).max() < 0.5
    assert np.isfinite(P.forward(read, w, [1, 2, 3])).all()


def test_stretched_frequencies_against_the_plain_ones():
    from gophonic_b200.config import LinearStretch, RampStretch
    from gophonic_b200.parts.rope import scaled_frequencies, scaled_magnitude
    for dims, base, sc in ((8, 1000.0, RAMP), (64, 10000.0, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (2, 10.0, RAMP), (16, 50.0, {"factor": 3.0, "original": 8, "fast": 30.0, "slow": 20.0})):
        plain = P.frequencies(dims, base)
        want, mag = P.ramp_frequencies(dims, base, sc)
        stretch = RampStretch(**sc)
        assert np.allclose(scaled_frequencies(plain.copy(), stretch, base), want, rtol=1e-14, atol=0)
        assert abs(scaled_magnitude(stretch) - mag) < 1e-15
        assert np.allclose(scaled_frequencies(plain.copy(), LinearStretch(7.0), base), P.linear_frequencies(dims, base, {"factor": 7.0}), rtol=1e-15)
    f, p = P.ramp_frequencies(64, 10000.0, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0})[0], P.frequencies(64, 10000.0)
    assert (f == p).any() and np.isclose(f, p / 40.0).any() and ((f < p * 0.999) & (f > p / 40.0 * 1.001)).any()     # all three ranges occur
    assert scaled_magnitude(None) == scaled_magnitude(LinearStretch(4.0)) == 1.0


def test_the_cache_keeps_a_blocks_state_beside_its_mixers():
    from gophonic_b200.cache import Cache, CacheError
    from gophonic_b200.config import ZenoraxConfig
    from gophonic_b200 import parts, registry  # noqa: F401
    spec = ZenoraxConfig.from_dict(CONFIGS["mix"]).model_spec()
    reqs = [(registry.part_class("block", spec.layers[e.layer].block).cache_request(spec.layers[e.layer]), e.cache_of) for e in spec.schedule]
    cache = Cache(reqs, max_tokens=256, device="cpu", dtype=torch.bfloat16, max_slots=2)
    a, h, l = (cache.view(i) for i in range(3))
    assert tuple(a.mixer.k.shape[1:]) == tuple(a.mixer.v.shape[1:]) == (2, 64, 16)
    assert tuple(h.mixer.state.shape[1:]) == (2, 24 * 40) and h.mixer.state.dtype == torch.float32
    assert tuple(l.mixer.k.shape[1:]) == (1, 64, 64) and l.mixer.v.data_ptr() == l.mixer.k.data_ptr()
    views = [cache.view(i) for i in range(6)]
    assert all(tuple(v.state.shape[1:]) == (3 * 64,) and v.state.dtype == torch.float32 and v.writable for v in views)
    assert len({v.state.data_ptr() for v in views}) == 6               # a layer's own, none shared
    slot = cache.alloc_slot()
    for v in views:
        v.state[slot] = 1.0
    h.mixer.state[slot] = 2.0
    mark = cache.snapshot(slot)
    for v in views:
        v.state[slot] = 5.0
    h.mixer.state[slot] = 5.0
    cache.restore(slot, mark)
    assert all(float(v.state[slot].max()) == 1.0 for v in views) and float(h.mixer.state[slot].max()) == 2.0
    cache.free_slot(slot)
    assert cache.alloc_slot() == slot and all(float(v.state[slot].abs().max()) == 0.0 for v in views)     # a slot starts from zero again
    with pytest.raises(CacheError, match="block"):
        Cache([reqs[0], (reqs[0][0], 0)], max_tokens=64, device="cpu", dtype=torch.float32)
    odd = ZenoraxConfig.from_dict(CONFIGS["odd"]).model_spec()          # one tap: nothing to keep
    assert registry.part_class("block", "sandwich").cache_request(odd.layers[2]).shape == (1, 15)


def test_the_plain_convolution_and_average():
    h = np.array([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]])
    w = np.array([[0.5, 0.25, 1.0], [0.0, 1.0, 0.0]])
    assert np.allclose(P.input_convolution(h, w), [[2.0, 10.0], [4.25, 30.0], [9.0, 60.0]])
    assert np.allclose(P.depth_average([h, 2 * h, -h], [1.0, 0.5, 3.0]), -h)


def test_the_plain_choice_of_experts():
    """Groups by their two largest choice scores, among them the largest choice scores; negative ones count as they are."""
    w = {"router": np.eye(4) * 0.0, "correction": np.array([-0.6, -0.9, -0.5, -1.4])}
    index, weight = P.route(np.ones((1, 4)), w, "", {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert index.tolist() == [[0, 1]] and np.allclose(weight, 0.5)      # the best expert's group (2, 3) is the weaker one
    index, _ = P.route(np.ones((1, 4)), w, "", {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 2}})
    assert index.tolist() == [[2, 0]]


def test_the_plain_state_by_hand():
    cfg = CONFIGS["hgrn2"]
    w = P.random_weights(cfg, 3)
    m = cfg["layers"][0]["mixer"]
    h = np.random.default_rng(0).standard_normal((2, cfg["width"]))
    p, d, dv, H = "l0.mix.", m["dim"], m["vdim"], m["heads"]
    f = w[p + "lower"] + (1 - w[p + "lower"]) / (1 + np.exp(-(h @ w[p + "f"].T + w[p + "f.b"])))
    v, q = h @ w[p + "v"].T, h @ w[p + "q"].T
    q = q / (1 + np.exp(-q))
    heads = []
    for k in range(H):
        fs, vs, qs = f[:, k * d:(k + 1) * d], v[:, k * dv:(k + 1) * dv], q[:, k * d:(k + 1) * d]
        S = np.outer(1 - fs[0], vs[0]) * fs[1][:, None] + np.outer(1 - fs[1], vs[1])
        o = S.T @ qs[1]
        heads.append(o / np.sqrt((o * o).mean() + 1e-5) * w[p + "norm"])
    assert np.allclose(P.hgrn2(h, w, p, m, 1e-5)[1], w[p + "o"] @ np.concatenate(heads))
