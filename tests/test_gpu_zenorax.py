"""The Zenorax design on the GPU against the plain implementation (tests/plain/zenorax_plain.py): each mechanism
alone, whole prompts against token-by-token decoding, prompts in portions down to two tokens, batches of unequal
requests, slots and pages that are used again, keys and tokens far back, page borders, the first tokens, long decoding,
odd sizes, the kernels by themselves, and greedy generation through the entry point.  Every model here is made by
the test (its own sizes, random weights that bfloat16 holds exactly)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests.plain import zenorax_plain as P

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

RAMP = {"factor": 4.0, "original": 64, "fast": 6.0, "slow": 0.5}     # kept, blended and divided channels all occur


def moe(experts=8, top=2, ff=24, count=4, keep=2):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if count is not None:
        m["router"]["groups"] = {"count": count, "keep": keep}
    return m


def hgrn2(heads=3, dim=16, vdim=24, mlp=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=40, kv_rank=32, base=1000.0, scale=0.25, scaling=RAMP, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def attention(heads=4, kv_heads=2, dim=16, rot=8, base=100.0, scale=0.5, factor=None, vdim=True, mlp=None):
    m = {"heads": heads, "dim": dim, "scale": scale}
    if vdim:
        m["vdim"] = dim
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if rot is not None:
        m["rot"] = {"dims": rot, "base": base}
        if factor is not None:
            m["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, width=64, vocab=96, emb=0.7, eps=1e-5, taps=4, cap=20.0):
    cfg = {"architecture": "Zenorax", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "embedding": {"scale": emb}}
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


CONFIGS = {
    # each mechanism alone
    "hgrn2": config([hgrn2()]),
    "latent": config([latent()]),
    "attention": config([attention(factor=3.0)]),
    "moe": config([hgrn2(mlp=moe())]),
    # all together, the mixers in another order than the presets' and some layers without a feed-forward
    "mix": config([attention(factor=2.5, scale=0.3, mlp=moe(6, 3, 40, 3, 2)), hgrn2(heads=2, dim=24, vdim=40, mlp=moe(9, 2, 24, 3, 1)),
                   latent(heads=2, dim=24, rot_dim=16, vdim=8, q_rank=24, kv_rank=48, mlp=moe(4, 4, 16, 2, 2)), hgrn2(heads=5, dim=8, vdim=12),
                   attention(heads=6, kv_heads=1, dim=8, rot=4, scale=0.6), latent(mlp=moe(12, 3, 20, 2, 1))]),
    # sizes the tensor-core kernels take in bfloat16
    "tensor": config([hgrn2(heads=2, dim=128, vdim=128, mlp=moe(8, 2, 64, 4, 2)),
                      latent(heads=4, dim=64, rot_dim=32, vdim=64, q_rank=96, kv_rank=128, scale=0.1, mlp=moe(8, 3, 32, 2, 1)),
                      attention(heads=4, kv_heads=2, dim=128, rot=128, scale=0.3, factor=4.0, mlp=moe(4, 1, 32, 2, 1)),
                      attention(heads=4, kv_heads=4, dim=64, rot=64, scale=0.4), hgrn2(heads=1, dim=256, vdim=64)], width=128, vocab=80),
    # what a file may leave out (groups, scaling, rotation, kv_heads, vdim, the cap) and sizes that are odd, equal or 1: one
    # tap, one head, one expert, every expert used, groups of one expert, a width that no vector load fits
    "odd": config([attention(heads=3, kv_heads=None, dim=12, rot=None, vdim=False, mlp=moe(1, 1, 56, None)),
                   latent(heads=1, dim=20, rot_dim=0, vdim=17, q_rank=7, kv_rank=9, scale=1.0, mlp=moe(5, 3, 8, 5, 4)),
                   hgrn2(heads=1, dim=3, vdim=5, mlp=moe(3, 3, 8, 1, 1)), latent(heads=5, dim=6, rot_dim=2, vdim=10, q_rank=48, kv_rank=5, scaling=None),
                   hgrn2(heads=7, dim=20, vdim=33)], width=45, vocab=61, emb=1.0, eps=1e-6, taps=1, cap=None),
    # more taps than a short portion has tokens
    "taps": config([hgrn2(), attention()], taps=7, width=52),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(configuration, weights, folder) by (name, dtype): in bfloat16 the choice of experts is decided by their corrections
    (a near-tie that rounding turns would change every row behind it); the mixture's own tests let the scores choose."""
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        for dtype in ("float32", "bfloat16"):
            w = P.random_weights(cfg, seed=370 + i, decided=dtype == "bfloat16")
            out[name, dtype] = (cfg, w, P.write_model(str(tmp_path_factory.mktemp(f"zenorax_{name}_{dtype}")), cfg, w))
    return out


_engines = {}


def engine_for(models, name, dtype, graphs=True, max_tokens=4096):
    from gophonic_b200.engine.model import Model
    from gophonic_b200.engine.step import Engine
    key = (name, dtype, graphs, max_tokens)
    if key not in _engines:
        _engines[key] = Engine(Model.from_dir(models[name, dtype][2], dtype=dtype), max_tokens=max_tokens, use_graphs=graphs)
    return _engines[key]


def tokens_for(cfg, seed, n):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def feed(engine, tokens, cuts=None):
    """All logits of one sequence fed in portions of the sizes ``cuts`` (the rest in one piece)."""
    slot = engine.new_sequence()
    out, at = [], 0
    for n in list(cuts or []) + [len(tokens)]:
        n = min(n, len(tokens) - at)
        if n <= 0:
            break
        out.append(engine.step([(slot, tokens[at:at + n])], [list(range(n))]).cpu().numpy())
        at += n
    engine.end_sequence(slot)
    engine.check_kernels()
    return np.concatenate(out)


def close(got, want, tol, most=1.0):
    """Every row within ``tol``: a float32 row's largest difference relative to the largest wanted value, a bfloat16 row's (``tol``
    above 1e-3) root mean square relative to the wanted values' own (the norms behind the sublayers carry rounding on at full
    size, so the largest of thousands of differences says little).  With ``most`` < 1 that share of the rows must be, and the
    rest within five times as much: a router may take another expert than the plain model where two choice scores nearly tie."""
    rows = got.shape[0]
    diff, want = (got - want).reshape(rows, -1), want.reshape(rows, -1)
    if tol > 1e-3:
        err = np.sqrt((diff * diff).mean(-1)) / max(1e-3, np.sqrt((want * want).mean()))
        if rows >= 50:         # one row in fifty may be one whose small numbers a norm blows up
            most = min(most, 0.98)
    else:
        err = np.abs(diff).max(-1) / max(1.0, np.abs(want).max())
    if most >= 1.0:
        assert err.max() < tol, f"relative error {err.max():.3e} (tolerance {tol})"
    else:
        assert (err < tol).mean() >= most and err.max() < 5 * tol, f"{(err >= tol).sum()} of {len(err)} rows over {tol}, worst {err.max():.3e}"


TOL = {"float32": 5e-5, "bfloat16": 8e-2}
MOST = {"float32": 1.0, "bfloat16": 0.9}


# ---- each mechanism alone, and all together ---------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_match_the_plain_model(models, name, dtype):
    cfg, w, _ = models[name, dtype]
    toks = tokens_for(cfg, 1, 230)
    close(feed(engine_for(models, name, dtype), toks), P.forward(cfg, w, toks), TOL[dtype])


def test_what_goes_on_behind_every_layer(models):
    """The weighted sums of the results so far, as the block behind reads them."""
    from gophonic_b200.parts.sandwich import SandwichBlock
    cfg, w, _ = models["mix", "float32"]
    eng = engine_for(models, "mix", "float32", graphs=False)
    toks = tokens_for(cfg, 2, 70)
    seen, orig = [], SandwichBlock._open

    def spy(self, batch, planes, pending, state):
        start, x = orig(self, batch, planes, pending, state)
        seen.append(start.cpu().numpy())
        return start, x
    SandwichBlock._open = spy
    try:
        feed(eng, toks)
    finally:
        SandwichBlock._open = orig
    _, layers = P.forward(cfg, w, toks, return_layers=True)
    assert len(seen) == len(cfg["layers"])
    close(seen[0], w["embed"][toks] * cfg["embedding"]["scale"], 1e-6)
    for got, want in zip(seen[1:], layers):
        close(got, want, 2e-5)


# ---- prompts against decoding, portions, batches ----------------------------------------------
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["mix", "odd", "tensor", "taps"])
def test_token_by_token_equals_the_whole_prompt(models, name, graphs):
    cfg, w, _ = models[name, "float32"]
    eng = engine_for(models, name, "float32", graphs=graphs)
    toks = tokens_for(cfg, 3, 90)
    whole = feed(eng, toks)
    single = feed(eng, toks, cuts=[1] * len(toks))
    close(single, whole, 4e-5)
    close(single, P.forward(cfg, w, toks), TOL["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "odd", "tensor", "taps"])
@pytest.mark.parametrize("cuts", [[2] * 40, [3, 64, 1, 2, 61], [63, 1, 1, 64], [130, 2]])
def test_portions_of_a_prompt(models, cuts, dtype, name):
    cfg, w, _ = models[name, dtype]
    eng = engine_for(models, name, dtype)
    toks = tokens_for(cfg, 4, 140)
    got = feed(eng, toks, cuts=cuts)
    close(got, P.forward(cfg, w, toks), TOL[dtype])
    if dtype == "float32":
        close(got, feed(eng, toks), 4e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "tensor", "taps"])
def test_a_batch_of_unequal_requests_equals_each_alone(models, dtype, name):
    cfg, w, _ = models[name, dtype]
    eng = engine_for(models, name, dtype)
    prompts = [tokens_for(cfg, 10 + i, n) for i, n in enumerate([1, 70, 9, 33])]
    more = [tokens_for(cfg, 20 + i, 12) for i in range(4)]
    slots = [eng.new_sequence() for _ in prompts]
    got = [[] for _ in prompts]
    first = eng.step(list(zip(slots, prompts)), [list(range(len(p))) for p in prompts]).cpu().numpy()
    at = 0
    for i, p in enumerate(prompts):
        got[i].append(first[at:at + len(p)])
        at += len(p)
    live = list(range(len(prompts)))
    for t in range(12):
        if t == 5:                      # one request ends early; the others go on
            eng.end_sequence(slots[live.pop(1)])
        logits = eng.step([(slots[i], [more[i][t]]) for i in live]).cpu().numpy()
        for j, i in enumerate(live):
            got[i].append(logits[j:j + 1])
    for i in live:
        eng.end_sequence(slots[i])
    eng.cache.check()
    for i, p in enumerate(prompts):
        n = 12 if i != 1 else 5
        close(np.concatenate(got[i]), P.forward(cfg, w, p + more[i][:n]), TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_sequences_decode_together(models, dtype):
    """More sequences than a few-row step takes (the mixture's other paths, a captured step with filler rows)."""
    cfg, w, _ = models["mix", dtype]
    eng = engine_for(models, "mix", dtype)
    prompts = [tokens_for(cfg, 60 + i, 3 + i % 5) for i in range(21)]
    more = [tokens_for(cfg, 90 + i, 3) for i in range(21)]
    slots = [eng.new_sequence() for _ in prompts]
    eng.step(list(zip(slots, prompts)), [[] for _ in prompts])
    got = [eng.step([(s, [m[t]]) for s, m in zip(slots, more)]).cpu().numpy() for t in range(3)]
    for s in slots:
        eng.end_sequence(s)
    for i, p in enumerate(prompts):
        close(np.stack([g[i] for g in got]), P.forward(cfg, w, p + more[i])[-3:], TOL[dtype])


def test_slots_and_pages_that_are_used_again(models):
    """A sequence that takes over the slot and the pages of one that ended sees nothing of it."""
    cfg, w, _ = models["mix", "float32"]
    eng = engine_for(models, "mix", "float32", max_tokens=256)     # four pages: the second sequence must reuse them
    a, b = tokens_for(cfg, 30, 200), tokens_for(cfg, 31, 130)
    close(feed(eng, a, cuts=[100]), P.forward(cfg, w, a), TOL["float32"])
    assert eng.cache.pages.held() == 0
    close(feed(eng, b, cuts=[64, 1, 1]), P.forward(cfg, w, b), TOL["float32"])
    s1 = eng.new_sequence()
    eng.step([(s1, a[:50])])
    eng.end_sequence(s1)
    s2 = eng.new_sequence()
    assert s2 == s1
    got = eng.step([(s2, b[:2])], [[0, 1]]).cpu().numpy()          # the first tokens of a sequence
    got = np.concatenate([got, eng.step([(s2, b[2:20])], [list(range(18))]).cpu().numpy()])
    eng.end_sequence(s2)
    close(got, P.forward(cfg, w, b[:20]), TOL["float32"])


def test_a_sequence_goes_back_to_a_mark(models):
    """The convolution's rows and the matrix states go back with the keys."""
    cfg, w, _ = models["mix", "float32"]
    eng = engine_for(models, "mix", "float32")
    a, b = tokens_for(cfg, 32, 40), tokens_for(cfg, 33, 9)
    slot = eng.new_sequence()
    eng.step([(slot, a[:30])])
    mark = eng.checkpoint(slot)
    eng.step([(slot, a[30:])])
    eng.restore(slot, mark)
    got = eng.step([(slot, b)], [list(range(9))]).cpu().numpy()
    eng.end_sequence(slot)
    close(got, P.forward(cfg, w, a[:30] + b)[30:], TOL["float32"])


@pytest.mark.parametrize("name", ["mix", "tensor", "odd"])
def test_long_decoding_past_pages(models, name):
    for dtype in ("float32", "bfloat16"):
        cfg, w, _ = models[name, dtype]
        toks = tokens_for(cfg, 5, 40 + 230)
        got = feed(engine_for(models, name, dtype), toks, cuts=[40] + [1] * 230)
        close(got, P.forward(cfg, w, toks), TOL[dtype])


# ---- one token far back, through a whole model ---------------------------------------------------
def _standout(tmp_path, kind):
    """One layer whose attention picks out one key.  Every embedding row carries the same large share along one
    direction a, from which the query path makes queries along a fixed direction u (so every row asks for u);
    the token ``mark`` has an embedding that the key path turns into a key along u, ordinary tokens' keys point
    anywhere.  Whoever sees the marked token puts most of its weight on it; whoever does not, spreads it."""
    rng = np.random.default_rng(6)
    mark, width, d = 7, 32, 16
    u = rng.standard_normal(d)
    u /= np.linalg.norm(u)
    a = rng.standard_normal(width)
    a /= np.linalg.norm(a)
    if kind == "attention":
        cfg = config([attention(heads=2, kv_heads=1, dim=d, rot=None, scale=1.5)], width=width, vocab=50, cap=40.0)
    else:
        cfg = config([latent(heads=2, dim=d, rot_dim=0, vdim=16, q_rank=24, kv_rank=16, scale=0.5)], width=width, vocab=50, cap=40.0)
    w = P.random_weights(cfg, seed=5)
    w["l0.canon1"] *= 0.1
    w["l0.norm1"][:] = 1.0
    w["l0.dwa"][:] = (-1.0, 1.0)                              # what goes on is the mixer's normed output alone
    e = w["embed"][mark] - (w["embed"][mark] @ a) * a         # what only the marked token has much of
    e /= np.linalg.norm(e)
    others = np.arange(50) != mark
    w["embed"][others] -= np.outer(w["embed"][others] @ e, e)
    w["embed"] += 4.0 * a
    off_u = np.eye(d) - np.outer(u, u)                        # ordinary keys have no share along u
    if kind == "attention":
        w["l0.mix.k"] -= np.outer(w["l0.mix.k"] @ a, a)       # keys do not see the common share
        w["l0.mix.k"] = off_u @ w["l0.mix.k"] + np.outer(u, e) * 12.0
        w["l0.mix.q"] *= 0.05
        w["l0.mix.q"][0:d] += np.outer(u, a) * 3.0            # head 0: every query points along u
        w["l0.mix.sink"][:] = 0.5
    else:
        w["l0.mix.dkv.norm"][:] = 1.0
        w["l0.mix.dq.norm"][:] = 1.0
        w["l0.mix.dkv"] -= np.outer(w["l0.mix.dkv"] @ a, a)
        w["l0.mix.dkv"] = 0.3 * off_u @ w["l0.mix.dkv"] + np.outer(u, e) * 2.0    # the marked token's latent points along u
        w["l0.mix.uk"][:d] = np.eye(16) * 2.0                 # head 0 reads the latent as its key
        w["l0.mix.dq"] *= 0.05
        w["l0.mix.dq"][0] = a                                 # the first latent channel of every query is large and positive
        w["l0.mix.uq"][:d] = 0.0
        w["l0.mix.uq"][:d, 0] = 1.5 * u                       # head 0's queries point along u
    w = {k: P.from_bf16_bits(P.to_bf16_bits(v)).reshape(v.shape) for k, v in w.items()}
    return cfg, w, P.write_model(str(tmp_path), cfg, w), mark


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 130])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_key_far_back(tmp_path, kind, far, dtype):
    from gophonic_b200.engine.model import Model
    from gophonic_b200.engine.step import Engine
    cfg, w, d, mark = _standout(tmp_path / "far", kind)
    toks = [int(t) for t in np.random.default_rng(8).integers(8, cfg["vocab"], size=300)]
    toks[far] = mark
    middle = lambda z: z - z.mean(-1, keepdims=True)           # the embeddings' common share moves all logits alike
    want = middle(P.forward(cfg, w, toks))
    gone = middle(P.forward(cfg, w, toks[:far] + [9] + toks[far + 1:]))
    # (rows ahead of the marked key average many values to little, which the norm behind the mixer blows up with its rounding)
    tol = TOL[dtype] if dtype == "float32" else 1e-1
    # the plain model itself must tell at the end whether the key is there, by much more than the tolerance
    assert np.sqrt(((want[-1] - gone[-1]) ** 2).mean()) > 4 * tol * np.sqrt((want ** 2).mean())
    eng = Engine(Model.from_dir(d, dtype=dtype), max_tokens=1024)
    close(middle(feed(eng, toks)), want, tol)                                          # in a prompt
    close(middle(feed(eng, toks, cuts=[far + 1, 1, 1])), want, tol)                    # the first tokens behind the marked one
    close(middle(feed(eng, toks, cuts=[290] + [1] * 10)), want, tol)                   # decoded far behind it
    close(middle(feed(eng, toks, cuts=[64, 2, 126, 2, 70])), want, tol)                # in portions


def test_the_sink_shows(models):
    """A large sink takes the weight away from the keys: the model without it gives other logits."""
    cfg, w, _ = models["attention", "float32"]
    toks = tokens_for(cfg, 6, 20)
    less = dict(w)
    less["l0.mix.sink"] = w["l0.mix.sink"] - 30.0
    assert np.abs(P.forward(cfg, w, toks) - P.forward(cfg, less, toks)).max() > 0.05


def test_a_state_remembers_its_first_tokens(tmp_path):
    """Forget gates close to one (a bias that makes 1 - f a few thousandths): the first token still shows 250 tokens
    on, in a prompt, in portions and decoded."""
    from gophonic_b200.engine.model import Model
    from gophonic_b200.engine.step import Engine
    cfg = config([hgrn2(heads=2, dim=16, vdim=16)], width=32, vocab=50)
    w = P.random_weights(cfg, seed=9)
    w["l0.mix.f.b"][:] = 6.0
    w["l0.mix.lower"][:] = 0.5
    toks = tokens_for(cfg, 7, 250)
    want = P.forward(cfg, w, toks)
    other = P.forward(cfg, w, [(toks[0] + 1) % 50] + toks[1:])
    tol = 5e-5
    assert np.abs(want[-1] - other[-1]).max() > 10 * tol
    eng = Engine(Model.from_dir(P.write_model(str(tmp_path / "keep"), cfg, w), dtype="float32"), max_tokens=1024)
    for cuts in (None, [1] * 250, [100, 2, 3, 70]):
        close(feed(eng, toks, cuts=cuts), want, tol)


# ---- the kernels by themselves -------------------------------------------------------------------
def _f32(a):
    import torch
    return torch.tensor(np.asarray(a), dtype=torch.float32, device="cuda:0")


@pytest.mark.parametrize("out_dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows, width, planes", [(5, 45, 3), (700, 64, 0), (3, 2048, 6), (700, 2048, 5), (2, 4096, 9), (2, 5000, 1), (4, 1030, 2), (3, 9000, 2)])
def test_residual_rows_between_sublayers(rows, width, planes, out_dtype):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    rng = np.random.default_rng(rows + width)
    P_ = _f32(rng.standard_normal((planes + 2, rows, width)))
    y, yw, nw, avg = _f32(3 * rng.standard_normal((rows, width))), _f32(1 + 0.3 * rng.standard_normal(width)), _f32(1 + 0.3 * rng.standard_normal(width)), \
        _f32(rng.standard_normal(planes + 1))
    d = lambda t: t.double().cpu().numpy()
    base = d(P_[planes])
    v = base + P.rms_norm(d(y), d(yw), 1e-3)
    x = np.tensordot(d(avg), np.concatenate([d(P_[:planes]), v[None]]), axes=1)
    want = P.rms_norm(x, d(nw), 1e-4)
    tol = 2e-5 if out_dtype == "float32" else 4e-2
    out = torch.zeros((rows, width), dtype=getattr(torch, out_dtype), device="cuda:0")
    x_out = torch.zeros((rows, width), dtype=torch.float32, device="cuda:0")
    # gathered rows leave everything else as it is
    pick = [rows - 1, 0, rows // 2]
    gathered = torch.zeros((3, width), dtype=out.dtype, device="cuda:0")
    before = P_.clone()
    common = dict(base=P_[planes], norm_weight=nw, eps=1e-4, y=y, y_weight=yw, y_eps=1e-3, planes=P_, n_planes=planes, average=avg)
    ops.sandwich_rows(out=gathered, rows=torch.tensor(pick, dtype=torch.int32, device="cuda:0"), **common)
    assert torch.equal(P_, before)
    ops.sandwich_rows(out=out, result=P_[planes], x_out=x_out, **common)
    torch.cuda.synchronize()
    assert np.abs(d(P_[planes]) - v).max() < 2e-5 and np.abs(d(x_out) - x).max() < 5e-5 and np.abs(d(out) - want).max() < tol
    assert np.abs(d(gathered) - want[pick]).max() < tol
    assert torch.equal(P_[:planes], before[:planes]) and torch.equal(P_[planes + 1], before[planes + 1])
    # without an output and without an average: the norm alone
    ops.sandwich_rows(base=P_[planes], out=out, norm_weight=nw, eps=1e-4)
    torch.cuda.synchronize()
    assert np.abs(d(out) - P.rms_norm(v, d(nw), 1e-4)).max() < tol


class _Rows:
    def __init__(self, lengths, slots):
        import torch
        i32 = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda:0")
        self.nseq, self.max_q_len = len(lengths), max(lengths)
        self.row_seq = i32([s for s, n in enumerate(lengths) for _ in range(n)])
        self.seq_slot, self.seq_q_len = i32(slots), i32(lengths)
        self.seq_q_start = i32(np.concatenate([[0], np.cumsum(lengths)[:-1]]).astype(np.int32))


@pytest.mark.parametrize("width", [45, 64, 2048])
@pytest.mark.parametrize("taps", [1, 2, 4, 7, 16])
def test_the_convolution_in_portions_and_token_by_token(taps, width):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    rng = np.random.default_rng(taps)
    lengths = [90, 103]
    h = [rng.standard_normal((n, width)) for n in lengths]
    conv = _f32(0.4 * rng.standard_normal((taps, width)))
    hs = [_f32(a) for a in h]
    want = [P.input_convolution(a.double().cpu().numpy(), conv.double().cpu().numpy().T) for a in hs]
    ones = torch.ones(width, dtype=torch.float32, device="cuda:0")
    state = torch.zeros((3, max(taps - 1, 1) * width), dtype=torch.float32, device="cuda:0")
    got, at, slots = [[], []], [0, 0], [2, 0]
    for portion in ([3, 5], [2, 2], [1, 4], [20, 1], [2, 2], [40, 50], [2, 30]):      # few rows a step, and many (another kernel)
        x = torch.cat([hs[s][at[s]:at[s] + n] for s, n in enumerate(portion)]).contiguous()
        out = torch.zeros_like(x)
        ops.conv_rows(x, conv, state, out, _Rows(portion, slots))
        for s, part in enumerate(out.split(portion)):
            got[s].append(part.cpu().numpy())
            at[s] += portion[s]
    # the rest token by token, where the same kernel norms and convolves: rows already of unit mean square keep their values
    unit = [a / torch.sqrt((a * a).mean(-1, keepdim=True)) for a in hs]
    for s in range(2):
        err = np.abs(np.concatenate(got[s]) - want[s][:at[s]]).max()
        assert err < 2e-5, err
    assert state[1].abs().max().item() == 0.0
    for s in range(2):
        state.zero_()
        w1 = P.input_convolution(unit[s].double().cpu().numpy(), conv.double().cpu().numpy().T)
        for t in range(40):
            out = torch.zeros((1, width), dtype=torch.float32, device="cuda:0")
            ops.sandwich_rows(base=unit[s][t:t + 1].contiguous(), out=out, norm_weight=ones, eps=0.0, conv=conv, state=state, batch=_Rows([1], [slots[s]]))
            assert np.abs(out.cpu().numpy()[0] - w1[t]).max() < 3e-5


@pytest.mark.parametrize("sizes", [(2, 16, 24), (3, 20, 33), (1, 1, 1), (2, 128, 128), (1, 256, 40), (4, 100, 64)])
def test_the_state_whose_forget_gate_writes(sizes):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    H, d, dv = sizes
    lengths, slots = [37, 1, 12], [1, 3, 0]
    rows = sum(lengths)
    rng = np.random.default_rng(sum(sizes))
    buf = _f32(1.5 * rng.standard_normal((rows, 2 * H * d + H * dv + 3)))
    bias, low = _f32(1.0 + rng.standard_normal(H * d)), _f32(rng.uniform(0, 0.95, H * d))
    b = buf.double().cpu().numpy()
    q, v = P.silu(b[:, :H * d]).reshape(rows, H, d), b[:, H * d:H * d + H * dv].reshape(rows, H, dv)
    l = low.double().cpu().numpy()
    f = (l + (1 - l) * P.sigmoid(b[:, H * (d + dv):2 * H * d + H * dv] + bias.double().cpu().numpy())).reshape(rows, H, d)
    want, at, S_end = np.zeros((rows, H, dv)), 0, []
    for n in lengths:
        S = np.zeros((H, d, dv))
        for t in range(at, at + n):
            S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
            want[t] = np.einsum("hdv,hd->hv", S, q[t])
        S_end.append(S)
        at += n

    def run(x, batch, state, single):
        out = torch.zeros((x.shape[0], H * dv), dtype=torch.float32, device="cuda:0")
        ops.state_scan(x, 0, 0, H * d, H, d, dv, 1.0, state, out, batch.seq_slot, batch.seq_q_start, batch.seq_q_len, batch.nseq,
                       decay=x[:, H * (d + dv):2 * H * d + H * dv], gate_bias=bias, lower=low, max_q_len=1 if single else batch.max_q_len)
        return out.cpu().numpy().reshape(-1, H, dv)
    scale = max(1.0, np.abs(want).max())
    state = torch.zeros((4, H, d * dv), dtype=torch.float32, device="cuda:0")
    got = run(buf.clone(), _Rows(lengths, slots), state, False)
    assert np.abs(got - want).max() / scale < 2e-5
    for s, S in zip(slots, S_end):
        assert np.abs(state[s].cpu().numpy().reshape(H, d, dv) - S).max() < 2e-5
    assert state[2].abs().max().item() == 0.0
    state.zero_()
    for t in range(lengths[0]):         # token by token: the kernel for single tokens forms the gates itself
        got = run(buf[t:t + 1].clone(), _Rows([1], [2]), state, True)
        assert np.abs(got[0] - want[t]).max() / scale < 2e-5


@pytest.mark.parametrize("sizes", [(8, 2, 4, 2), (16, 4, 2, 1), (6, 3, 3, 2), (5, 3, 5, 4), (512, 8, 16, 3), (40, 6, 1, 1), (4, 4, 2, 2), (96, 10, 48, 7)])
@pytest.mark.parametrize("score", ["sigmoid", "softmax"])
def test_the_choice_by_corrected_scores_inside_the_best_groups(sizes, score):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    E, top, count, keep = sizes
    rows = 61
    rng = np.random.default_rng(sum(sizes))
    z, corr = _f32(2 * rng.standard_normal((rows, E))), _f32(0.4 * rng.standard_normal(E) - 0.5)      # negative choice scores too
    z[0, :] = -20.0                                                                                   # scores near zero: the correction decides
    dense, index, weight = torch.zeros((rows, E), device="cuda:0"), torch.zeros((rows, top), dtype=torch.int32, device="cuda:0"), torch.zeros((rows, top), device="cuda:0")
    ops.moe_route(z, top, 0.0, dense, index, weight, score=score, renorm=False, correction=corr, groups=count, keep_groups=keep)
    torch.cuda.synchronize()
    zz, cc = z.double().cpu().numpy(), corr.double().cpu().numpy()
    if score == "sigmoid":
        s = P.sigmoid(zz)
    else:
        s = np.exp(zz - zz.max(-1, keepdims=True))
        s /= s.sum(-1, keepdims=True)
    choice = s + cc
    got_i, got_w = index.cpu().numpy(), weight.cpu().numpy()
    for r in range(rows):
        g = choice[r].reshape(count, -1)
        strength = np.sort(g, -1)[:, -2:].sum(-1)
        kept = np.argsort(-strength, kind="stable")[:keep]
        c = np.where(np.isin(np.arange(E) // (E // count), kept), choice[r], -np.inf)
        want = np.argsort(-c, kind="stable")[:top]
        order = np.sort(strength)[::-1]
        if keep < count and order[keep - 1] - order[keep] < 1e-6 or np.diff(np.sort(-c)[:top + 1]).min(initial=1.0) < 1e-6:
            continue            # a near-tie: either is right
        assert (got_i[r] == want).all(), r
        assert np.abs(got_w[r] - s[r][want]).max() < 1e-5
        row = np.zeros(E)
        row[want] = s[r][want]
        assert np.abs(dense[r].cpu().numpy() - row).max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 3, 16, 17, 100, 230])
@pytest.mark.parametrize("sizes", [(8, 2, 24, 4, 2), (12, 1, 48, 3, 1), (3, 3, 8, None, None), (6, 4, 32, 2, 2)])
def test_mixture_rows(rows, sizes, dtype):
    """The mixture part by itself in every range of rows against the plain mixture."""
    import torch
    from gophonic_b200.config import ZenoraxConfig
    from gophonic_b200.engine.model import make_runtime
    from gophonic_b200.parts.moe import MoE
    hidden = 64
    cfg = config([hgrn2(mlp=moe(*sizes))], width=hidden)
    w = {k[len("l0.mlp."):]: v for k, v in P.random_weights(cfg, seed=rows + sizes[0]).items() if k.startswith("l0.mlp.")}
    spec = ZenoraxConfig.from_dict(cfg).model_spec().layers[0].feed_forward
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    part = MoE(spec, "", {k: torch.tensor(v, dtype=torch.float32).to(td).cuda() for k, v in w.items()}, make_runtime(dtype, "cuda:0"))
    x = torch.tensor(np.random.default_rng(rows).standard_normal((rows, hidden)), dtype=torch.float32).to(td).cuda()
    out = torch.zeros((rows, hidden), dtype=torch.float32, device="cuda:0")
    part.forward(None, x, out)
    torch.cuda.synchronize()
    close(out.cpu().numpy(), P.mixture(x.double().cpu().numpy(), w, "", cfg["layers"][0]["mlp"]), 3e-5 if dtype == "float32" else 4e-2, MOST[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 8), (3, 1, 12, 12), (4, 2, 128, 128), (2, 2, 128, 64)])
@pytest.mark.parametrize("rows", [3, 300])
def test_values_that_are_the_keys_in_the_cache(sizes, rows, dtype):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    H, G, d, rot = sizes
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    rng = np.random.default_rng(sum(sizes))
    buf = torch.tensor(rng.standard_normal((rows, (H + G) * d)), dtype=torch.float32).to(td).cuda()
    x = buf.double().cpu().numpy()
    freqs = P.linear_frequencies(rot, 200.0, {"factor": 2.0})
    ang = np.arange(512)[:, None] * freqs[None, :]
    pages = 6
    k_plane, v_plane = (torch.zeros((pages, G, 64, d), dtype=td, device="cuda:0") for _ in range(2))
    perm = [3, 0, 5, 1, 4, 2]
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda:0")
    ones = torch.ones(d, device="cuda:0")
    pos = [7 + r for r in range(rows)]
    ops.qk_norm_rope_kv_write(buf, H, G, d, ones, ones, 1e-5, _f32(np.cos(ang)), _f32(np.sin(ang)), rot, i32(pos), i32([0] * rows), i32([0]), i32([perm]),
                              k_plane, v_plane, True, value_from_key=True)
    torch.cuda.synchronize()
    q, k = x[:, :H * d].reshape(rows, H, d), x[:, H * d:].reshape(rows, G, d)
    turned = lambda t: P.unit_rms(P.rotate(t, pos, freqs, "half"), 1e-5)
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert np.abs(buf.double().cpu().numpy()[:, :H * d].reshape(rows, H, d) - turned(q)).max() < tol
    kd, vd = k_plane.double().cpu().numpy(), v_plane.double().cpu().numpy()
    at = lambda plane: np.stack([plane[perm[p // 64], :, p % 64] for p in pos])
    assert np.abs(at(kd) - turned(k)).max() < tol
    assert np.array_equal(at(vd), k)                        # as projected, bit for bit


@pytest.mark.parametrize("shape", [(5, 70, 64, 96), (16, 700, 128, 256), (3, 300, 520, 40)])
def test_squared_products_of_groups_in_one_launch(shape):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    groups, rows, K, N = shape
    rng = np.random.default_rng(sum(shape))
    sizes = rng.multinomial(rows, rng.dirichlet(np.ones(groups)))
    sizes[0] += sizes[1]
    sizes[1] = 0                                               # a group without rows
    offsets = torch.tensor(np.concatenate([[0], np.cumsum(sizes)]), dtype=torch.int32, device="cuda:0")
    a = torch.tensor(rng.standard_normal((rows, K)), dtype=torch.float32).bfloat16().cuda()
    w = torch.tensor(rng.standard_normal((groups * N, K)) / np.sqrt(K), dtype=torch.float32).bfloat16().cuda()
    out = torch.zeros((rows, N), dtype=torch.bfloat16, device="cuda:0")
    ops.gemm_grouped(a, w, out, offsets, groups, gate="relu2")
    torch.cuda.synchronize()
    assert ops.tc5_status() == 0
    z = np.concatenate([a.double().cpu().numpy()[o:o + n] @ w.double().cpu().numpy()[e * N:(e + 1) * N].T
                        for e, (o, n) in enumerate(zip(offsets.tolist(), sizes))])
    want = np.maximum(z, 0.0) ** 2
    assert (np.abs(out.double().cpu().numpy() - want) / (1.0 + want)).max() < 1e-2


@pytest.mark.parametrize("kind", ["relu2", "swiglu", "glu_clamp"])
@pytest.mark.parametrize("shape", [(5, 3, 16, 64, 96), (8, 2, 9, 72, 24), (4, 4, 3, 2048, 128), (3, 1, 16, 40, 1536)])
def test_few_rows_sorted_by_expert_on_the_tensor_cores(shape, kind):
    """Experts with no pair, with a few and with more than one tile of pairs; inner sizes that are no multiple of a step."""
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    E, top, rows, hidden, ff = shape
    rng = np.random.default_rng(sum(shape))
    per = 1 if kind == "relu2" else 2
    as_bf = lambda a: torch.tensor(a, dtype=torch.float32).bfloat16().cuda()
    x, up = as_bf(rng.standard_normal((rows, hidden))), as_bf(rng.standard_normal((E * per * ff, hidden)) / np.sqrt(hidden))
    down = as_bf(rng.standard_normal((hidden, E * ff)) / np.sqrt(ff))
    chosen = np.stack([np.sort(rng.permutation(E)[:top]) for _ in range(rows)])
    chosen[:, 0] = 0 if E > top else chosen[:, 0]              # one expert takes every row
    index = torch.tensor(chosen, dtype=torch.int32, device="cuda:0")
    i32 = lambda n: torch.zeros(n, dtype=torch.int32, device="cuda:0")
    offsets, place, src = i32(E + 1), i32(rows * top), i32(rows * top)
    ops.moe_group(index, E, offsets, place, src)
    ys = torch.zeros((rows * top, hidden), dtype=torch.float32, device="cuda:0")
    ops.moe_rows_grouped(x, up, down, offsets, src, ys, E, top, ff, kind=kind, limit=1.0, slope=1.7)
    torch.cuda.synchronize()
    X, U, D = (t.double().cpu().numpy() for t in (x, up, down))
    for r in range(rows):
        for j in range(top):
            e = chosen[r, j]
            z = U[e * per * ff:(e + 1) * per * ff] @ X[r]
            if kind == "relu2":
                a = np.maximum(z, 0) ** 2
            elif kind == "swiglu":
                a = P.silu(z[:ff]) * z[ff:]
            else:
                c = np.minimum(z[:ff], 1.0)
                a = c * P.sigmoid(1.7 * c) * (np.clip(z[ff:], -1.0, 1.0) + 1.0)
            want = D[:, e * ff:(e + 1) * ff] @ a
            got = ys[place[r * top + j].item()].double().cpu().numpy()
            assert np.abs(got - want).max() < 4e-2 * max(1.0, np.abs(want).max())


def test_capped_logits():
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    z = _f32(20 * np.random.default_rng(1).standard_normal((3, 777)))
    want = P.soft_cap(z.double().cpu().numpy(), 7.0)
    ops.soft_cap_(z, 7.0)
    assert np.abs(z.double().cpu().numpy() - want).max() < 1e-5


# ---- generation through the entry point, the trace program, the command line ----------------------
def test_greedy_generation_through_the_entry_point(models):
    import gophonic_b200 as g
    cfg, w, d = models["mix", "float32"]
    prompts = [tokens_for(cfg, 40, 9), tokens_for(cfg, 41, 1), tokens_for(cfg, 42, 75)]
    model = g.Open(d, g.Options(Format=g.FormatF32, CacheTokens=2048, Batch=4))
    got = g.Lane(model, g.TokensGenerator).Generate(prompts, g.ChatOptions(MaxTokens=10))
    model.Close()
    for p, out in zip(prompts, got):
        want, margins = P.greedy_generate(cfg, w, p, 10)
        for a, b, m in zip(out, want, margins):
            if m < 1e-3:
                break           # a near-tie of the plain logits: from here on either token is right
            assert a == b


def test_trace_program_on_a_folder(models, tmp_path):
    cfg = CONFIGS["mix"]
    a, b = tokens_for(cfg, 50, 70), tokens_for(cfg, 51, 5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": []}, {"id": "b", "tokens": b[3:4], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[67:68], "want": [0]}, {"id": "b", "tokens": b[4:5], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:70], "want": [1]}], "end": ["a"]}]
    out = tmp_path / "out"
    for dtype in ("float32", "bfloat16"):
        _, w, d = models["mix", dtype]
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                           timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        wa, wb = P.forward(cfg, w, a), P.forward(cfg, w, b)
        read = lambda n: np.fromfile(str(out / f"{n}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
        close(read(0), np.stack([wa[0], wa[65], wb[2]]), TOL[dtype])
        close(read(1), wb[3:4], TOL[dtype])
        close(read(2), np.stack([wa[67], wb[4]]), TOL[dtype])
        close(read(3), wa[69:70], TOL[dtype])


def test_the_command_line_writes_and_runs_a_named_configuration(tmp_path):
    """-random-config NAME -write-model DIR, then -model DIR: the plain model reads the written folder
    and would have chosen the same tokens."""
    out = tmp_path / "written"
    run = lambda *a: subprocess.run([sys.executable, "-m", "gophonic_b200", *a], cwd=ROOT, capture_output=True, text=True, timeout=600)
    r = run("-random-config", "zenorax-tiny", "-weights-seed", "4", "-write-model", str(out))
    assert r.returncode == 0, r.stderr[-2000:]
    cfg, w = P.read_model(str(out))
    assert cfg["architecture"] == "Zenorax" and {n: tuple(a.shape) for n, a in w.items()} == P.tensor_shapes(cfg)
    r = run("-model", str(out), "-format", "f32", "-max-tokens", "6", "3,9,27", "100")
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(l) for l in r.stdout.splitlines() if l.startswith("{")]
    assert [l["prompt"] for l in lines] == [[3, 9, 27], [100]]
    for l in lines:
        ids = list(l["prompt"])
        assert len(l["tokens"]) == 6
        for t in l["tokens"]:
            logits = P.forward(cfg, w, ids)[-1]
            assert logits.max() - logits[t] <= 1e-5
            ids.append(t)
