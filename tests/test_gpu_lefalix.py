"""The Lefalix design on the GPU against the plain implementation (tests/plain/lefalix_plain.py): each mechanism alone, whole
prompts against token-by-token decoding, prompts in portions down to two tokens, batches of unequal requests, slots and pages
that are used again, keys at the window's and the pages' edges, tokens far back in a state, the first tokens, long decoding,
odd sizes, the kernels by themselves, and greedy generation through the entry point.  Every model here is made by the test
(its own sizes, random weights that bfloat16 holds exactly)."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest

from tests.plain import lefalix_plain as P

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

RAMP = {"factor": 3.0, "original": 64, "fast": 6.0, "slow": 0.5}     # kept, blended and divided channels all occur


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=8, top=2, ff=24, count=4, keep=2):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if count is not None:
        m["router"]["groups"] = {"count": count, "keep": keep}
    return m


def part(heads, kv_heads, dim, vdim, conv):
    m = {"heads": heads, "dim": dim, "vdim": vdim}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if conv is not None:
        m["conv"] = conv
    return m


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, mlp=None):
    return {"type": "channel_delta", "mixer": part(heads, kv_heads, dim, vdim, conv), "mlp": mlp}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, size=20, rot=8, base=100.0, scale=1.2, scaling=RAMP):
    m = dict(part(heads, kv_heads, dim, vdim, conv), scale=scale)
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = {"dims": rot, "base": base}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    return m


def pair(left=None, right=None, mlp=None):
    return {"type": "parallel", "mixer": {"left": left or attention(), "right": right or part(3, 3, 12, 20, 2)}, "mlp": mlp}


def config(layers, width=64, vocab=96, eps=1e-5, loop=None):
    cfg = {"architecture": "Lefalix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIGS = {
    # each mechanism alone
    "delta": config([delta()]),
    "pair": config([pair()]),
    "dense": config([delta(mlp=dense())]),
    "moe": config([delta(mlp=moe())]),
    "loop": config([delta(heads=2), delta(kv_heads=4, dim=8, mlp=dense(24)), delta(heads=3, kv_heads=1)], loop=(1, 2, 3)),
    # all together: a stretch in the middle runs three times, layers with and without a feed-forward on both sides of its edges
    "mix": config([pair(attention(scale=0.7, size=33), mlp=moe(6, 3, 40, 3, 2)), delta(heads=6, kv_heads=3, dim=24, vdim=8, conv=2, mlp=moe(9, 2, 24, 3, 1)),
                   pair(attention(heads=6, kv_heads=1, dim=24, vdim=12, conv=4, size=64, rot=24, scale=1.5), part(4, 2, 20, 16, 3)),
                   delta(heads=2, kv_heads=2, dim=40, vdim=32, conv=3, mlp=dense(72)), pair(mlp=dense(24))], loop=(1, 3, 3)),
    # sizes the tensor-core kernels take in bfloat16
    "tensor": config([delta(heads=4, kv_heads=4, dim=64, vdim=64, conv=4, mlp=moe(8, 2, 64, 4, 2)),
                      pair(attention(heads=4, kv_heads=2, dim=128, vdim=128, conv=4, size=100, rot=64, scale=2.0, base=10000.0),
                           part(2, 1, 128, 128, 4), mlp=dense(128)),
                      pair(attention(heads=4, kv_heads=4, dim=64, vdim=64, conv=2, size=48, rot=32, scale=1.0), part(4, 2, 64, 32, 4), mlp=moe(4, 4, 32, 2, 2)),
                      delta(heads=2, kv_heads=1, dim=256, vdim=64)], width=128, vocab=80, loop=(0, 2, 2)),
    # what a file may leave out (groups, scaling, rotation, mask, kv_heads, convolutions, the loop) and sizes that are odd, equal or
    # 1: one tap, one head, one expert, every expert used, groups of one expert, a width that no vector load fits
    "odd": config([pair(attention(heads=3, kv_heads=None, dim=11, vdim=7, conv=None, size=None, rot=None), part(1, None, 2, 5, None), mlp=moe(1, 1, 56, None)),
                   delta(heads=1, kv_heads=None, dim=3, vdim=4, conv=1, mlp=moe(5, 3, 8, 5, 4)),
                   pair(attention(heads=1, kv_heads=1, dim=6, vdim=13, conv=1, size=1, rot=2, scaling=None), part(5, 1, 33, 6, 1), mlp=dense(9)),
                   delta(heads=7, kv_heads=7, dim=20, vdim=33, conv=5, mlp=moe(3, 3, 8, 1, 1))], width=45, vocab=61, eps=1e-6),
    # a norm behind a rotation that stretches what it turns, without a convolution
    "turned": config([pair(attention(conv=None, rot=12, size=None), part(2, 1, 16, 16, 3))]),
    # more taps than a short portion has tokens
    "taps": config([delta(conv=7), pair(attention(conv=6), part(2, 2, 16, 16, 9))], width=52, loop=(0, 2, 2)),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(configuration, weights, folder) by (name, dtype): in bfloat16 the experts' order is far from ties (see ``random_weights``);
    the mixture's own tests let the scores choose."""
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        for dtype in ("float32", "bfloat16"):
            w = P.random_weights(cfg, seed=810 + i, decided=dtype == "bfloat16")
            out[name, dtype] = (cfg, w, P.write_model(str(tmp_path_factory.mktemp(f"lefalix_{name}_{dtype}")), cfg, w))
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
    above 1e-3) root mean square relative to the wanted values' own.  With ``most`` < 1 that share of the rows must be, and the rest
    within five times as much."""
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


def test_the_residual_behind_every_layer_run(models):
    """The results of all runs in order, repeated layers included, as the block behind each completes them."""
    from gophonic_b200.parts.sandwich import SandwichBlock
    cfg, w, _ = models["mix", "float32"]
    eng = engine_for(models, "mix", "float32", graphs=False)
    toks = tokens_for(cfg, 2, 70)
    seen, starts, orig = [], [], SandwichBlock._open

    def spy(self, batch, planes, pending, state, enter=None):
        start, x = orig(self, batch, planes, pending, state, enter)
        if pending is not None:
            assert planes.shape[0] == 2              # nothing but the embedding output and the latest result is kept
            seen.append(planes[1].cpu().numpy())
        starts.append((start.cpu().numpy(), enter is not None))
        return start, x
    SandwichBlock._open = spy
    try:
        feed(eng, toks)
    finally:
        SandwichBlock._open = orig
    _, layers = P.forward(cfg, w, toks, return_layers=True)
    runs = P.layer_runs(cfg)
    assert len(starts) == len(runs) == 9 and [e for _, e in starts] == [again for _, again in runs]
    x0 = w["embed"][toks]
    close(starts[0][0], x0, 1e-6)
    for i, (got, want) in enumerate(zip(seen, layers)):
        close(got, want, 2e-5)
        close(starts[i + 1][0], want + (x0 if runs[i + 1][1] else 0.0), 2e-5)


# ---- prompts against decoding, portions, batches ----------------------------------------------
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["mix", "odd", "tensor", "taps", "turned"])
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
    prompts = [tokens_for(cfg, 10 + i, n) for i, n in enumerate([1, 70, 9, 133])]
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
    """The convolutions' rows and the matrix states go back with the keys."""
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
def test_long_decoding_past_pages_and_windows(models, name):
    for dtype in ("float32", "bfloat16"):
        cfg, w, _ = models[name, dtype]
        toks = tokens_for(cfg, 5, 40 + 230)
        got = feed(engine_for(models, name, dtype), toks, cuts=[40] + [1] * 230)
        close(got, P.forward(cfg, w, toks), TOL[dtype])


# ---- one token far back, through a whole model ---------------------------------------------------
def _rounded(w):
    return {k: P.from_bf16_bits(P.to_bf16_bits(v)).reshape(v.shape) for k, v in w.items()}


def _standout(tmp_path, window):
    """One layer whose attention picks out one key.  Every embedding row carries the same large share along one direction a,
    from which the query path makes queries along a fixed direction u of the unrotated channels; the token ``mark`` has an
    embedding that the key path turns into a key along u, ordinary tokens' keys have no share along u.  Whoever sees the marked
    token puts most of its weight on it; whoever does not, spreads it.  The other mixer is silent."""
    rng = np.random.default_rng(6)
    mark, width, d = 7, 32, 16
    u = np.concatenate([np.zeros(8), rng.standard_normal(8)])
    u /= np.linalg.norm(u)
    a = rng.standard_normal(width)
    a /= np.linalg.norm(a)
    cfg = config([pair(attention(heads=2, kv_heads=1, dim=d, vdim=16, conv=2, size=window, rot=8, scale=0.9), part(1, 1, 8, 8, 2))], width=width, vocab=50)
    w = P.random_weights(cfg, seed=5)
    q = "l0.mix.left."
    e = w["embed"][mark] - (w["embed"][mark] @ a) * a         # what only the marked token has much of
    e /= np.linalg.norm(e)
    others = np.arange(50) != mark
    w["embed"][others] -= np.outer(w["embed"][others] @ e, e)
    w["embed"] += 4.0 * a
    w["l0.norm1"][:] = 1.0
    w["l0.norm1b"] *= 8.0
    w["l0.mix.right.out"][:] = 0.0
    off_u = np.eye(d) - np.outer(u, u)
    w[q + "k"] = off_u @ (w[q + "k"] - np.outer(w[q + "k"] @ a, a)) + np.outer(u, e) * 12.0      # keys do not see the common share
    w[q + "k.b"] = 0.2 * off_u @ w[q + "k.b"]
    w[q + "q"] *= 0.05
    w[q + "q.b"] *= 0.05
    w[q + "q"][:d] += np.outer(u, a) * 3.0                    # head 0: every query points along u
    for n in "qkv":
        w[q + n + ".conv"][:] = (0.002, 1.0)
    w[q + "sink"][:] = 0.5
    w = _rounded(w)
    return cfg, w, P.write_model(str(tmp_path), cfg, w), mark


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 130])
@pytest.mark.parametrize("window", [5, 64, 100])
def test_one_key_just_inside_and_just_outside_the_window(tmp_path, window, far, dtype):
    from gophonic_b200.engine.model import Model
    from gophonic_b200.engine.step import Engine
    cfg, w, d, mark = _standout(tmp_path / "far", window)
    toks = [int(t) for t in np.random.default_rng(8).integers(8, cfg["vocab"], size=300)]
    toks[far] = mark
    middle = lambda z: z - z.mean(-1, keepdims=True)
    want = middle(P.forward(cfg, w, toks))
    gone = middle(P.forward(cfg, w, toks[:far] + [9] + toks[far + 1:]))
    tol = TOL[dtype]
    # the plain model itself must tell at the window's last row that the key is there and behind it that it is not
    shows = np.sqrt(((want - gone) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    last = far + window - 1
    assert shows[last] > 3 * tol and shows[last + 1] < 0.2 * shows[last], (shows[last], shows[last + 1])
    eng = Engine(Model.from_dir(d, dtype=dtype), max_tokens=1024)
    close(middle(feed(eng, toks)), want, tol)                                                  # in a prompt
    close(middle(feed(eng, toks, cuts=[far + 1, 1, 1])), want, tol)                            # the first tokens behind the marked one
    close(middle(feed(eng, toks, cuts=[max(1, last - 2)] + [1] * 6)), want, tol)               # decoded over the edge
    close(middle(feed(eng, toks, cuts=[64, 2, 126, 2, 70])), want, tol)                        # in portions


def test_the_sink_shows(models):
    """A large sink takes the weight away from the keys: the model without it gives other logits."""
    cfg, w, _ = models["pair", "float32"]
    toks = tokens_for(cfg, 6, 20)
    less = dict(w)
    less["l0.mix.left.sink"] = w["l0.mix.left.sink"] - 30.0
    less["l0.mix.left.o.b"] = w["l0.mix.left.o.b"]
    assert np.abs(P.forward(cfg, w, toks) - P.forward(cfg, less, toks)).max() > 0.02


@pytest.mark.parametrize("kind", ["channel", "head"])
def test_a_state_remembers_its_first_tokens(tmp_path, kind):
    """Decays close to one and small write strengths (made from a share that all embeddings have): the first token still shows
    250 tokens on, in a prompt, in portions and decoded."""
    from gophonic_b200.engine.model import Model
    from gophonic_b200.engine.step import Engine
    layer = delta(heads=2, kv_heads=1, dim=16, vdim=16) if kind == "channel" else pair(attention(size=8), part(2, 1, 16, 16, 3))
    cfg = config([layer], width=32, vocab=50)
    w = P.random_weights(cfg, seed=9)
    q = "l0.mix." if kind == "channel" else "l0.mix.right."
    a = np.random.default_rng(1).standard_normal(32)
    a /= np.linalg.norm(a)
    w["embed"] += 6.0 * a
    w["l0.norm1"][:] = 1.0
    w[q + "b"] = 0.1 * w[q + "b"] - 1.0 * a                    # strengths of a few hundredths
    w[q + "A_log"][:] = -3.0
    w[q + "dt_bias"][:] = -4.0
    w = _rounded(w)
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


def _i32(a):
    import torch
    return torch.tensor(np.asarray(a, dtype=np.int32), dtype=torch.int32, device="cuda:0")


def _rows(lengths, slots, firsts=None):
    """What the kernels read of a step: sequences of ``lengths`` rows that go on at positions ``firsts``."""
    firsts = firsts or [0] * len(lengths)
    return SimpleNamespace(nseq=len(lengths), max_q_len=max(lengths), row_seq=_i32([s for s, n in enumerate(lengths) for _ in range(n)]),
                           row_pos=_i32([f + i for n, f in zip(lengths, firsts) for i in range(n)]), seq_slot=_i32(slots), seq_q_len=_i32(lengths),
                           seq_q_start=_i32(np.concatenate([[0], np.cumsum(lengths)[:-1]])))


@pytest.mark.parametrize("narrow", [0, 1 << 30])
@pytest.mark.parametrize("per_channel", [True, False])
@pytest.mark.parametrize("sizes", [(2, 1, 16, 24), (3, 3, 20, 33), (1, 1, 1, 1), (2, 2, 128, 128), (4, 2, 256, 40), (6, 2, 100, 64), (2, 1, 64, 16), (2, 2, 32, 4)])
def test_the_gated_delta_rule(sizes, per_channel, narrow):
    """Prompts whose lengths are no multiples of the tokens taken together, in pieces that start anywhere among them, and token by
    token; decays from one down to zero."""
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    H, G, d, dv = sizes
    if d == 1 and per_channel:
        pytest.skip("one key channel: the two decays are one")
    lengths, slots = [37, 1, 12, 70], [1, 3, 0, 4]
    rows, D = sum(lengths), (H * d if per_channel else H)
    rng = np.random.default_rng(sum(sizes))
    unit = lambda *shape: P.unit_length(rng.standard_normal(shape))
    k = unit(rows, G, d)
    k[1::3] = P.unit_length(k[1::3] + 2.0 * k[0:-1:3][:len(k[1::3])])       # keys that share a direction with the one before
    x = _f32(np.concatenate([unit(rows, G, d).reshape(rows, -1), k.reshape(rows, -1), rng.standard_normal((rows, H * dv)), np.ones((rows, 2))], -1))
    z = _f32(np.concatenate([2.0 * rng.standard_normal((rows, H)), 2.0 * rng.standard_normal((rows, D))], -1))
    z[5, H:] += 60.0                                                         # decays of zero
    rate, bias = _f32(rng.uniform(-3.0, 1.5, H)), _f32(rng.uniform(-6.0, 1.0, D))
    b = lambda t: t.double().cpu().numpy()
    xs, of = b(x), np.arange(H) // (H // G)
    q, kk, v = xs[:, :G * d].reshape(rows, G, d)[:, of], xs[:, G * d:2 * G * d].reshape(rows, G, d)[:, of], xs[:, 2 * G * d:-2].reshape(rows, H, dv)
    g = np.exp(-np.exp(b(rate))[None, :, None] * P.softplus(b(z)[:, H:] + b(bias)).reshape(rows, H, -1))
    beta = P.sigmoid(b(z)[:, :H])
    starts = np.concatenate([[0], np.cumsum(lengths)])
    want = np.concatenate([P.delta_recurrence(q[a:e], kk[a:e], v[a:e], g[a:e], beta[a:e]) for a, e in zip(starts, starts[1:])])
    scale = max(1.0, np.abs(want).max())
    state = torch.zeros((5, H, d * dv), dtype=torch.float32, device="cuda:0")

    def run(pick, batch):
        out = torch.zeros((len(pick), H * dv), dtype=torch.float32, device="cuda:0")
        zz = z[pick].contiguous()
        ops.gated_delta(x[pick].contiguous(), H, G, d, dv, zz[:, H:], bias, rate, zz[:, :H], state, out, batch, narrow_below=narrow)
        return out.cpu().numpy().reshape(-1, H, dv)
    got = run(list(range(rows)), _rows(lengths, slots))
    assert np.abs(got - want).max() / scale < 2e-5
    assert state[2].abs().max().item() == 0.0
    whole = state.clone()
    state.zero_()
    at = [0] * 4
    for portion in ([3, 1, 2, 5], [2, 0, 4, 1], [1, 0, 1, 1], [20, 0, 5, 40], [1, 0, 0, 1]):
        live = [i for i in range(4) if portion[i] > 0]
        pick = [starts[i] + at[i] + j for i in live for j in range(portion[i])]
        got = run(pick, _rows([portion[i] for i in live], [slots[i] for i in live]))
        assert np.abs(got - want[pick]).max() / scale < 2e-5
        at = [a + n for a, n in zip(at, portion)]
    for t in range(at[0], 37):          # the rest of the first sequence token by token
        assert np.abs(run([t], _rows([1], [1]))[0] - want[t]).max() / scale < 2e-5
    assert (state[1] - whole[1]).abs().max().item() < 2e-5 * scale
    assert state[2].abs().max().item() == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(4, 2, 3, 16, 24), (3, 1, 1, 11, 7), (2, 2, 2, 64, 64), (1, 1, 2, 128, 200), (2, 2, 4, 128, 128)])
@pytest.mark.parametrize("taps", [None, 1, 2, 3, 4, 7, 16])
def test_the_short_convolution_in_portions_and_token_by_token(taps, sizes, dtype):
    """Bias, convolution, silu, unit queries and keys into packed float32 rows; few rows a step, many, and single tokens."""
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    QH, KH, VH, d, dv = sizes
    C = (QH + KH) * d + VH * dv
    td = getattr(torch, dtype)
    rng = np.random.default_rng(C + (taps or 0))
    n = [150, 168]
    u = [torch.tensor(rng.standard_normal((m, C + 3)), dtype=torch.float32).to(td).cuda() for m in n]
    bias = _f32(0.3 * rng.standard_normal(C))
    conv = None if taps is None else _f32(0.5 * rng.standard_normal((taps, C)))
    want = []
    for t in u:
        y = t.double().cpu().numpy()[:, :C] + bias.double().cpu().numpy()
        y = P.silu(y if conv is None else P.convolution(y, conv.double().cpu().numpy().T))
        q, k = P.unit_length(y[:, :QH * d].reshape(-1, QH, d)) * 0.25, P.unit_length(y[:, QH * d:(QH + KH) * d].reshape(-1, KH, d))
        want.append(np.concatenate([q.reshape(len(y), -1), k.reshape(len(y), -1), y[:, (QH + KH) * d:]], -1))
    state = torch.zeros((3, max(1, (taps or 1) - 1) * C), dtype=torch.float32, device="cuda:0")
    at, slots = [0, 0], [2, 0]
    for portion in ([3, 5], [1, 1], [2, 1], [1, 4], [60, 81], [1, 1], [2, 2], [60, 50], [2, 2]):
        x = torch.cat([u[s][at[s]:at[s] + portion[s]] for s in range(2)]).contiguous()
        out = torch.zeros((x.shape[0], C), dtype=torch.float32, device="cuda:0")
        ops.short_conv(x, out, QH, KH, VH, d, dv, conv, state, _rows(portion, slots, at), bias=bias, silu=True, norm=ops.HEAD_NORM_UNIT, eps=P.UNIT_EPS,
                       q_scale=0.25)
        w = np.concatenate([want[s][at[s]:at[s] + portion[s]] for s in range(2)])
        assert np.abs(out.cpu().numpy() - w).max() < 3e-5, portion
        at = [a + m for a, m in zip(at, portion)]
    assert state[1].abs().max().item() == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pairs", [True, False])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 8), (3, 1, 11, 7, 6), (4, 2, 128, 128, 64), (2, 2, 64, 32, 64), (1, 1, 200, 16, 0)])
def test_rotated_and_normed_heads_in_the_cache(sizes, pairs, dtype):
    """Rotation with a factor on cosines and sines, the norm behind it, queries in a buffer, keys and values in their pages."""
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    H, G, d, dv, rot = sizes
    td, C, taps = getattr(torch, dtype), (H + G) * d + G * dv, 3
    rng = np.random.default_rng(sum(sizes))
    conv = _f32(0.5 * rng.standard_normal((taps, C)))
    freqs, mag = P.frequencies(rot, 200.0, RAMP) if rot else (np.zeros(0), 1.0)
    ang = np.arange(512)[:, None] * freqs[None, :]
    cos, sin = (_f32(mag * np.cos(ang)), _f32(mag * np.sin(ang))) if rot else (None, None)
    T = 260
    x = torch.tensor(rng.standard_normal((T, C)), dtype=torch.float32).to(td).cuda()
    y = P.convolution(x.double().cpu().numpy(), conv.double().cpu().numpy().T)

    def turned(t):
        if rot and pairs:
            t = P.rotate_pairs(t, freqs, mag)
        elif rot:
            h = rot // 2
            c, s = mag * np.cos(ang[:T])[:, None], mag * np.sin(ang[:T])[:, None]
            a, b = t[..., :h].copy(), t[..., h:rot].copy()
            t = t.copy()
            t[..., :h], t[..., h:rot] = a * c - b * s, b * c + a * s
        return P.unit_rms(t, 1e-5)
    want_q, want_k = turned(y[:, :H * d].reshape(T, H, d)), turned(y[:, H * d:(H + G) * d].reshape(T, G, d))
    want_v = y[:, (H + G) * d:].reshape(T, G, dv)
    perm = [3, 0, 5, 1, 4, 2]
    k_plane, v_plane = (torch.zeros((6, G, 64, n), dtype=td, device="cuda:0") for n in (d, dv))
    state = torch.zeros((2, (taps - 1) * C), dtype=torch.float32, device="cuda:0")
    table = _i32([[0] * 6, perm])
    got_q, at = [], 0
    for n in (150, 1, 1, 2, 60, 1, 45):
        q = torch.zeros((n, H * d), dtype=td, device="cuda:0")
        ops.short_conv(x[at:at + n], q, H, G, G, d, dv, conv, state, _rows([n], [1], [at]), norm=ops.HEAD_NORM_RMS, eps=1e-5, cos=cos, sin=sin,
                       rotary_dim=rot, pairs=pairs, planes=(table, k_plane, v_plane))
        got_q.append(q.double().cpu().numpy())
        at += n
    tol = 2e-5 if dtype == "float32" else 2e-2
    from_pages = lambda plane: np.stack([plane.double().cpu().numpy()[perm[p // 64], :, p % 64] for p in range(T)])
    close_to = lambda got, want: np.abs(got - want).max() / max(1.0, np.abs(want).max()) < tol
    assert close_to(np.concatenate(got_q).reshape(T, H, d), want_q) and close_to(from_pages(k_plane), want_k) and close_to(from_pages(v_plane), want_v)


@pytest.mark.parametrize("out_dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows, width", [(5, 45), (700, 64), (3, 2048), (700, 2048), (2, 4096), (2, 5000), (4, 1030), (3, 9000)])
def test_two_outputs_between_sublayers(rows, width, out_dtype):
    """A sublayer that left two outputs; the planes' weighted sum where a pass begins again; the result in the place it is made from."""
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    rng = np.random.default_rng(rows + width)
    r = lambda *shape: _f32(rng.standard_normal(shape))
    weight = lambda: _f32(1 + 0.3 * rng.standard_normal(width))
    planes, y, y2 = r(2, rows, width), r(rows, width), 3 * r(rows, width)
    yw, w1, w2, nw = weight(), weight(), weight(), weight()
    d = lambda t: t.double().cpu().numpy()
    both = P.rms_norm(d(y), d(w1), 1e-3) + P.rms_norm(d(y2), d(w2), 1e-3)
    v = d(planes[1]) + P.rms_norm(both, d(yw), 1e-4)
    x = v + d(planes[0])
    want = P.rms_norm(x, d(nw), 1e-5)
    tol = 3e-5 if out_dtype == "float32" else 4e-2
    out = torch.zeros((rows, width), dtype=getattr(torch, out_dtype), device="cuda:0")
    start = torch.zeros((rows, width), dtype=torch.float32, device="cuda:0")
    common = dict(base=planes[1], norm_weight=nw, eps=1e-5, y=y, y_weight=yw, y_eps=1e-4, pair=(y2, w1, w2, 1e-3))
    pick = [rows - 1, 0, rows // 2]
    gathered = torch.zeros((3, width), dtype=out.dtype, device="cuda:0")
    ops.sandwich_rows(out=gathered, rows=_i32(pick), **common)
    ops.sandwich_rows(out=out, result=planes[1], planes=planes, n_planes=1, average=_f32([1.0, 1.0]), x_out=start, **common)
    torch.cuda.synchronize()
    assert np.abs(d(planes[1]) - v).max() < 3e-5 and np.abs(d(start) - x).max() < 3e-5 and np.abs(d(out) - want).max() < tol
    assert np.abs(d(gathered) - P.rms_norm(v, d(nw), 1e-5)[pick]).max() < tol


@pytest.mark.parametrize("sizes", [(8, 2, 4, 2), (16, 4, 2, 1), (6, 3, 3, 2), (5, 3, 5, 4), (512, 8, 16, 3), (40, 6, 1, 1), (4, 4, 2, 2), (96, 10, 48, 7)])
def test_the_choice_inside_the_groups_with_the_largest_scores(sizes):
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    E, top, count, keep = sizes
    rows = 61
    z = _f32(2 * np.random.default_rng(sum(sizes)).standard_normal((rows, E)))
    dense, index, weight = torch.zeros((rows, E), device="cuda:0"), torch.zeros((rows, top), dtype=torch.int32, device="cuda:0"), torch.zeros((rows, top), device="cuda:0")
    ops.moe_route(z, top, 0.0, dense, index, weight, renorm=False, groups=count, keep_groups=keep, group_rank="largest")
    torch.cuda.synchronize()
    # the plain route reads logits as a product with an identity
    want_i, want_w = P.route(z.double().cpu().numpy(), {"router": np.eye(E)}, "", {"experts": E, "top": top, "groups": {"count": count, "keep": keep}})
    assert (index.cpu().numpy() == want_i).all() and np.abs(weight.cpu().numpy() - want_w).max() < 1e-5
    full = np.zeros((rows, E))
    np.put_along_axis(full, want_i, want_w, -1)
    assert np.abs(dense.cpu().numpy() - full).max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 3, 16, 17, 100, 230])
@pytest.mark.parametrize("kind", [(8, 2, 24, 4, 2), (12, 1, 48, 3, 1), (3, 3, 8, None, None), (6, 4, 32, 2, 2), 56, 9])
def test_feed_forward_rows(rows, kind, dtype):
    """The feed-forwards by themselves in every range of rows."""
    import torch
    from gophonic_b200 import registry
    from gophonic_b200.config import LefalixConfig
    from gophonic_b200.engine.model import make_runtime
    hidden = 64
    cfg = config([delta(mlp=dense(kind) if isinstance(kind, int) else moe(*kind))], width=hidden)
    w = {k[len("l0.mlp."):]: v for k, v in P.random_weights(cfg, seed=rows + 7).items() if k.startswith("l0.mlp.")}
    spec = LefalixConfig.from_dict(cfg).model_spec().layers[0].feed_forward
    td = getattr(torch, dtype)
    ff = registry.part_class("feed_forward", spec.kind)(spec, "", {k: torch.tensor(v, dtype=torch.float32).to(td).cuda() for k, v in w.items()},
                                                        make_runtime(dtype, "cuda:0"))
    x = torch.tensor(np.random.default_rng(rows).standard_normal((rows, hidden)), dtype=torch.float32).to(td).cuda()
    out = torch.zeros((rows, hidden), dtype=torch.float32, device="cuda:0")
    ff.forward(None, x, out)
    torch.cuda.synchronize()
    h = x.double().cpu().numpy()
    want = P.dense(h, w, "") if isinstance(kind, int) else P.mixture(h, w, "", cfg["layers"][0]["mlp"])
    close(out.cpu().numpy(), want, 3e-5 if dtype == "float32" else 4e-2, MOST[dtype])


def test_gelu():
    import torch
    from gophonic_b200 import ops
    ops.use_device(0)
    for n in (777, 4096):
        z = _f32(np.concatenate([[-50.0, 50.0, 0.0], 3 * np.random.default_rng(1).standard_normal(n - 3)]))
        want = P.gelu(z.double().cpu().numpy())
        half = z.bfloat16()
        ops.gelu(z)
        assert np.abs(z.double().cpu().numpy() - want).max() < 1e-5
        want = P.gelu(half.double().cpu().numpy())
        ops.gelu(half)
        torch.cuda.synchronize()
        assert (np.abs(half.double().cpu().numpy() - want) / (1e-2 + np.abs(want))).max() < 5e-3


def test_an_added_start_ahead_of_plain_blocks():
    """The junction for blocks that keep one residual: what is still owed to it is added too, and the embedding output stays."""
    import torch
    from gophonic_b200.config import AddStartSpec
    from gophonic_b200.engine.model import make_runtime
    from gophonic_b200.parts import AddStart
    rng = np.random.default_rng(3)
    h, owed, x0 = (_f32(rng.standard_normal((5, 33))) for _ in range(3))
    junction = AddStart(AddStartSpec(hidden=33), "", {}, make_runtime("float32", "cuda:0"))
    before = x0.clone()
    assert torch.allclose(junction.forward(None, h, owed, x0), h + owed + x0, atol=1e-6)
    assert torch.allclose(junction.forward(None, h, None, x0), h + x0, atol=1e-6) and torch.equal(before, x0)


def test_mixers_side_by_side_under_any_block():
    """``forward`` leaves the two outputs' normed sum for blocks that take one output."""
    import torch
    from gophonic_b200.config import LefalixConfig
    from gophonic_b200.engine.model import make_runtime
    from gophonic_b200.parts import Parallel
    spec = LefalixConfig.from_dict(config([pair()])).model_spec().layers[0].mixer
    rng = np.random.default_rng(4)
    rt = make_runtime("float32", "cuda:0")
    tensors = {d.name: _f32(rng.standard_normal([n or 10 for n in d.shape])) for d in Parallel.declare(spec, "")}
    mixer = Parallel(spec, "", tensors, rt)
    a, b = (_f32(rng.standard_normal((7, 64))) for _ in range(2))
    mixer.forward_pair = lambda batch, x, cache: (a, b, *mixer.weights, float(spec.eps))
    out = torch.ones((7, 64), dtype=torch.float32, device="cuda:0")
    mixer.forward(None, None, out, None)
    d = lambda t: t.double().cpu().numpy()
    want = 0.5 * (P.rms_norm(d(a), d(tensors["left.out"]), spec.eps) + P.rms_norm(d(b), d(tensors["right.out"]), spec.eps))
    assert np.abs(d(out) - want).max() < 1e-5


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
    """-random-config NAME -write-model DIR, then -model DIR: the plain model reads the written folder and would have chosen the
    same tokens."""
    out = tmp_path / "written"
    run = lambda *a: subprocess.run([sys.executable, "-m", "gophonic_b200", *a], cwd=ROOT, capture_output=True, text=True, timeout=600)
    r = run("-random-config", "lefalix-tiny", "-weights-seed", "4", "-write-model", str(out))
    assert r.returncode == 0, r.stderr[-2000:]
    cfg, w = P.read_model(str(out))
    assert cfg["architecture"] == "Lefalix" and cfg["loop"]["times"] == 2
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
