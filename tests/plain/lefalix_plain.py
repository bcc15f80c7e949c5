"""A plain, slow Lefalix decoder in numpy float64: whole sequences, no cache, one function for each
mechanism.  It is the oracle of the Lefalix tests and shares no code with ``gophonic_b200``.

A Lefalix layer norms in front of and behind each sublayer,

    x <- x + norm1b(mixer(norm1(x))),   x <- x + norm2b(feed_forward(norm2(x))),

and a stretch of layers may run several times with the same weights; ahead of every pass but the first the embedding
output is added to x.  Mixers: a gated delta rule whose decay is a number per key channel, and a pair of mixers side by
side (windowed softmax attention behind a short convolution, with a learned sink; a gated delta rule whose decay is one
number per head) whose outputs are normed and averaged.  Feed-forwards: down(gelu(up x)), or a mixture of gated experts
chosen inside the best groups.

Everything takes the weights as a dict name -> float64 array and the configuration as the parsed config.json.
"""
from __future__ import annotations

import math
from typing import Dict, List, Tuple

import numpy as np

from .pugalix_plain import from_bf16_bits, read_model, to_bf16_bits, write_model  # noqa: F401  (file helpers of the tests)

UNIT_EPS = 1e-6      # under the root of a unit vector's length


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    """z times the normal law's distribution function at z."""
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def unit_length(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + UNIT_EPS)


# ---- the short convolution -------------------------------------------------------------------------
def convolution(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start.  u: [T, channels], w: [channels, taps]."""
    taps = w.shape[1]
    out = np.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        for t in range(back, u.shape[0]):
            out[t] += w[:, j] * u[t - back]
    return out


# ---- rotation --------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None) -> Tuple[np.ndarray, float]:
    """base^(-2i/dims) and the factor on cos and sin.  ``scaling`` {factor, original, fast, slow}: with c(t) the number of the
    channel pair whose wave turns t times in ``original`` positions, pairs up to c(fast) keep their frequency, pairs from
    c(slow) on have it divided by ``factor``, and a straight line in the pair's number blends the two between."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, original, fast, slow = scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"]

    def c(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(c(fast)), 0), min(math.ceil(c(slow)), dims - 1)
    out = f.copy()
    for i in range(len(f)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * r + f[i] * (1.0 - r)
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, freqs, magnitude=1.0):
    """x: [T, heads, d]; channels 2i and 2i + 1 turn by t * freqs[i], i < len(freqs); the rest stays."""
    n = len(freqs)
    out = x.copy()
    ang = np.arange(x.shape[0], dtype=np.float64)[:, None] * freqs[None, :]
    c, s = magnitude * np.cos(ang)[:, None, :], magnitude * np.sin(ang)[:, None, :]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


# ---- attention -------------------------------------------------------------------------------------
def windowed_attention(q, k, v, scale, window, sink):
    """q, k: [T, d], v: [T, dv] -> [T, dv].  i sees j with 0 <= i - j < window (None: every j <= i); the denominator
    holds exp(sink) besides the keys' terms."""
    T = q.shape[0]
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = back >= 0
    if window:
        seen &= back < window
    s = np.where(seen, (q @ k.T) * scale, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - top)
    return (e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))) @ v


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    proj = lambda n: convolution(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]) if m.get("conv") else h @ w[p + n].T + w[p + n + ".b"]
    q, k, v = proj("q").reshape(T, H, d), proj("k").reshape(T, G, d), proj("v").reshape(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"] > 0:
        f, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_pairs(q, f, mag), rotate_pairs(k, f, mag)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    window = (m.get("mask") or {}).get("size")
    out = np.zeros((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = windowed_attention(q[:, hd], k[:, g], v[:, g], m["scale"], window, w[p + "sink"][hd])
    return out.reshape(T, H * dv) @ w[p + "o"].T + w[p + "o.b"]


# ---- the gated delta rule --------------------------------------------------------------------------
def delta_recurrence(q, k, v, g, beta):
    """q, k: [T, H, d], v: [T, H, dv], g: [T, H, d] (or [T, H, 1]), beta: [T, H] -> [T, H, dv]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def delta_inputs(h, w, p, m):
    """Unit queries (scaled) and keys and the values, one row a head."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)

    def proj(n):
        u = h @ w[p + n].T
        return silu(convolution(u, w[p + n + ".conv"])) if m.get("conv") else silu(u)
    q, k = unit_length(proj("q").reshape(T, G, d)) * d ** -0.5, unit_length(proj("k").reshape(T, G, d))
    of = np.arange(H) // (H // G)
    return q[:, of], k[:, of], proj("v").reshape(T, H, dv)


def gated_delta(h, w, p, m, eps):
    """One decay a head; the output gate is silu of a projection."""
    T = h.shape[0]
    H, dv = m["heads"], m["vdim"]
    q, k, v = delta_inputs(h, w, p, m)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = delta_recurrence(q, k, v, g[:, :, None], sigmoid(h @ w[p + "b"].T))
    o = rms_norm(o, w[p + "norm"], eps) * silu(h @ w[p + "g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def channel_delta(h, w, p, m, eps):
    """A decay a head and key channel, out of two small matrices; the output gate is sigmoid of two more."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = delta_inputs(h, w, p, m)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(z.reshape(T, H, d)))
    o = delta_recurrence(q, k, v, g, sigmoid(h @ w[p + "b"].T))
    o = rms_norm(o, w[p + "norm"], eps) * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    left = attention(h, w, p + "left.", m["left"], eps)
    right = gated_delta(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


MIXERS = {"parallel": side_by_side, "channel_delta": channel_delta}


# ---- feed-forward ----------------------------------------------------------------------------------
def dense(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, router):
    """(chosen experts [T, top], their weights).  A group of neighbours counts as its largest score; the weights are the
    softmax scores over all experts."""
    z = h @ w[p + "router"].T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    groups = router.get("groups") or {"count": 1, "keep": 1}
    T, E = s.shape
    per = E // groups["count"]
    strength = s.reshape(T, groups["count"], per).max(axis=-1)
    kept = np.argsort(-strength, axis=-1, kind="stable")[:, :groups["keep"]]
    allowed = np.zeros((T, groups["count"]), dtype=bool)
    np.put_along_axis(allowed, kept, True, axis=-1)
    choice = np.where(np.repeat(allowed, per, axis=-1), s, -np.inf)
    index = np.argsort(-choice, axis=-1, kind="stable")[:, :router["top"]]
    return index, np.take_along_axis(s, index, axis=-1)


def mixture(h, w, p, mlp):
    index, weight = route(h, w, p, mlp["router"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, js = np.nonzero(index == e)
        if len(rows):
            out[rows] += weight[rows, js][:, None] * expert(h[rows], w, f"{p}e{e}.")
    return out


# ---- the model -------------------------------------------------------------------------------------
def layer_runs(cfg) -> List[Tuple[int, bool]]:
    """(layer, whether the embedding output is added ahead of it) in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": n, "times": 1}
    runs = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, return_layers: bool = False):
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][np.asarray(tokens)]
    x, after = x0, []
    for i, again in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        y = MIXERS[L["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            y = dense(h, w, p + "mlp.") if mlp["kind"] == "dense" else mixture(h, w, p + "mlp.", mlp)
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        after.append(x.copy())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(after)) if return_layers else logits


# ---- test models -----------------------------------------------------------------------------------
def _delta_shapes(q, m, W, taps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    out = {q + "q": (G * d, W), q + "k": (G * d, W), q + "v": (H * dv, W), q + "b": (H, W), q + "A_log": (H,), q + "norm": (dv,), q + "o": (W, H * dv)}
    if taps:
        out.update({q + "q.conv": (G * d, taps), q + "k.conv": (G * d, taps), q + "v.conv": (H * dv, taps)})
    return out


def tensor_shapes(cfg: dict, rank: int = 10, gate_rank: int = 14) -> Dict[str, tuple]:
    """``rank``, ``gate_rank``: inner sizes of the decays' and the gates' small matrices (a file's configuration does not name them)."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if L["type"] == "channel_delta":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            out.update(_delta_shapes(q, m, W, m.get("conv")))
            out.update({q + "a1": (rank, W), q + "a2": (H * d, rank), q + "dt_bias": (H * d,), q + "g1": (gate_rank, W), q + "g2": (H * dv, gate_rank)})
        else:
            a, r = m["left"], m["right"]
            H, d, dv = a["heads"], a["dim"], a["vdim"]
            G = a.get("kv_heads", H)
            for n, size in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out.update({f"{q}left.{n}": (size, W), f"{q}left.{n}.b": (size,)})
                if a.get("conv"):
                    out[f"{q}left.{n}.conv"] = (size, a["conv"])
            out.update({q + "left.sink": (H,), q + "left.o": (W, H * dv), q + "left.o.b": (W,)})
            out.update(_delta_shapes(q + "right.", r, W, r.get("conv")))
            out.update({q + "right.a": (r["heads"], W), q + "right.dt_bias": (r["heads"],), q + "right.g": (r["heads"] * r["vdim"], W),
                        q + "left.out": (W,), q + "right.out": (W,)})
        mlp = L.get("mlp")
        if mlp is None:
            continue
        out.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if mlp["kind"] == "dense":
            out.update({p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
            continue
        E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[p + "mlp.router"] = (E, W)
        for e in range(E):
            out.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return out


def random_weights(cfg: dict, seed: int, rank: int = 10, gate_rank: int = 14, decided: bool = False) -> Dict[str, np.ndarray]:
    """Random weights whose values bfloat16 holds exactly: matrices of deviation 1/sqrt(inputs), norms, biases and sinks
    that matter, decays from nearly one to a few tenths.  With ``decided`` all embeddings share a large part along one direction
    and the routers read that direction above all, so that the experts' order is nearly the same for every token and far from a
    tie: no rounding can turn a choice, which a layer with norms behind its sublayers would carry into every later row."""
    rng = np.random.default_rng(seed)
    common = rng.standard_normal(cfg["width"])
    common *= math.sqrt(cfg["width"]) / np.linalg.norm(common)
    w = {}
    for name, shape in tensor_shapes(cfg, rank, gate_rank).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in last or last == "out":
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "conv":
            v = 0.6 * rng.standard_normal(shape)
        elif last == "A_log":
            v = rng.uniform(-2.0, 1.0, shape)
        elif last == "dt_bias":
            v = rng.uniform(-4.0, 0.5, shape)
        elif last == "b" and len(shape) == 1:
            v = 0.5 * rng.standard_normal(shape)
        elif last == "sink":
            v = 1.0 + rng.standard_normal(shape)
        elif name == "embed":
            v = rng.standard_normal(shape) + (3.0 * common if decided else 0.0)
        elif last == "router" and decided:      # whole groups one behind the other
            count = (cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"].get("groups") or {"count": 1})["count"]
            per = shape[0] // count
            ranks = np.concatenate([r * per + rng.permutation(per) for r in rng.permutation(count)]) - shape[0] / 2.0
            v = 0.05 * rng.standard_normal(shape) / math.sqrt(shape[-1]) + np.outer(0.8 * ranks, common) / shape[-1]
        elif last == "router":
            v = 2.0 * rng.standard_normal(shape) / math.sqrt(shape[-1])
        elif last in ("q", "k"):
            v = 2.0 * rng.standard_normal(shape) / math.sqrt(shape[-1])
        else:
            v = rng.standard_normal(shape) / math.sqrt(shape[-1])
        w[name] = from_bf16_bits(to_bf16_bits(v)).reshape(shape)
    return w


def greedy_generate(cfg, w, prompt, n: int) -> Tuple[List[int], List[float]]:
    """``n`` greedy tokens after ``prompt`` and, for each, the margin of its logit over the runner-up."""
    ids, out, margins = list(prompt), [], []
    for _ in range(n):
        logits = forward(cfg, w, ids)[-1]
        order = np.argsort(logits)
        out.append(int(order[-1]))
        margins.append(float(logits[order[-1]] - logits[order[-2]]))
        ids.append(out[-1])
    return out, margins
