"""A plain, slow Zenorax decoder in numpy float64: whole sequences, no cache, one function for each
mechanism.  It is the oracle of the Zenorax tests and shares no code with ``gophonic_b200``.

A Zenorax layer norms in front of and behind each sublayer, adds to what its mixer reads a short causal
convolution of it, and hands on a weighted sum of the embedding output and of every layer's result so far:

    h = norm1(x),  h <- h + conv(h),  x <- x + norm1b(mixer(h)),  x <- x + norm2b(mixture(norm2(x)))
    X_(i+1) = x,   x <- sum_(j <= i+1) dwa_i[j] X_j          (X_0: the embedding output)

Mixers: latent attention (queries, keys and values from low-rank latents, an output gate), grouped-query
attention whose values are its unrotated keys (a norm without a weight behind the rotation, a learned sink) and
HGRN2 (a matrix state a head whose forget gate also decides what is written).  The feed-forward is a mixture of
squared-relu experts chosen inside the best groups by corrected sigmoid scores.  The head is the embedding table
and its logits are capped by a tanh.

Everything takes the weights as a dict name -> float64 array and the configuration as the parsed config.json.
"""
from __future__ import annotations

import math
from typing import Dict, List, Tuple

import numpy as np

from .pugalix_plain import from_bf16_bits, read_model, to_bf16_bits, write_model  # noqa: F401  (file helpers of the tests)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


# ---- what surrounds the sublayers ------------------------------------------------------------------
def input_convolution(h, w):
    """h_t + sum_j w[:, j] h_(t - taps + 1 + j), zeros before the start.  h: [T, width], w: [width, taps]."""
    taps = w.shape[1]
    out = h.copy()
    for j in range(taps):
        back = taps - 1 - j
        for t in range(back, h.shape[0]):
            out[t] += w[:, j] * h[t - back]
    return out


def depth_average(results, weights):
    """sum_j weights[j] results[j]; ``results`` holds X_0 .. X_(i+1)."""
    assert len(results) == len(weights)
    out = np.zeros_like(results[0])
    for x, a in zip(results, weights):
        out += a * x
    return out


# ---- rotations -------------------------------------------------------------------------------------
def frequencies(dims: int, base: float) -> np.ndarray:
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])


def linear_frequencies(dims, base, scaling=None):
    f = frequencies(dims, base)
    return f if not scaling else f / scaling["factor"]


def ramp_frequencies(dims, base, scaling=None) -> Tuple[np.ndarray, float]:
    """Frequencies and the factor on cos and sin.  ``scaling`` {factor, original, fast, slow}: the channel number at
    which a wave turns t times in ``original`` positions is dim(t); below dim(fast) a frequency stays, above
    dim(slow) it is divided by factor, and a straight line in the channel's number blends the two between."""
    f = frequencies(dims, base)
    if not scaling:
        return f, 1.0
    factor, original, fast, slow = scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"]

    def dim(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim(fast)), 0), min(math.ceil(dim(slow)), dims - 1)
    out = f.copy()
    for i in range(len(f)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * r + f[i] * (1.0 - r)
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, freqs, layout: str, magnitude: float = 1.0):
    """x: [T, heads, d]; the first 2 len(freqs) channels of every head turn.  layout "half": channel i with
    channel i + n; "pairs": channel 2i with channel 2i + 1 (n = len(freqs)); cos and sin times ``magnitude``."""
    n = len(freqs)
    out = x.copy()
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freqs[None, :]
    c, s = magnitude * np.cos(ang)[:, None, :], magnitude * np.sin(ang)[:, None, :]
    if layout == "half":
        u, v = x[..., :n], x[..., n:2 * n]
        out[..., :n], out[..., n:2 * n] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
        out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


# ---- mixers ----------------------------------------------------------------------------------------
def causal_attention(q, k, v, scale, sink=None):
    """q, k: [T, d], v: [T, dv] -> [T, dv]; ``sink``: the denominator holds exp(sink) besides the keys' terms."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    s = np.where(np.arange(T)[None, :] <= np.arange(T)[:, None], s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return (e / total) @ v


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dr, R, dv = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(T, H, d + dr)
    ckv = h @ w[p + "dkv"].T
    c = rms_norm(ckv[:, :R], w[p + "dkv.norm"], eps)
    k_rot, q_rot = ckv[:, R:], q[:, :, d:]
    if dr > 0:
        f, mag = ramp_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        k_rot = rotate(k_rot.reshape(T, 1, dr), np.arange(T), f, "pairs", mag)[:, 0]
        q_rot = rotate(q_rot, np.arange(T), f, "pairs", mag)
    k_plain = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        qq = np.concatenate([q[:, hd, :d], q_rot[:, hd]], axis=-1)
        kk = np.concatenate([k_plain[:, hd], k_rot], axis=-1)
        out[:, hd] = causal_attention(qq, kk, v[:, hd], m["scale"])
    gate = sigmoid(h @ w[p + "g"].T)
    return (out.reshape(T, H * dv) * gate) @ w[p + "o"].T


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, G, d)
    v = k.copy()                                       # as projected
    rot = m.get("rot")
    if rot and rot["dims"] > 0:
        f = linear_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate(q, np.arange(T), f, "half"), rotate(k, np.arange(T), f, "half")
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    out = np.zeros((T, H, d))
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = causal_attention(q[:, hd], k[:, g], v[:, g], m["scale"], w[p + "sink"][hd])
    return out.reshape(T, H * d) @ w[p + "o"].T


def hgrn2(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(T, H, d)
    S = np.zeros((H, d, dv))
    out = np.zeros((T, H, dv))
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return rms_norm(out, w[p + "norm"], eps).reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": attention, "hgrn2": hgrn2}


# ---- feed-forward ----------------------------------------------------------------------------------
def expert(h, w, p):
    return (np.maximum(h @ w[p + "up"].T, 0.0) ** 2) @ w[p + "down"].T


def route(h, w, p, router):
    """(chosen experts [T, top], their weights).  Scores s = sigmoid(z); an expert is chosen by s + correction among
    the experts of the groups whose two largest such numbers add up to most; the weights are s."""
    s = sigmoid(h @ w[p + "router"].T)
    choice = s + w[p + "correction"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    T, E = s.shape
    per = E // groups["count"]
    by_group = choice.reshape(T, groups["count"], per)
    strength = np.sort(by_group, axis=-1)[:, :, -2:].sum(-1)
    kept = np.argsort(-strength, axis=-1, kind="stable")[:, :groups["keep"]]
    allowed = np.zeros((T, groups["count"]), dtype=bool)
    np.put_along_axis(allowed, kept, True, axis=-1)
    choice = np.where(np.repeat(allowed, per, axis=-1), choice, -np.inf)
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
def soft_cap(z, cap):
    return z if cap is None else cap * np.tanh(z / cap)


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, return_layers: bool = False):
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    results, after = [x], []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(rms_norm(x, w[p + "norm1"], eps), w[p + "canon1"])
        x = x + rms_norm(MIXERS[L["type"]](h, w, p + "mix.", L["mixer"], eps), w[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            y = mixture(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        after.append(x.copy())
    logits = soft_cap(rms_norm(x, w["final.norm"], eps) @ w["embed"].T, cfg.get("logit_softcap"))
    return (logits, np.stack(after)) if return_layers else logits


# ---- test models -----------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "canon1": (W, cfg["canon"]["taps"]), p + "dwa": (i + 2,)})
        H, d = m["heads"], m["dim"]
        if L["type"] == "hgrn2":
            dv = m["vdim"]
            out.update({q + "q": (H * d, W), q + "f": (H * d, W), q + "f.b": (H * d,), q + "lower": (H * d,), q + "v": (H * dv, W),
                        q + "norm": (dv,), q + "o": (W, H * dv)})
        elif L["type"] == "attention":
            G = m.get("kv_heads", H)
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "sink": (H,), q + "o": (W, H * d)})
        else:
            R, Q, dr, dv = m["kv_rank"], m["q_rank"], m["rot_dim"], m["vdim"]
            out.update({q + "dq": (Q, W), q + "dq.norm": (Q,), q + "uq": (H * (d + dr), Q), q + "dkv": (R + dr, W), q + "dkv.norm": (R,),
                        q + "uk": (H * d, R), q + "uv": (H * dv, R), q + "g": (H * dv, W), q + "o": (W, H * dv)})
        mlp = L.get("mlp")
        if mlp is None:
            continue
        E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
        for e in range(E):
            out.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return out


def random_weights(cfg: dict, seed: int, decided: bool = False) -> Dict[str, np.ndarray]:
    """Random weights whose values bfloat16 holds exactly: matrices of deviation 1/sqrt(inputs), norms and averages
    that matter, corrections that move the choice (some choice scores are negative), lower bounds in [0, 1).  With
    ``decided`` the corrections lie further apart than scores reach, so that they alone choose the experts (and the scores
    still weigh them): no rounding can turn a choice, which a layer with norms behind its sublayers would carry into
    every later row."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in last:
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "dwa":
            v = 0.3 * rng.standard_normal(shape)
            v[-1] += 1.0
        elif last == "canon1":
            v = 0.4 * rng.standard_normal(shape)
        elif last == "lower":
            v = rng.uniform(0.0, 0.9, shape)
        elif last == "b":
            v = 1.0 + rng.standard_normal(shape)
        elif last == "sink":
            v = 1.0 + rng.standard_normal(shape)
        elif last == "correction":
            if decided:      # whole groups one behind the other, so that their sums of two lie apart as well
                router = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
                count = (router.get("groups") or {"count": 1})["count"]
                per = shape[0] // count
                ranks = np.concatenate([r * per + rng.permutation(per) for r in rng.permutation(count)])
                v = 1.5 * (ranks - shape[0] // 2)
            else:
                v = 0.4 * rng.standard_normal(shape) - 0.5
        elif name == "embed":
            v = rng.standard_normal(shape)
        elif last == "router":
            v = 2.0 * rng.standard_normal(shape) / math.sqrt(shape[-1])
        elif last in ("q", "k", "uq", "uk"):
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
