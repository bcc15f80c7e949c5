"""Typed configuration of the Lefalix decoder, read from the keys of its ``config.json``.

A Lefalix layer has a norm in front of and behind each sublayer (``SandwichLayerSpec``), and a stretch of layers may run several times
with the same weights, the embedding output being added to the residual ahead of every pass but the first (``AddStartSpec``).  The file
gives ``width``, ``vocab``, ``norm.eps``, ``loop`` {start, stop, times} (layers start .. stop - 1 run ``times`` times; absent: once) and, per entry of
``layers``, ``type`` (the mixer), ``mixer`` (its sizes and constants) and ``mlp``: ``{"kind": "dense", "ff": F}``, ``{"kind": "moe", "expert":
{"ff": F}, "router": {"experts": E, "top": K, "groups": {"count": C, "keep": G}}}`` (``groups`` absent: one) or null.

Mixer ``channel_delta`` (``GatedDeltaSpec``, a decay per key channel): ``heads``, ``kv_heads`` (absent: as many), ``dim``, ``vdim``, ``conv`` (taps;
absent: no convolution).  The ranks of the decays' and the gates' small matrices are the shapes of those tensors; a file may name them as
``rank`` and ``gate_rank``, which random weights need.

Mixer ``parallel`` (``ParallelSpec``): ``left``, windowed softmax attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``, ``scale``, ``mask.size``
(absent: every earlier key), ``rot`` {base, dims, optionally scaling {factor, original, fast, slow}}; biases, a norm without a weight behind
the rotation of neighbouring channels, a learned sink), beside ``right``, the gated delta rule with a decay per head (keys as for
``channel_delta``).

The constants the design fixes stand below and travel in the parts' specs.

Tensor names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.mix.q``, ``l<i>.mix.q.conv``, ``l<i>.mix.A_log``,
``l<i>.mix.left.q.b``, ``l<i>.mix.left.out``, ``l<i>.mix.right.dt_bias``, ``l<i>.mlp.up``, ``l<i>.mlp.e<j>.gate``, ``l<i>.mlp.router``.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, List, Optional, Tuple

from .pugalix import _freeze, _get, _int, _pos, _thaw
from .qwen3 import ConfigError
from .spec import (AddStartSpec, EmbeddingSpec, GatedAttentionSpec, GatedDeltaSpec, GeluSpec, HeadSpec, ModelSpec, MoESpec, NoPositionSpec,
                   PairRotarySpec, ParallelSpec, RMSNormSpec, RampStretch, SandwichLayerSpec, ScheduleEntry)

MIXERS = ("parallel", "channel_delta")
SCALING_KEYS = ("factor", "original", "fast", "slow")
UNIT_EPS = 1e-6         # under the root of a query's or key's length


def _object(d: dict, key: str, where: str) -> dict:
    v = _get(d, key, where)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: '{where}{key}' must be an object")
    return {k: x for k, x in v.items() if x is not None}


def _heads(m: dict, ma: str) -> None:
    heads = _int(m, "heads", ma)
    if "kv_heads" in m and heads % _int(m, "kv_heads", ma):
        raise ConfigError(f"config.json: '{ma}heads' {heads} is not a multiple of '{ma}kv_heads' {m['kv_heads']}")
    for k in ("dim", "vdim"):
        _int(m, k, ma)
    if "conv" in m:
        _int(m, "conv", ma)


def _delta(m: dict, ma: str) -> None:
    _heads(m, ma)
    for k in ("rank", "gate_rank"):
        if k in m:
            _int(m, k, ma)


def _attention(m: dict, ma: str) -> None:
    _heads(m, ma)
    _pos(m, "scale", ma)
    if "mask" in m:
        _int(_object(m, "mask", ma), "size", ma + "mask.")
    if "rot" in m:
        rot, ra = _object(m, "rot", ma), ma + "rot."
        dims = _int(rot, "dims", ra, low=0)
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"config.json: '{ra}dims' {dims} must be even and at most '{ma}dim' {m['dim']}")
        base = _pos(rot, "base", ra)
        if "scaling" in rot:
            for k in SCALING_KEYS:
                _pos(_object(rot, "scaling", ra), k, ra + "scaling.")
            if base == 1.0:
                raise ConfigError(f"config.json: '{ra}base' 1 has no logarithm to scale by")


def _feed_forward(mlp, fa: str) -> None:
    kind = _get(mlp, "kind", fa)
    if kind == "dense":
        _int(mlp, "ff", fa)
        return
    if kind != "moe":
        raise ConfigError(f"config.json: '{fa}kind' is {kind!r}; this design has dense and moe feed-forwards")
    _int(_get(mlp, "expert", fa), "ff", fa + "expert.")
    router, ra = _get(mlp, "router", fa), fa + "router."
    experts, top = _int(router, "experts", ra), _int(router, "top", ra)
    room = experts
    if router.get("groups") is not None:
        ga = ra + "groups."
        count, keep = _int(router["groups"], "count", ga), _int(router["groups"], "keep", ga)
        if experts % count:
            raise ConfigError(f"config.json: '{ra}experts' {experts} do not form {count} equal groups")
        if keep > count:
            raise ConfigError(f"config.json: '{ga}keep' {keep} exceeds its {count} groups")
        room = experts // count * keep
    if top > room:
        raise ConfigError(f"config.json: '{ra}top' {top} exceeds the {room} experts that can be chosen")


@dataclass(frozen=True)
class LefalixLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]      # the mixer's keys, as read (nested dicts as tuples of pairs)
    mlp: Optional[Tuple[Tuple[str, Any], ...]]


@dataclass(frozen=True)
class LefalixConfig:
    width: int
    vocab: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]    # first layer, the one behind the last, passes
    layers: Tuple[LefalixLayer, ...]
    architecture: str = "Lefalix"

    # ---- reading -------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LefalixConfig":
        width, vocab = _int(d, "width", ""), _int(d, "vocab", "")
        eps = _pos(_get(d, "norm", ""), "eps", "norm.")
        raw_layers = _get(d, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[LefalixLayer] = []
        for i, raw in enumerate(raw_layers):
            at = f"layers[{i}]."
            kind = _get(raw, "type", at)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: '{at}type' is {kind!r}; this design has {', '.join(MIXERS)}")
            m, ma = _object(raw, "mixer", at), at + "mixer."
            if kind == "parallel":
                for side, check in (("left", _attention), ("right", _delta)):
                    m[side] = _object(m, side, ma)
                    check(m[side], f"{ma}{side}.")
            else:
                _delta(m, ma)
            mlp = raw.get("mlp")
            if mlp is not None:
                _feed_forward(mlp, at + "mlp.")
                mlp = {k: v for k, v in mlp.items() if v is not None}
            layers.append(LefalixLayer(kind, _freeze(m), None if mlp is None else _freeze(mlp)))
        loop = None
        if d.get("loop") is not None:
            start = _int(d["loop"], "start", "loop.", low=0)
            stop, times = _int(d["loop"], "stop", "loop."), _int(d["loop"], "times", "loop.")
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: 'loop' runs layers {start} .. {stop} - 1 of {len(layers)}")
            loop = (start, stop, times)
        return cls(width=width, vocab=vocab, norm_eps=eps, loop=loop, layers=tuple(layers), architecture=str(d.get("architecture", "Lefalix")))

    # ---- writing -------------------------------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        out = {
            "architecture": self.architecture,
            "layers": [{"type": l.type, "mixer": _thaw(l.mixer), "mlp": None if l.mlp is None else _thaw(l.mlp)} for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def with_layers(self, n: int) -> "LefalixConfig":
        """The first ``n`` layers; a repeated stretch that reaches beyond them ends with them."""
        if not 0 < n <= len(self.layers):
            raise ValueError(f"layers={n} of a configuration with {len(self.layers)}")
        loop = self.loop
        if loop is not None:
            loop = (loop[0], min(loop[1], n), loop[2]) if loop[0] < n else None
        return replace(self, layers=self.layers[:n], loop=loop)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    # ---- derived -------------------------------------------------------------------------
    def _attention(self, m: dict) -> GatedAttentionSpec:
        W, eps, d = self.width, self.norm_eps, m["dim"]
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        position = NoPositionSpec(head_dim=d)
        if rot["dims"] > 0:
            sc = rot.get("scaling")
            position = PairRotarySpec(head_dim=d, rotary_dim=rot["dims"], theta=float(rot["base"]),
                                      scaling=None if sc is None else RampStretch(*(float(sc[k]) for k in SCALING_KEYS)))
        return GatedAttentionSpec(hidden=W, heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), head_dim=d, value_dim=m["vdim"],
                                  scale=float(m["scale"]), position=position, window=(m.get("mask") or {}).get("size", 0), sink=True,
                                  sink_learned=True, bias=True, out_bias=True, qk_norm=RMSNormSpec(size=d, eps=eps), qk_norm_weight=False,
                                  qk_norm_after=True, conv_taps=m.get("conv", 0))

    def _delta(self, m: dict, channel: bool) -> GatedDeltaSpec:
        return GatedDeltaSpec(hidden=self.width, heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), key_dim=m["dim"], value_dim=m["vdim"],
                              eps=self.norm_eps, conv_taps=m.get("conv", 0), unit_eps=UNIT_EPS, channel_decay=channel, rank=m.get("rank"),
                              gate="sigmoid" if channel else "silu", gate_low_rank=channel, gate_rank=m.get("gate_rank"))

    def _mixer(self, l: LefalixLayer):
        m = _thaw(l.mixer)
        if l.type == "channel_delta":
            return self._delta(m, channel=True)
        return ParallelSpec(hidden=self.width, mixers=(self._attention(m["left"]), self._delta(m["right"], channel=False)), eps=self.norm_eps, factor=0.5)

    def _feed_forward(self, l: LefalixLayer):
        if l.mlp is None:
            return None
        W, mlp = self.width, _thaw(l.mlp)
        if mlp["kind"] == "dense":
            return GeluSpec(hidden=W, intermediate=mlp["ff"])
        groups = mlp["router"].get("groups") or {"count": 1, "keep": 1}
        return MoESpec(hidden=W, experts=mlp["router"]["experts"], top=mlp["router"]["top"], intermediate=mlp["expert"]["ff"], score="softmax",
                       renorm=False, weight_on="output", act="swiglu", groups=groups["count"], keep_groups=groups["keep"], group_rank="largest")

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """Every run of a layer in order; the first of each pass but the first through the repeated stretch adds the embedding output."""
        n = len(self.layers)
        start, stop, times = self.loop or (0, n, 1)
        again = AddStartSpec(hidden=self.width)
        runs = [ScheduleEntry(layer=i) for i in range(start)]
        for t in range(times):
            runs += [ScheduleEntry(layer=i, enter=again if t > 0 and i == start else None) for i in range(start, stop)]
        return tuple(runs + [ScheduleEntry(layer=i) for i in range(stop, n)])

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = RMSNormSpec(size=W, eps=eps, tensor="")
        layers = []
        for i, l in enumerate(self.layers):
            ff = self._feed_forward(l)
            ff_norm = None if ff is None else norm
            layers.append(SandwichLayerSpec(prefix=f"l{i}.", mixer=self._mixer(l), feed_forward=ff, mixer_norm=norm, mixer_out_norm=norm,
                                            feed_forward_norm=ff_norm, feed_forward_out_norm=ff_norm))
        spec = ModelSpec(
            architecture=self.architecture, hidden=W, vocab=self.vocab, max_positions=1 << 30, embedding=EmbeddingSpec("embed", self.vocab, W),
            layers=tuple(layers), schedule=self.schedule(), final_norm=norm, final_norm_name="final.norm",
            head=HeadSpec("head", self.vocab, W, tied_to=None))
        spec.validate()
        return spec
