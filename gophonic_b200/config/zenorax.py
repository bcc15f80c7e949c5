"""Typed configuration of the Zenorax decoder, read from the keys of its ``config.json``.

A Zenorax layer has a norm in front of and behind each sublayer, adds a short causal convolution over time to what its
mixer reads, and hands on a learned weighted sum of the embedding output and of every layer's result so far
(``SandwichLayerSpec``).  The file gives ``width``, ``vocab``, ``embedding.scale`` (the factor on the embedding rows),
``norm.eps``, ``canon.taps`` (the convolution's taps), ``logit_softcap`` (cap * tanh(logits / cap); absent: none) and, per
entry of ``layers``, ``type`` (the mixer), ``mixer`` (its sizes and constants) and ``mlp``: ``{"kind": "moe", "expert":
{"ff": F}, "router": {"experts": E, "top": K, "groups": {"count": C, "keep": G}}}`` (``groups`` absent: one) or null.
The head is the embedding table.

Mixer ``latent_attention``: ``heads``, ``dim`` (plain query/key channels a head), ``rot_dim`` (rotated channels, one
rotated key part for all heads, neighbouring channels together), ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot``
(``base``, ``dims`` = ``rot_dim``, optionally ``scaling`` {factor, original, fast, slow}); a gate on the heads.

Mixer ``attention``: ``heads``, ``kv_heads`` (absent: as many as heads), ``dim``, ``vdim`` (``dim``: the values are the keys as
projected), ``scale``, ``rot`` (``dims``, ``base`` and optionally ``scaling`` {factor}; rotate-half over the first ``dims``
channels); a norm without a weight behind the rotation and a learned sink per head.

Mixer ``hgrn2``: ``heads``, ``dim`` (query and forget channels a head), ``vdim``.

The constants the design fixes stand below and travel in the parts' specs.

Tensor names: ``embed``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.canon1``, ``l<i>.dwa``, ``l<i>.mix.q``,
``l<i>.mix.sink``, ``l<i>.mix.dq.norm``, ``l<i>.mix.f.b``, ``l<i>.mix.lower``, ``l<i>.mlp.e<j>.up``, ``l<i>.mlp.router``,
``l<i>.mlp.correction``.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, List, Optional, Tuple

from .kimilix import _number
from .pugalix import _freeze, _get, _int, _pos, _thaw
from .qwen3 import ConfigError
from .spec import (EmbeddingSpec, ForgetStateSpec, GatedAttentionSpec, HeadSpec, LatentAttentionSpec, LinearStretch, ModelSpec, MoESpec,
                   NoPositionSpec, PairRotarySpec, RMSNormSpec, RampStretch, RotarySpec, SandwichLayerSpec, ScheduleEntry)

MIXERS = ("latent_attention", "attention", "hgrn2")
SCALING_KEYS = {"latent_attention": ("factor", "original", "fast", "slow"), "attention": ("factor",)}


def _rot(m: dict, ma: str, kind: str, width: int) -> None:
    """Checks ``m['rot']``: ``dims`` even and at most ``width``, a positive ``base``, a usable ``scaling``."""
    rot, ra = _get(m, "rot", ma), ma + "rot."
    dims = _int(rot, "dims", ra, low=0)
    if dims % 2 or dims > width:
        raise ConfigError(f"config.json: '{ra}dims' {dims} must be even and at most {width}")
    base = _pos(rot, "base", ra)
    if rot.get("scaling") is not None:
        for k in SCALING_KEYS[kind]:
            _pos(rot["scaling"], k, ra + "scaling.")
        if kind == "latent_attention" and base == 1.0:
            raise ConfigError(f"config.json: '{ra}base' 1 has no logarithm to scale by")


@dataclass(frozen=True)
class ZenoraxLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]      # the mixer's keys, as read (nested dicts as tuples of pairs)
    mlp: Optional[Tuple[Tuple[str, Any], ...]]


@dataclass(frozen=True)
class ZenoraxConfig:
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    taps: int
    logit_softcap: Optional[float]
    layers: Tuple[ZenoraxLayer, ...]
    architecture: str = "Zenorax"
    tie_word_embeddings = True              # the head is the embedding table (no field: the file has no such key)

    # ---- reading -------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZenoraxConfig":
        width, vocab = _int(d, "width", ""), _int(d, "vocab", "")
        eps = _pos(_get(d, "norm", ""), "eps", "norm.")
        emb = 1.0 if d.get("embedding") is None else _number(d["embedding"], "scale", "embedding.")
        taps = _int(_get(d, "canon", ""), "taps", "canon.")
        cap = None if d.get("logit_softcap") is None else _pos(d, "logit_softcap", "")
        raw_layers = _get(d, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[ZenoraxLayer] = []
        for i, raw in enumerate(raw_layers):
            at = f"layers[{i}]."
            kind = _get(raw, "type", at)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: '{at}type' is {kind!r}; this design has {', '.join(MIXERS)}")
            m = _get(raw, "mixer", at)
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: '{at}mixer' must be an object")
            ma = at + "mixer."
            m = {k: v for k, v in m.items() if v is not None}
            heads, dim = _int(m, "heads", ma), _int(m, "dim", ma)
            if kind == "hgrn2":
                _int(m, "vdim", ma)
            elif kind == "attention":
                _pos(m, "scale", ma)
                if "kv_heads" in m and heads % _int(m, "kv_heads", ma):
                    raise ConfigError(f"config.json: '{ma}heads' {heads} is not a multiple of '{ma}kv_heads' {m['kv_heads']}")
                if "vdim" in m and _int(m, "vdim", ma) != dim:
                    raise ConfigError(f"config.json: '{ma}vdim' {m['vdim']} must equal '{ma}dim' {dim}: the values are the keys")
                if "rot" in m:
                    _rot(m, ma, kind, dim)
            else:
                _pos(m, "scale", ma)
                for k in ("vdim", "q_rank", "kv_rank"):
                    _int(m, k, ma)
                rd = _int(m, "rot_dim", ma, low=0)
                if rd % 2:
                    raise ConfigError(f"config.json: '{ma}rot_dim' {rd} must be even")
                if rd > 0:
                    _rot(m, ma, kind, rd)
                    if m["rot"]["dims"] != rd:
                        raise ConfigError(f"config.json: '{ma}rot.dims' {m['rot']['dims']} must equal '{ma}rot_dim' {rd}")
            mlp = raw.get("mlp") if isinstance(raw, dict) else None
            if mlp is not None:
                fa = at + "mlp."
                if _get(mlp, "kind", fa) != "moe":
                    raise ConfigError(f"config.json: '{fa}kind' is {mlp['kind']!r}; this design has moe feed-forwards")
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
                mlp = {k: v for k, v in mlp.items() if v is not None}
            layers.append(ZenoraxLayer(kind, _freeze(m), None if mlp is None else _freeze(mlp)))
        return cls(width=width, vocab=vocab, norm_eps=eps, embedding_scale=emb, taps=taps, logit_softcap=cap, layers=tuple(layers),
                   architecture=str(d.get("architecture", "Zenorax")))

    # ---- writing -------------------------------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        out = {
            "architecture": self.architecture,
            "canon": {"taps": self.taps},
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": l.type, "mixer": _thaw(l.mixer), "mlp": None if l.mlp is None else _thaw(l.mlp)} for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    def with_layers(self, n: int) -> "ZenoraxConfig":
        if not 0 < n <= len(self.layers):
            raise ValueError(f"layers={n} of a configuration with {len(self.layers)}")
        return replace(self, layers=self.layers[:n])

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    # ---- derived -------------------------------------------------------------------------
    def _mixer(self, l: ZenoraxLayer):
        W, eps, m = self.width, self.norm_eps, _thaw(l.mixer)
        heads, d = m["heads"], m["dim"]
        if l.type == "hgrn2":
            return ForgetStateSpec(hidden=W, heads=heads, key_dim=d, value_dim=m["vdim"], eps=eps)
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        sc = rot.get("scaling")
        turn = dict(rotary_dim=rot["dims"], theta=float(rot["base"]))
        if l.type == "attention":
            turn["scaling"] = None if sc is None else LinearStretch(float(sc["factor"]))
            position = RotarySpec(head_dim=d, **turn) if rot["dims"] > 0 else NoPositionSpec(head_dim=d)
            return GatedAttentionSpec(hidden=W, heads=heads, kv_heads=m.get("kv_heads", heads), head_dim=d, value_dim=d, scale=float(m["scale"]),
                                      position=position, sink=True, sink_learned=True, qk_norm=RMSNormSpec(size=d, eps=eps),
                                      qk_norm_weight=False, qk_norm_after=True, value_from_key=True)
        turn["scaling"] = None if sc is None else RampStretch(*(float(sc[k]) for k in SCALING_KEYS[l.type]))
        position = PairRotarySpec(head_dim=m["rot_dim"], **turn) if m["rot_dim"] > 0 else NoPositionSpec(head_dim=0)
        return LatentAttentionSpec(hidden=W, heads=heads, head_dim=d, rot_dim=m["rot_dim"], value_dim=m["vdim"], q_rank=m["q_rank"],
                                   kv_rank=m["kv_rank"], scale=float(m["scale"]), position=position, eps=eps, gate=True)

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = RMSNormSpec(size=W, eps=eps, tensor="")
        layers = []
        for i, l in enumerate(self.layers):
            ff = None
            if l.mlp is not None:
                mlp = _thaw(l.mlp)
                groups = mlp["router"].get("groups") or {"count": 1, "keep": 1}
                ff = MoESpec(hidden=W, experts=mlp["router"]["experts"], top=mlp["router"]["top"], intermediate=mlp["expert"]["ff"], renorm_eps=0.0,
                             score="sigmoid", renorm=False, weight_on="output", act="relu2", correction=True, groups=groups["count"],
                             keep_groups=groups["keep"])
            ff_norm = None if ff is None else norm
            layers.append(SandwichLayerSpec(prefix=f"l{i}.", mixer=self._mixer(l), feed_forward=ff, mixer_norm=norm, mixer_out_norm=norm,
                                            feed_forward_norm=ff_norm, feed_forward_out_norm=ff_norm, conv_taps=self.taps, average=i + 2))
        spec = ModelSpec(
            architecture=self.architecture, hidden=W, vocab=self.vocab, max_positions=1 << 30,
            embedding=EmbeddingSpec("embed", self.vocab, W, scale=self.embedding_scale), layers=tuple(layers),
            schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))),
            final_norm=norm, final_norm_name="final.norm",
            head=HeadSpec("head", self.vocab, W, tied_to="embed", soft_cap=self.logit_softcap or 0.0))
        spec.validate()
        return spec
