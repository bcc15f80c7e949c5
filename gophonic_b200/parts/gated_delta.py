"""The gated delta rule as a mixer (``GatedDeltaSpec``): a matrix state per head that decays, per head or per key channel, has the
value it already holds along the token's unit key taken off what is written, and is read behind the write.

One product projects x to q | k | v | gate in the activation dtype.  A second, small product leaves float32: the write strengths' and
the decays' pre-activations (a decay per channel comes out of two small matrices, both products float32).  ``ops.short_conv`` takes the
projected q, k and v through their convolution over time (the sequence's last projected rows are part of the state) and silu and
leaves unit queries, unit keys and the values in float32; ``ops.gated_delta`` forms decays and strengths from their pre-activations
and walks the recurrence, its state in the cache's per-sequence storage.  Each head's output is divided by its root mean square,
multiplied by a weight and by the gate (``ops.head_norm_gate``), and projected back.
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from .base import Mixer, PartsRequest, Runtime, StateRequest, TensorDecl


class GatedDelta(Mixer):
    capturable = True

    @staticmethod
    def _sizes(spec):
        """Rows of q (and of k), of v, and the channels that are convolved."""
        kd, vd = spec.kv_heads * spec.key_dim, spec.heads * spec.value_dim
        return kd, vd, 2 * kd + vd

    @classmethod
    def declare(cls, spec, prefix: str) -> List[TensorDecl]:
        n = dict(spec.names)
        kd, vd, _ = cls._sizes(spec)
        H, W = spec.heads, spec.hidden
        decls = [TensorDecl(prefix + n["q"], (kd, W)), TensorDecl(prefix + n["k"], (kd, W)), TensorDecl(prefix + n["v"], (vd, W)),
                 TensorDecl(prefix + n["b"], (H, W)), TensorDecl(prefix + n["a_log"], (H,), role="vector"),
                 TensorDecl(prefix + n["norm"], (spec.value_dim,), role="norm"), TensorDecl(prefix + n["o"], (W, vd))]
        if spec.conv_taps > 0:
            decls += [TensorDecl(prefix + n[k] + spec.conv_suffix, (size, spec.conv_taps)) for k, size in (("q", kd), ("k", kd), ("v", vd))]
        if spec.channel_decay:      # a rank of None: whatever the checkpoint has
            decls += [TensorDecl(prefix + n["a1"], (spec.rank, W)), TensorDecl(prefix + n["a2"], (H * spec.key_dim, spec.rank)),
                      TensorDecl(prefix + n["dt_bias"], (H * spec.key_dim,), role="vector")]
        else:
            decls += [TensorDecl(prefix + n["a"], (H, W)), TensorDecl(prefix + n["dt_bias"], (H,), role="vector")]
        if spec.gate_low_rank:
            decls += [TensorDecl(prefix + n["g1"], (spec.gate_rank, W)), TensorDecl(prefix + n["g2"], (vd, spec.gate_rank))]
        else:
            decls.append(TensorDecl(prefix + n["g"], (vd, W)))
        return decls

    @classmethod
    def cache_request(cls, spec):
        matrix = StateRequest(shape=(spec.heads, spec.key_dim * spec.value_dim), dtype=torch.float32)
        rows = None
        if spec.conv_taps > 1:
            rows = StateRequest(shape=((spec.conv_taps - 1) * cls._sizes(spec)[2],), dtype=torch.float32)
        return PartsRequest((matrix, rows))

    def __init__(self, spec, prefix: str, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        if spec.heads % spec.kv_heads:
            raise ValueError(f"{prefix}: {spec.heads} heads are not a multiple of {spec.kv_heads} key heads")
        self.spec, self.rt = spec, runtime
        n = dict(spec.names)
        t = lambda key: tensors[prefix + n[key]]
        f32 = lambda key: t(key).to(torch.float32).contiguous()
        self.kd, self.vd, self.channels = self._sizes(spec)

        def stacked(keys):
            mats = [t(k) for k in keys]
            if len({m.dtype for m in mats}) != 1:
                raise ValueError(f"{prefix}: {', '.join(n[k] for k in keys)} are stored in different dtypes; they must agree")
            return torch.cat(mats, dim=0).contiguous()
        self.in_matrix = stacked(("q", "k", "v", "g1" if spec.gate_low_rank else "g"))      # x is read once
        self.small = stacked(("b", "a1" if spec.channel_decay else "a"))                    # strengths, then decays: a float32 product
        self.o = t("o").contiguous()
        self.a2 = self.g2 = None
        for low, high, on in (("a1", "a2", spec.channel_decay), ("g1", "g2", spec.gate_low_rank)):
            if on:
                if t(low).shape[0] != t(high).shape[1]:
                    raise ValueError(f"{prefix}: {n[low]} has {t(low).shape[0]} rows and {n[high]} {t(high).shape[1]} columns; they must agree")
                setattr(self, high, t(high).contiguous())
        self.a_log, self.dt_bias, self.norm_w = f32("a_log"), f32("dt_bias"), f32("norm")
        self.conv = None
        if spec.conv_taps > 0:      # [taps, channels]: a tap's weights lie together
            self.conv = torch.cat([tensors[prefix + n[k] + spec.conv_suffix] for k in ("q", "k", "v")], dim=0).to(torch.float32).t().contiguous()
        if spec.gate not in ("silu", "sigmoid"):
            raise ValueError(f"{prefix}: unknown gate '{spec.gate}'")
        self.gate_kind = runtime.ops.GATE_SILU if spec.gate == "silu" else runtime.ops.GATE_SIGMOID

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.in_matrix, self.small, self.o, self.a2, self.g2) if t is not None)

    def forward(self, batch, x: torch.Tensor, out: torch.Tensor, cache) -> None:
        buf = torch.empty((x.shape[0], self.in_matrix.shape[0]), dtype=x.dtype, device=x.device)
        self.rt.ops.gemm(x, self.in_matrix, buf)
        self.project_out(self.heads_of(batch, x, buf, cache), out)

    def project_out(self, heads: torch.Tensor, out: torch.Tensor) -> None:
        self.rt.ops.gemm(heads, self.o, out)

    def heads_of(self, batch, x: torch.Tensor, buf: torch.Tensor, cache) -> torch.Tensor:
        """The normed and gated heads, [rows, heads * value_dim], from the mixer's input and its projected rows ``buf``
        (q | k | v | gate; rows may lie further apart)."""
        ops, s = self.rt.ops, self.spec
        rows, dev, f32 = x.shape[0], x.device, torch.float32
        matrix, last_rows = cache.parts
        small = torch.empty((rows, self.small.shape[0]), dtype=f32, device=dev)
        ops.gemm(x, self.small, small)
        decay = small[:, s.heads:]
        if s.channel_decay:
            decay = torch.empty((rows, s.heads * s.key_dim), dtype=f32, device=dev)
            ops.gemm(small[:, s.heads:], self.a2, decay)
        qkv = torch.empty((rows, self.channels), dtype=f32, device=dev)
        ops.short_conv(buf, qkv, s.kv_heads, s.kv_heads, s.heads, s.key_dim, s.value_dim, self.conv,
                       None if last_rows is None else last_rows.state, batch, silu=True, norm=ops.HEAD_NORM_UNIT, eps=float(s.unit_eps),
                       q_scale=float(s.key_dim) ** -0.5)
        o = torch.empty((rows, self.vd), dtype=f32, device=dev)
        ops.gated_delta(qkv, s.heads, s.kv_heads, s.key_dim, s.value_dim, decay, self.dt_bias, self.a_log, small[:, :s.heads], matrix.state, o, batch)
        gate = buf[:, self.channels:]
        if s.gate_low_rank:
            gate = torch.empty((rows, self.vd), dtype=x.dtype, device=dev)
            ops.gemm(buf[:, self.channels:], self.g2, gate)
        y = torch.empty((rows, self.vd), dtype=x.dtype, device=dev)
        ops.head_norm_gate(o, gate, y, s.heads, s.value_dim, self.gate_kind, weight=self.norm_w, eps=float(s.eps))
        return y
