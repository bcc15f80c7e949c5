"""HGRN2 as a mixer (``ForgetStateSpec``): a matrix state per head whose forget gate also decides what is written,
S <- diag(f) S + (1 - f) v^T, o = S^T q.

One product projects x to q | v | f and leaves float32.  The kernel of the recurrence (``ops.state_scan``, state in the cache's
per-sequence storage) turns the pre-activations into silu(q) and the write gate 1 - f = (1 - l) sigmoid(-z), which keeps
its digits where f is close to one, and updates the state as S + (1 - f)(v - S).  Each head's output is RMS-normed
(``ops.head_norm_gate`` without a gate) and projected back.
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from .base import Runtime, TensorDecl
from .linear_state import _StateMixer


class ForgetState(_StateMixer):
    @classmethod
    def declare(cls, spec, prefix: str) -> List[TensorDecl]:
        n = dict(spec.names)
        kd, vd = spec.heads * spec.key_dim, spec.heads * spec.value_dim
        return [TensorDecl(prefix + n["q"], (kd, spec.hidden)), TensorDecl(prefix + n["v"], (vd, spec.hidden)),
                TensorDecl(prefix + n["f"], (kd, spec.hidden)), TensorDecl(prefix + n["f_bias"], (kd,), role="vector"),
                TensorDecl(prefix + n["lower"], (kd,), role="vector"), TensorDecl(prefix + n["norm"], (spec.value_dim,), role="norm"),
                TensorDecl(prefix + n["o"], (spec.hidden, vd))]

    def __init__(self, spec, prefix: str, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.spec, self.rt = spec, runtime
        n = dict(spec.names)
        self.kd, self.vd = spec.heads * spec.key_dim, spec.heads * spec.value_dim
        mats = [tensors[prefix + n[k]] for k in ("q", "v", "f")]
        if len({t.dtype for t in mats}) != 1:
            raise ValueError(f"{prefix}: the projections are stored in different dtypes; they must agree")
        self.qvf = torch.cat(mats, dim=0).contiguous()      # q | v | f: one product reads x once
        self.o = tensors[prefix + n["o"]].contiguous()
        self.f_bias = tensors[prefix + n["f_bias"]].to(torch.float32).contiguous()
        self.lower = tensors[prefix + n["lower"]].to(torch.float32).contiguous()
        self.norm_w = tensors[prefix + n["norm"]].to(torch.float32).contiguous()

    def _matrices(self):
        return (self.qvf, self.o)

    def _heads(self, batch, x: torch.Tensor, cache) -> torch.Tensor:
        """Everything up to the output projection: the normed heads, [rows, heads * value_dim]."""
        ops, s = self.rt.ops, self.spec
        rows = x.shape[0]
        buf = torch.empty((rows, self.qvf.shape[0]), dtype=torch.float32, device=x.device)
        ops.gemm(x, self.qvf, buf)
        o = torch.empty((rows, self.vd), dtype=torch.float32, device=x.device)
        ops.state_scan(buf, 0, 0, self.kd, s.heads, s.key_dim, s.value_dim, 1.0, cache.state, o, batch.seq_slot, batch.seq_q_start,
                       batch.seq_q_len, batch.nseq, decay=buf[:, self.kd + self.vd:], gate_bias=self.f_bias, lower=self.lower,
                       max_q_len=batch.max_q_len)
        y = torch.empty((rows, self.vd), dtype=x.dtype, device=x.device)
        ops.head_norm_gate(o, None, y, s.heads, s.value_dim, ops.GATE_NONE, weight=self.norm_w, eps=float(s.eps))
        return y
