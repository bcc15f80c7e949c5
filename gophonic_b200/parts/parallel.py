"""Two mixers side by side (``ParallelSpec``): both read the same input, and the result is the sum of their outputs, each normed over
the model width, times a factor.

The two first products are one (their matrices lie one above the other, x is read once); each mixer goes on from its columns of the
projected rows.  A block whose row-wise kernel takes two outputs (``forward_pair``) norms and adds them in the pass that adds the
sublayer to the residual; for any other block ``forward`` leaves the sum.
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from .. import registry
from .base import Mixer, PartsRequest, Runtime, TensorDecl


class Parallel(Mixer):
    @classmethod
    def _classes(cls, spec):
        return [registry.part_class("mixer", m.kind) for m in spec.mixers]

    @classmethod
    def declare(cls, spec, prefix: str) -> List[TensorDecl]:
        decls: List[TensorDecl] = []
        for part, m, name in zip(cls._classes(spec), spec.mixers, spec.prefixes):
            decls += part.declare(m, prefix + name)
            decls.append(TensorDecl(prefix + name + spec.out_name, (spec.hidden,), role="norm"))
        return decls

    @classmethod
    def cache_request(cls, spec):
        return PartsRequest(tuple(part.cache_request(m) for part, m in zip(cls._classes(spec), spec.mixers)))

    def __init__(self, spec, prefix: str, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        self.spec, self.rt = spec, runtime
        self.parts = [part(m, prefix + name, tensors, runtime) for part, m, name in zip(self._classes(spec), spec.mixers, spec.prefixes)]
        # the factor rides on the norms' weights
        self.weights = [(tensors[prefix + name + spec.out_name].to(torch.float32) * float(spec.factor)).contiguous() for name in spec.prefixes]
        self.in_matrix = None
        mats = [getattr(p, "in_matrix", None) for p in self.parts]
        if all(m is not None for m in mats) and len({m.dtype for m in mats}) == 1:
            # each mixer's columns start on 16 bytes, so that its kernels may load vectors; the rows between are zeros
            at, pieces, self.offsets = 0, [], []
            for m in mats:
                pad = (-at) % 8
                if pad:
                    pieces.append(torch.zeros((pad, m.shape[1]), dtype=m.dtype, device=m.device))
                self.offsets.append(at + pad)
                pieces.append(m)
                at += pad + m.shape[0]
            if at % 8:
                pieces.append(torch.zeros(((-at) % 8, mats[0].shape[1]), dtype=mats[0].dtype, device=mats[0].device))
            self.in_matrix = torch.cat(pieces, dim=0).contiguous()
            for p, m, o in zip(self.parts, mats, self.offsets):
                p.in_matrix = self.in_matrix[o:o + m.shape[0]]      # the same storage, no second copy

    @property
    def capturable(self) -> bool:
        return all(p.capturable for p in self.parts)

    def weight_bytes(self) -> int:
        return sum(p.weight_bytes() for p in self.parts if hasattr(p, "weight_bytes"))

    def mixers(self):
        return [m for p in self.parts for m in p.mixers()]

    def prepare(self, capacity: int) -> None:
        for p in self.parts:
            p.prepare(capacity)

    def forward_pair(self, batch, x: torch.Tensor, cache):
        """The two outputs (float32 [rows, hidden]), the weights of their norms (with the factor) and the norms' eps."""
        ops, rows = self.rt.ops, x.shape[0]
        outs = [torch.empty((rows, self.spec.hidden), dtype=torch.float32, device=x.device) for _ in self.parts]
        if self.in_matrix is None:
            for p, out, view in zip(self.parts, outs, cache.parts):
                p.forward(batch, x, out, view)
        else:
            buf = torch.empty((rows, self.in_matrix.shape[0]), dtype=x.dtype, device=x.device)
            ops.gemm(x, self.in_matrix, buf)
            for p, out, view, o in zip(self.parts, outs, cache.parts, self.offsets):
                p.project_out(p.heads_of(batch, x, buf[:, o:o + p.in_matrix.shape[0]], view), out)
        return outs[0], outs[1], self.weights[0], self.weights[1], float(self.spec.eps)

    def forward(self, batch, x: torch.Tensor, out: torch.Tensor, cache) -> None:
        a, b, wa, wb, eps = self.forward_pair(batch, x, cache)
        out.zero_()
        self.rt.ops.norm_scale_add(out, a, wa, eps)
        self.rt.ops.norm_scale_add(out, b, wb, eps)
