"""A block with a norm in front of and behind each sublayer, a short convolution on what its mixer reads and a weighted sum
over the depth behind it (``SandwichLayerSpec``).

The model keeps the results of all layer runs as float32 planes [runs + 1, rows, width]: plane 0 is the embedding output
X_0, plane i + 1 the result of the layer run at place i of the schedule.  Where no block weighs earlier results there are two planes:
the embedding output, and one that holds the latest result.  A sublayer's output is not added when it is there but
handed on, with the norm that stands behind it, to the row-wise kernel that reads the residual next
(``ops.sandwich_rows``): behind the mixer that kernel adds the normed output and norms the sum for the feed-forward;
behind a layer the next block's (or the model's last step) adds it, stores the layer's result in its plane, forms the
weighted sum of the planes and norms it, in one pass over the row.  In a step of single tokens the same kernel also applies
the next mixer's convolution, whose earlier inputs are then all in the sequence's state, and moves that state on; in a
prompt the normed rows are written once in float32 and a second kernel convolves them (``ops.conv_rows``), reaching back
into the step's own rows of the sequence and, before them, into the state.

A mixer that leaves two outputs to be normed apart and added (``forward_pair``) has that done by the same kernel on its way, and a
junction that adds planes to the residual where a pass through repeated layers begins (``over_planes``) is a weighted sum like a
layer's own.

The residual, the averages, the norms, the convolution's inputs and its state are float32; what the sublayers read is in
the activation dtype.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Mapping, Optional, Tuple

import torch

from .. import registry
from .base import BlockStateRequest, Part, Runtime, StateRequest, TensorDecl


@dataclass
class PendingResult:
    """A layer's last sublayer output ``y`` that has yet to be normed and added to ``base``; the sum is plane ``at`` of the
    results, and ``average`` weighs the planes 0 .. at into what goes on (None: the result itself)."""
    y: torch.Tensor
    norm: Tuple[torch.Tensor, float]
    base: torch.Tensor
    at: int
    average: Optional[torch.Tensor]
    pair: Optional[tuple] = None      # (second output, the two outputs' weights, eps) where ``y`` is the first of two


class SandwichBlock(Part):
    category = "block"
    takes_history = True     # forward gets the results of all layer runs as planes [runs + 1, rows, width]

    @classmethod
    def _norms(cls, layer):
        out = [("mixer_norm", layer.mixer_norm, layer.mixer_norm_prefix), ("mixer_out_norm", layer.mixer_out_norm, layer.mixer_out_norm_prefix)]
        if layer.feed_forward is not None:
            out += [("feed_forward_norm", layer.feed_forward_norm, layer.feed_forward_norm_prefix),
                    ("feed_forward_out_norm", layer.feed_forward_out_norm, layer.feed_forward_out_norm_prefix)]
        return out

    @classmethod
    def declare(cls, layer, prefix: str = "") -> List[TensorDecl]:
        p = layer.prefix
        decls: List[TensorDecl] = []
        for _, spec, name in cls._norms(layer):
            decls += registry.part_class("norm", spec.kind).declare(spec, p + name)
        decls += registry.part_class("mixer", layer.mixer.kind).declare(layer.mixer, p + layer.mixer_prefix)
        if layer.feed_forward is not None:
            decls += registry.part_class("feed_forward", layer.feed_forward.kind).declare(layer.feed_forward, p + layer.feed_forward_prefix)
        if layer.conv_taps > 0:
            decls.append(TensorDecl(p + layer.conv_name, (layer.mixer_norm.size, layer.conv_taps)))
        if layer.average > 0:
            decls.append(TensorDecl(p + layer.average_name, (layer.average,), role="norm"))
        return decls

    def __init__(self, layer, prefix: str, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        p = layer.prefix
        self.layer = layer
        self.rt = runtime
        self.mixer = registry.part_class("mixer", layer.mixer.kind)(layer.mixer, p + layer.mixer_prefix, tensors, runtime)
        self.feed_forward = None
        if layer.feed_forward is not None:
            self.feed_forward = registry.part_class("feed_forward", layer.feed_forward.kind)(
                layer.feed_forward, p + layer.feed_forward_prefix, tensors, runtime)
        self.norms = {}
        for name, spec, suffix in self._norms(layer):
            fold = registry.part_class("norm", spec.kind)(spec, p + suffix, tensors, runtime).rms_fold()
            if fold is None:
                raise ValueError(f"{p}{suffix}: this block's norms are RMS norms with a float32 weight")
            self.norms[name] = (fold[0].contiguous(), float(fold[1]))
        self.conv = None       # [taps, width]: a tap's weights lie together
        if layer.conv_taps > 0:
            self.conv = tensors[p + layer.conv_name].to(torch.float32).t().contiguous()
        self.average = None
        if layer.average > 0:
            self.average = tensors[p + layer.average_name].to(torch.float32).contiguous()

    @classmethod
    def cache_request(cls, layer):
        req = registry.part_class("mixer", layer.mixer.kind).cache_request(layer.mixer)
        if layer.conv_taps <= 1:
            return req
        return BlockStateRequest(req, StateRequest(shape=((layer.conv_taps - 1) * layer.mixer_norm.size,), dtype=torch.float32))

    def prepare(self, capacity: int) -> None:
        self.mixer.prepare(capacity)

    def mixers(self) -> List[Part]:
        return self.mixer.mixers() if hasattr(self.mixer, "mixers") else [self.mixer]

    @property
    def reads_history(self) -> bool:
        """Whether this block reads results other than the latest (and the embedding output)."""
        return self.average is not None

    def weight_bytes(self) -> int:
        return sum(p.weight_bytes() for p in (self.mixer, self.feed_forward) if p is not None and hasattr(p, "weight_bytes"))

    @property
    def capturable(self) -> bool:
        return all(p.capturable for p in (self.mixer, self.feed_forward) if p is not None)

    def _average_of(self, pending: PendingResult):
        if pending.average is not None and pending.average.numel() != pending.at + 1:
            raise ValueError(f"a weighted sum of {pending.average.numel()} results behind {pending.at} layer runs")
        return pending.average

    @staticmethod
    def _plane(planes: torch.Tensor, at: int) -> torch.Tensor:
        """The plane of result ``at`` (0: the embedding output); with two planes in all every result is the second."""
        return planes[min(at, planes.shape[0] - 1)]

    def _mix(self, batch, x: torch.Tensor, view):
        """The mixer's output, or its first output and what ``pair`` needs of the second."""
        if hasattr(self.mixer, "forward_pair"):
            y, *pair = self.mixer.forward_pair(batch, x, view)
            second, w, w2, eps = pair
            return y, (second, w, w2, eps)
        y = torch.empty((x.shape[0], x.shape[1]), dtype=torch.float32, device=x.device)
        self.mixer.forward(batch, x, y, view)
        return y, None

    def _open(self, batch, planes: torch.Tensor, pending: Optional[PendingResult], state: Optional[torch.Tensor], enter=None):
        """Finish the layer before, form what this layer starts from and norm and convolve it for the mixer: (the residual
        this layer starts from, the mixer's input).  ``enter``: a junction that weighs planes into what this layer starts from."""
        ops = self.rt.ops
        rows, width = planes.shape[1], planes.shape[2]
        weight, eps = self.norms["mixer_norm"]
        kw, start = {}, planes[0]
        n_planes, average = 0, None
        if pending is None:
            kw["base"] = start
        else:
            result = self._plane(planes, pending.at)
            n_planes, average = pending.at, self._average_of(pending)
            start = result
            kw = dict(base=pending.base, y=pending.y, y_weight=pending.norm[0], y_eps=pending.norm[1], result=result, pair=pending.pair)
        if enter is not None:
            if average is not None:
                raise ValueError("a junction behind a layer that weighs the results so far is not built")
            n_planes, average = enter.over_planes()
        if average is not None:
            start = torch.empty((rows, width), dtype=torch.float32, device=planes.device)
            kw.update(planes=planes, n_planes=n_planes, average=average, x_out=start)
        x = torch.empty((rows, width), dtype=self.rt.act_dtype, device=planes.device)
        if self.conv is None or batch.max_q_len == 1:
            if self.conv is not None:
                kw.update(conv=self.conv, state=state, batch=batch)
            ops.sandwich_rows(out=x, norm_weight=weight, eps=eps, **kw)
        else:
            normed = torch.empty((rows, width), dtype=torch.float32, device=planes.device)
            ops.sandwich_rows(out=normed, norm_weight=weight, eps=eps, **kw)
            ops.conv_rows(normed, self.conv, state, x, batch)
        return start, x

    def forward(self, batch, planes: torch.Tensor, at: int, pending: Optional[PendingResult], cache, enter=None) -> PendingResult:
        """Runs the layer as run ``at`` of the schedule.  ``pending``: what the run before left (None: this is the first
        run and starts from plane 0).  ``enter``: the junction ahead of this run, if there is one."""
        ops = self.rt.ops
        rows, width = planes.shape[1], planes.shape[2]
        state, view = None, cache
        if self.conv is not None and self.conv.shape[0] > 1:
            state, view = cache.state, cache.mixer
        start, x = self._open(batch, planes, pending, state, enter) if enter is not None else self._open(batch, planes, pending, state)
        y, pair = self._mix(batch, x, view)
        if self.feed_forward is None:
            return PendingResult(y, self.norms["mixer_out_norm"], start, at + 1, self.average, pair)
        result = self._plane(planes, at + 1)      # holds the residual between the two sublayers until the result is complete
        weight, eps = self.norms["feed_forward_norm"]
        out_weight, out_eps = self.norms["mixer_out_norm"]
        ops.sandwich_rows(base=start, y=y, y_weight=out_weight, y_eps=out_eps, result=result, out=x, norm_weight=weight, eps=eps, pair=pair)
        self.feed_forward.forward(batch, x, y)
        return PendingResult(y, self.norms["feed_forward_out_norm"], result, at + 1, self.average)

    def finish(self, planes: torch.Tensor, pending: PendingResult, norm, x_out: torch.Tensor, rows: torch.Tensor) -> None:
        """The model's last step: complete the last layer's result for the wanted rows and norm what goes on behind it."""
        weight, eps = norm.rms_fold()
        kw = {}
        average = self._average_of(pending)
        if average is not None:
            kw = dict(planes=planes, n_planes=pending.at, average=average)
        self.rt.ops.sandwich_rows(base=pending.base, y=pending.y, y_weight=pending.norm[0], y_eps=pending.norm[1], out=x_out,
                                  norm_weight=weight, eps=eps, rows=rows, pair=pending.pair, **kw)
