"""Several residual streams (hyper-connections).

A token has n float32 rows x_1 .. x_n of the model's width, all equal to the embedding's row at the start. A sublayer f
reads one combination of them and writes into all of them:

    u = sum_s a_s x_s;   y = f(norm(u));   x_t <- sum_s M[s, t] x_s + b_t y        (all t from the old x)

with ``in`` = a [n], ``out`` = b [n] and ``mix`` = M [from, to] per sublayer (family "connection", kind "hyper"); in front
of the head the streams are summed. Writing one sublayer's result, reading for the next one and the next one's norm are
ONE kernel over the rows: a block leaves its last result pending in the ``StreamRows`` it passes on, and whoever reads
next takes it in. ``names`` renames the three tensors by role.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.specs import PartSpec
from .base import Connection, Stream, register_connection, register_stream

_NAMES = {"in": "in", "out": "out", "mix": "mix"}


class StreamRows:
    """The streams of a step's tokens: float32 [T, n, width] (or [T, width] while all n are that row), and the sublayer
    result that they have yet to take in, with the connection it goes through."""

    def __init__(self, rows: torch.Tensor, n: int):
        self.rows, self.n = rows, n
        self.pending = None                    # (y float32 [T, width], connection)

    @property
    def device(self):
        return self.rows.device

    def _args(self):
        if self.pending is None:
            return {}
        y, link = self.pending
        return {"y": y, "mix": link.mix, "out_w": link.out_w}

    def read(self, link: "HyperConnection", norm, dtype: torch.dtype) -> torch.Tensor:
        """Takes in what is pending; returns norm(sum_s a_s x_s) in ``dtype``."""
        self.rows, normed = ops.stream_link(self.rows, self.n, dtype, in_w=link.in_w, norm_w=norm.weight, eps=norm.eps,
                                            groups=norm.groups, **self._args())
        self.pending = None
        return normed

    def write(self, link: "HyperConnection", y: torch.Tensor) -> None:
        assert self.pending is None, "a sublayer's result is pending already"
        self.pending = (y, link)

    def total(self) -> torch.Tensor:
        """float32 [T, width]: the sum of the streams, what is pending included."""
        return ops.stream_link(self.rows, self.n, torch.float32, store=False, **self._args())[1]

    def close(self, norm, rows: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
        return ops.stream_link(self.rows, self.n, dtype, norm_w=norm.weight, eps=norm.eps, groups=norm.groups, rows=rows, **self._args())[1]


@register_connection("hyper")
class HyperConnection(Connection):
    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.n = int(spec["streams"])
        if not 1 <= self.n <= ops.stream_link_max_streams():
            raise ValueError(f"a hyper connection takes 1 to {ops.stream_link_max_streams()} streams, got {self.n}")
        self.in_w = self.out_w = self.mix = None

    @classmethod
    def param_shapes(cls, spec):
        n, names = int(spec["streams"]), {**_NAMES, **dict(spec.get("names") or {})}
        return {names["in"]: (n,), names["out"]: (n,), names["mix"]: (n, n)}

    @classmethod
    def init_params(cls, spec, name, shape, gen):
        noise = 0.2 * torch.randn(shape, generator=gen, dtype=torch.float32, device=gen.device)
        names = {**_NAMES, **dict(spec.get("names") or {})}
        if name == names["mix"]:
            return torch.eye(shape[0], device=gen.device) + 0.3 * noise
        return (1.0 / shape[0] if name == names["in"] else 1.0) + noise

    def load(self, params):
        names = {**_NAMES, **dict(self.spec.get("names") or {})}
        f32 = dict(device=self.rt.device, dtype=torch.float32)
        self.in_w, self.out_w, self.mix = (params[names[r]].to(**f32).contiguous() for r in ("in", "out", "mix"))


@register_stream("copies")
class CopiedStream(Stream):
    """n streams that start as copies of the embedding's rows and end in their sum."""

    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.n = int(spec["streams"])
        if self.n < 1:
            raise ValueError("a model has at least one residual stream")

    def open(self, rows):
        return StreamRows(rows, self.n)

    def close(self, h, norm, rows):
        return h.close(norm, rows, self.rt.dtype)


# ----------------------------------------------------------------------------- one row per token, results pending

class PendingRows:
    """The residual rows of a step's tokens, float32 [T, width], and what the last layer's sublayers returned, each with the
    factor per channel it enters through: whoever reads next takes it in, in the same kernel as its norm."""

    def __init__(self, rows: torch.Tensor):
        self.rows = rows
        self.pending = []                      # [(y float32 [T, width], factors float32 [width])], at most two

    @property
    def device(self):
        return self.rows.device

    def _terms(self):
        flat = [t for pair in self.pending for t in pair]
        return flat + [None] * (4 - len(flat))

    def read(self, norm, dtype: torch.dtype) -> torch.Tensor:
        """Takes in what is pending; returns norm(rows) in ``dtype``."""
        out = ops.scaled_sum_norm(self.rows, *self._terms(), norm.weight, norm.eps, dtype)
        self.pending = []
        return out

    def write(self, link: "ChannelScale", y: torch.Tensor) -> None:
        assert len(self.pending) < 2, "two results are pending already"
        self.pending.append((y, link.weight))

    def total(self) -> torch.Tensor:
        """float32 [T, width]: the rows with what is pending taken in (a copy; the rows stay as they are)."""
        rows = self.rows.clone()
        for y, w in self.pending:
            rows += y * w
        return rows

    def close(self, norm, rows: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
        return ops.scaled_sum_norm(self.rows, *self._terms(), norm.weight, norm.eps, dtype, rows=rows)


@register_connection("channel_scale")
class ChannelScale(Connection):
    """A sublayer's result enters the residual stream times a stored factor per channel."""

    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.size = int(spec["size"])
        if self.size <= 0:
            raise ValueError("channel_scale needs a positive size")
        self.weight = None

    @classmethod
    def param_shapes(cls, spec):
        return {str(spec.get("weight_name", "scale")): (int(spec["size"]),)}

    @classmethod
    def init_params(cls, spec, name, shape, gen):
        return 1.0 + 0.2 * torch.randn(shape, generator=gen, dtype=torch.float32, device=gen.device)

    def load(self, params):
        self.weight = params[str(self.spec.get("weight_name", "scale"))].to(device=self.rt.device, dtype=torch.float32).contiguous()


@register_stream("pending_sum")
class PendingSum(Stream):
    """One row per token that starts as the embedding's; a layer's results stay pending until the next norm."""

    def open(self, rows):
        return PendingRows(rows)

    def close(self, h, norm, rows):
        return h.close(norm, rows, self.rt.dtype)
