"""Several residual streams that every sublayer mixes (hyper-connections: Zhu, Huang, Huang, Zeng, Mao, Wu, Min, Zhou,
"Hyper-Connections", 2024).

A token has n streams X_1 .. X_n, float32, all equal to the embedding's output before the first layer.  A sublayer f
with the stored numbers a [n], M [n, n] (indexed [from, to]) and b [n]:
    u = sum_s a[s] X_s;    y = f(norm(u));    X_t <- sum_s M[s, t] X_s + b[t] y      (all t from the old streams)
After the last layer the streams are added up.

`StreamValue` is what hyper-connected blocks hand on.  A sublayer's result is not written back at once: it waits until the
streams are read next, and one kernel (csrc/streams.cu) then adds the result up from wherever its sublayer left it, writes
the streams, reads them for the next sublayer and norms that.  The end of the model reads the wanted rows alone and writes no
stream.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import CONNECTIONS, STREAMS, Connection, Streams
from .norm import RMSNorm
from .spec import TensorSpec


MAX_STREAMS = 16           # the streams kernel keeps a column's streams in registers


@CONNECTIONS.register("hyper_connection")
class HyperConnection(Connection):
    """params: streams, name; the tensors are name + ".in" (a), ".mix" (M) and ".out" (b) under the prefix."""

    def __init__(self, params, prefix, runtime) -> None:
        super().__init__(params, prefix, runtime)
        self.n = int(params["streams"])
        self.name = prefix + params["name"]
        self.read = self.mix = self.back = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.name + ".in": TensorSpec((self.n,), init="one_plus_normal"),
                self.name + ".mix": TensorSpec((self.n, self.n), init="eye_plus_normal"),
                self.name + ".out": TensorSpec((self.n,), init="one_plus_normal")}

    def load(self, tensors) -> None:
        # part of the residual sum: float32 in every run
        self.read, self.mix, self.back = (tensors[self.name + s].float().contiguous() for s in (".in", ".mix", ".out"))


class StreamValue:
    """x: float32 [rows, n, width], or [rows, 1, width] while all streams are equal; `pending`: the last sublayer's
    (result, connection), not yet in x."""

    def __init__(self, rt, n: int, x: torch.Tensor) -> None:
        self.rt, self.n, self.x = rt, n, x
        self.pending = None

    def give(self, y, connection: HyperConnection) -> None:
        """A sublayer's result: float32 rows [rows, width] (a sum deferred on them is taken over when the streams are read
        next), or what `forward_unsummed` returns."""
        if self.pending is not None:
            raise RuntimeError("the streams were not read since the last sublayer's result")
        self.pending = (y, connection)

    def _take(self, ctx) -> dict:
        if self.pending is None:
            return {}
        y, c = self.pending
        self.pending = None
        if isinstance(y, torch.Tensor):
            d = ctx.take_deferred(y)
            if d is not None:
                if d[1] != "store":
                    raise RuntimeError("a sublayer of several streams leaves its result alone, not a sum with the residual")
                y = d[0]
        return {"y": y, "mix": c.mix, "back": c.back}

    def _norm_args(self, norm, rows: int) -> tuple:
        """(what the kernel is told, the rows it writes, whether the norm is still to be applied)."""
        width = self.x.shape[2]
        if isinstance(norm, RMSNorm) and not norm.offset:
            out = self.rt.empty(rows, width)
            return {"w": norm.weight, "eps": norm.eps, "out": out}, out, False
        out = torch.empty((rows, width), dtype=torch.float32, device=self.x.device)
        return {"out": out}, out, True

    def read(self, connection: HyperConnection, norm, ctx) -> torch.Tensor:
        """norm(sum_s a[s] X_s), every row, in the run's type; a result that was given is written back on the way."""
        pending = self._take(ctx)
        rows, n_in, width = self.x.shape
        args, out, plain = self._norm_args(norm, rows)
        x_out = None
        if pending:
            x_out = self.x if n_in == self.n else torch.empty((rows, self.n, width), dtype=torch.float32, device=self.x.device)
        self.rt.kernels.streams(self.x, x_out, self.n, read=connection.read, **pending, **args)
        if x_out is not None:
            self.x = x_out
        return norm.forward(out, ctx) if plain else out

    def total(self, ctx) -> torch.Tensor:
        pending = self._take(ctx)
        rows, n_in, width = self.x.shape
        out = torch.empty((rows, width), dtype=torch.float32, device=self.x.device)
        x_out = None
        if pending:
            x_out = self.x if n_in == self.n else torch.empty((rows, self.n, width), dtype=torch.float32, device=self.x.device)
        self.rt.kernels.streams(self.x, x_out, self.n, out=out, **pending)
        if x_out is not None:
            self.x = x_out
        return out

    def close(self, norm, ctx, row_index: torch.Tensor, rows: int) -> torch.Tensor:
        pending = self._take(ctx)
        args, out, plain = self._norm_args(norm, rows)
        self.rt.kernels.streams(self.x, None, self.n, row_index=row_index, **pending, **args)
        return norm.forward(out, ctx) if plain else out


@STREAMS.register("equal_start")
class EqualStart(Streams):
    """params: streams.  Every stream starts as the embedding's output; the end is their sum."""

    def __init__(self, params, prefix, runtime) -> None:
        super().__init__(params, prefix, runtime)
        self.n = int(params["streams"])
        if not 1 <= self.n <= MAX_STREAMS:
            raise ValueError(f"1 to {MAX_STREAMS} residual streams are built, not {self.n}")

    def open(self, h: torch.Tensor) -> StreamValue:
        return StreamValue(self.rt, self.n, h.unsqueeze(1))

    def total(self, value: StreamValue, ctx) -> torch.Tensor:
        return value.total(ctx)

    def close(self, value: StreamValue, norm, ctx, row_index: Optional[torch.Tensor] = None, rows: Optional[int] = None) -> torch.Tensor:
        return value.close(norm, ctx, row_index, rows)
