"""Several residual streams per token (hyper-connections) in place of one.

The model keeps n copies x_1 .. x_n of the stream, all equal to the embedding output at a step's start.  A sublayer with the
constants enter [n], leave [n] and mix [n, n] (indexed from, to) reads a weighted sum of them, and its output goes back into all of
them while they are mixed:

    u = sum_s enter_s x_s;   y = sublayer(norm(u));   x_t <- sum_s mix_st x_s + leave_t y     (every t from the old streams)

At a step's end the stream is the sum of the copies.  The update a sublayer leaves behind and the weighted sum and norm of the
next one walk the same rows, so the update is owed (like `parts.residual` leaves partial sums owed) until somebody reads the
streams: one kernel then completes the sublayer's split sum, mixes, writes the streams back and norms the weighted sum.  Until the
first update the copies are one tensor."""
from typing import Optional

import torch

from .. import ops
from ..weights.loader import ParamSpec
from .residual import Branch


class StreamMix:
    """The constants of one sublayer; `enter`, `leave` and `mix` are 32-bit once loaded."""

    def __init__(self, n: int):
        self.n = n
        self.enter = self.leave = self.mix = None

    def param_specs(self):
        return {"enter": ParamSpec((self.n,), "vector"), "leave": ParamSpec((self.n,), "vector"), "mix": ParamSpec((self.n, self.n), "vector")}

    def load(self, tensors):
        self._stored = {k: tensors[k] for k in ("enter", "leave", "mix")}
        self.enter, self.leave, self.mix = (self._stored[k].float().contiguous() for k in ("enter", "leave", "mix"))

    def export(self):
        return dict(self._stored)


class Streams:
    """The n streams of a step's T tokens.  x: the embedding output, float32 [T, dim]."""

    def __init__(self, x: torch.Tensor, n: int):
        if n < 1:
            raise ValueError(f"{n} residual streams")
        self.n = int(n)
        self.x, self.shared = x, True               # [T, dim] while the streams are equal, then [n, T, dim]
        self.owed = None                            # (Branch, StreamMix): an update still to be done
        self.closed = False

    @property
    def n_tokens(self) -> int:
        return self.x.shape[-2]

    @property
    def device(self):
        return self.x.device

    def leave(self, branch: Branch, mix: StreamMix) -> None:
        """A sublayer's output goes into the streams; done when they are next read."""
        self.resolve()
        self.owed = (branch, mix)

    def read(self, mix: Optional[StreamMix]) -> "StreamRead":
        """What the sublayer with these constants reads (None: the plain sum of the streams)."""
        return StreamRead(self, None if mix is None else mix.enter)

    def total(self) -> "StreamRead":
        """The sum of the streams at a step's end: nothing reads the streams themselves after it."""
        return StreamRead(self, None, last=True)

    def tensor(self) -> torch.Tensor:
        """The sum of the streams, complete, float32 [T, dim]."""
        return self.read(None).value()

    def resolve(self) -> None:
        if self.owed is not None:
            self.step()

    def step(self, enter=None, weight=None, eps: float = 0.0, out=None, rows=None, last: bool = False) -> None:
        """One kernel: the owed update, and out = norm(sum_s enter_s x_s) or the sum itself without a weight."""
        if self.closed:
            raise ValueError("the streams of this step have been summed up")
        if rows is not None and not last:
            self.resolve()                          # a gather of rows writes no streams
        kw = {}
        if self.owed is not None:
            (branch, mix), self.owed = self.owed, None
            kw = dict(mix=mix.mix, leave=mix.leave, branches=branch.values())
            if last:
                self.closed = True
            else:
                kw["x_out"] = torch.empty(self.n, *self.x.shape, dtype=torch.float32, device=self.x.device) if self.shared else self.x
        ops.streams(self.x, self.n, self.shared, enter=enter, weight=weight, eps=eps, out=out, rows=rows, **kw)
        if kw.get("x_out") is not None:
            self.x, self.shared = kw["x_out"], False


class StreamRead:
    """A weighted sum of the streams that has not been made yet: a norm makes it on its way (`into`)."""

    def __init__(self, streams: Streams, enter, last: bool = False):
        self.streams, self.enter, self.last = streams, enter, last

    def into(self, out, weight=None, eps: float = 0.0, rows=None) -> None:
        """out = the sum, divided by its root mean square and times `weight` (None: the sum itself); rows picks rows."""
        self.streams.step(self.enter, weight, eps, out, rows, self.last)

    def value(self) -> torch.Tensor:
        """The sum, float32 [T, dim]."""
        s = self.streams
        out = torch.empty(s.n_tokens, s.x.shape[-1], dtype=torch.float32, device=s.device)
        self.into(out)
        return out
