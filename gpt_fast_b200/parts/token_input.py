"""What a layer adds to the stream for the token itself, whatever the context.

'gated_side': the model has a side table with a row per token; a layer owns `side_dim` of its columns, from `offset` on.

    e = side[token][offset : offset + side_dim];   g = gelu_tanh(Wg x) * e;   y = Wp g;   x += y / rms(y) * norm

x is the stream as it stands (not normed); rms with eps inside the root.  The normed sum is left to the stream, whose next
norm does it on the way (`Residual.add_normed`)."""
import torch

from .. import ops
from ..weights.loader import ParamSpec
from . import register_token_input
from .norm import NoNorm, RMSNorm
from .residual import Branch, as_residual


@register_token_input("gated_side")
class GatedSide:
    def __init__(self, dim: int, side_dim: int, offset: int, eps: float, dtype: torch.dtype):
        if side_dim < 1 or offset < 0:
            raise ValueError(f"{side_dim} columns of the side table from column {offset}")
        self.dim, self.side_dim, self.offset, self.dtype = dim, int(side_dim), int(offset), dtype
        self._read, self._norm = NoNorm(dim, dtype), RMSNorm(dim, eps, dtype)
        self.gate = self.proj = self.table = None

    def param_specs(self):
        return {"gate": ParamSpec((self.side_dim, self.dim)), "proj": ParamSpec((self.dim, self.side_dim)),
                "norm": ParamSpec((self.dim,), "vector")}

    def load(self, tensors):
        self.gate, self.proj = tensors["gate"], tensors["proj"]
        self._norm.load({"weight": tensors["norm"]})

    def export(self):
        return {"gate": self.gate, "proj": self.proj, "norm": self._norm.export()["weight"]}

    def bind_token_table(self, table):
        """The model's side table [vocab, columns], handed over when the weights are loaded."""
        if table is None or self.offset + self.side_dim > table.shape[1]:
            raise ValueError(f"a side table with columns {self.offset} .. {self.offset + self.side_dim - 1} is needed, the model has "
                             f"{None if table is None else tuple(table.shape)}")
        self.table = table

    def forward(self, x, batch):
        x = as_residual(x)
        T, dev = x.x.shape[0], x.x.device
        h = torch.empty(T, self.dim, dtype=self.dtype, device=dev)
        self._read.forward(x, h)
        z = torch.empty(T, self.side_dim, dtype=torch.float32, device=dev)
        ops.linear(h, self.gate, z)
        g = torch.empty(T, self.side_dim, dtype=self.dtype, device=dev)
        ops.token_gate(z, batch.tokens, self.table, self.offset, g, batch.status)
        y = Branch(T, self.dim, dev)
        y.add_linear(g, self.proj)
        x.add_normed(y, self._norm, 1.0)
