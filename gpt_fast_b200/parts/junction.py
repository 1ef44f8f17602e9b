"""What happens to the stream between two layer runs.

'pass_entry': the entry of a pass of a loop of layers.  Ahead of pass t

    x <- W [x ; x0] + step_t

with x0 the embedding output, W [dim, 2 dim] (the stream's half first) and a vector per pass.  The stream starts anew in a
tensor of its own as step_t, to which the product is added in 32-bit like any sublayer's."""
import torch

from .. import ops
from ..weights.loader import ParamSpec
from . import register_junction
from .residual import Residual


@register_junction("pass_entry")
class PassEntry:
    def __init__(self, dim: int, passes: int, dtype: torch.dtype):
        self.dim, self.passes, self.dtype = dim, int(passes), dtype
        self.weight = self.step = None

    def param_specs(self):
        return {"weight": ParamSpec((self.dim, 2 * self.dim)), "step": ParamSpec((self.passes, self.dim))}

    def load(self, tensors):
        self.weight, self.step = tensors["weight"], tensors["step"]

    def export(self):
        return {"weight": self.weight, "step": self.step}

    def forward(self, x: Residual, x0, turn: int):
        """x: the stream, which goes on in a new tensor; x0 float32 [T, dim]: the embedding output, left as it is."""
        T, dev = x0.shape[0], x0.device
        cat = torch.empty(T, 2 * self.dim, dtype=self.dtype, device=dev)
        new = torch.empty(T, self.dim, dtype=torch.float32, device=dev)
        ops.pass_entry(x.tensor(), x0, self.step[turn], cat, new)
        x.x = new
        x.add_linear(cat, self.weight)
