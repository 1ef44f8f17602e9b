"""Gated linear attention: a linear recurrence over key-value products with a decay per head and key channel.

    q = head_dim^-1/2 Wq h, k = Wk h (heads x head_dim), v = Wv h (heads x v_head_dim), gate = Wg h (heads x v_head_dim)
    z = Wa2 (Wa1 h) + b                                          heads x head_dim, through `decay_rank` numbers
    S <- diag(sigmoid(z)^(1/tau)) S + k v^T;  o = S^T q          per head, S [head_dim, v_head_dim], zero at the start
    y = Wo concat_h (o / rms(o) * norm * silu(gate))             rms over v_head_dim, eps inside the root

The five projections of h are one product; everything behind it up to the gated read-out is 32-bit.  The state S is the
mixer's only memory: a fixed-size per-sequence state of the cache, carried from step to step."""
import torch

from .. import ops
from ..cache.needs import CacheNeeds, StateNeed
from ..weights.loader import ParamSpec
from . import register_mixer
from .residual import as_residual
from .state_space import _pad_rows


@register_mixer("gla")
class GatedLinearAttention:
    def __init__(self, dim: int, n_head: int, head_dim: int, v_head_dim: int, decay_rank: int, tau: float, eps: float,
                 dtype: torch.dtype, position=None):
        if not tau > 0:
            raise ValueError(f"the decays' exponent 1/tau needs a positive tau, got {tau}")
        self.dim, self.n_head, self.head_dim, self.v_head_dim, self.decay_rank = dim, n_head, head_dim, v_head_dim, decay_rank
        self.tau, self.eps, self.dtype = float(tau), float(eps), dtype
        self.state_floats = n_head * head_dim * v_head_dim
        self.w_in = self.a2 = self.a2_bias = self.norm = self.wo = None

    def _rows(self):
        H, d, dv = self.n_head, self.head_dim, self.v_head_dim
        return [H * d, H * d, H * dv, H * dv, self.decay_rank]                 # q, k, v, gate, low-rank decay inputs

    def param_specs(self):
        H, d, dv, D = self.n_head, self.head_dim, self.v_head_dim, self.dim
        return {"wq": ParamSpec((H * d, D)), "wk": ParamSpec((H * d, D)), "wv": ParamSpec((H * dv, D)), "wg": ParamSpec((H * dv, D)),
                "wa1": ParamSpec((self.decay_rank, D)), "wa2": ParamSpec((H * d, self.decay_rank)), "a2_bias": ParamSpec((H * d,), "vector"),
                "norm": ParamSpec((dv,), "vector"), "wo": ParamSpec((D, H * dv))}

    def load(self, tensors):
        self.w_in = _pad_rows(torch.cat([tensors[k] for k in ("wq", "wk", "wv", "wg", "wa1")]))
        self.a2, self.a2_bias, self.norm, self.wo = tensors["wa2"], tensors["a2_bias"], tensors["norm"], tensors["wo"]

    def export(self):
        rows = self._rows()
        out = dict(zip(("wq", "wk", "wv", "wg", "wa1"), self.w_in[:sum(rows)].split(rows)))
        out.update(wa2=self.a2, a2_bias=self.a2_bias, norm=self.norm, wo=self.wo)
        return out

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateNeed((self.state_floats,), torch.float32))

    def forward(self, h, batch, view, residual, append: bool = True):
        if not append:
            raise ValueError("a gated linear attention layer owns its state: it cannot run on another run's cache entry")
        T = batch.n_tokens
        H, d, dv = self.n_head, self.head_dim, self.v_head_dim
        proj = torch.empty(T, self.w_in.shape[0], dtype=self.dtype, device=h.device)
        ops.linear(h, self.w_in, proj)
        q_off, k_off, v_off, g_off = 0, H * d, 2 * H * d, 2 * H * d + H * dv
        y = torch.empty(T, H * dv, dtype=self.dtype, device=h.device)
        ops.gla(proj, (q_off, k_off, v_off, g_off + H * dv, g_off), self.decay_rank, self.a2, self.a2_bias, self.tau, view.state, 0,
                self.norm, self.eps, y, batch, H, d, dv, q_scale=float(d) ** -0.5)
        as_residual(residual).add_linear(y, self.wo)
