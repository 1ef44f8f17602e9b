"""Mixture of experts as a feed-forward: every token runs `top` of `n_experts` small gated feed-forwards.

    z = W_router h                      router logits, 32-bit
    s = sigmoid(z);  chosen = the `top` experts with the largest s + correction  (the correction counts for the choice only)
    w_e = s_e / (sum of the chosen s + 1e-20) * scale
    expert e:  g = min(W_gate h, limit),  u = clamp(W_up h, -limit, limit),  y = W_down (g * sigmoid(alpha g) * (u + shift))
    result = sum over the chosen e of w_e * y_e

Options: score 'softmax_top' chooses the `top` largest logits themselves (plus the correction, if there is one) and weighs
the chosen experts by the softmax over just their logits (times scale).  `shared_hidden`: one more expert of that size, a
plain SwiGLU that every token runs; with `shared_gate` its output is multiplied by sigmoid(w_s . h), one number per token,
whose row rides behind the router's rows in one product.

Score 'softmax' takes s = softmax(z) over all experts, chooses by s + correction and weighs by s * scale as it is.
Score 'sigmoid_plain' is 'sigmoid' with the chosen experts' s * scale as weights, not divided by their sum.
`groups` = (count, keep[, terms]): the experts are `count` equal groups of neighbours; a group's score is the largest choice score
in it (with terms = 2 the sum of its two largest) and only experts of the `keep` best groups can be chosen.  `activation` 'relu2': experts (and the shared one) of two products,
W_down max(W_up h, 0)^2.  A shared expert without a gate and of the experts' own size is one more expert that every token
chooses with weight 1, so the experts' products run it along; of another size it is a feed-forward of its own.

The experts have no biases.  Their gate and up rows alternate in one matrix per expert, so one product yields both and
applies the activation before anything is written; the weighted sum of the chosen experts' outputs is added to the
residual stream in 32-bit by the kernel that does the down products (or by the one behind it)."""
import torch

from .. import ops
from ..weights.loader import ParamSpec
from . import register_feed_forward
from .residual import Branch, as_residual


def _pad_rows(w: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    extra = -w.shape[0] % multiple
    return w.contiguous() if extra == 0 else torch.cat([w, w.new_zeros(extra, w.shape[1])]).contiguous()


@register_feed_forward("moe")
class MixtureOfExperts:
    def __init__(self, dim: int, hidden: int, n_experts: int, top: int, dtype: torch.dtype, router_scale: float = 1.0,
                 limit: float = 0.0, alpha: float = 1.0, shift: float = 0.0, correction: bool = True, score: str = "sigmoid",
                 shared_hidden: int = 0, shared_gate: bool = False, activation: str = "glu", groups=None):
        if not 1 <= top <= n_experts:
            raise ValueError(f"{top} of {n_experts} experts per token")
        if score not in ("sigmoid", "sigmoid_plain", "softmax_top", "softmax"):
            raise ValueError(f"a router score is 'sigmoid', 'sigmoid_plain', 'softmax_top' or 'softmax', not {score!r}")
        if activation not in ("glu", "relu2"):
            raise ValueError(f"the experts' activation is 'glu' or 'relu2', not {activation!r}")
        if groups is not None and (groups[0] < 1 or n_experts % groups[0] or not 1 <= groups[1] <= groups[0]
                                   or top > groups[1] * (n_experts // groups[0])):
            raise ValueError(f"{top} experts from {groups[1]} of {groups[0]} groups of {n_experts} experts in all")
        if groups is not None and len(groups) > 2 and groups[2] not in (1, 2):
            raise ValueError(f"a group's score is made of one or two choice scores, not {groups[2]}")
        self.activation, self.groups = activation, None if groups is None or groups[0] == 1 else tuple(int(g) for g in groups)
        if shared_gate and not shared_hidden:
            raise ValueError("a gate for a shared expert that is not there")
        self.score, self.shared_hidden, self.shared_gate = score, int(shared_hidden or 0), bool(shared_gate)
        # one more expert that every token chooses, in the experts' own stacks
        plain_glu = float(limit) <= 0 and float(alpha) == 1.0 and float(shift) == 0.0          # the shared expert is a plain SwiGLU
        self.shared_inside = (bool(self.shared_hidden) and not self.shared_gate and self.shared_hidden == hidden
                              and (activation == "relu2" or plain_glu))
        self.shared_w13 = self.shared_w2 = None
        self.dim, self.hidden, self.n_experts, self.top, self.dtype = dim, hidden, int(n_experts), int(top), dtype
        self.router_scale, self.limit, self.alpha, self.shift = float(router_scale), float(limit), float(alpha), float(shift)
        self.has_correction = bool(correction)
        self.router = self.correction = self.w13 = self.w2 = None

    def param_specs(self):
        E, F, D = self.n_experts, self.hidden, self.dim
        specs = {"router": ParamSpec((E, D)), "up": ParamSpec((E, F, D)), "down": ParamSpec((E, D, F))}
        if self.activation == "glu":
            specs["gate"] = ParamSpec((E, F, D))
        if self.has_correction:
            specs["correction"] = ParamSpec((E,), "vector")
        if self.shared_hidden:
            Fs = self.shared_hidden
            specs.update(shared_up=ParamSpec((Fs, D)), shared_down=ParamSpec((D, Fs)))
            if self.activation == "glu":
                specs["shared_gate"] = ParamSpec((Fs, D))
            if self.shared_gate:
                specs["shared_sg"] = ParamSpec((1, D))
        return specs

    def load(self, tensors):
        E, F, D = self.n_experts, self.hidden, self.dim
        self._router_stored = tensors["router"]
        self.router = _pad_rows(torch.cat([tensors["router"], tensors["shared_sg"]]) if self.shared_gate else tensors["router"])
        if self.shared_hidden and self.activation == "relu2":
            self.shared_w13, self.shared_w2 = tensors["shared_up"], tensors["shared_down"]
        elif self.shared_hidden:
            self.shared_w13 = torch.stack([tensors["shared_gate"], tensors["shared_up"]], dim=1).reshape(2 * self.shared_hidden, D).contiguous()
            self.shared_w2 = tensors["shared_down"]
        self.correction = tensors["correction"] if self.has_correction else torch.zeros(E, dtype=torch.float32, device=tensors["router"].device)
        if self.activation == "relu2":
            self.w13, self.w2 = tensors["up"], tensors["down"]
            if self.shared_inside:
                self.w13, self.w2 = torch.cat([self.w13, self.shared_w13[None]]), torch.cat([self.w2, self.shared_w2[None]])
                self.shared_w13 = self.shared_w2 = None
            return
        # rows alternate gate, up within every expert
        self.w13 = torch.stack([tensors["gate"], tensors["up"]], dim=2).reshape(E, 2 * F, D).contiguous()
        self.w2 = tensors["down"]
        if self.shared_inside:
            self.w13, self.w2 = torch.cat([self.w13, self.shared_w13[None]]), torch.cat([self.w2, self.shared_w2[None]])
            self.shared_w13 = self.shared_w2 = None

    def export(self):
        if self.activation == "relu2":
            E = self.n_experts
            out = {"router": self._router_stored, "up": self.w13[:E], "down": self.w2[:E]}
            if self.has_correction:
                out["correction"] = self.correction
            if self.shared_hidden:
                out.update(shared_up=self.w13[E] if self.shared_inside else self.shared_w13,
                           shared_down=self.w2[E] if self.shared_inside else self.shared_w2)
                if self.shared_gate:
                    out["shared_sg"] = self.router[E:E + 1]
            return out
        E = self.n_experts
        w = self.w13.view(-1, self.hidden, 2, self.dim)
        out = {"router": self._router_stored, "gate": w[:E, :, 0], "up": w[:E, :, 1], "down": self.w2[:E]}
        if self.has_correction:
            out["correction"] = self.correction
        if self.shared_hidden:
            sw = w[E] if self.shared_inside else self.shared_w13.view(self.shared_hidden, 2, self.dim)
            out.update(shared_gate=sw[:, 0], shared_up=sw[:, 1], shared_down=self.w2[E] if self.shared_inside else self.shared_w2)
            if self.shared_gate:
                out["shared_sg"] = self.router[self.n_experts:self.n_experts + 1]
        return out

    def forward(self, h, residual):
        T = h.shape[0]
        slots = self.top + (1 if self.shared_inside else 0)
        idx = torch.empty(T, slots, dtype=torch.int32, device=h.device)
        w = torch.empty(T, slots, dtype=torch.float32, device=h.device)
        gate = ops.moe_router(h, self.router, self.correction, self.top, self.router_scale, idx, w, score=self.score,
                              n_extra=1 if self.shared_gate else 0, groups=self.groups, shared=self.shared_inside)
        residual = as_residual(residual)
        x = residual.fresh() if isinstance(residual, Branch) else None       # an empty branch: the experts' kernel writes all of it
        store = x is not None
        if not store:
            x = residual.tensor()                              # complete: the experts' kernel adds into it
        ops.moe_experts(h, idx, w, self.w13, self.w2, x, self.limit, self.alpha, self.shift, act=self.activation, store=store)
        if self.shared_hidden and not self.shared_inside:
            act = torch.empty(T, self.shared_hidden, dtype=self.dtype, device=h.device)
            ops.linear(h, self.shared_w13, act, mode="swiglu" if self.activation == "glu" else "relu2")
            if self.shared_gate:
                # a factor per token commutes with the down product: it goes onto the activations
                ops.sigmoid_gate(act, gate[0], gate[1], self.shared_hidden)
            residual.add_linear(act, self.shared_w2)
