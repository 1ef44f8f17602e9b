"""The Pikalix decoder stated plainly: whole sequences, 64-bit, no cache, one function per mechanism.

It shares no code with the package; tests compare the package's results with it.  Weights come as a dict of
tensors under the checkpoint's own names, the configuration as the config.json dict.

    embedding        e_t = E[tok_t] / rms(E[tok_t]) * w;  all S streams start as e
    sublayer f with constants a [S], b [S], M [S, S] (from, to):
                     u = sum_s a_s x_s;   y = f(n(u));   x_t <- sum_s M_st x_s + b_t y   (all t from the old streams)
    layer            the mixer, then the feed-forward (where there is one), each such a sublayer
    'attention'      grouped-query attention with biases on q, k and v, q and k normed over the whole projection, interleaved
                     rotation of the first dimensions, a sliding window and exp(0) as one more term of the denominator;
                     with 'kv_from' the keys and values of another layer
    feed-forward     dense with the tanh form of GELU, or routed SwiGLU experts (sigmoid scores, groups by the sum of
                     their two best choice scores, weights as they are) beside a shared one
    output           head (n(sum_s x_s))
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, base, dims):
    """x [T, heads, d]: dimensions 2i and 2i + 1, i < dims / 2, are turned by position * base^(-2i/dims); the rest passes."""
    T, half = x.shape[0], dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    a = torch.arange(T, dtype=F64)[:, None, None] * f
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def visible(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if window is None else seen & (i - j < window)


def softmax_plus_one(s, mask):
    """s [..., T, T]: exp(s_j) / (1 + sum exp(s_j)) over the visible j."""
    s = s.masked_fill(~mask, -math.inf)
    top = s.amax(-1, keepdim=True).clamp(min=0.0)
    p = torch.exp(s - top)
    return p / (p.sum(-1, keepdim=True) + torch.exp(-top))


def keys_and_values(h, w, m, eps):
    T, G = h.shape[0], m["kv_heads"]
    k = norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps).view(T, G, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).view(T, G, m["vdim"])
    return rotate_pairs(k, m["rot"]["base"], m["rot"]["dims"]), v


def attention(h, w, m, eps, kv):
    """kv: (keys [T, G, d], values [T, G, dv]) as a cache holds them."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).view(T, H, m["dim"])
    q = rotate_pairs(q, m["rot"]["base"], m["rot"]["dims"])
    k, v = (t.repeat_interleave(H // G, 1) for t in kv)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    p = softmax_plus_one(s, visible(T, m["mask"]["size"] if m.get("mask") else None))
    return torch.einsum("hij,jhv->ihv", p, v).reshape(T, H * m["vdim"]) @ w["o"].T


def dense(h, w):
    return gelu_tanh(h @ w["up"].T) @ w["down"].T


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def group_score(c):
    """c: the choice scores of one group (a list)."""
    return sum(sorted(c, reverse=True)[:2])


def choose(z, correction, top, groups, keep):
    """(experts [T, top], weights [T, top], margin [T]) from router logits z [T, E].  margin: how far the choice is from
    another one, in score units: the gap between the last chosen and the first left-out expert of the kept groups, or
    between the last kept and the first dropped group if that is smaller (infinite where nothing is left out)."""
    T, E = z.shape
    s = torch.sigmoid(z)
    c = s + correction
    per = E // groups
    idx, wts, margins = [], [], []
    for t in range(T):
        row = c[t].tolist()
        score = [group_score(row[g * per:(g + 1) * per]) for g in range(groups)]
        order = sorted(range(groups), key=lambda g: (-score[g], g))
        cand = sorted((e for g in order[:keep] for e in range(g * per, (g + 1) * per)), key=lambda e: (-row[e], e))
        m = math.inf
        if keep < groups:
            m = score[order[keep - 1]] - score[order[keep]]
        if top < len(cand):
            m = min(m, row[cand[top - 1]] - row[cand[top]])
        idx.append(cand[:top])
        wts.append(s[t, cand[:top]])
        margins.append(m)
    return torch.tensor(idx), torch.stack(wts), torch.tensor(margins, dtype=F64)


def experts(h, mlp, w, margins=None):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    idx, wt, margin = choose(h @ w["router"].T, w["correction"], r["top"], g["count"], g["keep"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        t, j = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out.index_add_(0, t, wt[t, j][:, None] * expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]))
    if mlp.get("shared"):
        out = out + expert(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


def enter(x, a):
    """x [S, T, D]: what a sublayer reads."""
    return torch.einsum("s,std->td", a, x)


def leave(x, mix, b, y):
    """The new streams from the old ones and a sublayer's output; mix [from, to]."""
    return torch.einsum("sr,std->rtd", mix, x) + b[:, None, None] * y


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, streams=None, margins=None, act=None):
    """Logits [T, vocab] (64-bit) of one whole sequence; `streams` (a list) receives the sum of the streams behind every
    layer, `margins` (a list) the router's margin per token of every layer with experts.  act (torch.bfloat16): the normed
    input of every sublayer is rounded to that type, to measure how much the format's rounding moves the logits."""
    rnd = (lambda v: v) if act is None else (lambda v: v.to(act).to(F64))
    W = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    e = norm(W["embed"][torch.as_tensor(tokens, dtype=torch.long)], W["embed.norm"], eps)
    x = e.expand(cfg["streams"], *e.shape)
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        w = sub(W, p + "mix.")
        h = rnd(norm(enter(x, W[p + "hc1.in"]), W[p + "norm1"], eps))
        if m.get("kv_from") is None:
            kept[i] = keys_and_values(h, w, m, eps)
        y = attention(h, w, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        x = leave(x, W[p + "hc1.mix"], W[p + "hc1.out"], y)
        if L.get("mlp"):
            h = rnd(norm(enter(x, W[p + "hc2.in"]), W[p + "norm2"], eps))
            w = sub(W, p + "mlp.")
            y = experts(h, L["mlp"], w, margins) if L["mlp"]["kind"] == "moe" else dense(h, w)
            x = leave(x, W[p + "hc2.mix"], W[p + "hc2.out"], y)
        if streams is not None:
            streams.append(x.sum(0))
    return rnd(norm(x.sum(0), W["final.norm"], eps)) @ W["head"].T
