"""The Dufizen decoder stated plainly: whole sequences, 64-bit, no cache, one function per mechanism.

It shares no code with the package; tests compare the package's results with it.  Weights come as a dict of
tensors under the checkpoint's own names, the configuration as the config.json dict.

    embedding        x0_t = E[tok_t]
    loop             layers a .. b-1 run R times with the same weights; ahead of pass r:  x <- M [x ; x0] + step_r
    layer            x <- x + s1 * mixer(n1(x));  x <- x + s2 * ff(n2(x));  x <- x + token input;   n(v) = v / rms(v) (1 + w)
    token input      e = the layer's slice of the side table's row of the token;  y = P (gelu(G x) * e);  x <- x + y / rms(y) * u
    'gla'            per head S <- diag(a) S + k v^T, o = S^T q,  a = sigmoid(z)^(1/tau) per key channel, z = A2 A1 h + b;
                     o / rms(o) * w, times silu(Wg h)
    'latent_attention'
                     keys and values expanded from a normed latent, a rotated key part shared by all heads, a sliding
                     window, a learned sink per head in the softmax, a sigmoid gate per head
    feed-forward     `top` of E experts W_down relu(W_up h)^2, weighted by the softmax over ALL experts, chosen by that score
                     plus a correction among the groups whose best choice score is largest; plus a shared expert
    output           E n(x)
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def pass_entry(x, x0, w_in, step):
    """What happens ahead of a pass of the loop: the stream beside the embedding output, mixed, plus the pass's vector."""
    return torch.cat([x, x0], -1) @ w_in.T + step


def token_input(x, e, gate, proj, norm, eps):
    """What a layer adds for the token itself: e [T, n], gate [n, D], proj [D, n]."""
    y = (gelu_tanh(x @ gate.T) * e) @ proj.T
    return rms(y, eps) * norm


def channel_decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def linear_attention_scan(q, k, v, a):
    """q, k, a [T, H, d], v [T, H, dv] -> o [T, H, dv]; the state starts at zero."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64)
    out = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gla(h, w, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].T).view(T, H, d)
    v = (h @ w["v"].T).view(T, H, dv)
    a = channel_decay((h @ w["a1"].T) @ w["a2"].T + w["a2.b"], m["tau"]).view(T, H, d)
    o = rms(linear_attention_scan(q, k, v, a), eps) * w["norm"]
    return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def rotate_half(x, base, dims):
    """x [T, ..., r]: dimension i of the first `dims` is paired with i + dims/2 and turned by position * base^(-2i/dims)."""
    T, half = x.shape[0], dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    ang = (torch.arange(T, dtype=F64)[:, None] * f).view([T] + [1] * (x.dim() - 2) + [half])
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def visible(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if window is None else seen & (i - j < window)


def softmax_with_sink(s, mask, sink):
    """s [H, T, T]; one more term exp(sink_h) in every row's denominator."""
    s = s.masked_fill(~mask, -math.inf)
    top = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    p = torch.exp(s - top)
    return p / (p.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def latent_attention(h, w, m, eps):
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).view(T, H, d + r)
    dkv = h @ w["dkv"].T
    c = rms(dkv[:, :R], eps) * w["dkv.norm"]
    k_rot = rotate_half(dkv[:, R:], m["rot"]["base"], m["rot"]["dims"])
    q_rot = rotate_half(q[..., d:], m["rot"]["base"], m["rot"]["dims"])
    k = (c @ w["uk"].T).view(T, H, d)
    v = (c @ w["uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihr,jr->hij", q_rot, k_rot)) * m["scale"]
    p = softmax_with_sink(s, visible(T, m["mask"]["size"] if m.get("mask") else None), w["sink"])
    o = torch.einsum("hij,jhv->ihv", p, v) * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


def expert(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


def choose(z, correction, top, groups, keep):
    """(experts [T, top], weights [T, top], margin [T]) from router logits z [T, E].  margin: how far the choice is from
    another one, in score units: the gap between the last chosen and the first left-out expert of the kept groups, or
    between the last kept and the first dropped group if that is smaller (infinite where nothing is left out)."""
    T, E = z.shape
    s = torch.softmax(z, -1)
    c = s + correction
    idx, wts, margins = [], [], []
    per = E // groups
    for t in range(T):
        best = [float(c[t, g * per:(g + 1) * per].max()) for g in range(groups)]
        order = sorted(range(groups), key=lambda g: (-best[g], g))
        kept = order[:keep]
        cand = sorted((e for g in kept for e in range(g * per, (g + 1) * per)), key=lambda e: (-float(c[t, e]), e))
        m = math.inf
        if keep < groups:
            m = min(m, best[order[keep - 1]] - best[order[keep]])
        if top < len(cand):
            m = min(m, float(c[t, cand[top - 1]] - c[t, cand[top]]))
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
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = int(idx[t, j])
            out[t] += wt[t, j] * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if mlp.get("shared"):
        out = out + expert(h, w["shared.up"], w["shared.down"])
    return out


MIXERS = {"gla": gla, "latent_attention": latent_attention}


def runs(cfg):
    """(layer, pass or None, whether the pass begins with it) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None, False) for i in range(a)]
    for t in range(times):
        out += [(i, t, i == a) for i in range(a, b)]
    return out + [(i, None, False) for i in range(b, n)]


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, streams=None, margins=None, act=None):
    """Logits [T, vocab] (64-bit) of one whole sequence; `streams` (a list) receives x behind every layer run, `margins` (a
    list) the router's margin per token of every layer run with experts.  act (torch.bfloat16): the normed input of every
    sublayer is rounded to that type, to measure how much the format's rounding moves the logits."""
    rnd = (lambda v: v) if act is None else (lambda v: v.to(act).to(F64))
    W = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x0 = W["embed"][tok]
    x = x0
    side = cfg.get("token_side")
    for i, t, first in runs(cfg):
        if first:
            x = pass_entry(x, x0, W["loop.in"], W["loop.step"][t])
        L, p = cfg["layers"][i], f"l{i}."
        x = x + W[p + "ls1"] * MIXERS[L["type"]](rnd(one_plus_norm(x, W[p + "norm1"], eps)), sub(W, p + "mix."), L["mixer"], eps)
        if L.get("mlp"):
            x = x + W[p + "ls2"] * experts(rnd(one_plus_norm(x, W[p + "norm2"], eps)), L["mlp"], sub(W, p + "mlp."), margins)
        if side:
            e = W["side.embed"][tok][:, i * side["dim"]:(i + 1) * side["dim"]]
            x = x + token_input(x, e, W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"], eps)
        if streams is not None:
            streams.append(x.clone())
    return rnd(one_plus_norm(x, W["final.norm"], eps)) @ W["embed"].T
