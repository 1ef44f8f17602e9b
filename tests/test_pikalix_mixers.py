"""Each mechanism of the Pikalix design alone, as a part with a cache entry of its own, against the plain statement of the
mechanism in `plain_pikalix.py`: the input goes in whole, in portions and as a batch of two sequences, and what the part adds
to an empty stream is compared.  Where random inputs would hide a fault (a key at a window's edge or hundreds of positions back, the
one in the softmax denominator, a mixing matrix that is nearly the identity) the inputs are made so that it stands out.  Three back
ends as in `test_pikalix.py`."""
import pytest
import torch

from gpt_fast_b200 import ops
from gpt_fast_b200.cache import Cache, EntryView
from gpt_fast_b200.config.spec import PartSpec
from gpt_fast_b200.ops.types import BatchMeta
from gpt_fast_b200.parts import BLOCKS, EMBEDDINGS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS, build_part
from gpt_fast_b200.parts.residual import Branch, Residual
from gpt_fast_b200.parts.streams import StreamMix, Streams
import plain_ops
import plain_pikalix as pp

BACKENDS = [
    pytest.param(("cpu", torch.float32), id="cpu-standin-f32"),
    pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu),
]
D, EPS = 40, 1e-5


@pytest.fixture(params=BACKENDS)
def backend(request):
    device, dtype = request.param
    prev = ops.use_kernels(plain_ops.PlainOps()) if device == "cpu" else None
    yield device, dtype
    if device == "cpu":
        ops.use_kernels(prev)


def rand(shape, seed, scale=1.0, shift=0.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale + shift).to(torch.bfloat16)


def run(part, h, seqs, cuts, device, dtype, reader=None):
    """Feed the sequences (lists of row ranges of h) through a mixer as one batch, each cut at `cuts`; what it added, in h's
    row order.  reader: another mixer that attends over the first one's cache entry with queries of its own; what IT added."""
    cache = Cache({0: part.cache_needs()}, dtype, device, max_tokens=2048, max_seqs=4)
    for p in (part, reader):
        if p is not None and p.position is not None:
            p.position.prepare(cache.max_pages * cache.page_size, device)
    slots = cache.begin(len(seqs))
    out = torch.zeros(h.shape)
    bounds = [0] + list(cuts) + [max(len(s) for s in seqs)]
    for lo, hi in zip(bounds[:-1], bounds[1:]):
        live = [(slot, s[lo:hi]) for slot, s in zip(slots, seqs) if len(s[lo:hi])]
        if not live:
            continue
        rows = [r for _, p in live for r in p]
        q_lens = [len(p) for _, p in live]
        for slot, p in live:
            cache.reserve(slot, cache.lengths_host[slot] + len(p))
        cache.sync_tables()
        cu = [0]
        for q in q_lens:
            cu.append(cu[-1] + q)
        ids = [s for s, _ in live]
        batch = BatchMeta(torch.tensor(cu, dtype=torch.int32).to(device),
                          torch.tensor([i for i, q in enumerate(q_lens) for _ in range(q)], dtype=torch.int32).to(device),
                          torch.tensor(ids, dtype=torch.int32).to(device), cache.lengths, len(live), cu[-1], max(q_lens),
                          max(cache.lengths_host[s] + q for s, q in zip(ids, q_lens)), ops.new_status(device))
        x = h[rows].to(dtype).to(device).contiguous()
        y = Branch(len(rows), h.shape[1], device)
        part.forward(x, batch, cache.view(0), residual=y, append=True)
        if reader is not None:
            y = Branch(len(rows), h.shape[1], device)
            reader.forward(x, batch, EntryView(kv=cache.view(0).kv), residual=y, append=False)
        out[rows] = y.tensor().float().cpu()
        ops.advance_lengths(batch)
        cache.note_advance(ids, q_lens)
        ops.check_status(batch.status)
    cache.end(slots)
    return out


def judge(got, want, dtype, where, bf16=0.03, f32=2e-4):
    scale = float(want.pow(2).mean().sqrt())
    if dtype == torch.float32:
        assert float((got - want.float()).abs().max()) <= f32 * scale, f"{where}: {float((got - want.float()).abs().max()) / scale:.2e} of the scale"
    else:
        err = float((got - want.float()).pow(2).mean().sqrt()) / scale
        assert err <= bf16, f"{where}: {err:.4f} of the scale"


def load(part, weights, names, backend):
    """Matrices in the compute type, vectors in 32-bit, under the part's own parameter names."""
    device, dtype = backend
    specs = part.param_specs()
    part.load({k: weights[v].to(dtype if specs[k].role == "matrix" else torch.float32).to(device) for k, v in names.items()})


def f64(w):
    return {k: v.double() for k, v in w.items()}


CUTS = (([], "whole"), ([1, 3, 64, 66], "portions"), (list(range(60, 75)), "a prompt, then token by token"))

# ---- attention -----------------------------------------------------------------------------------------------------------------

def att_m(H=4, G=2, d=12, dv=10, W=19, rot=6, scale=0.3, base=500.0):
    return dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=scale, rot=dict(dims=rot, base=base), mask=None if W is None else dict(size=W))


def att_weights(m, seed, s=0.3):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": rand((H * d, D), seed, s), "k": rand((G * d, D), seed + 1, s), "v": rand((G * dv, D), seed + 2, s),
            "q.b": rand((H * d,), seed + 3, 0.7), "k.b": rand((G * d,), seed + 4, 0.7), "v.b": rand((G * dv,), seed + 5, 0.7),
            "q.norm": rand((H * d,), seed + 6, 0.4, 1.2), "k.norm": rand((G * d,), seed + 7, 0.4, 1.2), "o": rand((D, H * dv), seed + 8, s)}


def att_part(m, w, backend, reader=False):
    r = m["rot"]["dims"]
    pos = build_part(POSITIONS, PartSpec("rope", dict(head_dim=r, base=m["rot"]["base"], pairing="interleaved", freq_dtype="float64")))
    part = build_part(MIXERS, PartSpec("attention", dict(dim=D, n_head=m["heads"], n_kv=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                                                         window=m["mask"]["size"] if m["mask"] else None, scale=m["scale"], bias=True,
                                                         qk_norm_eps=EPS, qk_norm_whole=True, sink_value=0.0, shared_kv=reader)),
                      dtype=backend[1], position=pos)
    names = dict(wq="q", bq="q.b", q_norm="q.norm", wo="o")
    if not reader:
        names.update(wk="k", bk="k.b", k_norm="k.norm", wv="v", bv="v.b")
    load(part, w, names, backend)
    return part


def plain_attention(h, m, w, own=None):
    """own: (m, w) of the layer whose keys and values are read (None: its own)."""
    h, w = h.double(), f64(w)
    return pp.attention(h, w, m, EPS, pp.keys_and_values(h, w if own is None else f64(own[1]), m if own is None else own[0], EPS))


# heads of 64 and 128 with values of the same size are those the tensor-core attention takes in bfloat16
SHAPES = [att_m(), att_m(H=3, G=3, d=16, dv=16, W=65, rot=16), att_m(H=6, G=1, d=9, dv=20, W=1, rot=4), att_m(H=4, G=2, d=64, dv=64, W=64, rot=16, scale=0.125),
          att_m(H=2, G=1, d=128, dv=128, W=100, rot=128, scale=0.09, base=1e6), att_m(H=8, G=4, d=64, dv=64, W=33, rot=64, scale=0.2),
          att_m(H=5, G=5, d=7, dv=3, W=None, rot=2), att_m(H=18, G=2, d=64, dv=64, W=70, rot=32, scale=0.125)]


@pytest.mark.parametrize("m", SHAPES)
def test_attention(backend, m):
    w = att_weights(m, 21)
    part = att_part(m, w, backend)
    seqs = [list(range(140)), list(range(140, 229))]
    h = rand((229, D), 4)
    want = torch.cat([plain_attention(h[s], m, w) for s in seqs])
    for cuts, what in CUTS + (([2, 4, 6, 127, 129], "portions of two"),):
        judge(run(part, h, seqs, cuts, *backend), want, backend[1], f"{m['mask']} {what}")


@pytest.mark.parametrize("m", [SHAPES[0], SHAPES[3], SHAPES[4]])
@pytest.mark.parametrize("W", [7, 130, None])
def test_a_reader_of_anothers_keys(backend, m, W):
    """Queries with a window and weights of their own over the keys and values that another layer normed, rotated and cached; the
    window is smaller and larger than the other layer's."""
    w, w2 = att_weights(m, 31), att_weights(m, 91)
    m2 = dict(m, scale=0.7 * m["scale"], mask=None if W is None else dict(size=W))
    part, reader = att_part(m, w, backend), att_part(m2, w2, backend, reader=True)
    seqs = [list(range(140)), list(range(140, 229))]
    h = rand((229, D), 6)
    want = torch.cat([plain_attention(h[s], m2, w2, (m, w)) for s in seqs])
    for cuts, what in CUTS:
        judge(run(part, h, seqs, cuts, *backend, reader=reader), want, backend[1], f"reader with {m2['mask']}, {what}")
    with pytest.raises(ValueError, match="reads another run's cache entry"):
        reader.forward(h[:1].to(backend[1]).to(backend[0]), type("B", (), dict(n_tokens=1))(), None, residual=None, append=True)


def loud_case(m, seed, backend, T, key, query):
    """Inputs and weights with which the positions from `query` on look for position `key`: the first dimension behind the rotated
    ones copies one input channel into every query head and another one into every key head, and everything else is quiet."""
    H, G, d, r = m["heads"], m["kv_heads"], m["dim"], m["rot"]["dims"]
    w = att_weights(m, seed)
    w["q"], w["k"] = rand((H * d, D), seed + 1, 0.02), rand((G * d, D), seed + 2, 0.02)
    w["q.b"], w["k.b"] = rand((H * d,), seed + 3, 0.3), rand((G * d,), seed + 4, 0.3)
    for hd in range(H):
        w["q"][hd * d + r, 1] = 2.0
    for g in range(G):
        w["k"][g * d + r, 0] = 2.0
    w["q.norm"], w["k.norm"] = torch.ones(H * d).to(torch.bfloat16), torch.ones(G * d).to(torch.bfloat16)
    h = rand((T, D), seed + 10, 0.3)
    h[:, 0], h[:, 1] = 0.0, 0.0
    h[key, 0] = 5.0
    h[query:, 1] = 5.0
    return att_part(m, w, backend), w, h


@pytest.mark.parametrize("shape", [dict(), dict(d=64, dv=64, rot=16), dict(H=2, G=1, d=128, dv=128, rot=64)])
@pytest.mark.parametrize("W,key", [(19, 60), (64, 63), (65, 64), (200, 3), (5, 127), (96, 0), (2, 63)])
def test_the_windows_edge(backend, shape, W, key):
    """A loud key W - 1 positions back is seen, one position later it is gone: in a prompt, in portions whose borders fall
    between them, and in decode steps."""
    m = att_m(W=W, scale=1.0, **shape)
    last = key + W - 1                                          # the last position that sees the key
    T = last + 4
    part, w, h = loud_case(m, 91, backend, T, key, max(key + 1, last - 2))
    want = plain_attention(h, m, w)
    wider, narrower = (plain_attention(h, dict(m, mask=dict(size=W + e)), w) for e in (1, -1))
    scale = float(want.pow(2).mean().sqrt())
    assert float((wider[last + 1] - want[last + 1]).abs().max()) > 0.3 * scale and float((narrower[last] - want[last]).abs().max()) > 0.3 * scale
    for cuts in ([], [last], [last + 1], list(range(last - 2, T)), [key, key + 1, last - 1]):
        got = run(part, h, [list(range(T))], sorted({c for c in cuts if 0 < c < T}), *backend)
        judge(got, want, backend[1], f"window {W}, key {key}, cuts {cuts[:4]}")
        judge(got[-6:], want[-6:], backend[1], f"window {W}, key {key}, cuts {cuts[:4]}, the last rows")


def test_one_joins_the_denominator(backend):
    """Scores far below zero leave almost everything to the one in the denominator, whose value is nothing; scores far above
    leave it nothing.  The first token of a sequence, alone with itself, shows it most."""
    for shape in (dict(), dict(d=64, dv=64, rot=16)):
        m = att_m(H=2, G=1, W=40, scale=1.0, **shape)
        w = att_weights(m, 61)
        w["k"], w["q"] = torch.zeros_like(w["k"]), torch.zeros_like(w["q"])
        d, r = m["dim"], m["rot"]["dims"]
        w["k.norm"], w["q.norm"] = torch.ones(d).to(torch.bfloat16), torch.ones(2 * d).to(torch.bfloat16)
        w["k.b"], w["q.b"] = torch.zeros(d).to(torch.bfloat16), torch.zeros(2 * d).to(torch.bfloat16)
        w["k.b"][r], w["q.b"][r], w["q.b"][d + r] = 1.0, 1.0, -1.0          # head 0 scores high, head 1 low, whatever the token
        part, h = att_part(m, w, backend), rand((90, D), 12)
        want = plain_attention(h, m, w)
        kv = pp.keys_and_values(h.double(), f64(w), m, EPS)
        assert float((want[0] - f64(w)["o"] @ torch.cat([kv[1][0, 0], 0 * kv[1][0, 0]])).abs().max()) < 0.05 * float(want[0].abs().max())
        for cuts in ([], list(range(1, 90)), [1, 3, 80]):
            got = run(part, h, [list(range(90))], cuts, *backend)
            judge(got, want, backend[1], f"cuts {cuts[:3]}")
            judge(got[:4], want[:4], backend[1], "the first tokens")


def test_a_far_key_in_a_long_sequence(backend):
    """One loud key near the start, hundreds of quiet ones behind it, no window in the way: found from a prompt, a portion and
    decode steps."""
    m = att_m(H=2, G=1, d=64, dv=64, rot=16, W=2000, scale=1.0)
    T = 700
    part, w, h = loud_case(m, 17, backend, T, 5, 690)
    want = plain_attention(h, m, w)
    quiet = h.clone()
    quiet[5, 0] = 0
    assert float((plain_attention(quiet, m, w) - want)[690:].pow(2).mean().sqrt()) > 0.5 * float(want[690:].pow(2).mean().sqrt())
    for cuts in ([], [300, 302, 688] + list(range(689, 700))):
        judge(run(part, h, [list(range(T))], cuts, *backend)[690:], want[690:], backend[1], f"far back, cuts {cuts[:3]}")


def test_attention_options_that_exclude_each_other():
    base = dict(dim=8, n_head=2, n_kv=1, head_dim=4, dtype=torch.float32, position=None)
    for extra in (dict(bias=True, conv_taps=3), dict(bias=True, values_are_keys=True), dict(sink=True, sink_value=0.0)):
        with pytest.raises(ValueError):
            MIXERS["attention"](**base, **extra)


# ---- the feed-forwards -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("T,width,ff", [(1, 40, 72), (3, 37, 21), (70, 64, 200), (300, 48, 136), (600, 128, 320)])
def test_dense(backend, T, width, ff):
    """Every form of the product that has the tanh GELU as its epilogue (split over K and not, tiles of one block and of pairs)."""
    device, dtype = backend
    w = {"up": rand((ff, width), 1, 1.5 * width ** -0.5), "down": rand((width, ff), 2, ff ** -0.5)}
    part = build_part(FEED_FORWARDS, PartSpec("dense", dict(dim=width, hidden=ff, activation="gelu_tanh")), dtype=dtype)
    load(part, w, dict(up="up", down="down"), backend)
    h = rand((T, width), 3)
    y = Branch(T, width, device)
    part.forward(h.to(dtype).to(device).contiguous(), residual=y)
    judge(y.tensor().float().cpu(), pp.dense(h.double(), f64(w)), dtype, f"dense {T} x {width} x {ff}", bf16=0.01)


def moe_case(mlp, seed, backend, s=0.3, D=D):
    r, F = mlp["router"], mlp["expert"]["ff"]
    E, Fs = r["experts"], (mlp.get("shared") or {}).get("ff", 0)
    g = r.get("groups") or dict(count=1, keep=1)
    w = {"router": rand((E, D), seed, s), "correction": rand((E,), seed + 1, 1.0, -1.0)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = rand((F, D), seed + 10 + e, s), rand((F, D), seed + 600 + e, s), rand((D, F), seed + 300 + e, s)
    if Fs:
        w["shared.gate"], w["shared.up"], w["shared.down"] = rand((Fs, D), seed + 2, s), rand((Fs, D), seed + 3, s), rand((D, Fs), seed + 4, s)
    part = build_part(FEED_FORWARDS, PartSpec("moe", dict(dim=D, hidden=F, n_experts=E, top=r["top"], score="sigmoid_plain",
                                                          groups=(g["count"], g["keep"], 2), shared_hidden=Fs)), dtype=backend[1])
    device, dtype = backend
    t = {"router": w["router"]}
    t.update({n: torch.stack([w[f"e{e}.{n}"] for e in range(E)]) for n in ("gate", "up", "down")})
    if Fs:
        t.update({f"shared_{n}": w[f"shared.{n}"] for n in ("gate", "up", "down")})
    t = {**{k: v.to(dtype).to(device) for k, v in t.items()}, "correction": w["correction"].float().to(device)}
    part.load(t)
    back = part.export()
    assert set(back) == set(part.param_specs()) and all(torch.equal(back[k], t[k]) for k in back)
    return part, w


def mlp_of(E, top, ff, groups=None, shared=None):
    return dict(expert=dict(ff=ff), router=dict(experts=E, top=top, groups=None if groups is None else dict(count=groups[0], keep=groups[1])),
                shared=None if shared is None else dict(ff=shared))


@pytest.mark.parametrize("T", [1, 3, 20, 70, 300])
@pytest.mark.parametrize("mlp", [mlp_of(14, 3, 16, (2, 1), 16), mlp_of(9, 4, 24, (3, 2), 40), mlp_of(5, 5, 11), mlp_of(40, 1, 8, (20, 3), 8),
                                 mlp_of(6, 2, 13, (6, 2), 9)])
def test_experts(backend, mlp, T):
    part, w = moe_case(mlp, 13, backend)
    device, dtype = backend
    h = rand((T, D), 5)
    margins = []
    want = pp.experts(h.double(), mlp, f64(w), margins)
    for into in ("branch", "stream"):
        y = Branch(T, D, device) if into == "branch" else Residual(torch.full((T, D), 2.0, device=device))
        part.forward(h.to(dtype).to(device).contiguous(), residual=y)
        got = y.tensor().float().cpu() - (0.0 if into == "branch" else 2.0)
        # the router's product is 32-bit of the same inputs here, so only a tie to rounding may fall otherwise
        sure = margins[0] > 1e-5
        judge(got[sure], want[sure], dtype, f"{into}, {T} tokens", f32=3e-4)
    assert part.shared_inside == (mlp["shared"] is not None and mlp["shared"]["ff"] == mlp["expert"]["ff"])


def test_the_choice_and_its_weights(backend):
    """Groups by the sum of their two best corrected scores, negative choice scores, ties and weights by hand: 6 experts in 3
    groups."""
    device, _ = backend
    z = torch.tensor([[4.0, -4.0, 0.5, 0.4, -5.0, -5.0], [0.0, 0.0, 0.0, 0.0, 0.0, 0.0], [3.0, 0.0, 0.0, 0.0, 2.9, 2.8]])
    s = torch.sigmoid(z.double())

    def choose(c, top, groups, shared=False):
        idx = torch.empty(3, top + shared, dtype=torch.int32, device=device)
        w = torch.empty(3, top + shared, dtype=torch.float32, device=device)
        ops.moe_route(z.to(device).contiguous(), c.to(device), top, 1.0, idx, w, score="sigmoid_plain", groups=groups, shared=shared)
        return idx.cpu().long(), w.cpu().double()
    none = torch.zeros(6)
    idx, w = choose(none, 2, (3, 1, 2))
    assert idx.tolist() == [[2, 3], [0, 1], [4, 5]]            # the best PAIR, although expert 0 is the best single one
    torch.testing.assert_close(w, s.gather(1, idx), rtol=1e-5, atol=1e-7)          # as they are, not divided by their sum
    idx, _ = choose(none, 2, (3, 1, 1))
    assert idx.tolist() == [[0, 1], [0, 1], [0, 1]]            # by the largest single score it is the other group
    idx, _ = choose(none, 2, (3, 2, 2))
    assert idx.tolist() == [[0, 2], [0, 1], [0, 4]]
    # all choice scores negative: the kept groups' experts are chosen all the same, none of a dropped group
    corr = torch.tensor([-3.0, -2.0, -1.5, -4.0, -2.5, -2.6])
    idx, w = choose(corr, 3, (3, 2, 2), shared=True)
    assert idx[:, 3].tolist() == [6, 6, 6] and w[:, 3].tolist() == [1.0, 1.0, 1.0]
    torch.testing.assert_close(w[:, :3], s.gather(1, idx[:, :3]), rtol=1e-5, atol=1e-7)      # the weights leave the correction out
    for t in range(3):
        want, _, _ = pp.choose(z[t:t + 1].double(), corr.double(), 3, 3, 2)
        assert idx[t, :3].tolist() == want[0].tolist()
    # groups of one expert: the sum of what there is
    idx, _ = choose(none, 2, (6, 2, 2))
    assert idx.tolist() == [[0, 2], [0, 1], [0, 4]]


def test_router_options():
    base = dict(dim=8, hidden=8, n_experts=6, top=2, dtype=torch.float32)
    with pytest.raises(ValueError, match="one or two"):
        FEED_FORWARDS["moe"](**base, groups=(3, 2, 3))
    with pytest.raises(ValueError, match="router score"):
        FEED_FORWARDS["moe"](**base, score="tanh")


# ---- the embedding behind its norm -----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("width", [40, 37, 2100])
def test_normed_embedding(backend, width):
    device, dtype = backend
    table, w = rand((30, width), 1, 2.0), rand((width,), 2, 0.4, 1.0)
    table[7] = 0.0                                               # eps inside the root keeps a row of zeros finite
    part = build_part(EMBEDDINGS, PartSpec("normed", dict(dim=width, eps=1e-3)), dtype=dtype)
    part.load({"weight": w.float().to(device)})
    tokens = torch.randint(0, 30, (50,), generator=torch.Generator().manual_seed(5)).to(torch.int32)
    tokens[3] = 7
    out = torch.empty(50, width, device=device)
    batch = type("B", (), dict(status=ops.new_status(device)))()
    part.forward(tokens.to(device), table.to(dtype).to(device), out, batch, None)
    ops.check_status(batch.status)
    want = pp.norm(table[tokens.long()].double(), w.double(), 1e-3)
    assert float((out.cpu().double() - want).abs().max()) <= 2e-6 * float(want.abs().max())


# ---- several streams ---------------------------------------------------------------------------------------------------------------

def mix_of(n, seed, device):
    """Constants far from an ordinary residual sum: no stream stays with itself, some shares are negative, and [from, to] matters."""
    t = {"enter": rand((n,), seed, 0.7, 0.2), "leave": rand((n,), seed + 1, 0.8), "mix": rand((n, n), seed + 2, 0.7)}
    part = StreamMix(n)
    part.load({k: v.float().to(device) for k, v in t.items()})
    return part, f64(t)


@pytest.mark.parametrize("n", [1, 2, 3, 4, 7, 8, 11, 16])
@pytest.mark.parametrize("T,width", [(1, 1024), (5, 40), (140, 1024), (3, 37), (2, 2049), (130, 64), (7, 4096)])
def test_streams(backend, n, T, width):
    """Three sublayers in a row, each with an output in another form (a tensor, partial sums, both), and what the next one reads; the
    sum of the streams at the end, all rows and some of them."""
    device, dtype = backend
    if device == "cpu" and T * width * n > 400000:
        pytest.skip("large rows are for the kernels")
    x0 = rand((T, width), 1).float()
    s = Streams(x0.clone().to(device), n)
    norm = build_part(NORMS, PartSpec("rmsnorm", dict(dim=width, eps=EPS)), dtype=dtype)
    nw = rand((width,), 2, 0.4, 1.0)
    norm.load({"weight": nw.float().to(device)})
    x = x0.double().expand(n, T, width)
    for q in range(3):
        c, cd = mix_of(n, 10 * q + n, device)
        h = torch.empty(T, width, dtype=dtype, device=device)
        norm.forward(s.read(c), h)
        judge(h.float().cpu(), pp.norm(pp.enter(x, cd["enter"]), nw.double(), EPS), dtype, f"what sublayer {q} reads", bf16=0.01, f32=2e-5)
        y = Branch(T, width, device)
        whole, parts = rand((T, width), 50 + q).float(), rand((3, T, width), 60 + q).float()
        total = torch.zeros(T, width, dtype=torch.float64)
        if q != 1:
            y.add(whole.to(device))
            total += whole.double()
        if q != 0:                                                # partial sums that are still owed to the branch
            if q == 1:
                y.empty, y.partials = False, parts.to(device)
            else:
                y.pending = parts.to(device)
            total += parts.double().sum(0)
        s.leave(y, c)
        x = pp.leave(x, cd["mix"], cd["leave"], total)
        if q == 1:
            judge(s.tensor().cpu(), x.sum(0), torch.float32, "the sum of the streams on the way", f32=2e-5)
    rows = torch.tensor([T - 1, 0], dtype=torch.int32, device=device)
    want = pp.norm(x.sum(0), nw.double(), EPS)
    out = torch.empty(2, width, dtype=dtype, device=device)
    norm.forward(s.total(), out, rows)
    judge(out.float().cpu(), want[[T - 1, 0]], dtype, "the end, two rows", bf16=0.01, f32=2e-5)
    with pytest.raises(ValueError, match="summed up"):
        s.tensor()


def test_streams_start_as_one_tensor(backend):
    """Nothing is copied until the first update, which leaves the embedding output as it is."""
    device, dtype = backend
    x0 = rand((4, 24), 3).float().to(device)
    kept = x0.clone()
    s = Streams(x0, 3)
    c, cd = mix_of(3, 5, device)
    for _ in range(2):                                           # reading does not change anything
        torch.testing.assert_close(s.tensor().cpu().double(), 3 * kept.cpu().double(), rtol=1e-6, atol=1e-6)
    assert s.x.data_ptr() == x0.data_ptr() and s.shared
    y = Branch(4, 24, device)
    y.add(torch.ones(4, 24, device=device))
    s.leave(y, c)
    want = pp.leave(kept.cpu().double().expand(3, 4, 24), cd["mix"], cd["leave"], torch.ones(4, 24, dtype=torch.float64)).sum(0)
    torch.testing.assert_close(s.tensor().cpu().double(), want, rtol=1e-5, atol=1e-5)
    assert not s.shared and torch.equal(x0, kept)


@pytest.mark.parametrize("kind,extra", [("layernorm", dict(bias=False)), ("none", {})])
def test_other_norms_read_streams(backend, kind, extra):
    device, dtype = backend
    x0 = rand((6, 32), 3).float().to(device)
    s = Streams(x0, 2)
    c, cd = mix_of(2, 9, device)
    norm = build_part(NORMS, PartSpec(kind, dict(dim=32, **({"eps": EPS} if kind == "layernorm" else {}), **extra)), dtype=dtype)
    norm.load({"weight": torch.full((32,), 1.5, device=device)} if kind == "layernorm" else {})
    out = torch.empty(6, 32, dtype=dtype, device=device)
    norm.forward(s.read(c), out)
    u = pp.enter(x0.cpu().double().expand(2, 6, 32), cd["enter"])
    if kind == "layernorm":
        u = pp.rms(u - u.mean(-1, keepdim=True), EPS) * 1.5
    judge(out.float().cpu(), u, dtype, kind, bf16=0.01, f32=2e-5)


def test_streams_block_takes_a_norm_with_its_feed_forward():
    with pytest.raises(ValueError, match="feed-forward with its norm"):
        BLOCKS["streams"](parts=dict(mixer=None, mixer_norm=None, ffn_norm=None), dim=8, dtype=torch.float32, streams=2)
