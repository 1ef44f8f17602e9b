"""Each mechanism of the Dufizen design alone, as a part with a cache entry of its own, against the plain statement of the
mechanism in `plain_dufizen.py`: the input goes in whole, in portions and as a batch of two sequences, and what the part adds
to an empty stream is compared.  Where random inputs would hide a fault (a key at a window's edge or hundreds of positions back, a
sink, a token far behind a recurrence) the inputs are made so that it stands out.  Three back ends as in `test_dufizen.py`."""
import pytest
import torch

from gpt_fast_b200 import ops
from gpt_fast_b200.cache import Cache
from gpt_fast_b200.config.spec import PartSpec
from gpt_fast_b200.ops.types import BatchMeta
from gpt_fast_b200.parts import BLOCKS, FEED_FORWARDS, JUNCTIONS, MIXERS, POSITIONS, TOKEN_INPUTS, build_part
from gpt_fast_b200.parts.residual import Branch, Residual
import plain_dufizen as pd
import plain_ops

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


def run(part, h, seqs, cuts, device, dtype):
    """Feed the sequences (lists of row ranges of h) through a mixer as one batch, each cut at `cuts`; what it added, in h's
    row order."""
    cache = Cache({0: part.cache_needs()}, dtype, device, max_tokens=2048, max_seqs=4)
    if getattr(part, "position", None) is not None:
        part.position.prepare(cache.max_pages * cache.page_size, device)
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
        y = Branch(len(rows), h.shape[1], device)
        part.forward(h[rows].to(dtype).to(device).contiguous(), batch, cache.view(0), residual=y, append=True)
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

# ---- gated linear attention ------------------------------------------------------------------------------------------------

GLA_NAMES = dict(wq="q", wk="k", wv="v", wg="g", wa1="a1", wa2="a2", a2_bias="a2.b", norm="norm", wo="o")


def gla_case(m, rank, seed, backend, bias_shift=0.0, s=0.3):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    w = {"q": rand((H * d, D), seed, s), "k": rand((H * d, D), seed + 1, s), "v": rand((H * dv, D), seed + 2, s),
         "g": rand((H * dv, D), seed + 3, s), "a1": rand((rank, D), seed + 4, s), "a2": rand((H * d, rank), seed + 5, 1.0),
         "a2.b": rand((H * d,), seed + 6, 1.0, bias_shift), "norm": rand((dv,), seed + 7, 0.2, 1.0), "o": rand((D, H * dv), seed + 8, s)}
    part = build_part(MIXERS, PartSpec("gla", dict(dim=D, n_head=H, head_dim=d, v_head_dim=dv, decay_rank=rank, tau=m["tau"], eps=EPS)),
                      dtype=backend[1], position=None)
    load(part, w, GLA_NAMES, backend)
    return part, w


@pytest.mark.parametrize("H,d,dv,tau,rank", [(2, 16, 24, 16.0, 5), (3, 9, 7, 1.0, 1), (1, 70, 36, 0.5, 12), (4, 5, 130, 40.0, 8)])
def test_gla(backend, H, d, dv, tau, rank):
    m = dict(heads=H, dim=d, vdim=dv, tau=tau)
    part, w = gla_case(m, rank, 11, backend)
    seqs = [list(range(140)), list(range(140, 229))]
    h = rand((229, D), 3)
    want = torch.cat([pd.gla(h[s].double(), f64(w), m, EPS) for s in seqs])
    for cuts, what in CUTS + ((list(range(1, 40)), "token by token"), ([2, 4, 6, 127, 129], "portions of two")):
        judge(run(part, h, seqs, cuts, *backend), want, backend[1], what)


@pytest.mark.parametrize("shift,tau,what", [(-30.0, 0.5, "decays that leave nothing of the state"), (-6.0, 1.0, "strong decays"),
                                            (9.0, 16.0, "decays of almost one"), (0.0, 0.05, "decays from everything to nothing")])
def test_gla_extreme_decays(backend, shift, tau, what):
    """Whatever the decays, nothing overflows and nothing that counts is lost: the sums of their logarithms inside a chunk
    reach from almost zero to minus thousands."""
    m = dict(heads=2, dim=16, vdim=20, tau=tau)
    part, w = gla_case(m, 4, 31, backend, bias_shift=shift)
    h = rand((200, D), 5)
    want = pd.gla(h.double(), f64(w), m, EPS)
    for cuts in ([], [70, 71, 72, 130]):
        got = run(part, h, [list(range(200))], cuts, *backend)
        assert bool(torch.isfinite(got).all())
        judge(got, want, backend[1], what, bf16=0.05)


def test_gla_remembers_far_back(backend):
    """One strong key-value product at the third position, decays of almost one and weak other keys: hundreds of positions on it
    still decides the output, through chunks, portions and decode steps."""
    m = dict(heads=2, dim=8, vdim=12, tau=16.0)
    part, w = gla_case(m, 3, 51, backend, bias_shift=12.0)
    T = 330
    h = rand((T, D), 6, 0.05)
    h[2] = rand((D,), 7, 3.0)
    want = pd.gla(h.double(), f64(w), m, EPS)
    other = h.clone()
    other[2] = h[3]
    moved = pd.gla(other.double(), f64(w), m, EPS)
    assert float((moved[-40:] - want[-40:]).pow(2).mean().sqrt()) > 0.3 * float(want[-40:].pow(2).mean().sqrt())
    for cuts in ([], [100, 102, 290] + list(range(291, 330))):
        judge(run(part, h, [list(range(T))], cuts, *backend)[-40:], want[-40:], backend[1], f"far back, cuts {cuts[:3]}")


def test_channel_decay_acts_on_key_channels(backend):
    """Half of the key channels forget at once, half never: a fault that laid decays along the value columns, or head by head,
    would show."""
    m = dict(heads=2, dim=8, vdim=8, tau=1.0)
    part, w = gla_case(m, 2, 71, backend)
    w["a2"] = torch.zeros_like(w["a2"])
    w["a2.b"] = torch.tensor([20.0, -20.0] * 8).to(torch.bfloat16)
    load(part, w, GLA_NAMES, backend)
    h = rand((150, D), 8)
    want = pd.gla(h.double(), f64(w), m, EPS)
    for cuts in ([], [64, 65, 66]):
        judge(run(part, h, [list(range(150))], cuts, *backend), want, backend[1], "alternating channels")


# ---- latent attention with a window, a sink and a gate per head ---------------------------------------------------------------

LAT_NAMES = dict(wq="q", wdkv="dkv", latent_norm="dkv.norm", wuk="uk", wuv="uv", sink="sink", wg="g", wo="o")


def lat_m(H=3, d=12, r=6, dv=10, R=20, W=19, scale=0.3, base=500.0):
    return dict(heads=H, dim=d, rot_dim=r, vdim=dv, kv_rank=R, scale=scale, rot=dict(dims=r, base=base), mask=dict(size=W))


def lat_case(m, seed, backend, s=0.3, sink=1.0):
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    w = {"q": rand((H * (d + r), D), seed, s), "dkv": rand((R + r, D), seed + 1, s), "dkv.norm": rand((R,), seed + 2, 0.2, 1.0),
         "uk": rand((H * d, R), seed + 3, s), "uv": rand((H * dv, R), seed + 4, s), "sink": rand((H,), seed + 5, sink),
         "g": rand((H, D), seed + 6, s), "o": rand((D, H * dv), seed + 7, s)}
    pos = build_part(POSITIONS, PartSpec("rope", dict(head_dim=r, base=m["rot"]["base"], pairing="half", freq_dtype="float64")))
    part = build_part(MIXERS, PartSpec("latent_attention", dict(dim=D, n_head=H, head_dim=d, rot_dim=r, v_head_dim=dv, rank=R, scale=m["scale"],
                                                                eps=EPS, window=m["mask"]["size"], sink=True, head_gate=True)),
                      dtype=backend[1], position=pos)
    load(part, w, LAT_NAMES, backend)
    return part, w


# the second and third shapes are those the tensor-core attention takes in bfloat16
@pytest.mark.parametrize("m", [lat_m(), lat_m(H=4, d=16, r=16, dv=8, R=32, W=65), lat_m(H=5, d=8, r=16, dv=12, R=48, W=1),
                               lat_m(H=1, d=7, r=2, dv=3, R=9, W=1000, base=30000.0), lat_m(H=2, d=16, r=16, dv=16, R=16, W=64)])
def test_latent_attention(backend, m):
    part, w = lat_case(m, 21, backend)
    seqs = [list(range(140)), list(range(140, 229))]
    h = rand((229, D), 4)
    want = torch.cat([pd.latent_attention(h[s].double(), f64(w), m, EPS) for s in seqs])
    for cuts, what in CUTS + (([2, 4, 6, 127, 129], "portions of two"),):
        judge(run(part, h, seqs, cuts, *backend), want, backend[1], f"{m['mask']} {what}")


def loud_case(m, seed, backend, T, key, query):
    """Inputs and weights with which position `query` looks for position `key`: the query and latent maps copy input channels,
    the two positions share a loud channel and everything else is quiet."""
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    part, w = lat_case(m, seed, backend, sink=0.3)
    w["q"], w["uk"] = torch.zeros_like(w["q"]), torch.zeros_like(w["uk"])
    dkv = rand((R + r, D), seed + 9, 0.05)
    dkv[:, 0] = 0
    dkv[0] = 0
    dkv[0, 0] = 1.0                                            # latent number 0 copies input channel 0
    w["dkv"] = dkv
    for hd in range(H):
        w["uk"][hd * d, 0] = 1.0                               # every head's first key number is latent number 0
        w["q"][hd * (d + r), 1] = 1.0                          # and its first query number input channel 1
    load(part, w, LAT_NAMES, backend)
    h = rand((T, D), seed + 10, 0.3)
    h[:, 0], h[:, 1] = 0.02, 0.0
    h[key, 0] = 4.0                                            # the one loud key (its normed latent is mostly number 0)
    h[query:, 1] = 6.0                                         # queries from `query` on look for it
    return part, w, h


@pytest.mark.parametrize("shape", [dict(), dict(H=4, d=16, r=16, dv=8, R=32)])
@pytest.mark.parametrize("W,key,query", [(19, 60, 78), (64, 63, 126), (65, 64, 128), (200, 3, 202), (5, 127, 131), (100, 40, 135)])
def test_the_windows_edge(backend, shape, W, key, query):
    """A loud key W - 1 positions back is seen, one position later it is gone: in a prompt, in portions whose borders fall
    between them, and in decode steps."""
    m = lat_m(W=W, scale=1.0, **shape)
    assert query - key == W - 1 or W == 100
    T = query + 4
    part, w, h = loud_case(m, 91, backend, T, key, query - 2 if W > 2 else query)
    want = pd.latent_attention(h.double(), f64(w), m, EPS)
    wider = pd.latent_attention(h.double(), f64(w), dict(m, mask=dict(size=W + 1)), EPS)
    narrower = pd.latent_attention(h.double(), f64(w), dict(m, mask=dict(size=W - 1)), EPS)
    scale = float(want.pow(2).mean().sqrt())
    last = key + W - 1                                          # the last position that sees the key
    if last + 1 < T:
        assert float((wider[last + 1] - want[last + 1]).abs().max()) > 0.3 * scale and float((narrower[last] - want[last]).abs().max()) > 0.3 * scale
    for cuts in ([], [query], [query + 1], list(range(query - 3, T)), [key, key + 1, query - 1]):
        got = run(part, h, [list(range(T))], [c for c in cuts if 0 < c < T], *backend)
        judge(got, want, backend[1], f"window {W}, key {key}, cuts {cuts[:4]}")
        judge(got[-6:], want[-6:], backend[1], f"window {W}, key {key}, cuts {cuts[:4]}, the last rows")


def test_sinks_take_their_share(backend):
    """Sinks far above, among and far below the scores, one per head: the first tokens of a sequence, where the sink weighs most,
    and a decode step."""
    m = lat_m(H=4, d=16, r=16, dv=8, R=32, W=40)
    part, w = lat_case(m, 61, backend)
    w["sink"] = torch.tensor([6.0, 1.0, -1.0, -40.0]).to(torch.bfloat16)
    load(part, w, LAT_NAMES, backend)
    h = rand((90, D), 12)
    want = pd.latent_attention(h.double(), f64(w), m, EPS)
    without = pd.latent_attention(h.double(), dict(f64(w), sink=torch.full((4,), -1e4, dtype=torch.float64)), m, EPS)
    assert float((want - without)[:5].abs().mean()) > 0.1 * float(want.abs().mean())
    for cuts in ([], list(range(1, 90)), [1, 3, 80]):
        got = run(part, h, [list(range(90))], cuts, *backend)
        judge(got, want, backend[1], f"sinks, cuts {cuts[:3]}")
        judge(got[:4], want[:4], backend[1], "sinks, the first tokens")


# ---- the router and the experts -----------------------------------------------------------------------------------------------

def moe_case(mlp, seed, backend, s=0.3, corr=0.05, D=D):
    r, F = mlp["router"], mlp["expert"]["ff"]
    E, Fs = r["experts"], (mlp.get("shared") or {}).get("ff", 0)
    g = r.get("groups") or dict(count=1, keep=1)
    w = {"router": rand((E, D), seed, s), "correction": rand((E,), seed + 1, corr)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = rand((F, D), seed + 10 + e, s), rand((D, F), seed + 300 + e, s)
    if Fs:
        w["shared.up"], w["shared.down"] = rand((Fs, D), seed + 2, s), rand((D, Fs), seed + 3, s)
    part = build_part(FEED_FORWARDS, PartSpec("moe", dict(dim=D, hidden=F, n_experts=E, top=r["top"], score="softmax", activation="relu2",
                                                          groups=(g["count"], g["keep"]), shared_hidden=Fs)), dtype=backend[1])
    device, dtype = backend
    t = {"router": w["router"], "up": torch.stack([w[f"e{e}.up"] for e in range(E)]), "down": torch.stack([w[f"e{e}.down"] for e in range(E)])}
    if Fs:
        t.update(shared_up=w["shared.up"], shared_down=w["shared.down"])
    part.load({**{k: v.to(dtype).to(device) for k, v in t.items()}, "correction": w["correction"].float().to(device)})
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
    want = pd.experts(h.double(), mlp, f64(w), margins)
    for into in ("branch", "stream"):
        y = Branch(T, D, device) if into == "branch" else Residual(torch.full((T, D), 2.0, device=device))
        part.forward(h.to(dtype).to(device).contiguous(), residual=y)
        got = y.tensor().float().cpu() - (0.0 if into == "branch" else 2.0)
        # the router's product is 32-bit of the same inputs here, so only a tie to rounding may fall otherwise
        sure = margins[0] > 1e-5
        judge(got[sure], want[sure], dtype, f"{into}, {T} tokens", f32=3e-4)
    assert part.shared_inside == (mlp["shared"] is not None and mlp["shared"]["ff"] == mlp["expert"]["ff"])


def test_the_choice_and_its_weights(backend):
    """Group limits, the correction and ties by hand: 6 experts in 3 groups."""
    device, _ = backend
    z = torch.tensor([[2.0, 0.0, 1.9, 1.8, -5.0, -5.0], [0.0, 0.0, 0.0, 0.0, 0.0, 0.0], [3.0, 0.0, 0.0, 0.0, 2.9, 2.8]])
    corr = torch.tensor([0.0, -2.0, -2.0, -2.0, -1.0, -2.0])
    s = torch.softmax(z.double(), -1)

    def choose(c, top, groups, shared=False):
        idx = torch.empty(3, top + shared, dtype=torch.int32, device=device)
        w = torch.empty(3, top + shared, dtype=torch.float32, device=device)
        ops.moe_route(z.to(device).contiguous(), c.to(device), top, 1.0, idx, w, score="softmax", groups=groups, shared=shared)
        return idx.cpu().long(), w.cpu().double()
    idx, w = choose(torch.zeros(6), 2, (3, 1))
    assert idx.tolist() == [[0, 1], [0, 1], [0, 1]]            # the best group's second expert, not the best of another group
    torch.testing.assert_close(w, s.gather(1, idx), rtol=1e-5, atol=1e-7)          # as they are, not divided by their sum
    idx, w = choose(torch.zeros(6), 2, (3, 2))
    assert idx.tolist() == [[0, 2], [0, 1], [0, 4]]
    # corrected scores are negative but for expert 0: the kept groups' experts are chosen all the same, none of a dropped group
    idx, w = choose(corr, 3, (3, 2), shared=True)
    assert idx[:, 0].tolist() == [0, 0, 0]
    assert idx[:, 3].tolist() == [6, 6, 6] and w[:, 3].tolist() == [1.0, 1.0, 1.0]
    torch.testing.assert_close(w[:, :3], s.gather(1, idx[:, :3]), rtol=1e-5, atol=1e-7)      # the weights leave the correction out
    for t in range(3):
        want, _, _ = pd.choose(z[t:t + 1].double(), corr.double(), 3, 3, 2)
        assert idx[t, :3].tolist() == want[0].tolist()


# ---- the token input, the entry of a pass, the block --------------------------------------------------------------------------

@pytest.mark.parametrize("T,n,width", [(1, 5, 40), (9, 8, 64), (130, 16, 72)])
def test_token_input(backend, T, n, width):
    device, dtype = backend
    V, off = 30, 2 * n
    w = {"gate": rand((n, width), 1, 0.3), "proj": rand((width, n), 2, 0.3), "norm": rand((width,), 3, 0.3, 1.0)}
    table = rand((V, 4 * n), 4)
    part = build_part(TOKEN_INPUTS, PartSpec("gated_side", dict(dim=width, side_dim=n, offset=off, eps=EPS)), dtype=dtype)
    load(part, w, dict(gate="gate", proj="proj", norm="norm"), backend)
    part.bind_token_table(table.to(dtype).to(device))
    tokens = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(5)).to(torch.int32)
    x = rand((T, width), 6).float()
    owed, scale = rand((T, width), 7).float(), rand((width,), 8)
    full = x.double() + owed.double() * scale.double()
    want = pd.token_input(full, table[tokens.long()][:, off:off + n].double(), *(w[k].double() for k in ("gate", "proj", "norm")), EPS)
    stream, b = Residual(x.clone().to(device)), Branch(T, width, device)
    b.add(owed.to(device))
    stream.add_scaled(b, scale.float().to(device))             # a scaled branch the stream still owes as the token input reads it
    batch = type("B", (), dict(tokens=tokens.to(device), status=ops.new_status(device)))()
    part.forward(stream, batch)
    got = stream.tensor().cpu()
    ops.check_status(batch.status)
    judge(got.double() - full, want, dtype, "token input")


@pytest.mark.parametrize("T", [1, 7, 140])
def test_pass_entry(backend, T):
    device, dtype = backend
    width, passes = 48, 3
    w = {"in": rand((width, 2 * width), 1, 0.2), "step": rand((passes, width), 2)}
    part = build_part(JUNCTIONS, PartSpec("pass_entry", dict(dim=width, passes=passes)), dtype=dtype)
    part.load({"weight": w["in"].to(dtype).to(device), "step": w["step"].to(dtype).to(device)})
    x, x0 = rand((T, width), 3).float(), rand((T, width), 4).float()
    for t in range(passes):
        stream, kept = Residual(x.clone().to(device)), x0.clone().to(device)
        part.forward(stream, kept, t)
        want = pd.pass_entry(x.double(), x0.double(), w["in"].double(), w["step"][t].double())
        judge(stream.tensor().cpu().double(), want, dtype, f"pass {t}", bf16=0.01)
        assert torch.equal(kept.cpu(), x0)                      # the embedding output stays as it is
        first = Residual(kept)                                  # the loop begins at the first layer: the stream IS the embedding output
        part.forward(first, kept, t)
        want = pd.pass_entry(x0.double(), x0.double(), w["in"].double(), w["step"][t].double())
        judge(first.tensor().cpu().double(), want, dtype, f"pass {t}, from the embedding", bf16=0.01)
        assert torch.equal(kept.cpu(), x0)


def test_prenorm_block_takes_a_norm_with_its_feed_forward():
    with pytest.raises(ValueError, match="feed-forward with its norm"):
        BLOCKS["prenorm"](parts=dict(mixer=None, mixer_norm=None, ffn_norm=None), dim=8, dtype=torch.float32)
