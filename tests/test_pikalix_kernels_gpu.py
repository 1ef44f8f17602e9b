"""The kernels behind the Pikalix decoder one at a time at sizes of real models, against plain 64-bit statements: several residual
streams in each of the kernel's forms, q/k/v with biases and a norm over the whole projection (in registers, through shared
memory, a warp per head; from the product or from its partial sums), the router by the sum of a group's two best scores, products
with the tanh GELU as their epilogue, the embedding behind its norm.  And guard words around every new output."""
import dataclasses

import pytest
import torch

from gpt_fast_b200 import ops
from gpt_fast_b200.ops.types import PagedKV
from test_kernels_canary_gpu import Guarded
from test_kernels_gpu import DEV, DTYPES, REF, make_batch, rnd

pytestmark = pytest.mark.gpu


def d64(t):
    return t.detach().double().cpu()


def cpu_batch(batch):
    return dataclasses.replace(batch, **{f: getattr(batch, f).cpu() for f in ("cu_seqlens", "tok_seq", "slots", "lengths", "status")})


def rel(got, want):
    return float((d64(got) - d64(want)).abs().max() / d64(want).abs().max())


# ---- several streams ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 2048), (64, 2048), (300, 2048), (129, 4096), (9, 8192), (3, 12000), (5, 1030), (2, 192), (400, 33)])
@pytest.mark.parametrize("n,shared,splits", [(4, False, 7), (4, True, 1), (3, False, 1), (2, False, 16), (8, False, 2), (1, True, 3), (13, False, 2)])
def test_streams(out_dtype, T, D, n, shared, splits):
    x = rnd(T, D, seed=1) if shared else rnd(n, T, D, seed=1)
    mix, leave, enter, w = rnd(n, n, seed=2), rnd(n, seed=3), rnd(n, seed=4), rnd(D, seed=5)
    branches = [rnd(splits, T, D, seed=6) if splits > 1 else rnd(T, D, seed=6)] + ([rnd(T, D, seed=7)] if n == 4 else [])
    want_x, want = torch.empty(n, T, D), torch.empty(T, D, dtype=torch.float64)
    host = dict(mix=mix.cpu(), leave=leave.cpu(), branches=[b.cpu() for b in branches])
    REF.streams(x.cpu(), n, shared, want_x, enter=enter.cpu(), weight=w.cpu(), eps=1e-5, out=want, **host)
    # the sum of the streams behind the update, some rows, nothing written back
    rows = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
    picked, want_rows, before = torch.empty(2, D, dtype=out_dtype, device=DEV), torch.empty(2, D, dtype=torch.float64), x.clone()
    REF.streams(x.cpu(), n, shared, None, weight=w.cpu(), eps=1e-5, out=want_rows, rows=rows.cpu(), **host)
    ops.streams(x, n, shared, None, mix, leave, branches, None, w, 1e-5, picked, rows)
    tol = 4e-6 if out_dtype == torch.float32 else 5e-3
    assert rel(picked, want_rows) < tol and torch.equal(x, before)
    x_out, out = torch.empty(n, T, D, device=DEV) if shared else x, torch.empty(T, D, dtype=out_dtype, device=DEV)
    ops.streams(x, n, shared, x_out, mix, leave, branches, enter, w, 1e-5, out)
    assert rel(x_out, want_x) < 4e-6 and rel(out, want) < tol
    # reading alone: a weighted sum without a norm
    plain, want_plain = torch.empty(T, D, device=DEV), torch.empty(T, D, dtype=torch.float64)
    ops.streams(x_out, n, enter=enter, out=plain)
    REF.streams(want_x, n, enter=enter.cpu(), out=want_plain)
    assert rel(plain, want_plain) < 1e-5


def test_streams_say_what_does_not_fit():
    x = rnd(2, 3, 16)
    for kw in (dict(mix=rnd(2, 2)), dict(x_out=x), dict(rows=torch.zeros(1, dtype=torch.int32, device=DEV)), dict(enter=rnd(3), out=rnd(3, 16)),
               dict(mix=rnd(2, 2), leave=rnd(2), branches=[rnd(3, 15)], x_out=x), dict(mix=rnd(2, 2), leave=rnd(2), branches=[rnd(3, 16)] * 3, x_out=x)):
        with pytest.raises(ops.KernelError):
            ops.streams(x, 2, **kw)
    with pytest.raises(ops.KernelError, match="streams"):
        ops.streams(rnd(17, 3, 16), 17, out=rnd(3, 16))


# ---- q, k and v --------------------------------------------------------------------------------------------------------

def table_of(P, dims):
    t = torch.empty(P, dims // 2, 2, device=DEV)
    ops.rope_table((1000.0 ** (-torch.arange(dims // 2).float() * 2 / dims)).to(DEV), t)
    return t


# columns per token from a few to more than one block's registers; odd head sizes; half-split pairs go through shared memory
QKV = [(16, 4, 128, 128, 64), (6, 2, 20, 12, 8), (3, 3, 33, 7, 6), (64, 8, 128, 128, 128), (8, 8, 64, 64, 0), (2, 1, 256, 64, 32), (80, 8, 128, 128, 16), (120, 8, 128, 128, 32)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_lens,starts", [([1, 1, 1], [0, 63, 64]), ([70, 1, 65], [5, 128, 31])], ids=["decode", "portions"])
@pytest.mark.parametrize("pairing", ["interleaved", "half"])
@pytest.mark.parametrize("splits", [0, 5])
@pytest.mark.parametrize("H,G,dk,dv,rot", QKV)
def test_qkv_prepare_with_biases_and_a_whole_norm(dtype, q_lens, starts, pairing, splits, H, G, dk, dv, rot):
    batch, table, n_pages = make_batch(q_lens, starts, 5, 64, 6, seed=3)
    T, W = batch.n_tokens, H * dk + G * (dk + dv)
    W += -W % 8
    src = rnd(T, W, dtype=dtype, seed=1)
    partials = rnd(splits, T, W, seed=2) if splits else None
    bias, qn, kn = rnd(W, seed=4), rnd(H * dk, dtype=dtype, seed=5), rnd(G * dk, dtype=dtype, seed=6)
    rope = table_of(300, rot) if rot else None
    for append in (True, False):
        pools = [torch.zeros(n_pages, G, 64, d, dtype=dtype, device=DEV) for d in (dk, dv)]
        kv, ref_kv = PagedKV(*pools, table, 64), PagedKV(*[torch.zeros(p.shape, dtype=torch.float64) for p in pools], table.cpu(), 64)
        q, want = torch.empty(T, H, dk, dtype=dtype, device=DEV), torch.empty(T, H, dk, dtype=torch.float64)
        off = (0, H * dk, (H + G) * dk)
        kw = dict(rot_dims=rot, pairing=pairing, norm_eps=1e-5, append=append, norm_whole=True)
        REF.qkv_prepare(src.cpu(), None if partials is None else partials.cpu(), off, want, ref_kv, cpu_batch(batch), H, G, dk, dv,
                        table=None if rope is None else rope.cpu(), q_norm=qn.cpu(), k_norm=kn.cpu(), bias=bias.cpu(), **kw)
        ops.qkv_prepare(src, partials, off, q, kv, batch, H, G, dk, dv, table=rope, q_norm=qn, k_norm=kn if append else None, bias=bias, **kw)
        ops.check_status(batch.status)
        tol = 5e-6 if dtype == torch.float32 else 5e-3
        assert rel(q, want) < tol
        if append:
            assert rel(kv.k_pool, ref_kv.k_pool) < tol and rel(kv.v_pool, ref_kv.v_pool) < tol
        else:
            assert not bool(pools[0].any()) and not bool(pools[1].any())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("head_norm", [False, True])
def test_qkv_prepare_with_biases_alone(dtype, head_norm):
    """Biases without a norm, and ahead of a norm per head: the form with a warp per head."""
    H, G, dk, dv = 4, 2, 24, 40
    batch, table, n_pages = make_batch([9, 1], [60, 3], 4, 64, 4, seed=3)
    T, W = batch.n_tokens, H * dk + G * (dk + dv)
    src, bias = rnd(T, W, dtype=dtype, seed=1), rnd(W, dtype=dtype, seed=4)
    qn, kn = (rnd(dk, seed=5), rnd(dk, seed=6)) if head_norm else (None, None)
    pools = [torch.zeros(n_pages, G, 64, d, dtype=dtype, device=DEV) for d in (dk, dv)]
    kv, ref_kv = PagedKV(*pools, table, 64), PagedKV(*[torch.zeros(p.shape, dtype=torch.float64) for p in pools], table.cpu(), 64)
    q, want = torch.empty(T, H, dk, dtype=dtype, device=DEV), torch.empty(T, H, dk, dtype=torch.float64)
    off, kw = (0, H * dk, (H + G) * dk), dict(rot_dims=8, pairing="half", norm_eps=1e-5)
    rope = table_of(100, 8)
    REF.qkv_prepare(src.cpu(), None, off, want, ref_kv, cpu_batch(batch), H, G, dk, dv, table=rope.cpu(), bias=bias.cpu(),
                    q_norm=None if qn is None else qn.cpu(), k_norm=None if kn is None else kn.cpu(), **kw)
    ops.qkv_prepare(src, None, off, q, kv, batch, H, G, dk, dv, table=rope, q_norm=qn, k_norm=kn, bias=bias, **kw)
    ops.check_status(batch.status)
    tol = 5e-6 if dtype == torch.float32 else 5e-3
    assert rel(q, want) < tol and rel(kv.k_pool, ref_kv.k_pool) < tol and rel(kv.v_pool, ref_kv.v_pool) < tol


@pytest.mark.parametrize("H,G,dk,dv,pairing", [(4, 2, 32, 32, "interleaved"), (4, 2, 32, 32, "half"), (3, 1, 9, 5, "interleaved")])
def test_a_token_without_a_page_is_reported(H, G, dk, dv, pairing):
    batch, table, n_pages = make_batch([3], [62], 2, 64, 4, seed=3)
    table[int(batch.slots[0]), 1] = -1                            # positions 64 on have no page
    kv = PagedKV(*[torch.zeros(n_pages, G, 64, d, device=DEV) for d in (dk, dv)], table, 64)
    W = H * dk + G * (dk + dv)
    q = torch.full((3, H, dk), 7.0, device=DEV)
    ops.qkv_prepare(rnd(3, W), None, (0, H * dk, (H + G) * dk), q, kv, batch, H, G, dk, dv, table=table_of(200, 4), rot_dims=4, pairing=pairing,
                    q_norm=rnd(H * dk), k_norm=rnd(G * dk), norm_eps=1e-5, norm_whole=True)
    with pytest.raises(ops.KernelError, match="position"):
        ops.check_status(batch.status)
    assert bool((q[2] == 0).all()) and bool((q[:2] != 7.0).any())


# ---- the router, products, embedding --------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,groups,D", [(1, 15, 4, (3, 1), 40), (7, 40, 3, (8, 2), 200), (64, 96, 8, (32, 5), 72), (300, 160, 6, (5, 3), 64),
                                              (9, 7, 3, (7, 3), 24), (70, 512, 8, (8, 4), 64), (5, 66, 2, (2, 1), 48)])
def test_router_with_groups_of_two_best(dtype, T, E, top, groups, D):
    h, router = rnd(T, D, dtype=dtype, seed=E), rnd(E, D, dtype=dtype, scale=D ** -0.5, seed=E + 1)
    corr = rnd(E, seed=E + 2) - 1.0
    pad = torch.cat([router, torch.zeros(-E % 8, D, dtype=dtype, device=DEV)]).contiguous()
    idx = torch.empty(T, top + 1, dtype=torch.int32, device=DEV)
    w = torch.empty(T, top + 1, dtype=torch.float32, device=DEV)
    ops.moe_router(h, pad, corr, top, 1.0, idx, w, score="sigmoid_plain", groups=groups + (2,), shared=True)
    idx, w = idx.cpu().long(), d64(w)
    s = torch.sigmoid(d64(h) @ d64(router).T)
    c = s + d64(corr)
    assert idx[:, top].tolist() == [E] * T and w[:, top].tolist() == [1.0] * T
    torch.testing.assert_close(w[:, :top], s.gather(1, idx[:, :top]), rtol=1e-4, atol=1e-7)
    per = E // groups[0]
    checked = 0
    for t in range(T):
        best = [float(c[t, g * per:(g + 1) * per].sort(descending=True).values[:2].sum()) for g in range(groups[0])]
        order = sorted(range(groups[0]), key=lambda g: (-best[g], g))
        cand = sorted((e for g in order[:groups[1]] for e in range(g * per, (g + 1) * per)), key=lambda e: (-float(c[t, e]), e))
        gaps = [float(c[t, cand[i]] - c[t, cand[i + 1]]) for i in range(min(top, len(cand) - 1))]
        if groups[1] < groups[0]:
            gaps.append(best[order[groups[1] - 1]] - best[order[groups[1]]])
        if min(gaps, default=1.0) > 2e-6:
            checked += 1
            assert idx[t, :top].tolist() == cand[:top], f"token {t}"
    assert checked > T // 2


def test_a_groups_two_best_scores_may_be_equal():
    """Both of them count, also where one lane of the kernel holds both."""
    z = torch.zeros(1, 66, device=DEV)
    z[0, 0] = z[0, 32] = 2.0                                       # group 0, both with one lane: the best pair
    z[0, 40] = 3.0                                                 # group 1, the best single score
    corr = torch.full((66,), -5.0, device=DEV)
    idx, w = torch.empty(1, 2, dtype=torch.int32, device=DEV), torch.empty(1, 2, device=DEV)
    ops.moe_route(z, corr, 2, 1.0, idx, w, score="sigmoid_plain", groups=(2, 1, 2))
    assert idx.tolist() == [[0, 32]]
    ops.moe_route(z, corr, 2, 1.0, idx, w, score="sigmoid_plain", groups=(2, 1, 1))
    assert idx[0, 0].item() == 40


@pytest.mark.parametrize("M,N,K", [(1, 8192, 2048), (8, 1024, 640), (40, 264, 72), (100, 512, 4096), (200, 1000, 512), (300, 136, 320), (600, 520, 264), (2048, 1024, 512)])
def test_tanh_gelu_in_the_products_epilogue(M, N, K):
    """Split over K and reduced, tiles of one block and of pairs of blocks; inputs that reach both tails."""
    a, w = rnd(M, K, dtype=torch.bfloat16, seed=1), rnd(N, K, dtype=torch.bfloat16, scale=3.0 * K ** -0.5, seed=2)
    out = torch.empty(M, N, dtype=torch.bfloat16, device=DEV)
    with ops.trace() as rec:
        ops.linear(a, w, out, mode="gelu_tanh")
    assert len(rec) == 1                                           # no activation kernel behind the product
    ops.check_status(ops.kernels().status)
    z = d64(a) @ d64(w).T
    want = REF._unary(z, "gelu_tanh")
    assert float((d64(out) - want).abs().max()) <= 2.0 ** -8 * float(want.abs().max())
    torch.testing.assert_close(d64(out), want, rtol=1e-2, atol=2e-3)


def test_tanh_gelu_far_out():
    """Beyond both tails: the argument itself, and nothing."""
    a = torch.zeros(2, 64, dtype=torch.bfloat16, device=DEV)
    a[0, 0], a[1, 0] = 1.0, -1.0
    w = torch.zeros(8, 64, dtype=torch.bfloat16, device=DEV)
    w[:, 0] = torch.tensor([0.0, 1e-3, 5.0, 20.0, 100.0, 1e4, 1e10, 1e12])
    out = torch.empty(2, 8, dtype=torch.bfloat16, device=DEV)
    ops.linear(a, w, out, mode="gelu_tanh")
    want = REF._unary(d64(a) @ d64(w).T, "gelu_tanh")
    assert bool(torch.isfinite(out).all())
    torch.testing.assert_close(d64(out), want, rtol=1e-2, atol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 2048), (70, 200), (300, 4096), (3, 37)])
def test_normed_embedding(dtype, T, D):
    table, w = rnd(50, D, dtype=dtype), rnd(D, dtype=dtype, seed=2)
    tokens = torch.randint(0, 50, (T,), dtype=torch.int32, device=DEV)
    out, want, st = torch.empty(T, D, device=DEV), torch.empty(T, D, dtype=torch.float64), ops.new_status(DEV)
    ops.embed_normed(tokens, table, w, 1e-5, out, st, 1.5)
    REF.embed_normed(tokens.cpu(), table.cpu(), w.cpu(), 1e-5, want, st.cpu(), 1.5)
    assert rel(out, want) < 2e-6
    ops.check_status(st)
    tokens[T - 1] = 50
    ops.embed_normed(tokens, table, w, 1e-5, out, st)
    with pytest.raises(ops.KernelError, match="token id out of range"):
        ops.check_status(st)
    assert not bool(out[T - 1].any())


@pytest.mark.parametrize("dtype", DTYPES)
def test_shared_expert_inside_the_stacks(dtype):
    """A shared SwiGLU expert of the experts' size runs as one more expert of weight 1 and gives what it gives as a feed-forward of
    its own."""
    from gpt_fast_b200.config.spec import PartSpec
    from gpt_fast_b200.parts import FEED_FORWARDS, build_part
    from gpt_fast_b200.parts.residual import Branch
    E, F, D = 6, 64, 128
    t = {"router": rnd(E, D, dtype=dtype, scale=0.2), "correction": rnd(E, seed=1)}
    t.update({k: rnd(E, *s, dtype=dtype, scale=0.1, seed=i) for i, (k, s) in enumerate((("gate", (F, D)), ("up", (F, D)), ("down", (D, F))))})
    t.update({f"shared_{k}": rnd(*s, dtype=dtype, scale=0.1, seed=9 + i) for i, (k, s) in enumerate((("gate", (F, D)), ("up", (F, D)), ("down", (D, F))))})
    spec = PartSpec("moe", dict(dim=D, hidden=F, n_experts=E, top=2, score="sigmoid_plain", groups=(3, 2, 2), shared_hidden=F))
    inside, beside = build_part(FEED_FORWARDS, spec, dtype=dtype), build_part(FEED_FORWARDS, spec, dtype=dtype)
    assert inside.shared_inside
    beside.shared_inside = False
    inside.load(t)
    beside.load(t)
    for T in (1, 40, 300):
        h, ys = rnd(T, D, dtype=dtype, seed=3), []
        for part in (inside, beside):
            y = Branch(T, D, DEV)
            part.forward(h, y)
            ys.append(y.tensor().clone())
        assert rel(ys[0], ys[1]) < (1e-5 if dtype == torch.float32 else 6e-3)


# ---- nothing is written outside an output -----------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_new_kernels_stay_inside_their_outputs(dtype):
    for T, D, n in ((13, 200, 3), (5, 33, 2), (3, 1056, 4), (300, 1056, 4), (2, 9000, 2), (4, 44, 11)):
        x, h = Guarded(n, T, D, fill=rnd(n, T, D)), Guarded(T, D, dtype=dtype)
        ops.streams(x.t, n, False, x.t, rnd(n, n), rnd(n), [rnd(2, T, D, seed=1), rnd(T, D, seed=2)], rnd(n), rnd(D), 1e-5, h.t)
        x.check(f"streams, {T} x {D}")
        h.check(f"streams (normed), {T} x {D}")
        new, h = Guarded(n, T, D), Guarded(2, D, dtype=dtype)
        ops.streams(rnd(T, D), n, True, new.t, rnd(n, n), rnd(n), [rnd(T, D, seed=2)])
        new.check(f"streams from one, {T} x {D}")
        ops.streams(new.t, n, weight=rnd(D), eps=1e-5, out=h.t, rows=torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV))
        h.check(f"streams (rows), {T} x {D}")
    for H, G, dk, dv, pairing in ((6, 2, 20, 12, "interleaved"), (3, 3, 33, 7, "interleaved"), (4, 1, 64, 64, "half"), (16, 4, 128, 128, "interleaved")):
        for q_lens in ([1, 1], [70, 3]):
            batch, table, n_pages = make_batch(q_lens, [62, 5], 3, 64, 4, seed=2)
            T, W = batch.n_tokens, H * dk + G * (dk + dv)
            k, v, q = Guarded(n_pages, G, 64, dk, dtype=dtype, fill=0), Guarded(n_pages, G, 64, dv, dtype=dtype, fill=0), Guarded(T, H, dk, dtype=dtype)
            ops.qkv_prepare(rnd(T, W, dtype=dtype), rnd(3, T, W) if len(q_lens) == T else None, (0, H * dk, (H + G) * dk), q.t, PagedKV(k.t, v.t, table, 64), batch,
                            H, G, dk, dv, table=table_of(200, 6), rot_dims=6, pairing=pairing, q_norm=rnd(H * dk), k_norm=rnd(G * dk), norm_eps=1e-5,
                            norm_whole=True, bias=rnd(W))
            ops.check_status(batch.status)
            for g, what in ((q, "q"), (k, "keys"), (v, "values")):
                g.check(f"qkv_prepare {what}, {H} heads of {dk}")
    e = Guarded(9, 77)
    ops.embed_normed(torch.arange(9, dtype=torch.int32, device=DEV), rnd(9, 77, dtype=dtype), rnd(77), 1e-5, e.t, ops.new_status(DEV))
    e.check("normed embedding")
    for T, E in ((5, 12), (200, 12)):
        idx, w = Guarded(T, 4, dtype=torch.int32), Guarded(T, 4)
        ops.moe_router(rnd(T, 24, dtype=dtype), rnd(16, 24, dtype=dtype, seed=2), rnd(E), 3, 1.0, idx.t, w.t, score="sigmoid_plain", groups=(3, 2, 2), shared=True)
        idx.check("router's choice")
        w.check("router's weights")
