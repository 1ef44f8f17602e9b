"""The kernels behind the Dufizen decoder one at a time at sizes of real models, against plain 64-bit statements: gated linear
attention in chunks and in decode steps (unequal sequences that start from a carried state), the tensor-core latent attention
with a window and sinks (prompts, portions, decode steps in several slices), per-head products with one gate per head, the
grouped squared-ReLU products, the router with groups, one row with scaled branches in its root-mean-square form."""
import dataclasses

import pytest
import torch

from gpt_fast_b200 import ops
from gpt_fast_b200.ops.types import PagedKV
from test_kernels_gpu import DEV, DTYPES, REF, make_batch, rnd

pytestmark = pytest.mark.gpu


def d64(t):
    return t.detach().double().cpu()


def cpu_batch(batch):
    return dataclasses.replace(batch, **{f: getattr(batch, f).cpu() for f in ("cu_seqlens", "tok_seq", "slots", "lengths", "status")})


def rel(got, want):
    return float((d64(got) - d64(want)).abs().max() / d64(want).abs().max())


# ---- gated linear attention --------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_lens", [[1, 1, 1], [130, 1, 64, 65], [2, 17]], ids=["decode", "chunks", "short"])
@pytest.mark.parametrize("H,d,dv,rank,shift", [(3, 128, 128, 16, 2.0), (2, 64, 256, 16, -3.0), (2, 33, 70, 5, 0.0), (1, 200, 12, 8, 8.0)])
def test_gla(dtype, q_lens, H, d, dv, rank, shift):
    batch, _, _ = make_batch(q_lens, [5] * len(q_lens), 6, 64, 8, seed=1)
    T, C = batch.n_tokens, H * d
    W = 2 * C + 2 * H * dv + rank + 3                             # three columns nobody reads
    src = rnd(T, W, dtype=dtype, seed=2)
    a2, bias, norm = rnd(C, rank, dtype=dtype, seed=3), rnd(C, dtype=torch.float32, seed=4) + shift, rnd(dv, seed=5)
    state = rnd(6, H * d * dv + 4, seed=6)
    before = state.clone()
    ref_state, want = state.cpu(), torch.empty(T, H * dv, dtype=torch.float64)
    offs = (0, C, 2 * C, 2 * C + 2 * H * dv, 2 * C + H * dv)      # q, k, v, low, gate
    REF.gla(src.cpu(), offs, rank, a2.cpu(), bias.cpu(), 4.0, ref_state, 4, norm.cpu(), 1e-5, want, cpu_batch(batch), H, d, dv, d ** -0.5)
    out = torch.empty(T, H * dv, dtype=dtype, device=DEV)
    ops.gla(src, offs, rank, a2, bias, 4.0, state, 4, norm, 1e-5, out, batch, H, d, dv, d ** -0.5)
    assert rel(state, ref_state) < 1e-5
    assert rel(out, want) < (5e-5 if dtype == torch.float32 else 1e-2)
    used = batch.slots.long()
    idle = [s for s in range(6) if s not in used.tolist()]
    assert torch.equal(state[idle], before[idle]) and torch.equal(state[:, :4], before[:, :4])


# ---- latent attention with a window and sinks ----------------------------------------------------------------------------

@pytest.mark.parametrize("q_lens,starts", [([70, 33, 2, 5], [0, 61, 31, 640]), ([1, 1, 1, 1], [0, 31, 64, 644]), ([300, 1], [0, 200])],
                         ids=["portions", "decode", "prompt"])
@pytest.mark.parametrize("H,R,r,window", [(16, 512, 64, 128), (6, 160, 32, 100), (3, 48, 16, 1), (40, 32, 16, 33), (5, 64, 32, 1000)])
def test_latent_attention_with_window_and_sink(H, R, r, window, q_lens, starts):
    dtype = torch.bfloat16
    batch, table, n_pages = make_batch(q_lens, starts, 6, 64, 12, seed=3)
    kv = PagedKV(rnd(n_pages, 1, 64, R + r, dtype=dtype, scale=0.5, seed=1), torch.zeros(n_pages, 1, 64, 0, dtype=dtype, device=DEV), table, 64)
    q, sink = rnd(batch.n_tokens, H, R + r, dtype=dtype, scale=0.5, seed=2), rnd(H, seed=4, scale=2.0)
    # the last sequence's last query meets one loud key just inside its window, and one just outside
    slot, t, p = int(batch.slots[-1]), batch.n_tokens - 1, starts[-1] + q_lens[-1] - 1
    inside = p - window + 1
    if inside > 0:
        loud = q[t, H - 1] * 20.0 / float(q[t, H - 1].float().norm())
        for key, sign in ((inside, 1.0), (inside - 1, 2.0)):
            kv.k_pool[int(table[slot, key // 64]), 0, key % 64] = (loud * sign).to(dtype)
    out = torch.empty(batch.n_tokens, H * R, dtype=dtype, device=DEV)
    with ops.trace() as rec:
        ops.attention(q, kv, batch, out, H, 1, R + r, 0.3, window, sink=sink, v_head_dim=R, values_in_keys=True)
    assert [label for label, _, _ in rec] == ["gfb_latent_attention"]
    ops.check_status(batch.status)
    want = torch.empty(batch.n_tokens, H * R, dtype=torch.float64)
    REF.attention(q.cpu(), PagedKV(kv.k_pool.cpu(), kv.v_pool.cpu(), table.cpu(), 64), cpu_batch(batch), want, H, 1, R + r, 0.3, window,
                  sink=sink.cpu(), v_head_dim=R, values_in_keys=True)
    torch.testing.assert_close(d64(out), want, rtol=3e-2, atol=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,K,N", [(4, 96, 56), (3, 20, 10), (16, 512, 128)])
def test_headwise_linear_with_one_gate_per_head(dtype, H, K, N):
    T = 70
    a, w, gate = rnd(T, H * K, dtype=dtype, seed=1), rnd(H, K, N, dtype=dtype, scale=K ** -0.5, seed=2), rnd(T, H + 5, dtype=dtype, seed=3)
    out, want = torch.empty(T, H * N, dtype=dtype, device=DEV), torch.empty(T, H * N, dtype=torch.float64)
    ops.headwise_linear(a, w, out, H, K, N, gate=gate, gate_off=5, gate_per_head=True)
    REF.headwise_linear(a.cpu(), w.cpu(), want, H, K, N, gate=gate.cpu(), gate_off=5, gate_per_head=True)
    assert rel(out, want) < (2e-5 if dtype == torch.float32 else 1e-2)


# ---- experts of two products ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,F,D", [(1, 4, 2, 200, 328), (20, 5, 2, 24, 40), (40, 5, 3, 64, 72), (130, 2, 1, 264, 72), (300, 6, 2, 136, 320),
                                         (900, 2, 1, 136, 320), (33, 3, 2, 13, 21)],
                         ids=["one-token", "tiles-of-32", "tiles-of-64", "two-row-tiles", "several-tiles", "tiles-of-256-rows", "odd-sizes"])
def test_squared_relu_experts(dtype, T, E, top, F, D):
    """Every form of the grouped products, stored and added; the last experts get no token at all."""
    g = torch.Generator().manual_seed(T + E)
    up, down, h = (rnd(*s, dtype=dtype, scale=c, seed=i) for i, (s, c) in enumerate((((E, F, D), D ** -0.5), ((E, D, F), F ** -0.5), ((T, D), 1.0))))
    busy = max(top, E - 2)
    idx = torch.stack([torch.randperm(busy, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    w = torch.rand(T, top, generator=g) + 0.1
    want = torch.empty(T, D)
    REF.moe_experts(h.cpu(), idx, w, up.cpu(), down.cpu(), want, 0.0, 1.0, 0.0, act="relu2", store=True)
    for store, start in ((True, float("nan")), (False, 0.25)):
        x = torch.full((T, D), start, dtype=torch.float32, device=DEV)
        ops.moe_experts(h, idx.to(DEV), w.to(DEV), up, down, x, 0.0, 1.0, 0.0, act="relu2", store=store)
        ops.check_status(ops.kernels().status)
        assert rel(x - (0.0 if store else 0.25), want) < (2e-5 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,groups,D", [(1, 15, 4, (3, 1), 40), (7, 40, 3, (8, 2), 200), (64, 96, 8, (32, 5), 72), (300, 160, 6, (5, 3), 64), (9, 7, 7, (7, 7), 24)])
def test_router_with_groups(dtype, T, E, top, groups, D):
    """Softmax scores over all experts, the choice within the best groups (corrected scores may be negative), weights as they
    are, the shared expert behind them: in one launch for few tokens, as product and choice for many."""
    h, router = rnd(T, D, dtype=dtype, seed=E), rnd(E, D, dtype=dtype, scale=D ** -0.5, seed=E + 1)
    corr = rnd(E, seed=E + 2, scale=2.0 / E) - 1.5 / E
    pad = torch.cat([router, torch.zeros(-E % 8, D, dtype=dtype, device=DEV)]).contiguous()
    idx = torch.empty(T, top + 1, dtype=torch.int32, device=DEV)
    w = torch.empty(T, top + 1, dtype=torch.float32, device=DEV)
    ops.moe_router(h, pad, corr, top, 1.0, idx, w, score="softmax", groups=groups, shared=True)
    idx, w = idx.cpu().long(), d64(w)
    s = torch.softmax(d64(h) @ d64(router).T, -1)
    c = s + d64(corr)
    assert bool((c < 0).any())
    assert idx[:, top].tolist() == [E] * T and w[:, top].tolist() == [1.0] * T
    torch.testing.assert_close(w[:, :top], s.gather(1, idx[:, :top]), rtol=1e-4, atol=1e-7)
    per = E // groups[0]
    for t in range(T):
        best = [float(c[t, g * per:(g + 1) * per].max()) for g in range(groups[0])]
        order = sorted(range(groups[0]), key=lambda g: (-best[g], g))
        cand = sorted((e for g in order[:groups[1]] for e in range(g * per, (g + 1) * per)), key=lambda e: (-float(c[t, e]), e))
        gaps = [float(c[t, cand[i]] - c[t, cand[i + 1]]) for i in range(min(top, len(cand) - 1))]
        if groups[1] < groups[0]:
            gaps.append(best[order[groups[1] - 1]] - best[order[groups[1]]])
        if min(gaps, default=1.0) > 1e-6:
            assert idx[t, :top].tolist() == cand[:top], f"token {t}"


# ---- one row with scaled branches, root-mean-square form -----------------------------------------------------------------------

@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(3, 2048), (300, 2048), (5, 192), (2, 44), (400, 33), (2, 7000), (1, 9000)])
@pytest.mark.parametrize("n_branch,splits,plain_row", [(1, 1, False), (2, 5, False), (2, 1, True), (0, 1, False)])
def test_row_with_scaled_branches(out_dtype, T, D, n_branch, splits, plain_row):
    x = rnd(T, D, seed=1)
    branches = [(rnd(splits, T, D, seed=2 + i) if i == 0 and splits > 1 else rnd(T, D, seed=2 + i), rnd(D, seed=9 + i)) for i in range(n_branch)]
    weight = None if plain_row else rnd(D, seed=5)
    out, ref_x = torch.empty(T, D, dtype=out_dtype, device=DEV), x.cpu()
    want = torch.empty(T, D, dtype=torch.float64)
    REF.layernorm_multi(ref_x, [(y.cpu(), s.cpu()) for y, s in branches], [(None if weight is None else weight.cpu(), 1e-5, want)], rms=True)
    ops.layernorm_multi(x, branches, [(weight, 1e-5, out)], rms=True)
    assert rel(x, ref_x) < 2e-6
    assert rel(out, want) < (3e-6 if out_dtype == torch.float32 else 5e-3)


def test_bad_token_is_reported_by_the_token_gate():
    z, table = rnd(3, 8), rnd(10, 16)
    tokens = torch.tensor([1, 12, 3], dtype=torch.int32, device=DEV)
    out, st = torch.empty(3, 8, device=DEV), ops.new_status(DEV)
    ops.token_gate(z, tokens, table, 8, out, st)
    with pytest.raises(ops.KernelError, match="token id out of range"):
        ops.check_status(st)
    assert out[1].abs().sum() == 0 and out[0].abs().sum() > 0


# ---- nothing is written outside an output -----------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_new_kernels_stay_inside_their_outputs(dtype):
    from test_kernels_canary_gpu import Guarded
    H, rank = 3, 5
    for q_lens, d, dv in (([1, 1], 33, 36), ([70, 1, 129], 33, 36), ([3, 64], 130, 71), ([65], 20, 130)):
        batch, _, _ = make_batch(q_lens, [2] * len(q_lens), 3, 64, 4, seed=2)
        T, C = batch.n_tokens, H * d
        src = rnd(T, 2 * C + 2 * H * dv + rank, dtype=dtype, seed=1)
        offs = (0, C, 2 * C, 2 * C + 2 * H * dv, 2 * C + H * dv)
        state, out = Guarded(3, H * d * dv, fill=rnd(3, H * d * dv, seed=3)), Guarded(T, H * dv, dtype=dtype)
        ops.gla(src, offs, rank, rnd(C, rank, dtype=dtype, seed=4), rnd(C, seed=5), 2.0, state.t, 0, rnd(dv, seed=6), 1e-5, out.t, batch, H, d, dv, 0.2)
        state.check(f"gla state, {q_lens}")
        out.check(f"gla, {q_lens}")
    T, n, D, V = 13, 7, 44, 20
    tokens = torch.randint(0, V, (T,), dtype=torch.int32, device=DEV)
    g = Guarded(T, n, dtype=dtype)
    ops.token_gate(rnd(T, n), tokens, rnd(V, 3 * n, dtype=dtype), 2 * n, g.t, ops.new_status(DEV))
    g.check("token gate")
    cat, y = Guarded(T, 2 * D, dtype=dtype), Guarded(T, D)
    ops.pass_entry(rnd(T, D), rnd(T, D), rnd(D, dtype=dtype), cat.t, y.t)
    cat.check("pass entry")
    y.check("pass entry (the new stream)")
    for T, F, D in ((1, 13, 21), (70, 13, 21), (9, 24, 40), (300, 40, 72)):
        E, top = 5, 2
        idx = torch.stack([torch.randperm(E)[:top] for _ in range(T)]).int().to(DEV)
        x = Guarded(T, D)
        ops.moe_experts(rnd(T, D, dtype=dtype), idx, torch.rand(T, top, device=DEV), rnd(E, F, D, dtype=dtype), rnd(E, D, F, dtype=dtype), x.t, 0.0, 1.0,
                        0.0, act="relu2", store=True)
        x.check(f"squared-ReLU experts, {T} tokens")
    for T, E in ((5, 12), (200, 12)):
        idx, w = Guarded(T, 4, dtype=torch.int32), Guarded(T, 4)
        ops.moe_router(rnd(T, 24, dtype=dtype), rnd(16, 24, dtype=dtype, seed=2), rnd(E), 3, 1.0, idx.t, w.t, score="softmax", groups=(3, 2), shared=True)
        idx.check("router's choice")
        w.check("router's weights")
