"""The Pikalix decoder through the whole engine, against the plain statement in `plain_pikalix.py`: small configurations that
differ in every size and option (one to four streams, layers that read another layer's keys and values under a window of their own,
value heads smaller and larger than key heads and of the same size, rotations of a few dimensions and of the whole head, windows of
one position, inside a page and across pages, one to eight heads, dense layers and experts, all experts chosen and one of them, with
and without groups, groups of one expert, a shared expert of the experts' size, of another size and none, layers without a
feed-forward), random weights.

Every test runs three ways: the host logic on the CPU against the plain statement of the kernels, and the kernels
themselves in 32-bit and in bfloat16 on a GPU."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch
from safetensors.torch import load_file, save_file

import gpt_fast_b200 as gf
from gpt_fast_b200 import ops
from gpt_fast_b200.engine.step import Stepper
import plain_pikalix as pp
import plain_ops
import traces

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
NAMES = ["pikalix-tiny-a", "pikalix-tiny-b"]
BACKENDS = [
    pytest.param(("cpu", "float32"), id="cpu-standin-f32"),
    pytest.param(("cuda", "float32"), id="cuda-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu),
]


@pytest.fixture(params=BACKENDS)
def backend(request):
    device, dtype = request.param
    prev = ops.use_kernels(plain_ops.PlainOps()) if device == "cpu" else None
    yield device, dtype
    if device == "cpu":
        ops.use_kernels(prev)


def make_folder(d, config, seed, vector_dtype="bfloat16", std=0.11):
    """A model folder whose router corrections lie apart and whose router is weak, so that few choices are close calls, with
    mixing constants that are no identity: every stream goes its own way, some with a negative share."""
    gf.write_model_folder(d, config, seed=seed, std=std, jitter=0.25, vector_dtype=vector_dtype)
    path = os.path.join(d, "model.safetensors")
    w = load_file(path)
    g = torch.Generator().manual_seed(seed)
    for k in w:
        if k.endswith(".correction"):
            E = w[k].shape[0]
            w[k] = ((torch.randperm(E, generator=g) / E) ** 1.4 * 4.0 - 3.0).to(w[k].dtype)     # most are negative; sums differ too
        elif k.endswith(".router"):
            w[k] = (w[k] * 0.5).contiguous()
        elif k.endswith(".q") or k.endswith(".k"):
            w[k] = (w[k] * 2).contiguous()
    save_file(w, path, metadata={"format": "pt"})
    return d


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: make_folder(str(tmp_path_factory.mktemp(name.replace("-", "_"))), name, 41 + i, "float32" if i else "bfloat16")
            for i, name in enumerate(NAMES)}


_plain_cache = {}
CLOSE_CALL = 0.006         # a router margin (in scores) that the rounding of a bfloat16 run may tip


def plain(folder, tokens, with_first_close_call=False):
    key = (folder, tuple(tokens))
    if key not in _plain_cache:
        with open(os.path.join(folder, "config.json")) as f:
            cfg = json.load(f)
        margins = []
        logits = pp.forward(cfg, load_file(os.path.join(folder, "model.safetensors")), tokens, margins=margins).float()
        close = torch.stack(margins).min(0).values < CLOSE_CALL if margins else torch.zeros(len(tokens), dtype=torch.bool)
        _plain_cache[key] = (logits, int(close.nonzero()[0]) if close.any() else len(tokens))
    return _plain_cache[key] if with_first_close_call else _plain_cache[key][0]


def judge(got, folder, tokens, rows, dtype, where):
    """32-bit: equal to rounding.  bfloat16: up to the sequence's first token at which a router's choice is a close call every
    row within a few per cent of the logits' own scale; from there on (another expert moves that token, and attention carries
    it on) half of the rows.  A wrong key, page, expert or stream moves the rows by about the scale."""
    want, first_close = plain(folder, tokens, True)
    positions = torch.arange(len(tokens))[rows]
    want = want[rows]
    got = got.float().cpu()
    scale = float(want.pow(2).mean().sqrt())
    if dtype == "float32":
        assert float((got - want).abs().max()) <= 2e-4 * max(scale, 1.0), f"{where}: off by {float((got - want).abs().max()):.2e}, scale {scale:.2f}"
    else:
        per_row = (got - want).pow(2).mean(-1).sqrt() / scale
        over = (per_row > 0.06) & (positions < first_close)
        assert not bool(over.any()), f"{where}: rows {positions[over].tolist()[:5]} are off by {per_row[over].tolist()[:5]}"
        assert float(per_row.median()) <= 0.06, f"{where}: half of the rows are off by {float(per_row.median()):.3f} of the scale or more"


def tokens_of(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def stepped(stepper, slot, toks, cuts):
    outs, at = [], 0
    for c in list(cuts) + [len(toks)]:
        if c > at:
            outs.append(stepper.step([slot], [toks[at:c]], "all"))
            at = c
    stepper.check()
    return torch.cat(outs)


def make(folder, backend, max_tokens=2048, max_seqs=8):
    device, dtype = backend
    model = gf.load(folder, dtype=dtype, device=device)
    cache = model.new_cache(max_tokens=max_tokens, max_seqs=max_seqs)
    return model, cache, Stepper(model, cache)


# ---- whole prompts, and the first tokens of a sequence ------------------------------------------------

@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(folders, backend, name):
    model, cache, st = make(folders[name], backend)
    for n in (1, 2, 3, 5, 6, 37, 38, 64, 65, 150):
        toks = tokens_of(model.vocab_size, n, seed=n)
        (slot,) = cache.begin(1)
        got = st.step([slot], [toks], "all")
        st.check()
        cache.end([slot])
        judge(got, folders[name], toks, slice(None), backend[1], f"{name}: prompt of {n}")


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer_run(folders, backend, name):
    """The sum of the streams behind each layer, not only the logits: a layer that is wrong by little does not hide
    behind the layers after it."""
    model, cache, st = make(folders[name], backend)
    toks = tokens_of(model.vocab_size, 75, seed=8)
    kept = []
    model.after_layer = lambda x: kept.append(x.tensor().float().cpu().clone())
    (slot,) = cache.begin(1)
    st.step([slot], [toks], "all")
    cache.end([slot])
    model.after_layer = None
    with open(os.path.join(folders[name], "config.json")) as f:
        cfg = json.load(f)
    want = []
    pp.forward(cfg, load_file(os.path.join(folders[name], "model.safetensors")), toks, want)
    assert len(kept) == len(want) == {"pikalix-tiny-a": 5, "pikalix-tiny-b": 4}[name]
    sure = len(toks) if backend[1] == "float32" else max(1, plain(folders[name], toks, True)[1])      # up to the first close call
    for i, got in enumerate(kept):
        tol = (1e-4 if backend[1] == "float32" else 0.03) * float(want[i].float().pow(2).mean().sqrt())
        assert float((got[:sure] - want[i][:sure].float()).pow(2).mean().sqrt()) <= tol, f"the stream behind run {i}"


def test_one_token_repeated(folders, backend):
    """Positions count from 0 in every sequence and go on across steps: one token repeated."""
    name = NAMES[0]
    model, cache, st = make(folders[name], backend)
    for toks in ([7, 7, 7, 7, 7], [9], [9, 9]):
        (slot,) = cache.begin(1)
        got = stepped(st, slot, toks, range(1, len(toks)))
        cache.end([slot])
        judge(got, folders[name], toks, slice(None), backend[1], f"{name}: {toks}")


# ---- prefill against token-by-token decoding, portions down to two tokens, long decoding ----------------

@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("cuts", [
    pytest.param(lambda n: range(1, n), id="token-by-token"),
    pytest.param(lambda n: [20] + list(range(21, n)), id="prefill-then-long-decode"),
    pytest.param(lambda n: [2, 4, 5, 9, 10, 36, 38, 64, 66, 69, 70, 72, 128, 130, 139, 141], id="portions"),
    pytest.param(lambda n: [63, 65, 140], id="page-edges"),
])
def test_cuts_agree_with_the_whole(folders, backend, name, cuts):
    model, cache, st = make(folders[name], backend)
    toks = tokens_of(model.vocab_size, 143, seed=5)
    (slot,) = cache.begin(1)
    got = stepped(st, slot, toks, cuts(len(toks)))
    cache.end([slot])
    judge(got, folders[name], toks, slice(None), backend[1], f"{name}: cut prompt")
    if backend[1] == "float32":
        (slot,) = cache.begin(1)
        whole = st.step([slot], [toks], "all")
        cache.end([slot])
        scale = float(whole.pow(2).mean().sqrt())
        assert float((got - whole).abs().max()) <= 1e-4 * max(scale, 1.0)


def test_long_decoding(folders, backend):
    """Windows pass over decoded tokens several times."""
    name = NAMES[0]
    model, cache, st = make(folders[name], backend)
    toks = tokens_of(model.vocab_size, 260, seed=9)
    (slot,) = cache.begin(1)
    got = stepped(st, slot, toks, [5] + list(range(6, len(toks))))
    cache.end([slot])
    judge(got[-40:], folders[name], toks, slice(len(toks) - 40, len(toks)), backend[1], f"{name}: the last of 255 decode steps")


# ---- batches of unequal requests against each alone; slots, pages and state used again ------------------

@pytest.mark.parametrize("name", NAMES)
def test_batches_and_reuse(folders, backend, name):
    model, cache, st = make(folders[name], backend, max_tokens=1024, max_seqs=4)
    V = model.vocab_size
    for turn in range(3):                                  # the later rounds get slots, pages and state that were used before
        lens = [[70, 3, 131], [1, 66, 9, 20], [129, 2]][turn]
        reqs = [tokens_of(V, n + 6, seed=100 * turn + n) for n in lens]
        slots = cache.begin(len(reqs))
        rows = {i: [] for i in range(len(reqs))}
        out = st.step(slots, [r[:n] for r, n in zip(reqs, lens)], "all")       # packed prefill
        at = 0
        for i, n in enumerate(lens):
            rows[i].append(out[at:at + n])
            at += n
        live = list(range(len(reqs)))
        for k in range(6):                                   # decode together; the shorter ones (by index) leave early
            live = [i for i in live if not (k >= 2 + 2 * i and i < len(reqs) - 1)]
            out = st.step([slots[i] for i in live], [[reqs[i][lens[i] + k]] for i in live], "all")
            for j, i in enumerate(live):
                rows[i].append(out[j:j + 1])
        st.check()
        cache.end(slots)
        for i, r in enumerate(reqs):
            got = torch.cat(rows[i])
            judge(got, folders[name], r, slice(0, got.shape[0]), backend[1], f"{name}: pass {turn}, request {i}")
    assert cache.slots.n_free == cache.n_slots and all(g.pages.n_free == cache.n_pages for g in cache.kv_groups)


# ---- greedy generation through the library's entry point and scheduler -----------------------------------

@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation(folders, backend, name):
    device, dtype = backend
    model = gf.load(folders[name], dtype=dtype, device=device)
    prompts = [tokens_of(model.vocab_size, n, seed=7 * n) for n in (5, 1, 68, 12)]
    seqs, stats = gf.generate(model, prompts, 9, temperature=0.0, batch_size=3)
    assert stats.batches == 2 and [len(s) for s in seqs] == [len(p) + 9 for p in prompts]
    for p, s in zip(prompts, seqs):
        assert s[:len(p)] == p
        logits = plain(folders[name], s[:-1])
        for j in range(len(p) - 1, len(s) - 1):
            margin = (1e-3 if dtype == "float32" else 0.25) * float(logits[j].pow(2).mean().sqrt())
            assert logits[j, s[j + 1]] >= logits[j].max() - margin, f"{name}: token {j + 1} is not the plain argmax"


# ---- what the model asks of the cache -----------------------------------------------------------------------

def test_cache_entries_and_schedule(folders, backend):
    model, cache, st = make(folders[NAMES[0]], backend)
    needs, sched = model.cache_needs(), model.spec.schedule
    assert [e.layer for e in sched] == [e.cache for e in sched] == [0, 1, 2, 3, 4]
    assert [e.kv_from for e in sched] == [None, None, 0, None, 1]
    assert needs[2].kv is None and needs[4].kv is None and all(needs[i].state is None for i in range(5))     # readers keep nothing
    assert (needs[0].kv.n_kv, needs[0].kv.head_dim, needs[0].kv.v_head_dim, needs[0].kv.window) == (2, 20, 12, 37)
    assert model.blocks[2].mixer.window == 70 and model.blocks[4].mixer.window == 65      # ... and have windows of their own
    assert all(model.blocks[i].mixer.wqkv.shape[0] == -(-rows // 8) * 8 for i, rows in ((0, 184), (2, 120), (4, 48)))
    assert sorted(len(g.entries) for g in cache.kv_groups) == [1, 1, 1]


# ---- configuration and weights ------------------------------------------------------------------------------

def test_config_errors_name_the_key():
    cfg = gf.config_from_name("pikalix-tiny-a")
    for path, value, word in [(("layers", 0, "type"), "gla", "type"), (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
                              (("layers", 0, "mixer", "vdim"), None, "vdim"), (("layers", 1, "mixer", "rot", "dims"), 7, "dims"),
                              (("layers", 1, "mixer", "rot", "dims"), 18, "dims"), (("layers", 1, "mixer", "rot", "base"), 0, "base"),
                              (("layers", 1, "mixer", "mask"), 5, "mask"), (("layers", 1, "mixer", "mask", "size"), 0, "size"),
                              (("layers", 1, "mixer", "scale"), "big", "scale"), (("layers", 2, "mixer", "kv_from"), 2, "kv_from"),
                              (("layers", 4, "mixer", "kv_from"), 2, "kv_from"), (("layers", 2, "mixer", "kv_from"), 1, "kv_heads"),
                              (("layers", 0, "mlp", "kind"), "sparse", "mlp"), (("layers", 1, "mlp", "ff"), 0, "ff"),
                              (("layers", 0, "mlp", "router", "groups", "count"), 3, "groups"),
                              (("layers", 0, "mlp", "router", "groups", "keep"), 6, "groups"),
                              (("layers", 0, "mlp", "router", "top"), 5, "top"), (("layers", 0, "mlp", "shared"), 3, "shared"),
                              (("norm",), 1e-5, "norm"), (("streams",), 0, "streams"), (("width",), None, "width")]:
        bad = json.loads(json.dumps(cfg))
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(gf.ConfigError, match=word):
            gf.load(bad, device="cpu", random_weights=True)


@pytest.mark.parametrize("name", NAMES)
def test_weights_roundtrip(folders, tmp_path, name):
    model = gf.load(folders[name], dtype="bfloat16", device="cpu")
    gf.save_folder(model, str(tmp_path / "again"))
    a, b = load_file(os.path.join(folders[name], "model.safetensors")), load_file(str(tmp_path / "again" / "model.safetensors"))
    assert set(a) == set(b) and all(torch.equal(a[k], b[k]) for k in a)


def test_one_error_for_all_faults(folders, tmp_path):
    name = NAMES[0]
    broken = dict(load_file(os.path.join(folders[name], "model.safetensors")))
    del broken["l1.hc2.mix"]
    broken["l0.hc1.out"] = torch.zeros(3)
    broken["l2.mix.k"] = torch.zeros(1)                        # a reader of another layer's keys has none of its own
    broken["l2.hc2.in"] = torch.zeros(4)                       # constants of a sublayer the layer does not have: dropped
    os.makedirs(tmp_path / "broken")
    save_file(broken, str(tmp_path / "broken" / "model.safetensors"))
    with open(tmp_path / "broken" / "config.json", "w") as f:
        json.dump(gf.config_from_name(name), f)
    with pytest.raises(gf.WeightError) as e:
        gf.load(str(tmp_path / "broken"), device="cpu")
    assert e.value.missing == ["l1.hc2.mix"] and e.value.unexpected == ["l2.mix.k"] and e.value.wrong_shape[0][0] == "l0.hc1.out"


def test_streams_and_blocks_agree():
    import dataclasses
    from gpt_fast_b200.config.registry import architecture_for
    cfg = gf.config_from_name("pikalix-tiny-a")
    arch = architecture_for(cfg)
    spec = arch.build_spec(arch.parse(cfg))
    with pytest.raises(ValueError, match="several residual streams"):
        gf.Transformer(dataclasses.replace(spec, streams=0), device="cpu")
    with pytest.raises(ValueError, match="streams"):
        dataclasses.replace(spec, streams=-1).validate()


# ---- the trace program and the command line as a user runs them ----------------------------------------------

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run(folders, tmp_path, dtype):
    name = NAMES[1]
    folder = folders[name]
    V = gf.config_from_name(name)["vocab"]
    reqs = traces.make_requests(V, [40, 3, 77, 65], seed=3)
    for cut, steps in (("whole", traces.whole(reqs)), ("stepped", traces.stepped(reqs)), ("batched", traces.batched(reqs, 3))):
        out_dir = str(tmp_path / cut)
        cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out_dir,
               "--max-tokens", str(traces.peak_tokens(steps))]
        proc = subprocess.Popen(cmd, stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
        try:
            for s in steps:
                proc.stdin.write(json.dumps(s) + "\n")
                proc.stdin.flush()
                assert proc.stdout.readline().strip() == f"done {s['step']}"
            proc.stdin.close()
            assert proc.wait(timeout=120) == 0
        finally:
            if proc.poll() is None:
                proc.kill()
        outputs = {}
        for s in steps:
            wanted = sum(len(e["want"]) for e in s["entries"])
            if wanted:
                outputs[s["step"]] = np.fromfile(os.path.join(out_dir, f"{s['step']}.f32"), dtype="<f4").reshape(wanted, V)
        by_request = {}
        for (rid, j), row in traces.collect(steps, outputs, V).items():
            by_request.setdefault(rid, []).append((j, row))
        for rid, rows in by_request.items():
            rows.sort(key=lambda x: x[0])
            got = torch.from_numpy(np.stack([r for _, r in rows]))
            judge(got, folder, reqs[rid], [j for j, _ in rows], dtype, f"{cut}: {rid}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_cli_greedy(folders, tmp_path, dtype):
    from test_cli_gpu import read_lines, run_cli
    name = NAMES[1]
    out = tmp_path / "tokens.jsonl"
    r = run_cli("--checkpoint_path", folders[name], "--prompt", "4,13", "--max_new_tokens", "7", "--temperature", "0",
                "--dtype", dtype, "--output", str(out))
    assert r.returncode == 0, r.stderr[-2000:]
    rows = read_lines(out)
    assert [len(x["prompt"]) for x in rows] == [4, 13]
    for x in rows:
        assert len(x["tokens"]) == 7


# ---- widths of whole 16-byte rows, at which the tensor-core products run, through the whole engine ------------------------

def _moe(E, top, ff, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _att(heads, kv, dim, vdim, size, dims, base, scale, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}, "rot": {"base": base, "dims": dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


WIDE = {
    "architecture": "Pikalix", "vocab": 223, "width": 160, "norm": {"eps": 1e-5}, "streams": 5,
    "layers": [_att(8, 2, 64, 64, 150, 48, 10000.0, 0.125, _moe(8, 2, 64, (4, 2), 64)), _att(4, 4, 128, 128, 33, 128, 500.0, 0.1, _dense(264)),
               _att(8, 2, 64, 64, 300, 48, 10000.0, 0.1, _moe(6, 3, 96, None, 40), 0), _att(2, 1, 80, 48, 90, 16, 1000.0, 0.11, None),
               _att(4, 4, 128, 128, 128, 128, 500.0, 0.1, _moe(16, 4, 40, (8, 3)), 1)]}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_sizes_through_the_engine(tmp_path, dtype):
    """Sizes at which bfloat16 runs the tensor-core products (the grouped expert products among them) and the tensor-core
    attention: prompts longer than every window, portions, a batch of unequal requests, decode steps."""
    folder = make_folder(str(tmp_path / "wide"), WIDE, seed=77, std=0.06)
    model, cache, st = make(folder, ("cuda", dtype))
    toks = tokens_of(WIDE["vocab"], 520, seed=8)
    (slot,) = cache.begin(1)
    whole = st.step([slot], [toks], "all")
    st.check()
    cache.end([slot])
    judge(whole, folder, toks, slice(None), dtype, "a prompt longer than every window")
    (slot,) = cache.begin(1)
    cut = stepped(st, slot, toks, [130, 132, 389] + list(range(390, 401)))
    cache.end([slot])
    judge(cut, folder, toks, slice(None), dtype, "portions and decode steps")
    others = [tokens_of(WIDE["vocab"], n, seed=n) for n in (77, 9)]
    slots = cache.begin(3)
    got = st.step(slots, [toks[:300], others[0][:71], others[1][:3]], "all")
    steps = [st.step(slots, [[toks[300 + i]], [others[0][71 + i]], [others[1][3 + i]]], "all") for i in range(6)]   # decoded together
    st.check()
    cache.end(slots)
    judge(got[:300], folder, toks, slice(0, 300), dtype, "the long request of a batch")
    judge(got[300:371], folder, others[0], slice(0, 71), dtype, "the second request of a batch")
    decoded = torch.stack(steps)                                 # [step, request, vocab]
    judge(decoded[:, 0], folder, toks, slice(300, 306), dtype, "the long request decoded in a batch")
    judge(decoded[:, 1], folder, others[0], slice(71, 77), dtype, "the second request decoded in a batch")
    judge(decoded[:, 2], folder, others[1], slice(3, 9), dtype, "the short request decoded in a batch")


# ---- random configurations -------------------------------------------------------------------------------------------------

def random_config(seed):
    g = torch.Generator().manual_seed(seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for i in range(pick(1, 2, 3, 4)):
        count = pick(1, 1, 2, 3)
        per = pick(1, 2, 3, 5)
        keep = pick(*range(1, count + 1))
        ff = pick(8, 16, 17, 40)
        mlp = pick(None, _dense(pick(5, 48)), 0, 0)
        if mlp == 0:
            mlp = _moe(count * per, pick(*range(1, keep * per + 1)), ff, (count, keep) if pick(0, 1) or count > 1 else None, pick(None, ff, 24))
        own = [j for j, L in enumerate(layers) if "kv_from" not in L["mixer"]]
        size, scale = pick(1, 2, 17, 64, 65, 300), pick(0.1, 0.5)
        if own and pick(0, 1):
            m = layers[pick(*own)]["mixer"]
            layers.append(_att(m["heads"], m["kv_heads"], m["dim"], m["vdim"], size, m["rot"]["dims"], m["rot"]["base"], scale, mlp,
                               [j for j in own if layers[j]["mixer"] is m][0]))
        else:
            kv, dim = pick(1, 2, 3), pick(6, 16, 33, 64)
            layers.append(_att(kv * pick(1, 2, 3), kv, dim, pick(dim, dim, 4, 21), size, pick(2, 4, 6), pick(100.0, 30000.0), scale, mlp))
    return {"architecture": "Pikalix", "vocab": pick(50, 97, 128), "width": pick(24, 37, 64), "norm": {"eps": pick(1e-6, 1e-3)},
            "streams": pick(1, 2, 3, 6, 9), "layers": layers}


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations(backend, tmp_path, seed):
    cfg = random_config(seed)
    folder = make_folder(str(tmp_path / "m"), cfg, seed=seed, std=0.15)
    model, cache, st = make(folder, backend)
    toks = tokens_of(cfg["vocab"], 100, seed=seed)
    (slot,) = cache.begin(1)
    got = stepped(st, slot, toks, [70, 72, 91, 92, 93, 94, 95])
    cache.end([slot])
    judge(got, folder, toks, slice(None), backend[1], f"random configuration {seed}")
