"""Windowed attention (differential, with a sink, with shared keys), mixtures of experts and the Zurevik model on the GPU
against the plain CPU restatement (oracle/layered_oracle.py).  Every mixer alone is in test_gpu_decoder.py."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import femtochat_b200 as fb
from femtochat_b200 import _lib
from oracle import layered_oracle as lo

import decoder_cases as dc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 3e-5, "bfloat16": 6e-2}
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def cache_for(model, n, B=1):
    return fb.KVCache(model.state(B), B, n)


def ok(model):
    assert model.state(1).status_word() == 0


_decided = {}


def decided(cfg, w, n, seed=0):
    key = (json.dumps(cfg), n, seed)
    if key not in _decided:
        _decided[key] = dc.decided_tokens(cfg, w, n, seed)
    return _decided[key]


@BOTH
@pytest.mark.parametrize("name", sorted(dc.EXPERTS))
def test_each_feed_forward(name, dtype):
    """Whole prompts (sorted rows), token by token and in small portions (lists of the chosen experts), and both."""
    cfg = dc.EXPERTS[name]
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=31)
    t, want = decided(cfg, w, 70)
    c = cache_for(model, 70)
    for cuts in ((70,), (1,) * 69, (2, 3, 2, 31, 2, 2, 9), (33,), (32, 8)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_mixed_model_residuals_and_portions(dtype):
    model, w = dc.model_and_weights(dc.ZMIXED, (8, 8), dtype, seed=33)
    t, want = decided(dc.ZMIXED, w, 90)
    ref = lo.Sequence(dc.ZMIXED, w)
    assert (ref.feed(t) - want).abs().max() < 1e-9
    c = cache_for(model, 90)
    z, res = fb.extend(model, c, t[None, :], want=list(range(90)), residuals=True)
    for i, (a, b) in enumerate(zip(res.cpu().double(), ref.residuals)):
        assert float((a - b).abs().max() / b.abs().max()) < TOL[dtype], i
    assert dc.rel_error(z, want) < TOL[dtype]
    for cuts in ((1,) * 89, (2,) * 44, (7, 2, 31, 2, 5), (3, 3, 64, 3), (9, 10, 11, 12, 13)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_large_sizes_long_prompt(dtype):
    """Sizes at which products and the attention of prompts run their tensor-core kernels; lengths around tile and window
    edges; more kept tokens than a tile holds; decoding after it."""
    model, w = dc.model_and_weights(dc.ZLARGE, (8, 8), dtype, seed=35)
    t, want = decided(dc.ZLARGE, w, 420)
    c = cache_for(model, 420)
    for cuts in ((420,), (256, 40), (127, 1, 128), (129, 64, 65), (9, 200, 2, 100), (391,) + (1,) * 28):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_columns_equal_each_alone(dtype):
    """Several columns of one length with different tokens give what each gives alone; prompts, portions, decoding."""
    cfg = dc.ZMIXED
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=33)
    B, n = 3, 47
    seqs = [decided(cfg, w, n, 10 + b) for b in range(B)]
    t, want = torch.stack([s[0] for s in seqs]), torch.stack([s[1] for s in seqs])
    c = cache_for(model, n, B)
    at = 0
    for k in (20, 2, 9, 1, 1, 14):
        z = fb.extend(model, c, t[:, at:at + k], want=list(range(B * k))).cpu().view(B, k, -1)
        assert dc.rel_error(z.reshape(B * k, -1), want[:, at:at + k].reshape(B * k, -1)) < TOL[dtype], at
        at += k
    z = fb.prefill(model, c, t[:, :30])
    assert dc.rel_error(z, want[:, 29]) < TOL[dtype]
    for k in range(30, 36):
        assert dc.rel_error(fb.decode_step(model, c, t[:, k]), want[:, k]) < TOL[dtype]
    assert len(c) == 36
    ok(model)


@BOTH
def test_more_query_tiles_than_multiprocessors(dtype):
    """Every block of the prompt's attention works through several items; columns with the same tokens agree."""
    cfg = dc.zurevik(dc.sinks(heads=12, kv_heads=3, dim=32, vdim=40, size=100), dc.differential(heads=12, kv_heads=4, dim=16, vdim=24, size=70, keep=3), width=48)
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=37)
    B, n = 9, 300
    t = dc.tokens(n, cfg["vocab"], 8)
    want = lo.Sequence(cfg, w).feed(t)
    z = fb.extend(model, cache_for(model, n, B), t[None].repeat(B, 1), want=list(range(B * n))).cpu().view(B, n, -1)
    for b in range(B):
        assert dc.rel_error(z[b], want) < TOL[dtype], b
    ok(model)


def test_internal_portions():
    """A prompt longer than one internal pass, several columns, a ragged choice of positions."""
    cfg = dc.ZMIXED
    model, w = dc.model_and_weights(cfg, (8, 8), "float32", seed=33, max_rows=26)
    t = torch.stack([dc.tokens(61, cfg["vocab"], 20 + b) for b in range(2)])
    ref = torch.cat([lo.Sequence(cfg, w).feed(t[b]) for b in range(2)])
    c = cache_for(model, 61, 2)
    want = [0, 12, 13, 14, 25, 26, 60, 61, 62, 73, 100, 121]
    assert dc.rel_error(fb.extend(model, c, t, want=want), ref[want]) < TOL["float32"]


@BOTH
def test_a_used_cache_gives_what_a_fresh_one_gives(dtype):
    model, w = dc.model_and_weights(dc.ZMIXED, (8, 8), dtype, seed=33)
    a, want_a = decided(dc.ZMIXED, w, 40, 30)
    b, want_b = decided(dc.ZMIXED, w, 33, 31)
    c, fresh = cache_for(model, 64), cache_for(model, 64)
    dc.feed(model, c, a, (5, 1, 1))
    c.reset()
    assert torch.equal(dc.feed(model, c, b, (12, 1, 2)), dc.feed(model, fresh, b, (12, 1, 2)))
    # two requests of different lengths in turn, each with its own cache
    c.reset(); fresh.reset()
    za, zb, i = [], [], 0
    for k in (3, 1, 10, 2, 17):
        za.append(fb.extend(model, c, a[None, i:i + k], want=list(range(k))).cpu())
        zb.append(fb.extend(model, fresh, b[None, i:i + k], want=list(range(k))).cpu())
        i += k
    zb.append(fb.extend(model, c, a[None, 33:], want=list(range(7))).cpu())
    assert dc.rel_error(torch.cat(za + zb[-1:]), want_a) < TOL[dtype]
    assert dc.rel_error(torch.cat(zb[:-1]), want_b) < TOL[dtype]


# ---- what a position sees ---------------------------------------------------------------------------------------------
def matching_model(kind, size, keep, dtype):
    """One attention layer in which the query of token A fits the key of token B alone: queries see the input through a
    rotation R, keys as it is, and the embedding of B is R times that of A."""
    n, vocab, A, B = 64, 700, 11, 622
    if kind == "differential":
        layers = [dc.differential(heads=2, kv_heads=1, dim=n, vdim=n, size=size, keep=keep, scale=0.25, diff=0.5)]
    elif kind == "sinks":
        layers = [dc.sinks(heads=2, kv_heads=1, dim=n, vdim=n, size=size, scale=0.25)]
    else:       # keys of a layer with a shorter window
        layers = [dc.sinks(heads=2, kv_heads=1, dim=n, vdim=n, size=9, scale=0.25), dc.sinks(heads=2, kv_heads=1, dim=n, vdim=n, size=size, scale=0.25, kv_from=0)]
    cfg = dc.zurevik(*layers, width=n, vocab=vocab, embed_scale=1.0, softcap=30.0)
    last = f"l{len(layers) - 1}.mix."

    def edit(w):
        g = torch.Generator().manual_seed(5)
        ortho = lambda: torch.linalg.qr(torch.randn(n, n, generator=g, dtype=torch.float64))[0]
        R, M = ortho(), ortho()
        for name in w:
            if name.endswith(("norm1", "q.norm", "k.norm")):
                w[name].fill_(1.0)
            if name.endswith((".q.b", ".k.b")):
                w[name].zero_()
        w["embed"][B] = (R @ w["embed"][A].double()).bfloat16()
        if kind == "shared":
            w["l0.mix.o"].zero_()
        maps = 2 if kind == "differential" else 1
        for h in range(2):
            w[last + "q"].view(2, maps, n, n)[h, 0] = M @ R
        w["l0.mix.k"].view(1, maps, n, n)[0, 0] = M
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=13, edit=edit)
    return cfg, model, w, A, B


def with_mask(cfg, **mask):
    cfg = copy.deepcopy(cfg)
    cfg["layers"][-1]["mixer"]["mask"].update(mask)
    return cfg


EDGES = [("differential", 37, 5), ("differential", 128, 0), ("differential", 130, 129), ("sinks", 37, 0), ("sinks", 129, 0), ("shared", 64, 0)]


@BOTH
@pytest.mark.parametrize("kind,size,keep", EDGES)
@pytest.mark.parametrize("edge", ["window in", "window out", "window one inside", "keep in", "keep out", "first"])
def test_key_at_an_edge(kind, size, keep, edge, dtype):
    """The last token's query fits one key only, which lies just inside or just outside the window or the kept tokens.  A
    prompt, decoding, and last portions of two and of twenty tokens must all agree with the restatement."""
    n = 300
    place = {"window in": n - size, "window out": n - size - 1, "window one inside": n - size + 1, "keep in": keep - 1, "keep out": keep,
             "first": 0}[edge]
    if place < 0:
        pytest.skip("no kept tokens")
    cfg, model, w, A, B = matching_model(kind, size, keep, dtype)
    t = dc.tokens(n, cfg["vocab"], 50)
    t[(t == A) | (t == B)] = 3
    t[n - 1], t[place] = A, B
    want = lo.Sequence(cfg, w).feed(t)[-3:]
    # a mask that is one token off gives another answer
    off = {"window in": dict(size=size - 1), "window out": dict(size=size + 1), "keep in": dict(keep_first=keep - 1), "keep out": dict(keep_first=keep + 1)}
    if edge in off and (kind == "differential" or "keep" not in edge):
        assert dc.rel_error(lo.Sequence(with_mask(cfg, **off[edge]), w).feed(t)[-1:], want[-1:]) > 0.4
    c = cache_for(model, n)
    for cuts in ((n,), (n - 1,), (n - 3, 1, 1), (n - 2,), (n - 20,), (128, 1, 128)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts)[-3:], want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_kept_tokens_from_far_away(dtype):
    """Decoding long after the kept tokens left the window: they stay, and only they."""
    cfg, model, w, A, B = matching_model("differential", 24, 3, dtype)
    n = 700
    for place, seen in ((2, True), (3, False)):
        t = dc.tokens(n, cfg["vocab"], 51)
        t[(t == A) | (t == B)] = 3
        u = t.clone()
        t[place] = B
        t[n - 30::4] = A
        u[n - 30::4] = A
        want, without = lo.Sequence(cfg, w).feed(t)[-20:], lo.Sequence(cfg, w).feed(u)[-20:]
        assert (dc.rel_error(without, want) > 0.4) == seen
        assert dc.rel_error(dc.feed(model, cache_for(model, n), t, (n - 40,) + (1,) * 39)[-20:], want) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("level", [-30.0, 0.0, 6.0, 40.0])
def test_sinks_of_every_size(level, dtype):
    """A sink far below the scores, among them, above them and far above: each head has its own."""
    cfg = dc.zurevik(dc.sinks(heads=4, kv_heads=2, dim=32, vdim=32, size=20, scale=0.3), width=64, vocab=100)

    def edit(w):
        w["l0.mix.sink"].copy_(level + torch.tensor([0.0, 1.0, -1.0, 0.5]))
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=41, edit=edit)
    t = dc.tokens(60, 100, 3)
    want = lo.Sequence(cfg, w).feed(t)
    if level == 6.0:
        other = dict(w)
        other["l0.mix.sink"] = torch.full((4,), -100.0)
        assert dc.rel_error(lo.Sequence(cfg, other).feed(t), want) > 0.3
    c = cache_for(model, 60)
    for cuts in ((60,), (1,) * 59, (30, 2, 2)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts


@BOTH
def test_lambda_and_its_factor(dtype):
    """Lambda far from `diff` (each of the four vectors counts) and maps that differ."""
    cfg = dc.zurevik(dc.differential(heads=2, kv_heads=2, dim=32, vdim=32, size=16, keep=2, scale=0.4, diff=0.3), width=64, vocab=100)

    def edit(w):
        for n, v in (("lq1", 0.2), ("lk1", 0.25), ("lq2", -0.2), ("lk2", 0.15)):
            w["l0.mix." + n].fill_(v)
            w["l0.mix." + n][::3] *= 0.5
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=43, edit=edit)
    assert float(lo.differential_lambda({k[7:]: v.double() for k, v in w.items() if k.startswith("l0.mix.l")}, 0.3)) > 2.0
    t = dc.tokens(50, 100, 4)
    want = lo.Sequence(cfg, w).feed(t)
    c = cache_for(model, 50)
    for cuts in ((50,), (1,) * 49):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    # new lambda vectors take effect
    spec = model.layout["l0.mix.lq1"]
    model.params.theta[spec.offset:spec.offset + spec.size].mul_(0.0)
    w["l0.mix.lq1"].zero_()
    c.reset()
    assert dc.rel_error(dc.feed(model, c, t), lo.Sequence(cfg, w).feed(t)) < TOL[dtype]


# ---- experts ------------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("crowd", [False, True])
def test_many_rows_and_crowded_experts(crowd, dtype):
    """More rows than one tile per expert; all tokens at one expert, most experts empty."""
    cfg = dc.zurevik(dc.sinks(heads=1, kv_heads=1, dim=16, vdim=16, size=2, mlp=dc.moe(ff=72, experts=9, top=2)), width=64, vocab=64)

    def edit(w):
        if crowd:
            w["l0.mlp.router.b"].copy_(torch.tensor([0.0, 0, 0, 0, 40.0, 0, 0, 60.0, 0]))
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=45, edit=edit)
    t, want = decided(cfg, w, 900, 100 + crowd)
    c = cache_for(model, 900)
    for cuts in ((900,), (600, 40, 1, 200)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


def test_rows_do_not_depend_on_their_neighbours():
    """The same token sequence in one column and among others gives the same bits from the experts' few-row path."""
    cfg = dc.zurevik(dc.sinks(heads=2, kv_heads=2, dim=32, vdim=32, size=8, mlp=dc.moe(ff=64, experts=6, top=3)), width=64, vocab=64)
    model, w = dc.model_and_weights(cfg, (8, 8), "bfloat16", seed=47)
    t = torch.stack([dc.tokens(12, 64, 60 + b) for b in range(4)])
    many, one = cache_for(model, 12, 4), cache_for(model, 12, 4)
    for k in range(12):
        z = fb.extend(model, many, t[:, k:k + 1])
        y = fb.extend(model, one, t[:, k:k + 1].flip(0))
        assert torch.equal(z, y.flip(0)), k


# ---- long runs, generation, folders ---------------------------------------------------------------------------------
@BOTH
def test_long_decoding(dtype):
    model, w = dc.model_and_weights(dc.ZMIXED, (8, 8), dtype, seed=33)
    t, want = decided(dc.ZMIXED, w, 300, 7)
    assert dc.rel_error(dc.feed(model, cache_for(model, 300), t, (4,) + (1,) * 295), want) < TOL[dtype]
    ok(model)


def test_greedy_generation_matches_the_oracle():
    model, w = dc.model_and_weights(dc.ZMIXED, (8, 8), "float32", seed=33)
    prompt = [5, 0, 112, 7, 7, 60]
    got = fb.generate(model, prompt, max_new_tokens=40, temperature=0.0)
    ref, toks = lo.Sequence(dc.ZMIXED, w), list(prompt)
    z = ref.feed(toks)[-1]
    for _ in range(40):
        toks.append(int(z.argmax()))
        z = ref.feed(toks[-1:])[-1]
    assert got == toks
    assert fb.generate(model, prompt, max_new_tokens=40, temperature=0.0, use_cache=False) == toks


@BOTH
def test_trace_replay_and_command_line(tmp_path, dtype):
    """bin/trace_run on a folder: whole, decoded and cut requests, one after another and in turn; the command line."""
    cfg = dc.ZMIXED
    w = lo.random_weights(cfg, 33)
    os.makedirs(tmp_path / "m")
    (tmp_path / "m" / "config.json").write_text(json.dumps(cfg))
    fb.save_safetensors(str(tmp_path / "m" / "model.safetensors"), w)
    ref = {r: decided(cfg, w, n, s) for r, n, s in (("a", 40, 30), ("b", 33, 31), ("c", 47, 10))}
    plan = [[("a", 40)], [("b", 10)], [("c", 20)], [("b", 1)], [("c", 2)], [("b", 1)], [("c", 25)], [("b", 21)]]
    at, steps, rows = dict.fromkeys(ref, 0), [], []
    for n, step in enumerate(plan):
        entries, mine, end = [], [], []
        for r, k in step:
            pick = [] if n == 5 else [i for i in range(k) if i % 3 == 0 or i == k - 1]
            entries.append(dict(id=r, tokens=ref[r][0][at[r]:at[r] + k].tolist(), want=pick))
            mine += [ref[r][1][at[r] + i] for i in pick]
            at[r] += k
            if at[r] == len(ref[r][0]):
                end.append(r)
        steps.append(json.dumps(dict(step=n, entries=entries, end=end)))
        rows.append(mine)
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(steps) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    for n, mine in enumerate(rows):
        f = out / f"{n}.f32"
        assert f.exists() == bool(mine)
        if mine:
            got = torch.frombuffer(bytearray(f.read_bytes()), dtype=torch.float32).view(len(mine), cfg["vocab"])
            assert dc.rel_error(got, torch.stack(mine)) < TOL[dtype], n
    p = subprocess.run([sys.executable, "-m", "femtochat_b200", "generate", "--model", str(tmp_path / "m"), "--tokens", "5,17,3",
                        "--max-new-tokens", "5", "--temperature", "0", "--dtype", dtype], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    model = fb.load_model(str(tmp_path / "m"), compute_type=dtype)
    assert [int(x) for x in p.stdout.strip().split(",")] == fb.generate(model, [5, 17, 3], max_new_tokens=5, temperature=0.0)[3:]


def test_misuse_is_an_error_not_a_fault():
    model, w = dc.model_and_weights(dc.ZMIXED, (8, 8), "float32", seed=33)
    c = cache_for(model, 8)
    with pytest.raises(_lib.FemtoError, match="exceed the cache"):
        fb.extend(model, c, dc.tokens(9, 113)[None, :])
    fb.extend(model, c, dc.tokens(8, 113)[None, :])
    with pytest.raises(_lib.FemtoError, match="cache is full"):
        fb.decode_step(model, c, torch.tensor([1]))
