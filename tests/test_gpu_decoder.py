"""Layer-listing decoders on the GPU against the plain CPU restatement (oracle/layered_oracle.py)."""
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
TOL = {"float32": 3e-5, "bfloat16": 8e-2}     # rounding the weights of the small mixed model to bf16 once more moves its logits by 5e-2
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def cache_for(model, n, B=1):
    return fb.KVCache(model.state(B), B, n)


def ok(model):
    assert model.state(1).status_word() == 0


@BOTH
@pytest.mark.parametrize("name", sorted(dc.SINGLE))
def test_each_mixer_alone(name, dtype):
    """One layer: a whole prompt, the same prompt token by token, and in portions (two tokens and more)."""
    cfg, ranks = dc.SINGLE[name]
    model, w = dc.model_and_weights(cfg, ranks, dtype, seed=3)
    n = 150 if "aligned" in name else 75
    t = dc.tokens(n, cfg["vocab"])
    want = lo.Sequence(cfg, w).feed(t)
    c = cache_for(model, n)
    assert dc.rel_error(dc.feed(model, c, t), want) < TOL[dtype]
    for cuts in ((1,) * 40, (2, 3, 2, 17, 2, 2, 9), (33,), (n - 2,), (64, 2)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_mixed_model_residuals_and_portions(dtype):
    """All mixers together, two of them twice with one set of weights: residual stream after every layer, and logits
    however the sequence is cut."""
    model, w = dc.model_and_weights(dc.MIXED, dc.MIXED_RANKS, dtype, seed=5)
    t = dc.tokens(90, dc.MIXED["vocab"], 1)
    ref = lo.Sequence(dc.MIXED, w)
    want = ref.feed(t)
    c = cache_for(model, 90)
    z, res = fb.extend(model, c, t[None, :], want=list(range(90)), residuals=True)
    for i, (a, b) in enumerate(zip(res.cpu().double(), ref.residuals)):
        assert float((a - b).abs().max() / b.abs().max()) < TOL[dtype], i
    assert dc.rel_error(z, want) < TOL[dtype]
    for cuts in ((1,) * 89, (2,) * 44, (7, 2, 31, 2, 5), (3, 3, 64, 3)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    ok(model)


@BOTH
def test_large_sizes_long_prompt(dtype):
    """Sizes at which products, attention and recurrences of a prompt run their tensor-core kernels; prompt lengths
    around tile edges; decoding after it."""
    model, w = dc.model_and_weights(dc.LARGE, dc.LARGE_RANKS, dtype, seed=7)
    t = dc.tokens(330, dc.LARGE["vocab"], 2)
    want = lo.Sequence(dc.LARGE, w).feed(t)
    c = cache_for(model, 330)
    for cuts in ((330,), (256, 40), (127, 1, 128), (129, 64, 65), (9, 200, 2, 100), (16, 17, 63, 65)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts
    c.reset()
    assert dc.rel_error(dc.feed(model, c, t, (300,) + (1,) * 29), want) < TOL[dtype]
    ok(model)


@BOTH
def test_columns_equal_each_alone(dtype):
    """Several columns of one length with different tokens give what each gives alone; prompts, portions, decoding."""
    cfg, ranks = dc.MIXED, dc.MIXED_RANKS
    model, w = dc.model_and_weights(cfg, ranks, dtype, seed=8)
    B, n = 3, 47
    t = torch.stack([dc.tokens(n, cfg["vocab"], 10 + b) for b in range(B)])
    want = torch.stack([lo.Sequence(cfg, w).feed(t[b]) for b in range(B)])
    c = cache_for(model, n, B)
    at = 0
    for k in (20, 2, 9, 1, 1, 14):
        z = fb.extend(model, c, t[:, at:at + k], want=list(range(B * k))).cpu().view(B, k, -1)
        assert dc.rel_error(z.reshape(B * k, -1), want[:, at:at + k].reshape(B * k, -1)) < TOL[dtype], at
        at += k
    # the plain entry points: last positions only
    z = fb.prefill(model, c, t[:, :30])
    assert dc.rel_error(z, want[:, 29]) < TOL[dtype]
    for k in range(30, 36):
        assert dc.rel_error(fb.decode_step(model, c, t[:, k]), want[:, k]) < TOL[dtype]
    assert len(c) == 36
    ok(model)


def test_wanted_positions_and_internal_portions():
    """A prompt longer than one internal pass, several columns, a ragged choice of positions."""
    cfg, ranks = dc.MIXED, dc.MIXED_RANKS
    model, w = dc.model_and_weights(cfg, ranks, "float32", seed=9, max_rows=26)
    t = torch.stack([dc.tokens(61, cfg["vocab"], 20 + b) for b in range(2)])
    ref = torch.cat([lo.Sequence(cfg, w).feed(t[b]) for b in range(2)])
    c = cache_for(model, 61, 2)
    want = [0, 12, 13, 14, 25, 26, 60, 61, 62, 73, 100, 121]
    assert dc.rel_error(fb.extend(model, c, t, want=want), ref[want]) < TOL["float32"]
    assert fb.extend(model, cache_for(model, 61, 2), t, want=[]) is None
    c.reset()
    assert dc.rel_error(fb.extend(model, c, t), ref[[60, 121]]) < TOL["float32"]
    for bad in ([3, 3], [5, 2], [-1], [122]):
        c.reset()
        with pytest.raises(_lib.FemtoError, match="ascend"):
            fb.extend(model, c, t, want=bad)


@BOTH
def test_a_used_cache_gives_what_a_fresh_one_gives(dtype):
    model, w = dc.model_and_weights(dc.MIXED, dc.MIXED_RANKS, dtype, seed=11)
    a, b = dc.tokens(40, dc.MIXED["vocab"], 30), dc.tokens(33, dc.MIXED["vocab"], 31)
    c, fresh = cache_for(model, 64), cache_for(model, 64)
    dc.feed(model, c, a, (5, 1, 1))
    c.reset()
    assert len(c) == 0
    assert torch.equal(dc.feed(model, c, b, (12, 1, 2)), dc.feed(model, fresh, b, (12, 1, 2)))
    # two requests in turn, each with its own cache
    c.reset(); fresh.reset()
    za, zb, i = [], [], 0
    for k in (3, 1, 10, 2, 17):
        za.append(fb.extend(model, c, a[None, i:i + k], want=list(range(k))).cpu())
        zb.append(fb.extend(model, fresh, b[None, i:i + k], want=list(range(k))).cpu())
        i += k
    assert dc.rel_error(torch.cat(za), lo.Sequence(dc.MIXED, w).feed(a[:33])) < TOL[dtype]
    assert dc.rel_error(torch.cat(zb), lo.Sequence(dc.MIXED, w).feed(b)) < TOL[dtype]


def matching_model(dtype):
    """One attention layer whose query of token A fits the key of token B alone: queries see the input through a random
    rotation R, keys as it is, and the embedding of B is R times that of A."""
    n, vocab = 64, 700
    cfg = dc.config(dc.latent(heads=2, dim=n, rot_dim=32, vdim=n, q_rank=n, kv_rank=n, scale=0.25, ff=0, base=500.0), width=n, vocab=vocab, mult=1.0)
    A, B = 11, 622

    def edit(w):
        g = torch.Generator().manual_seed(5)
        R = torch.linalg.qr(torch.randn(n, n, generator=g, dtype=torch.float64))[0]
        for name in ("l0.norm1", "l0.mix.dq.norm", "l0.mix.dkv.norm"):
            w[name].fill_(1.0)
        w["embed"][B] = (R @ w["embed"][A].double()).bfloat16()
        w["l0.mix.dq"].copy_(R)
        w["l0.mix.dkv"][:n] = torch.eye(n)
        for h in range(2):
            M = torch.linalg.qr(torch.randn(n, n, generator=g, dtype=torch.float64))[0]
            w["l0.mix.uq"].view(2, n + 32, n)[h, :n] = M
            w["l0.mix.uk"].view(2, n, n)[h] = M
        w["l0.mix.uq"].view(2, n + 32, n)[:, n:] *= 0.1
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=13, edit=edit)
    return cfg, model, w, A, B


@BOTH
@pytest.mark.parametrize("place", [0, 1, 15, 16, 127, 128, 129, 255, 256, 300])
def test_far_key_stands_out(dtype, place):
    """The last token's query fits one far key among hundreds, which lies at the start or at a tile's edge.  A prompt,
    decoding, and a last portion of two tokens must all find it."""
    cfg, model, w, A, B = matching_model(dtype)
    n = 400
    t = dc.tokens(n, cfg["vocab"], 50)
    t[(t == A) | (t == B)] = 3
    t[n - 1] = A
    u = t.clone()
    t[place] = B
    want = lo.Sequence(cfg, w).feed(t)[-3:]
    assert dc.rel_error(lo.Sequence(cfg, w).feed(u)[-1:], want[-1:]) > 0.4      # without the key the answer is another
    c = cache_for(model, n)
    for cuts in ((n,), (n - 1,), (n - 3, 1, 1), (n - 2,), (130, 128, 140)):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts)[-3:], want) < TOL[dtype], cuts
    ok(model)


@BOTH
@pytest.mark.parametrize("kind", ["long memory", "fast decay", "mixed decay"])
def test_delta_rule_decays(kind, dtype):
    """Decays next to 1 (a token hundreds back still shows), decays that underflow within a few tokens, and both in
    neighbouring channels: no overflow anywhere in the chunked form."""
    cfg = dc.config(dc.delta(heads=2, kv_heads=1, dim=64, vdim=64, conv=3, ff=0), width=64, vocab=200, mult=1.0)

    def edit(w):
        b = w["l0.mix.dt_bias"]
        if kind == "long memory":
            b.fill_(-9.0)
        elif kind == "fast decay":
            b.fill_(6.0); w["l0.mix.A_log"].fill_(3.0)
        else:
            b.copy_(torch.where(torch.arange(b.numel()) % 2 == 0, -9.0, 8.0)); w["l0.mix.A_log"].copy_(torch.tensor([2.5, -1.0]))
        w["l0.mix.a2"].mul_(0.3)

    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=17, edit=edit)
    t = dc.tokens(330, 200, 5)
    ref = lo.Sequence(cfg, w)
    want = ref.feed(t)
    if kind == "long memory":
        u = t.clone()
        u[3] = (u[3] + 1) % 200
        assert dc.rel_error(lo.Sequence(cfg, w).feed(u)[-1:], want[-1:]) > 10 * TOL["float32"]
    c = cache_for(model, 330)
    for cuts in ((330,), (64, 64, 64), (63, 65, 2), (300,) + (1,) * 29):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts


@BOTH
def test_lightning_decays(dtype):
    cfg = dc.config(dc.lightning(heads=6, dim=64, vdim=64, decay=[1.0, 0.9999, 0.5, 1e-3, 1e-20, 0.0], ff=0), width=64, vocab=200, mult=1.0)
    model, w = dc.model_and_weights(cfg, (8, 8), dtype, seed=19)
    t = dc.tokens(400, 200, 6)
    want = lo.Sequence(cfg, w).feed(t)
    c = cache_for(model, 400)
    for cuts in ((400,), (64, 64, 64), (63, 65, 2, 128), (380,) + (1,) * 19):
        c.reset()
        assert dc.rel_error(dc.feed(model, c, t, cuts), want) < TOL[dtype], cuts


@BOTH
def test_long_decoding(dtype):
    cfg, ranks = dc.MIXED, dc.MIXED_RANKS
    model, w = dc.model_and_weights(cfg, ranks, dtype, seed=21)
    t = dc.tokens(300, cfg["vocab"], 7)
    want = lo.Sequence(cfg, w).feed(t)
    assert dc.rel_error(dc.feed(model, cache_for(model, 300), t, (4,) + (1,) * 295), want) < TOL[dtype]
    ok(model)


def test_greedy_generation_matches_the_oracle():
    model, w = dc.model_and_weights(dc.MIXED, dc.MIXED_RANKS, "float32", seed=23)
    prompt = [5, 0, 112, 7, 7, 60]
    got = fb.generate(model, prompt, max_new_tokens=24, temperature=0.0)
    ref, toks = lo.Sequence(dc.MIXED, w), list(prompt)
    z = ref.feed(toks)[-1]
    for _ in range(24):
        toks.append(int(z.argmax()))
        z = ref.feed(toks[-1:])[-1]
    assert got == toks
    assert fb.generate(model, prompt, max_new_tokens=24, temperature=0.0, use_cache=False) == toks
    a, b = torch.Generator().manual_seed(1), torch.Generator().manual_seed(1)
    kw = dict(max_new_tokens=10, temperature=0.9, top_k=7)
    assert fb.generate(model, prompt, generator=a, **kw) == fb.generate(model, prompt, generator=b, use_cache=False, **kw)


def test_misuse_is_an_error_not_a_fault():
    model, w = dc.model_and_weights(dc.MIXED, dc.MIXED_RANKS, "float32", seed=25)
    st = model.state(1)
    c = cache_for(model, 8)
    with pytest.raises(_lib.FemtoError, match="exceed the cache"):
        fb.extend(model, c, dc.tokens(9, 113)[None, :])
    fb.extend(model, c, dc.tokens(8, 113)[None, :])
    with pytest.raises(_lib.FemtoError, match="cache is full"):
        fb.decode_step(model, c, torch.tensor([1]))
    with pytest.raises(_lib.FemtoError, match="positions"):
        fb.prefill(model, c, dc.tokens(4, 113)[None, :], torch.arange(4)[None, :])
    with pytest.raises(_lib.FemtoError, match="does not train|runs through"):
        x = torch.zeros(8, device="cuda")
        i = torch.zeros(8, device="cuda", dtype=torch.int32)
        _lib.check(_lib.lib().femto_loss_and_gradient(st.h, _lib.ptr(x), _lib.ptr(x), _lib.ptr(i), _lib.ptr(i), None, 1, 0, 0, _lib.ptr(x),
                                                      _lib.ptr(i), None))
    c.reset()
    fb.extend(model, c, torch.tensor([[3, 113, 2]]))       # an id outside the vocabulary is clamped and reported
    assert st.status_word() & 1


def test_updated_parameters_are_packed_again():
    model, w = dc.model_and_weights(dc.MIXED, dc.MIXED_RANKS, "float32", seed=27)
    t = dc.tokens(12, 113)[None, :]
    c = cache_for(model, 12)
    before = fb.prefill(model, c, t).cpu()
    spec = model.layout["l1.mix.uv"]
    model.params.theta[spec.offset:spec.offset + spec.size].mul_(-1)
    w["l1.mix.uv"].mul_(-1)
    after = fb.prefill(model, c, t).cpu()
    assert not torch.equal(before, after)
    assert dc.rel_error(after, lo.Sequence(dc.MIXED, w).feed(t[0])[-1:]) < TOL["float32"]


def write_model(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    fb.save_safetensors(os.path.join(path, "model.safetensors"), w)


@BOTH
def test_trace_replay_and_command_line(tmp_path, dtype):
    """bin/trace_run on a folder: whole, decoded and cut requests, one after another and in turn."""
    cfg, ranks = dc.MIXED, dc.MIXED_RANKS
    w = lo.random_weights(cfg, 29, *ranks)
    write_model(str(tmp_path / "m"), cfg, w)
    seqs = {r: dc.tokens(n, cfg["vocab"], 40 + n).tolist() for r, n in (("a", 31), ("b", 12), ("c", 44))}
    want = {r: lo.Sequence(cfg, w).feed(s) for r, s in seqs.items()}
    plan = [[("a", 31)], [("b", 10)], [("c", 20)], [("b", 1)], [("c", 2)], [("b", 1)], [("c", 1)], [("c", 21)]]
    at, steps, rows = dict.fromkeys(seqs, 0), [], []
    for n, step in enumerate(plan):
        entries, mine, end = [], [], []
        for r, k in step:
            pick = [] if n == 6 else [i for i in range(k) if i % 3 == 0 or i == k - 1]
            entries.append(dict(id=r, tokens=seqs[r][at[r]:at[r] + k], want=pick))
            mine += [want[r][at[r] + i] for i in pick]
            at[r] += k
            if at[r] == len(seqs[r]):
                end.append(r)
        steps.append(json.dumps(dict(step=n, entries=entries, end=end)))
        rows.append(mine)
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(steps) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(len(plan))]
    for n, mine in enumerate(rows):
        f = out / f"{n}.f32"
        assert f.exists() == bool(mine)
        if mine:
            got = torch.frombuffer(bytearray(f.read_bytes()), dtype=torch.float32).view(len(mine), cfg["vocab"])
            assert dc.rel_error(got, torch.stack(mine)) < TOL[dtype], n
    if dtype == "float32":
        p = subprocess.run([sys.executable, "-m", "femtochat_b200", "generate", "--model", str(tmp_path / "m"), "--tokens", "5,17,3",
                            "--max-new-tokens", "5", "--temperature", "0", "--dtype", dtype], cwd=ROOT, capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        model = fb.load_model(str(tmp_path / "m"), compute_type=dtype)
        assert [int(x) for x in p.stdout.strip().split(",")] == fb.generate(model, [5, 17, 3], max_new_tokens=5, temperature=0.0)[3:]


def test_gpt_loads_through_the_registry(tmp_path):
    """The framework's GPT through the same folder format and generation entry point."""
    from oracle import femto_oracle as fo
    kw = dict(sequence_len=64, max_document_tokens=128, vocab_size=100, n_layer=3, n_head=4, n_kv_head=2, n_embed=64, window_pattern="SL")
    cfg = fb.GPTConfig(**kw)
    lay = fb.parameter_layout(cfg)
    th = torch.zeros(lay.nparams)
    fo.initialize(th, fo.GPTConfig(**kw), fo.parameter_layout(fo.GPTConfig(**kw)), 2, all_nonzero=True)
    write_model(str(tmp_path), dict(kw, architecture="GPT"), {n: th[s.offset:s.offset + s.size].clone() for n, s in lay.named()})
    model = fb.load_model(str(tmp_path), compute_type="float32")
    assert torch.equal(model.params.theta.cpu(), th)
    direct = fb.GPT(fb.Params(th.cuda()), cfg, lay)
    assert fb.generate(model, [5, 17, 3], max_new_tokens=6, temperature=0.0) == fb.generate(direct, [5, 17, 3], max_new_tokens=6, temperature=0.0)
    c = fb.KVCache(model.state(1), 1, 64)
    z = fb.extend(model, c, torch.tensor([[5, 17, 3]]))
    assert torch.equal(z, fb.prefill(direct, fb.KVCache(direct.state(1), 1, 64), torch.tensor([[5, 17, 3]])))
