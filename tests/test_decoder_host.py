"""Layer-listing decoders without a GPU: the oracle's own invariants, configuration, layout, loading, command line."""
import json
import struct

import pytest
import torch

import femtochat_b200 as fb
from femtochat_b200 import _lib
from oracle import layered_oracle as lo

import decoder_cases as dc


@pytest.mark.parametrize("name", ["lightning", "delta", "latent"])
def test_oracle_portions_equal_the_whole(name):
    cfg, ranks = dc.SINGLE[name]
    w, t = lo.random_weights(cfg, 1, *ranks), dc.tokens(17, cfg["vocab"])
    whole = lo.Sequence(cfg, w).feed(t)
    for cuts in ((2, 5, 2), (1,) * 16, (16,)):
        s, at, out = lo.Sequence(cfg, w), 0, []
        for n in cuts + (99,):
            out.append(s.feed(t[at:at + n])) if at < 17 else None
            at += n
        assert (torch.cat(out) - whole).abs().max() < 1e-10


def test_oracle_recurrences_against_closed_forms():
    g = torch.Generator().manual_seed(3)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    T, H, D, E = 7, 2, 3, 4
    q, k, v, S0 = r(T, H, D), r(T, H, D), r(T, H, E), r(H, D, E)
    decay = torch.tensor([0.3, 0.9], dtype=torch.float64)
    o, S = lo.decayed_outer_recurrence(q, k, v, decay, S0)
    for h in range(H):       # o_t = decay^(t+1) S0^T q + sum_j decay^(t-j) (q_t . k_j) v_j
        for t in range(T):
            want = decay[h] ** (t + 1) * (S0[h].T @ q[t, h])
            for j in range(t + 1):
                want = want + decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h]
            assert torch.allclose(o[t, h], want)
    # with g = 1, beta = 1 and a unit key the delta rule stores v under k exactly: reading k back gives v
    k1 = lo.unit_vector(k)
    one = torch.ones(T, H, D, dtype=torch.float64)
    o, S = lo.gated_delta_recurrence(k1, k1, v, one, torch.ones(T, H, dtype=torch.float64), S0)
    assert torch.allclose(o, v, atol=1e-3)


def test_rotation_keeps_relative_positions():
    g = torch.Generator().manual_seed(4)
    a, b = torch.randn(1, 1, 8, generator=g, dtype=torch.float64), torch.randn(1, 1, 8, generator=g, dtype=torch.float64)
    dot = lambda i, j: float((lo.rotate_half(a, torch.tensor([i]), 6, 100.0) * lo.rotate_half(b, torch.tensor([j]), 6, 100.0)).sum())
    assert dot(3, 1) == pytest.approx(dot(12, 10)) and dot(3, 1) != pytest.approx(dot(3, 2))


@pytest.mark.parametrize("name", sorted(dc.SINGLE))
def test_layout_names_and_shapes(name):
    cfg, ranks = dc.SINGLE[name]
    shapes = lo.tensor_shapes(cfg, *ranks)
    c = fb.DecoderConfig.from_json(cfg, shapes)
    lay = fb.decoder_layout(c)
    assert {n: s.shape for n, s in lay.items()} == shapes
    spans = sorted((s.offset, s.offset + s.size) for s in lay.values())
    assert all(a[1] <= b[0] for a, b in zip(spans, spans[1:])) and all(o % 4 == 0 for o, _ in spans)
    assert spans[-1][1] <= _lib.lib().femto_decoder_nparams(c.c_struct())


def test_shared_weights_have_one_set_of_tensors():
    shapes = lo.tensor_shapes(dc.MIXED, *dc.MIXED_RANKS)
    lay = fb.decoder_layout(fb.DecoderConfig.from_json(dc.MIXED, shapes))
    assert set(lay) == set(shapes) and not any(n.startswith(("l3.", "l5.")) for n in lay)
    ranks = [(l.decay_rank, l.gate_rank) for l in fb.DecoderConfig.from_json(dc.MIXED, shapes).layers]
    assert ranks[0] == ranks[3] == dc.MIXED_RANKS      # sizes that only the owner's tensors give


def test_bad_configurations_are_refused():
    def layout(*layers, **kw):
        cfg = dc.config(*layers, **kw)
        return fb.decoder_layout(fb.DecoderConfig.from_json(cfg, lo.tensor_shapes(cfg)))
    with pytest.raises(_lib.FemtoError, match="multiple of kv_heads"):
        layout(dc.delta(heads=3, kv_heads=2))
    with pytest.raises(_lib.FemtoError, match="256"):
        layout(dc.lightning(dim=300))
    with pytest.raises(_lib.FemtoError, match="differs in its sizes"):
        layout(dc.lightning(), dc.lightning(dim=20, weights_of=0))
    with pytest.raises(_lib.FemtoError, match="circle"):
        fb.decoder_layout(fb.DecoderConfig.from_json(dc.config(dc.lightning(weights_of=1), dc.lightning(weights_of=0)), {}))
    with pytest.raises(_lib.FemtoError, match="even"):
        layout(dc.latent(rot_dim=8, rot_dims=3))
    with pytest.raises(ValueError, match="decays"):
        layout(dc.lightning(heads=3, decay=[0.5]))
    with pytest.raises(ValueError, match="unknown mixer"):
        fb.DecoderConfig.from_json(dc.config(dict(dc.lightning(), type="windmill")), {})


def test_safetensors_round_trip_and_format(tmp_path):
    path = str(tmp_path / "w.safetensors")
    t = {"a": torch.randn(3, 5).bfloat16(), "b.c": torch.arange(7, dtype=torch.int32), "e": torch.zeros(2, 0)}
    fb.save_safetensors(path, t)
    f = fb.SafeTensors(path)
    assert f.shapes == {k: tuple(v.shape) for k, v in t.items()} and set(f) == set(t)
    for k in t:
        assert f[k].dtype == t[k].dtype and torch.equal(f[k], t[k])
    raw = open(path, "rb").read()
    n, = struct.unpack("<Q", raw[:8])
    assert json.loads(raw[8:8 + n])["a"]["dtype"] == "BF16"
    (tmp_path / "bad").write_bytes(struct.pack("<Q", 1 << 40) + b"{}")
    with pytest.raises(ValueError, match="header"):
        fb.SafeTensors(str(tmp_path / "bad"))


def test_registry(tmp_path):
    assert fb.MODELS["Virolorn"] is fb.MODELS["Zurevik"] is fb.Decoder and fb.MODELS["GPT"] is fb.GPT
    (tmp_path / "config.json").write_text(json.dumps(dict(architecture="Nothing")))
    with pytest.raises(ValueError, match="unknown architecture"):
        fb.load_model(str(tmp_path))


def test_sample_token_counts_from_the_models_base():
    z = torch.tensor([0.0, 3.0, 1.0])
    assert fb.sample_token(None, z, 0, 1) == 2 and fb.sample_token(None, z, 0, 1, 0) == 1
    g = torch.Generator().manual_seed(0)
    assert all(0 <= fb.sample_token(g, z, 1.0, 3, 0) <= 2 for _ in range(20))


def test_no_cpu_fallback():
    if torch.cuda.is_available():
        pytest.skip("GPU present")
    cfg, ranks = dc.SINGLE["lightning"]
    c = fb.DecoderConfig.from_json(cfg, lo.tensor_shapes(cfg, *ranks))
    with pytest.raises(_lib.FemtoError, match="no CUDA device"):
        fb.DecoderState(c, 1)


# ---- windows, sinks, differential attention, mixtures of experts ------------------------------------------------------
@pytest.mark.parametrize("name", ["differential", "sinks", "sinks, shared keys"])
def test_oracle_portions_of_windowed_layers(name):
    cfg, ranks = dc.SINGLE[name]
    w, t = lo.random_weights(cfg, 1, *ranks), dc.tokens(60, cfg["vocab"])
    whole = lo.Sequence(cfg, w).feed(t)
    for cuts in ((2, 5, 2), (1,) * 59, (21,)):
        s, at, out = lo.Sequence(cfg, w), 0, []
        for n in cuts + (99,):
            out.append(s.feed(t[at:at + n])) if at < 60 else None
            at += n
        assert (torch.cat(out) - whole).abs().max() < 1e-10


def test_oracle_windowed_attention_against_masked_softmax():
    g = torch.Generator().manual_seed(6)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    N, T, H, G, D, E, size, keep = 23, 9, 4, 2, 5, 3, 6, 2
    q, k, v, sink = r(T, H, D), r(N, G, D), r(N, G, E), r(H)
    i, j = torch.arange(N - T, N)[:, None], torch.arange(N)[None, :]
    see = (j <= i) & ((i - j < size) | (j < keep))
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("thd,nhd->htn", q, kk) * 0.7
    s = s.masked_fill(~see, -torch.inf)
    p = torch.softmax(torch.cat([s, sink[:, None, None].expand(H, T, 1)], -1), -1)[..., :-1]
    assert torch.allclose(lo.windowed_attention(q, k, v, 0.7, N - T, size, keep, sink), torch.einsum("htn,nhe->the", p, vv))
    assert torch.allclose(lo.windowed_attention(q, k, v, 0.7, N - T, size, keep), torch.einsum("htn,nhe->the", torch.softmax(s, -1), vv))
    # an unreachable sink changes nothing, an overwhelming one leaves nothing
    assert torch.allclose(lo.windowed_attention(q, k, v, 0.7, N - T, size, keep, sink - 100), lo.windowed_attention(q, k, v, 0.7, N - T, size, keep))
    assert lo.windowed_attention(q, k, v, 0.7, N - T, size, keep, sink + 100).abs().max() < 1e-30


def test_oracle_routing():
    best, weight = lo.route(torch.tensor([[1.0, 3.0, 3.0, -2.0], [0.0, -1.0, 5.0, 4.0]], dtype=torch.float64), 2)
    assert best.tolist() == [[1, 2], [2, 3]] and torch.allclose(weight[0], torch.tensor([0.5, 0.5], dtype=torch.float64))
    assert torch.allclose(weight[1], torch.softmax(torch.tensor([5.0, 4.0], dtype=torch.float64), 0))


@pytest.mark.parametrize("name", sorted(dc.EXPERTS))
def test_layout_of_mixtures(name):
    cfg = dc.EXPERTS[name]
    shapes = lo.tensor_shapes(cfg)
    assert {n: s.shape for n, s in fb.decoder_layout(fb.DecoderConfig.from_json(cfg, shapes)).items()} == shapes


def test_a_layer_that_reads_anothers_keys_has_none():
    lay = fb.decoder_layout(fb.DecoderConfig.from_json(dc.ZMIXED, lo.tensor_shapes(dc.ZMIXED)))
    assert "l0.mix.k" in lay and "l0.mix.v.b" in lay and "l2.mix.q.b" in lay and "head" in lay
    assert not any(n.startswith(("l2.mix.k", "l2.mix.v")) or n.endswith("norm1b") for n in lay)


def test_bad_windowed_configurations_are_refused():
    def layout(*layers, **kw):
        return fb.decoder_layout(fb.DecoderConfig.from_json(dc.zurevik(*layers, **kw), {}))
    with pytest.raises(_lib.FemtoError, match="multiple of kv_heads"):
        layout(dc.differential(heads=3, kv_heads=2))
    with pytest.raises(_lib.FemtoError, match="earlier layer"):
        layout(dc.sinks(kv_from=1), dc.sinks())
    with pytest.raises(_lib.FemtoError, match="of its own"):
        layout(dc.sinks(), dc.sinks(kv_from=0), dc.sinks(kv_from=1))
    with pytest.raises(_lib.FemtoError, match="key or value sizes"):
        layout(dc.sinks(), dc.sinks(kv_from=0, vdim=24))
    with pytest.raises(_lib.FemtoError, match="window"):
        layout(dc.sinks(size=0))
    with pytest.raises(_lib.FemtoError, match="256"):
        layout(dc.differential(dim=300))
    with pytest.raises(_lib.FemtoError, match="experts"):
        layout(dc.sinks(mlp=dc.moe(experts=3, top=4)))
    with pytest.raises(ValueError, match="unknown mixer"):
        layout(dc.lightning())
    with pytest.raises(ValueError, match="unknown feed-forward"):
        layout(dc.sinks(mlp=dict(kind="spline")))
