"""Prefill and decode throughput of the layer-listing decoders beside the framework's GPT at equal size, random weights: the
GPT with full attention (Virolorn's counterpart) and with the window that Zurevik's layers have.

Times are CUDA events around whole calls of the public entry points (`extend` / `prefill` / `decode_step`), after warm-up;
every call reads weights and caches larger than L2.  `--kernels` lists where a call's device time goes."""
from __future__ import annotations

import argparse
import json

SIZES = {
    # width, layers, feed-forward of the gated MLP (the GPT's has 4 x width: equal weights), heads of 128
    "d20": dict(width=1280, n_layer=20, ff=3456, heads=10, kv_heads=5, q_rank=768, kv_rank=512, vocab=65536),
    "w2560": dict(width=2560, n_layer=12, ff=6912, heads=20, kv_heads=10, q_rank=1536, kv_rank=512, vocab=65536),
}
MIX = ("lightning", "channel_delta", "channel_delta", "latent_attention")
WINDOW, KEEP, EXPERTS, TOP = 1024, 4, 8, 2      # Zurevik: two experts of 2 x width, the weights a token uses in the GPT's 4 x width
MODELS = ("Virolorn", "Zurevik", "GPT", "GPT window")


def decoder_config(s, mix=MIX):
    import femtochat_b200 as fb
    layers = []
    for i in range(s["n_layer"]):
        kind = mix[i % len(mix)]
        lc = fb.LayerConfig(mixer=kind, heads=s["heads"], dim=128, vdim=128, ff=s["ff"])
        if kind == "lightning":
            lc.decay = tuple(2.718281828 ** (-2.0 ** (-8.0 * (h + 1) / s["heads"])) for h in range(s["heads"]))
        elif kind == "channel_delta":
            lc.kv_heads, lc.conv, lc.decay_rank, lc.gate_rank = s["kv_heads"], 4, 128, 128
        else:
            lc.q_rank, lc.kv_rank, lc.rot_dim, lc.rot_dims, lc.rot_base, lc.scale = s["q_rank"], s["kv_rank"], 64, 64, 500000.0, 192 ** -0.5
        layers.append(lc)
    return fb.DecoderConfig(vocab_size=s["vocab"], width=s["width"], norm_eps=1e-6, residual_mult=0.5, layers=layers)


def zurevik_config(s):
    import femtochat_b200 as fb
    layers = []
    for i in range(s["n_layer"]):
        kw = dict(mixer="attention", heads=s["heads"], kv_heads=s["kv_heads"], vdim=128, window=WINDOW, ff=2 * s["width"], experts=EXPERTS, top=TOP)
        if i % 4 < 2:       # the second reads the keys and values of the first
            layers.append(fb.LayerConfig(dim=128, scale=128 ** -0.5, qkv_bias=True, sink=True, gate="head", kv_from=i - 1 if i % 4 else None, **kw))
        else:
            layers.append(fb.LayerConfig(dim=64, scale=64 ** -0.5, maps=2, qk_norm=True, gate="element", diff=0.5, keep_first=KEEP, **kw))
    return fb.DecoderConfig(vocab_size=s["vocab"], width=s["width"], norm_eps=1e-6, layers=layers, block="parallel", untied=True,
                            embed_scale=1.0, logit_softcap=15.0)


def random_decoder(s, cfg=None, max_rows=16384):
    import torch
    import femtochat_b200 as fb
    from femtochat_b200 import _lib
    cfg = cfg or decoder_config(s)
    lay = fb.decoder_layout(cfg)
    theta = torch.zeros(int(_lib.lib().femto_decoder_nparams(cfg.c_struct())), device="cuda")
    g = torch.Generator(device="cuda").manual_seed(1)
    for name, spec in lay.items():
        v = theta[spec.offset:spec.offset + spec.size]
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            v.fill_(1.0)
        elif leaf in ("sink", "b", "lq1", "lk1", "lq2", "lk2"):
            v.normal_(0.0, 0.1, generator=g)
        elif leaf == "dt_bias":
            v.normal_(-3.0, 1.0, generator=g)
        elif leaf == "A_log":
            v.normal_(0.0, 0.5, generator=g)
        else:
            v.normal_(0.0, spec.shape[-1] ** -0.5, generator=g)
    return fb.Decoder(fb.Params(theta, delta=False), cfg, lay, compute_type="bfloat16", max_rows=max_rows)


def random_gpt(s, T, window=None):
    import torch
    import femtochat_b200 as fb
    cfg = fb.GPTConfig(sequence_len=T, max_document_tokens=16384, vocab_size=s["vocab"], n_layer=s["n_layer"], n_head=s["heads"],
                       n_kv_head=s["kv_heads"], n_embed=s["width"], window_pattern="L" if window is None else "S")
    lay = fb.parameter_layout(cfg)
    theta = torch.empty(lay.nparams, device="cuda")
    fb.initialize_(theta, lay, seed=1, all_nonzero=True)
    return fb.GPT(fb.Params(theta, delta=False), cfg, lay, compute_type="bfloat16", **({"short_window": window} if window else {}))


def timed(fn, iters, warm=3):
    import torch
    for _ in range(warm):
        fn()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def kernel_times(fn):
    """(name, launches, milliseconds) of the kernels of one call, longest first."""
    import torch
    from torch.profiler import ProfilerActivity, profile
    fn()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as p:
        fn()
        torch.cuda.synchronize()
    rows = [(e.key.replace("(anonymous namespace)::", "").split("(")[0], e.count, e.device_time_total / 1e3) for e in p.key_averages() if e.device_time_total > 0]
    return sorted(rows, key=lambda r: -r[2])


def measure(model, B, T, vocab, n_decode=32, kernels=False):
    import torch
    import femtochat_b200 as fb
    g = torch.Generator(device="cuda").manual_seed(2)
    tok = torch.randint(model.index_base, vocab + model.index_base, (B, T), generator=g, device="cuda", dtype=torch.int32)
    model.state(B).refresh_weights(model.params.theta)
    model.state(B).refresh_weights = lambda theta: None      # Θ does not change: no cast inside the timed calls
    c = fb.KVCache(model.state(B), B, T + 4 * n_decode + 64)
    pre = timed(lambda: fb.prefill(model, c, tok), 5)
    one = tok[:, 0].contiguous()
    dec = timed(lambda: fb.decode_step(model, c, one), n_decode, warm=8)
    out = dict(B=B, T=T, prefill_ms=pre, prefill_tokens_per_s=B * T / pre * 1e3, decode_ms=dec, decode_tokens_per_s=B / dec * 1e3)
    if kernels:
        for name, fn in (("prefill", lambda: fb.prefill(model, c, tok)), ("decode", lambda: fb.decode_step(model, c, one))):
            rows = kernel_times(fn)
            print(f"-- {name} B={B} T={T}: {sum(r[2] for r in rows):.3f} ms in {sum(r[1] for r in rows)} launches")
            for k, n, ms in rows[:22]:
                print(f"   {ms:9.4f} ms {n:5d} x {k[:100]}")
    c.close()
    return out


def run(size="d20", shapes=((1, 8192), (8, 2048)), kernels=False, which=MODELS):
    import torch
    s, out = SIZES[size], dict(size=size)
    for name in which:
        out[name] = []
        for B, T in shapes:
            if name == "Zurevik":
                model = random_decoder(s, zurevik_config(s), max_rows=B * T)
            elif name == "Virolorn":
                model = random_decoder(s, max_rows=B * T)
            else:
                model = random_gpt(s, T + 192, WINDOW if name == "GPT window" else None)
            if kernels:
                print(f"== {name} {size}")
            out[name].append(measure(model, B, T, s["vocab"], kernels=kernels))
            if model._state is not None:
                model._state.close()
            del model
            torch.cuda.empty_cache()
    return out


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default="d20", choices=sorted(SIZES))
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--shapes", default="1x8192,8x2048")
    ap.add_argument("--which", default=",".join(MODELS))
    a = ap.parse_args()
    shapes = [tuple(int(v) for v in x.split("x")) for x in a.shapes.split(",")]
    print(json.dumps(run(a.size, shapes, a.kernels, a.which.split(","))))


if __name__ == "__main__":
    main()
