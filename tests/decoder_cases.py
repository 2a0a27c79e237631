"""Small configurations and helpers shared by the tests of the layer-listing decoders."""
import torch

from oracle import layered_oracle as lo


def lightning(heads=3, dim=16, vdim=24, decay=None, ff=48, **kw):
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay or [0.5, 0.97, 1.0, 0.9995, 0.02][:heads]),
                mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, ff=48, **kw):
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
                mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def latent(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=28, scale=0.2, base=10000.0, ff=48, rot_dims=None, **kw):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                                                   scale=scale, rot=dict(dims=rot_dim if rot_dims is None else rot_dims, base=base)),
                mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def moe(ff=24, experts=5, top=2):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def differential(heads=4, kv_heads=2, dim=16, vdim=24, size=20, keep=3, scale=0.3, diff=0.45, mlp=None, **kw):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff,
                                             mask=dict(size=size, keep_first=keep)), mlp=mlp, **kw)


def sinks(heads=6, kv_heads=2, dim=24, vdim=16, size=17, scale=0.2, mlp=None, kv_from=None, **kw):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention_2", mixer=m, mlp=mlp, **kw)


def zurevik(*layers, vocab=96, width=40, eps=1e-5, embed_scale=1.7, softcap=9.0):
    return dict(architecture="Zurevik", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=embed_scale), logit_softcap=softcap,
                layers=list(layers))


def config(*layers, vocab=96, width=40, eps=1e-5, mult=0.7):
    return dict(architecture="Virolorn", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, layers=list(layers))


# name -> (config, ranks of the two low-rank projections)
SINGLE = {
    "lightning": (config(lightning()), (8, 8)),
    "lightning without feed-forward": (config(lightning(ff=0)), (8, 8)),
    "lightning, aligned sizes": (config(lightning(heads=2, dim=128, vdim=128, ff=512, decay=[0.9, 0.999]), width=256, vocab=320), (8, 8)),
    "lightning, one head, odd sizes": (config(lightning(heads=1, dim=7, vdim=5, decay=[0.83], ff=33), width=30, vocab=61), (8, 8)),
    "lightning, wide": (config(lightning(heads=2, dim=200, vdim=72, ff=64, decay=[0.3, 0.99])), (8, 8)),
    "delta": (config(delta()), (5, 11)),
    "delta without feed-forward": (config(delta(ff=0)), (3, 8)),
    "delta, one tap": (config(delta(conv=1)), (8, 8)),
    "delta, two taps, heads of their own": (config(delta(conv=2, kv_heads=4, dim=24, vdim=16)), (16, 2)),
    "delta, aligned sizes": (config(delta(heads=4, kv_heads=2, dim=128, vdim=128, ff=512), width=256, vocab=320), (64, 64)),
    "delta, dim 64": (config(delta(heads=2, kv_heads=1, dim=64, vdim=96, conv=3, ff=256), width=128), (24, 40)),
    "delta, wide": (config(delta(heads=2, kv_heads=2, dim=200, vdim=136, conv=3)), (8, 24)),
    "delta, one head, odd sizes": (config(delta(heads=1, kv_heads=1, dim=9, vdim=5, conv=5, ff=20), width=34), (1, 1)),
    "latent": (config(latent()), (8, 8)),
    "latent without feed-forward": (config(latent(ff=0)), (8, 8)),
    "latent, partly rotated": (config(latent(rot_dim=12, rot_dims=6)), (8, 8)),
    "latent, aligned sizes": (config(latent(heads=4, dim=128, rot_dim=64, vdim=128, q_rank=192, kv_rank=128, ff=512, scale=0.07), width=256, vocab=320), (8, 8)),
    "latent, dim 64": (config(latent(heads=2, dim=64, rot_dim=64, vdim=64, q_rank=64, kv_rank=256, ff=256), width=128), (8, 8)),
    "latent, vdim 96": (config(latent(heads=5, dim=48, rot_dim=16, vdim=96, q_rank=40, kv_rank=72, ff=256), width=128), (8, 8)),
    "latent, wide values": (config(latent(heads=2, dim=64, rot_dim=16, vdim=160, q_rank=40, kv_rank=72)), (8, 8)),
    "latent, one head, odd sizes": (config(latent(heads=1, dim=5, rot_dim=2, vdim=3, q_rank=7, kv_rank=9, ff=20), width=34), (8, 8)),
    "differential": (zurevik(differential()), (8, 8)),
    "differential, one key head": (zurevik(differential(heads=6, kv_heads=1, dim=8, vdim=40, size=5, keep=1, scale=0.5, diff=0.2)), (8, 8)),
    "differential, a window of one": (zurevik(differential(size=1, keep=0)), (8, 8)),
    "differential, a window of one and kept tokens": (zurevik(differential(size=1, keep=9)), (8, 8)),
    "differential, a window beyond the prompt": (zurevik(differential(size=500, keep=2, diff=0.8)), (8, 8)),
    "differential, kept tokens beyond the prompt": (zurevik(differential(size=3, keep=300)), (8, 8)),
    "differential, aligned sizes": (zurevik(differential(heads=4, kv_heads=2, dim=64, vdim=128, size=50, keep=6, scale=0.15), width=256, vocab=320), (8, 8)),
    "differential, dim 128": (zurevik(differential(heads=2, kv_heads=2, dim=128, vdim=64, size=33, keep=2, scale=0.1), width=128), (8, 8)),
    "differential, wide": (zurevik(differential(heads=2, kv_heads=1, dim=200, vdim=136, scale=0.05)), (8, 8)),
    "differential, one head, odd sizes": (zurevik(differential(heads=1, kv_heads=1, dim=5, vdim=3, scale=0.7), width=34, vocab=61), (8, 8)),
    "sinks": (zurevik(sinks()), (8, 8)),
    "sinks, heads of their own": (zurevik(sinks(heads=3, kv_heads=3, dim=40, vdim=32, size=9)), (8, 8)),
    "sinks, one key head": (zurevik(sinks(heads=20, kv_heads=1, dim=8, vdim=8, size=30, scale=0.4)), (8, 8)),
    "sinks, a window of one": (zurevik(sinks(size=1)), (8, 8)),
    "sinks, no softcap": (zurevik(sinks(size=400), softcap=None, embed_scale=0.3), (8, 8)),
    "sinks, aligned sizes": (zurevik(sinks(heads=4, kv_heads=2, dim=128, vdim=128, size=70, scale=0.09), width=256, vocab=320), (8, 8)),
    "sinks, wide": (zurevik(sinks(heads=2, kv_heads=1, dim=256, vdim=200, scale=0.05)), (8, 8)),
    "sinks, wide values": (zurevik(sinks(heads=4, kv_heads=2, dim=64, vdim=200, scale=0.12), width=64), (8, 8)),
    "sinks, one head, odd sizes": (zurevik(sinks(heads=1, kv_heads=1, dim=7, vdim=5, scale=0.6), width=34, vocab=61), (8, 8)),
    "sinks, shared keys": (zurevik(sinks(size=9), sinks(size=30, kv_from=0, scale=0.35), sinks(size=4, kv_from=0, heads=2)), (8, 8)),
}

# mixtures of experts: tokens are chosen so that no router is near a tie (decided_tokens)
EXPERTS = {
    "two of five": zurevik(sinks(mlp=moe())),
    "one of three": zurevik(differential(mlp=moe(experts=3, top=1))),
    "all of four": zurevik(sinks(mlp=moe(experts=4, top=4, ff=9))),
    "one expert": zurevik(sinks(mlp=moe(experts=1, top=1))),
    "three of twenty": zurevik(sinks(mlp=moe(experts=20, top=3, ff=16))),
    "five of forty": zurevik(sinks(mlp=moe(experts=40, top=5, ff=16))),
    "one of seventy": zurevik(sinks(mlp=moe(experts=70, top=1, ff=8))),
    "two of three hundred": zurevik(sinks(mlp=moe(experts=300, top=2, ff=8))),
    "odd sizes": zurevik(sinks(heads=1, kv_heads=1, dim=7, vdim=5, mlp=moe(ff=13, experts=6, top=3)), width=34, vocab=61),
    "aligned sizes": zurevik(sinks(heads=2, kv_heads=2, dim=64, vdim=64, mlp=moe(ff=256, experts=4, top=2)), width=256, vocab=320),
    "between norms": config(latent(ff=0), latent(ff=0)),
    "gated feed-forward beside the mixer": zurevik(sinks(mlp=dict(kind="dense", ff=40)), differential(mlp=dict(kind="dense", ff=24))),
}
EXPERTS["between norms"]["layers"][0]["mlp"] = moe(experts=4, top=2)

ZMIXED = zurevik(sinks(heads=4, kv_heads=2, dim=24, vdim=32, size=13, mlp=moe()), differential(heads=2, kv_heads=1, dim=16, vdim=40, size=11, keep=4, mlp=moe(ff=32, experts=4, top=1)),
                 sinks(heads=2, kv_heads=2, dim=24, vdim=32, size=25, kv_from=0, mlp=moe(experts=3, top=3)), differential(size=7, keep=0, diff=0.7),
                 vocab=113, width=72, embed_scale=0.8, softcap=5.0)
# sizes at which every product and the attention of prompts run their tensor-core kernels; the second mixture fills runs of 256 rows
ZLARGE = zurevik(sinks(heads=4, kv_heads=2, dim=128, vdim=128, size=150, scale=0.1, mlp=moe(ff=256, experts=6, top=2)),
                 differential(heads=4, kv_heads=2, dim=64, vdim=128, size=90, keep=5, scale=0.15, mlp=moe(ff=384, experts=2, top=2)),
                 sinks(heads=8, kv_heads=2, dim=128, vdim=128, size=260, scale=0.1, kv_from=0),
                 differential(heads=2, kv_heads=2, dim=96, vdim=72, size=129, keep=140, scale=0.12), vocab=512, width=512)



MIXED = config(delta(heads=2, kv_heads=1, dim=32, vdim=40, conv=3), latent(heads=4, dim=24, rot_dim=16, vdim=32), lightning(heads=2, dim=24, vdim=32),
               delta(heads=2, kv_heads=1, dim=32, vdim=40, conv=3, weights_of=0), lightning(heads=3, dim=16, vdim=24, ff=0),
               latent(heads=4, dim=24, rot_dim=16, vdim=32, weights_of=1), vocab=113, width=72)
MIXED_RANKS = (12, 20)
# sizes at which every product, the attention of prompts and the chunked recurrences run their tensor-core kernels
LARGE = config(lightning(heads=4, dim=64, vdim=128, ff=512, decay=[0.5, 0.9, 0.99, 0.9999]),
               delta(heads=4, kv_heads=2, dim=128, vdim=128, conv=4, ff=512),
               latent(heads=4, dim=128, rot_dim=64, vdim=128, q_rank=192, kv_rank=256, scale=0.0722, ff=512),
               delta(heads=4, kv_heads=2, dim=128, vdim=128, conv=4, ff=512, weights_of=1), vocab=512, width=512, mult=0.5)
LARGE_RANKS = (64, 64)


class Tensors(dict):
    """A dict of tensors with the face of a weights file."""

    @property
    def shapes(self):
        return {k: tuple(v.shape) for k, v in self.items()}


def model_and_weights(cfg, ranks, dtype, seed=0, edit=None, **options):
    import femtochat_b200 as fb
    w = lo.random_weights(cfg, seed, *ranks)
    if edit:
        edit(w)
    return fb.Decoder.from_weights(cfg, Tensors(w), compute_type=dtype, **options), w


def tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, vocab, (n,), generator=g)


def decided_tokens(cfg, w, n, seed=0, margin=0.1):
    """(tokens, logits): a sequence in which the last expert that any router chose leads the next one by `margin`, so that
    rounding in 16 bits chooses the same experts."""
    g = torch.Generator().manual_seed(2000 + seed)
    s, toks, out = lo.Sequence(cfg, w), [], []
    while len(toks) < n:
        kept = [dict(x) for x in s.state]
        t = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
        z = s.feed([t])
        if s.margins and float(torch.cat(s.margins).min()) < margin:
            s.state = kept
            continue
        toks.append(t)
        out.append(z)
    return torch.tensor(toks), torch.cat(out)


def rel_error(got, want):
    """Largest root mean square error of a row of logits (means removed), in units of the logits' own spread."""
    got, want = got.detach().cpu().double(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max())


def feed(model, cache, toks, cuts=(), want_all=True):
    """Feeds a sequence in portions and returns the logits of all its positions."""
    import femtochat_b200 as fb
    out, at = [], 0
    for n in list(cuts) + [None]:
        part = toks[at:] if n is None else toks[at:at + n]
        if len(part):
            out.append(fb.extend(model, cache, part[None, :], want=list(range(len(part)))).cpu())
        at += len(part)
    return torch.cat(out)
