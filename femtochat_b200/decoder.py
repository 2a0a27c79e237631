"""Host side of the decoders that list their layers (femto_decoder_*): configuration, flat parameter layout, handle and
model call.  Two models are of this kind.  "Virolorn": lightning attention, the gated delta rule with channel decays and
latent attention in any order, an RMS norm before and after every sublayer, tied embedding.  "Zurevik": differential
attention with kept first tokens and attention with a sink, both in sliding windows, beside a mixture of experts.  All
arithmetic runs in the library; the cache is the framework's KVCache and generation its `prefill`, `decode_step` and
`generate`."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

from . import _lib
from .handle import Handle
from .parameters import Params, ParamSpec

MIXERS = {"lightning": 1, "channel_delta": 2, "latent_attention": 3, "attention": 4}
BLOCKS = {"sandwich": 0, "parallel": 1}
GATES = {None: 0, "head": 1, "element": 2}
NO_WINDOW = 1 << 30


@dataclass
class LayerConfig:
    """One layer of the list; sizes that its mixer does not have stay 0."""
    mixer: str
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0
    decay: Tuple[float, ...] = ()
    conv: int = 0
    decay_rank: int = 0
    gate_rank: int = 0
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_dims: int = 0
    rot_base: float = 1.0
    scale: float = 1.0
    ff: int = 0
    weights_of: Optional[int] = None
    # "attention": one map or two (differential), a window, what it adds to plain softmax attention
    maps: int = 1
    window: int = NO_WINDOW
    keep_first: int = 0
    kv_from: Optional[int] = None
    qkv_bias: bool = False
    qk_norm: bool = False
    sink: bool = False
    gate: Optional[str] = None
    diff: float = 0.0
    # feed-forward: 0 experts = one gated feed-forward
    experts: int = 0
    top: int = 0


def _attention(m: dict, **features) -> LayerConfig:
    mask = m.get("mask") or {}
    return LayerConfig(mixer="attention", heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_heads=m["kv_heads"], scale=float(m["scale"]),
                       window=mask.get("size", NO_WINDOW), keep_first=mask.get("keep_first", 0), kv_from=m.get("kv_from"), **features)


def _zurevik_mixer(kind: str, m: dict, where: str) -> LayerConfig:
    if kind == "attention":
        return _attention(m, maps=2, qk_norm=True, gate="element", diff=float(m["diff"]))
    if kind == "attention_2":
        return _attention(m, qkv_bias=True, sink=True, gate="head")
    raise ValueError(f"{where}: unknown mixer {kind!r}")


def _virolorn_mixer(kind: str, m: dict, where: str, shapes, x: str) -> LayerConfig:
    if kind not in ("lightning", "channel_delta", "latent_attention"):
        raise ValueError(f"{where}: unknown mixer {kind!r}")
    lc = LayerConfig(mixer=kind, heads=m["heads"], dim=m["dim"], vdim=m["vdim"])
    if kind == "lightning":
        lc.decay = tuple(float(v) for v in m["decay"])
        if len(lc.decay) != lc.heads:
            raise ValueError(f"{where}: {len(lc.decay)} decays for {lc.heads} heads")
    elif kind == "channel_delta":
        lc.kv_heads, lc.conv = m["kv_heads"], m["conv"]
        lc.decay_rank, lc.gate_rank = shapes[x + "a1"][0], shapes[x + "g1"][0]
    else:
        lc.q_rank, lc.kv_rank, lc.rot_dim, lc.scale = m["q_rank"], m["kv_rank"], m["rot_dim"], float(m["scale"])
        lc.rot_dims, lc.rot_base = m["rot"]["dims"], float(m["rot"]["base"])
    return lc


def _feed_forward(lc: LayerConfig, mlp: Optional[dict], where: str) -> None:
    if mlp is None:
        return
    if mlp["kind"] == "dense":
        lc.ff = mlp["ff"]
    elif mlp["kind"] == "moe":
        lc.ff, lc.experts, lc.top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
    else:
        raise ValueError(f"{where}: unknown feed-forward {mlp['kind']!r}")


@dataclass
class DecoderConfig:
    vocab_size: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    layers: List[LayerConfig] = field(default_factory=list)
    index_base: int = 0
    sequence_len: Optional[int] = None      # no limit of its own: the cache's length is the limit
    block: str = "sandwich"                 # how mixer and feed-forward of a layer are arranged
    untied: bool = False                    # the output head is a tensor of its own
    embed_scale: float = 1.0
    logit_softcap: float = 0.0              # 0 = none

    @classmethod
    def from_json(cls, d: dict, shapes: Dict[str, tuple]) -> "DecoderConfig":
        """From a parsed config.json; `shapes` (name -> shape of the weights) gives the sizes that exist only there."""
        zurevik = d.get("architecture") == "Zurevik"
        layers = []
        for i, e in enumerate(d["layers"]):
            own = i
            for _ in d["layers"]:
                if d["layers"][own].get("weights_of") is None:
                    break
                own = d["layers"][own]["weights_of"]
            where = f"layer {i}"
            lc = _zurevik_mixer(e["type"], e["mixer"], where) if zurevik else _virolorn_mixer(e["type"], e["mixer"], where, shapes, f"l{own}.mix.")
            lc.weights_of = e.get("weights_of")
            _feed_forward(lc, e.get("mlp"), where)
            layers.append(lc)
        out = cls(vocab_size=d["vocab"], width=d["width"], norm_eps=float(d["norm"]["eps"]), layers=layers)
        if zurevik:
            out.block, out.untied = "parallel", True
            out.embed_scale, out.logit_softcap = float(d["embedding"]["scale"]), float(d.get("logit_softcap") or 0.0)
        else:
            out.residual_mult = float(d["residual_mult"])
        return out

    def c_struct(self, *, compute_dtype="float32", max_batch=1, max_rows=1) -> _lib.DecoderConfigC:
        arr = (_lib.LayerConfigC * len(self.layers))()
        keep = []
        for a, l in zip(arr, self.layers):
            a.mixer, a.weights_of = MIXERS[l.mixer], -1 if l.weights_of is None else l.weights_of
            for n in ("heads", "kv_heads", "dim", "vdim", "conv", "decay_rank", "gate_rank", "q_rank", "kv_rank", "rot_dim", "rot_dims",
                      "ff", "scale", "rot_base", "maps", "window", "keep_first", "qkv_bias", "qk_norm", "sink", "diff", "experts", "top"):
                setattr(a, n, getattr(l, n))
            a.kv_from, a.gate = -1 if l.kv_from is None else l.kv_from, GATES[l.gate]
            if l.decay:
                buf = (C.c_float * len(l.decay))(*l.decay)
                keep.append(buf)
                a.h_decay = C.cast(buf, C.POINTER(C.c_float))
        c = _lib.DecoderConfigC()
        c.vocab, c.width, c.n_layer = self.vocab_size, self.width, len(self.layers)
        c.compute_dtype = _lib.BF16 if str(compute_dtype).endswith("bfloat16") or compute_dtype == "bf16" else _lib.F32
        c.index_base, c.max_batch, c.max_rows = self.index_base, max_batch, max_rows
        c.norm_eps, c.residual_mult = self.norm_eps, self.residual_mult
        c.block, c.untied, c.embed_scale, c.logit_softcap = BLOCKS[self.block], self.untied, self.embed_scale, self.logit_softcap
        c.h_layers = C.cast(arr, C.POINTER(_lib.LayerConfigC))
        c._keep = (arr, keep)
        return c


def decoder_layout(config: DecoderConfig) -> Dict[str, ParamSpec]:
    """name -> offset and (out, in) shape of every tensor in the flat fp32 parameter vector (femto_decoder_layout)."""
    L, c = _lib.lib(), config.c_struct()
    n = L.femto_decoder_layout(c, None, 0)
    if n < 0:
        _lib.check(n)
    arr = (_lib.DecoderTensorC * n)()
    L.femto_decoder_layout(c, arr, n)
    return {t.name.decode(): ParamSpec(int(t.offset), (int(t.rows), int(t.cols)) if t.cols else (int(t.rows),)) for t in arr}


class DecoderState(Handle):
    """The library handle of a decoder: packed weights and the workspace of one pass of up to `max_rows` tokens."""

    def __init__(self, config: DecoderConfig, max_batch: int, compute_type="float32", max_rows: int = 8192):
        super().__init__()
        self.config, self.max_batch, self.compute_type = config, max_batch, compute_type
        self.c = config.c_struct(compute_dtype=compute_type, max_batch=max_batch, max_rows=max(max_rows, max_batch))
        h = C.c_void_p()
        _lib.check(_lib.lib().femto_decoder_create(C.byref(self.c), C.byref(h)))
        self.h = h
        self._packed = None

    def refresh_weights(self, theta) -> None:
        """Packs Θ into the compute type unless this very content is packed already."""
        now = (theta.data_ptr(), theta._version)
        if self._packed != now:
            super().refresh_weights(theta)
            self._packed = now


class Decoder:
    """The model: Θ (flat fp32 on the device), its configuration and layout.  Same face as GPT towards `prefill`,
    `decode_step`, `extend` and `generate`."""

    def __init__(self, params: Params, config: DecoderConfig, layout: Dict[str, ParamSpec] = None, compute_type="float32", **options):
        self.params, self.config = params, config
        self.layout = layout if layout is not None else decoder_layout(config)
        self.compute_type, self.options = compute_type, options
        self._state: Optional[DecoderState] = None

    @property
    def index_base(self) -> int:
        return self.config.index_base

    def state(self, B: int) -> DecoderState:
        if self._state is None or self._state.max_batch < B:
            self._state = DecoderState(self.config, max_batch=B, compute_type=self.compute_type, **self.options)
        return self._state

    @classmethod
    def from_weights(cls, config_json: dict, tensors, compute_type="float32", **options) -> "Decoder":
        """`tensors`: a SafeTensors file, or anything with `shapes` and item access by name."""
        import sys
        import torch
        config = DecoderConfig.from_json(config_json, tensors.shapes)
        layout = decoder_layout(config)
        missing = sorted(n for n in layout if n not in tensors.shapes)
        wrong = sorted(n for n in layout if n in tensors.shapes and tuple(tensors.shapes[n]) != layout[n].shape)
        if missing or wrong:
            raise ValueError("weights do not fit the configuration: missing %s; wrong shape %s" % (
                missing, [(n, tuple(tensors.shapes[n]), layout[n].shape) for n in wrong]))
        unused = sorted(n for n in tensors.shapes if n not in layout)
        if unused:
            print("weights that the configuration does not use: " + ", ".join(unused), file=sys.stderr)
        n = int(_lib.lib().femto_decoder_nparams(config.c_struct()))
        theta = torch.zeros(n, dtype=torch.float32, device="cuda")
        for name, spec in layout.items():
            theta[spec.offset:spec.offset + spec.size].copy_(tensors[name].reshape(-1))
        params = Params(theta, delta=False)
        return cls(params, config, layout, compute_type=compute_type, **options)
