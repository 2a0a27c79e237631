"""Plain restatement, on the CPU, of the decoders whose configuration lists their layers one by one (Virolorn, Zurevik).

One function per mechanism, written from its equations and token by token wherever the mechanism is a recurrence.  It is
slow on purpose and shares no code with the product: only `tests/` use it.  All arithmetic is in the dtype of the tensors
it is given (float64 in the tests).  Weights are [out, in] matrices applied as x W^T.

A model is a plain dict (the parsed config.json) and a dict of tensors by name; `Sequence` carries one sequence's caches
and states so that a prompt can be fed in portions."""
from __future__ import annotations

import math

import torch


# ---- elementary pieces ---------------------------------------------------------------------------------------------
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps), times the weight when there is one."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def causal_conv(x, taps, tail):
    """y[t, c] = sum_i taps[c, i] * x[t - (n - 1) + i, c]; `tail` holds the n - 1 inputs before x.  Returns (y, new tail)."""
    n = taps.shape[1]
    full = torch.cat([tail, x], 0)
    y = torch.zeros_like(x)
    for i in range(n):
        y = y + full[i:i + x.shape[0]] * taps[:, i]
    return y, full[full.shape[0] - (n - 1):].clone()


def rotate_half(x, positions, dims, base):
    """Rotates the first `dims` entries of the last axis: entry i with entry i + dims/2 by the angle p * base^(-2i/dims)."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = positions.to(x.dtype) * (base ** (-2.0 * i / dims))
        while a.dim() < x.dim() - 1:
            a = a[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ---- the recurrences -----------------------------------------------------------------------------------------------
def decayed_outer_recurrence(q, k, v, decay, state):
    """Per head: S <- decay S + k v^T, o = S^T q.  q, k [T, H, D], v [T, H, E], decay [H], state [H, D, E]."""
    S, out = state.clone(), []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gated_delta_recurrence(q, k, v, g, beta, state):
    """Per head: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.
    q, k, g [T, H, D], v [T, H, E], beta [T, H], state [H, D, E]."""
    S, out = state.clone(), []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def softmax_attention(q, k, v, scale, first):
    """q [T, H, D] at positions first .. first + T - 1 against k [N, H, D], v [N, H, E]; key j is seen when j <= position."""
    T, N = q.shape[0], k.shape[0]
    out = []
    for t in range(T):
        n = min(N, first + t + 1)
        s = (k[:n] * q[t]).sum(-1) * scale              # [n, H]
        p = torch.exp(s - s.max(0, keepdim=True).values)
        p = p / p.sum(0, keepdim=True)
        out.append((p[:, :, None] * v[:n]).sum(0))
    return torch.stack(out)


# ---- the mixers ----------------------------------------------------------------------------------------------------
def lightning(h, w, m, eps, state):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(T, H, D)
    k = silu(h @ w["k"].T).view(T, H, D)
    v = silu(h @ w["v"].T).view(T, H, E)
    if not state:
        state["S"] = torch.zeros(H, D, E, dtype=h.dtype)
    o, state["S"] = decayed_outer_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype), state["S"])
    o = rms_norm(o.reshape(T, H * E), w["norm"], eps) * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def channel_delta(h, w, m, eps, state):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if not state:
        for n in "qkv":
            state[n] = torch.zeros(m["conv"] - 1, w[n].shape[0], dtype=h.dtype)
        state["S"] = torch.zeros(H, D, E, dtype=h.dtype)
    x = {}
    for n in "qkv":
        y, state[n] = causal_conv(h @ w[n].T, w[n + ".conv"], state[n])
        x[n] = silu(y)
    group = torch.arange(H) // (H // G)                  # query/key head of every head
    q = (unit_vector(x["q"].view(T, G, D)) * D ** -0.5)[:, group]
    k = unit_vector(x["k"].view(T, G, D))[:, group]
    v = x["v"].view(T, H, E)
    beta = torch.sigmoid(h @ w["b"].T)
    step = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
    o, state["S"] = gated_delta_recurrence(q, k, v, g, beta, state["S"])
    gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T).view(T, H, E)
    o = rms_norm(o, w["norm"], eps) * gate
    return o.reshape(T, H * E) @ w["o"].T


def latent_attention(h, w, m, eps, state):
    T, H, D, R, E, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    first = state.get("n", 0)
    pos = torch.arange(first, first + T)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate_half(q[..., D:], pos, dims, base)], -1)
    ckv = h @ w["dkv"].T
    c = rms_norm(ckv[:, :L], w["dkv.norm"], eps)
    r = rotate_half(ckv[:, L:], pos, dims, base)
    c = torch.cat([state["c"], c]) if first else c
    r = torch.cat([state["r"], r]) if first else r
    state["c"], state["r"], state["n"] = c, r, first + T
    N = c.shape[0]
    k = torch.cat([(c @ w["uk"].T).view(N, H, D), r[:, None, :].expand(N, H, R)], -1)
    v = (c @ w["uv"].T).view(N, H, E)
    o = softmax_attention(q, k, v, m["scale"], first)
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * E) @ w["o"].T


def sees(i, j, size, keep_first=0):
    """A sliding window of `size` tokens, itself included, and the first `keep_first` tokens of the sequence."""
    return j <= i and (i - j < size or j < keep_first)


def windowed_attention(q, k, v, scale, first, size, keep_first=0, sink=None):
    """q [T, H, D] at positions first .., k [N, G, D], v [N, G, E]; query head h reads key/value head h // (H / G).  `sink` [H]:
    one more term exp(sink) in the denominator."""
    T, H, per = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        see = torch.tensor([j for j in range(k.shape[0]) if sees(first + t, j, size, keep_first)])
        for h in range(H):
            s = (k[see, h // per] @ q[t, h]) * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            total = e.sum() if sink is None else e.sum() + torch.exp(sink[h] - top)
            out[t, h] = (e / total) @ v[see, h // per]
    return out


def differential_lambda(w, diff):
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def append_kv(state, k, v):
    """Adds rows to a layer's cached keys and values; returns (position of the first new row, all keys, all values)."""
    first = state["k"].shape[0] if "k" in state else 0
    state["k"] = torch.cat([state["k"], k]) if first else k
    state["v"] = torch.cat([state["v"], v]) if first else v
    return first


def differential_attention(h, w, m, eps, state):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w["q"].T).view(T, H, 2, D), w["q.norm"], eps)
    k = rms_norm((h @ w["k"].T).view(T, G, 2, D), w["k.norm"], eps)
    first = append_kv(state, k, (h @ w["v"].T).view(T, G, E))
    a = [windowed_attention(q[:, :, i], state["k"][:, :, i], state["v"], m["scale"], first, m["mask"]["size"], m["mask"]["keep_first"])
         for i in range(2)]
    o = a[0] - differential_lambda(w, m["diff"]) * a[1]
    o = rms_norm(o, None, eps) * (1.0 - m["diff"])
    return (o.reshape(T, H * E) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def sink_attention(h, w, m, eps, state, shared=None):
    """`shared`: the state of the layer whose keys and values this one reads (that layer has added its rows already)."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, D)
    if shared is None:
        append_kv(state, (h @ w["k"].T + w["k.b"]).view(T, G, D), (h @ w["v"].T + w["v.b"]).view(T, G, E))
        shared = state
    o = windowed_attention(q, shared["k"], shared["v"], m["scale"], shared["k"].shape[0] - T, m["mask"]["size"], sink=w["sink"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * E) @ w["o"].T


def gated_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z, top):
    """The `top` largest logits of every row: (expert indices, softmax over the chosen ones)."""
    best = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    s = torch.gather(z, 1, best)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return best, e / e.sum(-1, keepdim=True)


def expert_mlp(h, up, down):
    return torch.clamp(h @ up.T, min=0) ** 2 @ down.T


def mixture_mlp(h, w, top, margins=None):
    """`margins` collects, per row, the gap between the last logit that was chosen and the first that was not."""
    z = h @ w["router"].T + w["router.b"]
    best, weight = route(z, top)
    if margins is not None and top < z.shape[1]:
        s = torch.sort(z, dim=-1, descending=True).values
        margins.append(s[:, top - 1] - s[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(best[t].tolist(), weight[t]):
            out[t] = out[t] + p * expert_mlp(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    return out


MIXERS = dict(lightning=lightning, channel_delta=channel_delta, latent_attention=latent_attention, attention=differential_attention,
              attention_2=sink_attention)


# ---- the model -----------------------------------------------------------------------------------------------------
def _sub(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def feed_forward(h, w, mlp, margins=None):
    return gated_mlp(h, w) if mlp["kind"] == "dense" else mixture_mlp(h, w, mlp["router"]["top"], margins)


def sandwich_layer(x, w, layer, eps, mult, mix, margins=None):
    """A norm before and after each sublayer, one after the other."""
    x = x + mult * rms_norm(mix(rms_norm(x, w["norm1"], eps)), w["norm1b"], eps)
    if layer["mlp"] is not None:
        x = x + mult * rms_norm(feed_forward(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."), layer["mlp"], margins), w["norm2b"], eps)
    return x


def parallel_layer(x, w, layer, eps, mix, margins=None):
    """Mixer and feed-forward side by side, each behind a norm of its own."""
    y = mix(rms_norm(x, w["norm1"], eps))
    if layer["mlp"] is not None:
        y = y + feed_forward(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."), layer["mlp"], margins)
    return x + y


class Sequence:
    """One sequence: `feed(tokens)` returns the logits [T, vocab] of these tokens and keeps the state."""

    def __init__(self, config, weights, dtype=torch.float64):
        self.cfg = config
        self.w = {n: t.to(dtype) for n, t in weights.items()}
        self.state = [dict() for _ in config["layers"]]
        self.residuals = []           # the residual stream after every layer of the last call
        self.margins = []             # of the last call's routers

    def feed(self, tokens):
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = self.w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg.get("embedding", {}).get("scale", 1.0)
        self.residuals, self.margins = [], []
        for i, layer in enumerate(cfg["layers"]):
            own = i
            while cfg["layers"][own].get("weights_of") is not None:
                own = cfg["layers"][own]["weights_of"]
            w, m = _sub(self.w, f"l{own}."), layer["mixer"]
            shared = {} if m.get("kv_from") is None else dict(shared=self.state[m["kv_from"]])
            mix = lambda h: MIXERS[layer["type"]](h, _sub(w, "mix."), m, eps, self.state[i], **shared)
            if cfg["architecture"] == "Zurevik":
                x = parallel_layer(x, w, layer, eps, mix, self.margins)
            else:
                x = sandwich_layer(x, w, layer, eps, cfg["residual_mult"], mix, self.margins)
            self.residuals.append(x)
        z = rms_norm(x, self.w["final.norm"], eps) @ self.w["head" if "head" in self.w else "embed"].T
        cap = cfg.get("logit_softcap")
        return z if cap is None else cap * torch.tanh(z / cap)


# ---- small random models for the tests -------------------------------------------------------------------------------
def tensor_shapes(cfg, decay_rank=8, gate_rank=8):
    """name -> shape of every tensor of a model; the two low-rank projections' ranks exist only as shapes."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    if cfg["architecture"] == "Zurevik":
        out["head"] = out["embed"]
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = (d,)
        if cfg["architecture"] == "Virolorn":
            out[p + "norm1b"] = (d,)
        if layer["type"] == "lightning":
            H, D, E = m["heads"], m["dim"], m["vdim"]
            out.update({x + "q": (H * D, d), x + "k": (H * D, d), x + "v": (H * E, d), x + "g": (H * E, d),
                        x + "o": (d, H * E), x + "norm": (H * E,)})
        elif layer["type"] == "channel_delta":
            H, G, D, E, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            out.update({x + "q": (G * D, d), x + "q.conv": (G * D, n), x + "k": (G * D, d), x + "k.conv": (G * D, n),
                        x + "v": (H * E, d), x + "v.conv": (H * E, n), x + "b": (H, d), x + "A_log": (H,), x + "norm": (E,),
                        x + "a1": (decay_rank, d), x + "a2": (H * D, decay_rank), x + "dt_bias": (H * D,),
                        x + "g1": (gate_rank, d), x + "g2": (H * E, gate_rank), x + "o": (d, H * E)})
        elif layer["type"] == "attention":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({x + "q": (H * 2 * D, d), x + "k": (G * 2 * D, d), x + "v": (G * E, d), x + "q.norm": (D,), x + "k.norm": (D,),
                        x + "g": (H * E, d), x + "o": (d, H * E)})
            out.update({x + n: (D,) for n in ("lq1", "lk1", "lq2", "lk2")})
        elif layer["type"] == "attention_2":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({x + "q": (H * D, d), x + "q.b": (H * D,), x + "sink": (H,), x + "g": (H, d), x + "o": (d, H * E)})
            if m.get("kv_from") is None:
                out.update({x + "k": (G * D, d), x + "k.b": (G * D,), x + "v": (G * E, d), x + "v.b": (G * E,)})
        else:
            H, D, R, E, L, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            out.update({x + "dq": (Q, d), x + "dq.norm": (Q,), x + "uq": (H * (D + R), Q), x + "dkv": (L + R, d),
                        x + "dkv.norm": (L,), x + "uk": (H * D, L), x + "uv": (H * E, L), x + "g": (H, d), x + "o": (d, H * E)})
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            f, n = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"]
            out.update({p + "norm2": (d,), p + "mlp.router": (n, d), p + "mlp.router.b": (n,)})
            if cfg["architecture"] == "Virolorn":
                out[p + "norm2b"] = (d,)
            for e in range(n):
                out.update({p + f"mlp.e{e}.up": (f, d), p + f"mlp.e{e}.down": (d, f)})
        elif layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out[p + "norm2"] = (d,)
            if cfg["architecture"] == "Virolorn":
                out[p + "norm2b"] = (d,)
            out.update({p + "mlp.gate": (f, d), p + "mlp.up": (f, d), p + "mlp.down": (d, f)})
    return out


def random_weights(cfg, seed=0, decay_rank=8, gate_rank=8):
    """bfloat16 weights, so that every build of the product reads the same numbers."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, decay_rank, gate_rank).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(*shape, generator=g, dtype=torch.float64)
        if leaf == "norm" or leaf.startswith("norm"):
            t = 1.0 + 0.2 * r
        elif leaf == "A_log":
            t = 0.5 * r
        elif leaf == "dt_bias":
            t = r - 2.0
        elif leaf in ("sink", "b") and len(shape) == 1:
            t = r
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.6 * r / math.sqrt(shape[0]) ** 0.5
        elif leaf == "conv":
            t = r / math.sqrt(shape[1])
        elif name == "embed":
            t = r
        else:
            t = r * 1.5 / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16)
    return out
