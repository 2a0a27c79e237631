"""Plain restatement, on the CPU, of the decoders whose configuration lists their layers one by one (Virolorn).

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


def gated_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = dict(lightning=lightning, channel_delta=channel_delta, latent_attention=latent_attention)


# ---- the model -----------------------------------------------------------------------------------------------------
def _sub(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


class Sequence:
    """One sequence: `feed(tokens)` returns the logits [T, vocab] of these tokens and keeps the state."""

    def __init__(self, config, weights, dtype=torch.float64):
        self.cfg = config
        self.w = {n: t.to(dtype) for n, t in weights.items()}
        self.state = [dict() for _ in config["layers"]]
        self.residuals = []           # the residual stream after every layer of the last call

    def feed(self, tokens):
        cfg, eps, m = self.cfg, self.cfg["norm"]["eps"], self.cfg["residual_mult"]
        x = self.w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
        self.residuals = []
        for i, layer in enumerate(cfg["layers"]):
            own = i
            while cfg["layers"][own].get("weights_of") is not None:
                own = cfg["layers"][own]["weights_of"]
            w = _sub(self.w, f"l{own}.")
            y = MIXERS[layer["type"]](rms_norm(x, w["norm1"], eps), _sub(w, "mix."), layer["mixer"], eps, self.state[i])
            x = x + m * rms_norm(y, w["norm1b"], eps)
            if layer["mlp"] is not None:
                y = gated_mlp(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."))
                x = x + m * rms_norm(y, w["norm2b"], eps)
            self.residuals.append(x)
        return rms_norm(x, self.w["final.norm"], eps) @ self.w["embed"].T


# ---- small random models for the tests -------------------------------------------------------------------------------
def tensor_shapes(cfg, decay_rank=8, gate_rank=8):
    """name -> shape of every tensor of a model; the two low-rank projections' ranks exist only as shapes."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = out[p + "norm1b"] = (d,)
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
        else:
            H, D, R, E, L, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            out.update({x + "dq": (Q, d), x + "dq.norm": (Q,), x + "uq": (H * (D + R), Q), x + "dkv": (L + R, d),
                        x + "dkv.norm": (L,), x + "uk": (H * D, L), x + "uv": (H * E, L), x + "g": (H, d), x + "o": (d, H * E)})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (d,)
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
        elif leaf == "conv":
            t = r / math.sqrt(shape[1])
        elif name == "embed":
            t = r
        else:
            t = r * 1.5 / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16)
    return out
