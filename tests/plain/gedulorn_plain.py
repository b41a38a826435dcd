"""A plain, slow implementation of the Gedulorn decoder in float64: one function a mechanism, attention and the recurrence
as loops over tokens.  It shares no code with the package: it reads a configuration as the plain dictionary of config.json
and the weights as a dictionary name -> tensor.

Notation: x is the residual, h what a mixer or feed-forward reads (x itself), W_a the tensor '<layer>.mix.a' (or '.mlp.a'),
stored [out, in] and applied as W h."""
from __future__ import annotations

import json
import math
import os

import torch

F = torch.float64


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_weights(folder: str, dtype=F):
    from safetensors import safe_open
    out = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            out[name] = f.get_tensor(name).to(dtype)
    return out


def sample_greedy(logits):
    return int(torch.argmax(logits))


def rms_norm(v, w, eps):
    """w * v / sqrt(mean(v^2) + eps) over the last dimension."""
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1.0 + torch.exp(-z))


def turn_halves(v, positions, dims, base, factor=1.0):
    """v [T, ..., n]: dimensions i and i + dims/2 of the first ``dims`` form a pair, which the token at position p turns by
    the angle p base^(-2i/dims) / factor; the other dimensions pass."""
    if not dims:
        return v.clone()
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) / factor for i in range(half)], dtype=F)
    ang = positions.to(F)[:, None] * freq[None, :]
    shape = [v.shape[0]] + [1] * (v.dim() - 2) + [half]
    cos, sin = torch.cos(ang).reshape(shape), torch.sin(ang).reshape(shape)
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, v[..., dims:]], dim=-1)


def first_seen(p, window):
    """The first position that the token at position p sees: its window holds itself and the window - 1 tokens before it."""
    return 0 if window is None else max(0, p - window + 1)


def windowed_attention(q, k, v, q_positions, scale, window, softcap=None, sinks=None):
    """q [T, H, d], k [S, G, d], v [S, G, e] (key j at position j; query head h reads key/value head h // (H / G)).  A score
    is scaled, then capped as c tanh(score / c); a sink adds exp(sink_h) to head h's denominator."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[2], dtype=F)
    for t in range(q.shape[0]):
        p = int(q_positions[t])
        lo = first_seen(p, window)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:p + 1, g] @ q[t, h]) * scale
            if softcap is not None:
                s = softcap * torch.tanh(s / softcap)
            if sinks is None:
                w = torch.softmax(s, dim=0)
            else:
                w = torch.softmax(torch.cat([s, sinks[h:h + 1]]), dim=0)[:-1]
            out[t, h] = w @ v[lo:p + 1, g]
    return out


class Kept:
    """Rows that a layer keeps of a sequence, one a token: ``a`` (keys, or latents) and ``b`` (values, or rotated parts)."""

    def __init__(self):
        self.a = self.b = None

    def extend(self, a, b):
        self.a = a if self.a is None else torch.cat([self.a, a])
        self.b = b if self.b is None else torch.cat([self.b, b])


def _window(m):
    return m["mask"]["size"] if m.get("mask") is not None else None


def attention(h, positions, w, m, eps, kept):
    """Queries and keys are normed head by head and turned; a value is its key's projection before either."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    factor = rot["scaling"]["factor"] if rot.get("scaling") is not None else 1.0
    turn = lambda v: turn_halves(v, positions, rot["dims"], rot["base"], factor)
    q = (h @ w["q"].T).reshape(-1, H, d)
    k = (h @ w["k"].T).reshape(-1, G, d)
    kept.extend(turn(rms_norm(k, w["k.norm"], eps)), k)
    o = windowed_attention(turn(rms_norm(q, w["q.norm"], eps)), kept.a, kept.b, positions, m["scale"], _window(m), softcap=m.get("softcap"))
    return o.reshape(-1, H * d) @ w["o"].T


def latent_attention(h, positions, w, m, eps, kept):
    """``kept``: the layer's own latents and shared rotated key parts, or, for a layer with 'kv_from', those of that layer
    (which hold this step's tokens already)."""
    H, d, r, e, kv = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    turn = lambda v: turn_halves(v, positions, m["rot"]["dims"], m["rot"]["base"])
    cq = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (cq @ w["uq"].T).reshape(-1, H, d + r)
    if m.get("kv_from") is None:
        down = h @ w["dkv"].T
        kept.extend(rms_norm(down[:, :kv], w["dkv.norm"], eps), turn(down[:, kv:]))
    keys = torch.cat([(kept.a @ w["uk"].T).reshape(-1, H, d), kept.b[:, None, :].expand(-1, H, -1)], dim=-1)
    values = (kept.a @ w["uv"].T).reshape(-1, H, e)
    queries = torch.cat([q[..., :d], turn(q[..., d:])], dim=-1)
    o = windowed_attention(queries, keys, values, positions, m["scale"], _window(m), sinks=w["sink"])
    return o.reshape(-1, H * e) @ w["o"].T


def causal_convolution(u, before, w, b):
    """u [T, C] with the taps - 1 rows ``before`` in front of it (zeros at a sequence's start), w [C, taps] (the last tap the
    present row's), b [C]: silu(b + sum_j w[:, j] u_(t - taps + 1 + j)), and the rows to keep."""
    taps = w.shape[1]
    rows = torch.cat([before, u], dim=0)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        out[t] = b
        for j in range(taps):
            out[t] = out[t] + w[:, j] * rows[t + j]
    return silu(out), rows[rows.shape[0] - (taps - 1):].clone()


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def state_space(x, B, C, dt, A_log, D, S, groups):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (positive), S [H, N, P] (the state before):
    S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t, head h with group h // (H / G)."""
    T, H, P = x.shape
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // groups)
            S[h] = math.exp(-math.exp(float(A_log[h])) * float(dt[t, h])) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """y silu(z), cut into ``groups`` equal parts, each divided by its own root mean square, times w."""
    v = (y * silu(z)).reshape(y.shape[0], groups, -1)
    return (v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)).reshape(y.shape) * w


class Recurrent:
    """What a state-space layer keeps of a sequence: the state of every head and the convolution's last inputs."""

    def __init__(self, m, channels):
        self.S = torch.zeros(m["heads"], m["state"], m["vdim"], dtype=F)
        self.rows = torch.zeros(m["conv"] - 1, channels, dtype=F)


def mamba2(h, w, m, eps, kept):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    y = h @ w["in"].T
    z, u, dt = y[:, :inner], y[:, inner:2 * inner + 2 * G * N], y[:, 2 * inner + 2 * G * N:]
    u, kept.rows = causal_convolution(u, kept.rows, w["conv"], w["conv.b"])
    x, B, C = u[:, :inner].reshape(-1, H, P), u[:, inner:inner + G * N].reshape(-1, G, N), u[:, inner + G * N:].reshape(-1, G, N)
    o, kept.S = state_space(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"], kept.S, G)
    return gated_group_norm(o.reshape(-1, inner), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, bias, top, margins=None):
    """(ids [T, top], weights [T, top]): the experts with the largest logits W h + bias, weighted by the softmax over the
    chosen logits.  ``margins`` gets, for every token, how far the last chosen logit lies above the first that is not, as a
    part of the largest logit's size."""
    z = h @ router.T + bias
    if margins is not None and top < z.shape[1]:
        ranked = torch.sort(z, dim=1, descending=True).values
        margins.append((ranked[:, top - 1] - ranked[:, top]) / z.abs().max(dim=1).values.clamp_min(1e-9))
    chosen = torch.topk(z, top, dim=-1)
    return chosen.indices, torch.softmax(chosen.values, dim=-1)


def moe_ff(h, w, f, margins=None):
    ids, weights = route(h, w["router"], w["router.b"], f["router"]["top"], margins)
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=F)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), weights[t]):
            out[t] += wt * expert(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if f.get("shared") is not None:
        out = out + expert(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


def sub(weights, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in weights.items() if k.startswith(prefix)}


class Sequence:
    """What every layer keeps of one sequence, and how many tokens it has seen."""

    def __init__(self, config):
        self.length = 0
        self.layers = []
        for layer in config["layers"]:
            m = layer["mixer"]
            if layer["type"] == "mamba2":
                self.layers.append(Recurrent(m, m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]))
            else:
                self.layers.append(self.layers[m["kv_from"]] if m.get("kv_from") is not None else Kept())


def forward(config, weights, tokens, seq=None, trace=None, margins=None):
    """Runs ``tokens`` after what ``seq`` has seen; returns logits [T, vocab].  ``trace``: a list that takes the residual
    after every layer.  ``margins``: a list that takes every router's margins (see ``route``)."""
    seq = seq if seq is not None else Sequence(config)
    eps = config["norm"]["eps"]
    g = lambda name: weights[name].to(F)
    positions = torch.arange(seq.length, seq.length + len(tokens))
    x = g("embed")[torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p, kept, m, f = f"l{i}.", seq.layers[i], layer["mixer"], layer.get("mlp")
        w = sub(weights, p + "mix.")
        if layer["type"] == "mamba2":
            y = mamba2(x, w, m, eps, kept)
        else:
            y = (attention if layer["type"] == "attention" else latent_attention)(x, positions, w, m, eps, kept)
        x = x + rms_norm(y, g(p + "norm1"), eps)
        if f is not None:
            x = x + rms_norm(moe_ff(x, sub(weights, p + "mlp."), f, margins), g(p + "norm2"), eps)
        if trace is not None:
            trace.append(x.clone())
    seq.length += len(tokens)
    return rms_norm(x, g("final.norm"), eps) @ g("head").T
