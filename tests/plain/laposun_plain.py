"""A plain, slow implementation of the Laposun decoder in float64: one function a mechanism, the convolution and the
streams as loops, attention as a loop over queries.  It shares no code with the package: it reads a configuration as the
plain dictionary of config.json and the weights as a dictionary name -> tensor.

Notation: x_s is a token's vector in stream s, h what a sublayer reads, W_a the tensor '<layer>.mix.a' (or '.mlp.a'),
stored [out, in] and applied as W h."""
from __future__ import annotations

import json
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


def bigram_rows(tokens, before, bigram):
    """The row of the second table for every token: (token in front * mul_prev + token * mul_cur) mod buckets, and row
    number ``buckets`` for a token with none in front of it.  ``before``: the token in front of tokens[0], or None."""
    rows = []
    for t in tokens:
        rows.append(bigram["buckets"] if before is None else (before * bigram["mul_prev"] + t * bigram["mul_cur"]) % bigram["buckets"])
        before = t
    return rows


def embed(tokens, before, table, second, bigram, w, eps):
    rows = torch.as_tensor(bigram_rows(tokens, before, bigram), dtype=torch.long)
    return rms_norm(table[torch.as_tensor(tokens, dtype=torch.long)] + second[rows], w, eps)


def short_convolution(h, kept, w):
    """h [T, W] with the ``taps`` - 1 rows ``kept`` in front of it (zeros at a sequence's start), w [W, taps], the last
    tap the present row's: returns h_t + sum_j w[:, j] h_(t - taps + 1 + j) and the rows to keep."""
    taps = w.shape[1]
    rows = torch.cat([kept, h], dim=0)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        out[t] = h[t]
        for j in range(taps):
            out[t] = out[t] + w[:, j] * rows[t + j]
    return out, rows[rows.shape[0] - (taps - 1):].clone()


def read_streams(x, w_in):
    """x [streams, T, W]: sum_s w_in[s] x_s."""
    u = torch.zeros_like(x[0])
    for s in range(x.shape[0]):
        u = u + w_in[s] * x[s]
    return u


def write_streams(x, mix, w_out, y):
    """The new streams, all from the old ones: x_t <- sum_s mix[s, t] x_s + w_out[t] y."""
    new = torch.zeros_like(x)
    for t in range(x.shape[0]):
        new[t] = w_out[t] * y
        for s in range(x.shape[0]):
            new[t] = new[t] + mix[s, t] * x[s]
    return new


def rotate_interleaved(v, positions, dims, base):
    """v [T, ..., n]: the first ``dims`` dimensions in pairs (2i, 2i + 1), pair i of the token at position p turned by the
    angle p base^(-2i/dims); the other dimensions pass."""
    if not dims:
        return v.clone()
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    ang = positions.to(F)[:, None] * freq[None, :]
    shape = [v.shape[0]] + [1] * (v.dim() - 2) + [dims // 2]
    cos, sin = torch.cos(ang).reshape(shape), torch.sin(ang).reshape(shape)
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out = v.clone()
    out[..., 0:dims:2] = a * cos - b * sin
    out[..., 1:dims:2] = b * cos + a * sin
    return out


def window_attention(q, k, v, q_positions, scale, window):
    """q [T, H, d], k [S, H, d], v [S, H, e], key j at position j: the query at position p sees the keys j <= p with
    p - j < window.  Softmax over the seen keys."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=F)
    for t in range(q.shape[0]):
        p = int(q_positions[t])
        lo = max(0, p - window + 1)
        s = torch.einsum("hd,jhd->hj", q[t], k[lo:p + 1]) * scale
        out[t] = torch.einsum("hj,jhe->he", torch.softmax(s, dim=1), v[lo:p + 1])
    return out


class LatentCache:
    """What an attention layer keeps of a sequence: the normed latent and the rotated shared key part of every token."""

    def __init__(self):
        self.c = None
        self.kr = None

    def extend(self, c, kr):
        self.c = c if self.c is None else torch.cat([self.c, c])
        self.kr = kr if self.kr is None else torch.cat([self.kr, kr])


def latent_attention(h, positions, w, m, eps, cache):
    H, d, r, e, kv = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    turn = lambda v: rotate_interleaved(v, positions, m["rot"]["dims"], m["rot"]["base"])
    cq = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (cq @ w["uq"].T).reshape(-1, H, d + r)
    down = h @ w["dkv"].T
    cache.extend(rms_norm(down[:, :kv], w["dkv.norm"], eps), turn(down[:, kv:]))
    k_plain = (cache.c @ w["uk"].T).reshape(-1, H, d)
    values = (cache.c @ w["uv"].T).reshape(-1, H, e)
    keys = torch.cat([k_plain, cache.kr[:, None, :].expand(-1, H, -1)], dim=-1)
    queries = torch.cat([q[..., :d], turn(q[..., d:])], dim=-1)
    o = window_attention(queries, keys, values, positions, m["scale"], m["mask"]["size"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(-1, H * e) @ w["o"].T


def dense_ff(h, w):
    z = h @ w["gate"].T
    return (z * torch.sigmoid(z) * (h @ w["up"].T)) @ w["down"].T


def expert(h, up, down):
    z = torch.clamp(h @ up.T, min=0.0)
    return (z * z) @ down.T


def route(h, router, top, scale, margins=None):
    """(ids [T, top], weights [T, top]): the experts with the largest softmax scores (over all experts), the chosen scores
    over their sum, scaled.  ``margins`` gets, for every token, how far the last chosen logit lies above the first that is
    not, as a part of the largest logit's size."""
    z = h @ router.T
    s = torch.softmax(z, dim=1)
    if margins is not None and top < z.shape[1]:
        ranked = torch.sort(z, dim=1, descending=True).values
        margins.append((ranked[:, top - 1] - ranked[:, top]) / z.abs().max(dim=1).values.clamp_min(1e-9))
    chosen = torch.topk(s, top, dim=-1)
    return chosen.indices, chosen.values / (chosen.values.sum(dim=-1, keepdim=True) + 1e-20) * scale


def moe_ff(h, w, f, margins=None):
    ids, weights = route(h, w["router"], f["router"]["top"], f["router"]["scale"], margins)
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=F)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), weights[t]):
            out[t] += wt * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if f.get("shared") is not None:
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * expert(h, w["shared.up"], w["shared.down"])
    return out


def sub(weights, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in weights.items() if k.startswith(prefix)}


class Sequence:
    """What every layer keeps of one sequence, its last token and how many it has seen."""

    def __init__(self, config):
        self.length, self.before = 0, None
        rows = lambda: torch.zeros(config["canon"]["taps"] - 1, config["width"], dtype=F)
        self.layers = [{"mix": LatentCache(), "conv1": rows(), "conv2": rows()} for _ in config["layers"]]


def forward(config, weights, tokens, seq=None, trace=None, margins=None):
    """Runs ``tokens`` after what ``seq`` has seen; returns logits [T, vocab].  ``trace``: a list that takes the sum of the
    streams after every layer.  ``margins``: a list that takes every router's margins (see ``route``)."""
    seq = seq if seq is not None else Sequence(config)
    eps = config["norm"]["eps"]
    g = lambda name: weights[name].to(F)
    positions = torch.arange(seq.length, seq.length + len(tokens))
    first = embed(tokens, seq.before, g("embed"), g("bigram"), config["embedding"]["bigram"], g("embed.norm"), eps)
    x = torch.stack([first] * config["streams"])

    def sublayer(p, q, kept, fn):
        nonlocal x
        u = read_streams(x, g(f"{p}hc{q}.in"))
        h, kept[f"conv{q}"] = short_convolution(rms_norm(u, g(f"{p}norm{q}"), eps), kept[f"conv{q}"], g(f"{p}canon{q}"))
        x = write_streams(x, g(f"{p}hc{q}.mix"), g(f"{p}hc{q}.out"), fn(h))

    for i, layer in enumerate(config["layers"]):
        p, kept, f = f"l{i}.", seq.layers[i], layer.get("mlp")
        w = sub(weights, p + "mix.")
        sublayer(p, 1, kept, lambda h: latent_attention(h, positions, w, layer["mixer"], eps, kept["mix"]))
        if f is not None:
            wf = sub(weights, p + "mlp.")
            sublayer(p, 2, kept, lambda h: dense_ff(h, wf) if f["kind"] == "dense" else moe_ff(h, wf, f, margins))
        if trace is not None:
            trace.append(x.sum(dim=0))
    seq.length += len(tokens)
    if len(tokens):
        seq.before = tokens[-1]
    return rms_norm(x.sum(dim=0), g("final.norm"), eps) @ g("embed").T
