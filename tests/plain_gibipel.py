"""A plain, slow Gibipel: whole sequences, no cache, one function per mechanism.

The yardstick for the engine's Gibipel parts.  It shares no code with the package: config.json
is read with ``json``, the weights with the ``safetensors`` library, and everything is
elementary torch arithmetic on the CPU in float64 (or float32).

Notation: ``x`` [S, D] is the residual stream of one sequence of S tokens at positions
0 .. S-1; a linear map is stored [out, in] and applied as ``x @ W.T``;
``unit(x) = x / sqrt(mean(x**2) + eps)`` over the last axis.

* input: ``x = c * embed[id]``;
* block: ``x += n1 * unit(mixer(x))``, then (where the layer has one) ``x += n2 * unit(ff(x))``
  with one number ``n`` a norm;
* the mixer: two side by side on the same input, ``a * left + b * right``.  Left: grouped-query
  attention with biases, a norm over the whole query and key projections, a rotation with
  stretched wavelengths, a window whose far past is seen as means of blocks, a learned per-head
  term in the softmax's denominator.  Right: a matrix memory with exponential gates and a
  running maximum;
* the feed-forward: routed experts, some of which hand their input back, chosen in two stages
  with a correction that only the choice sees, and an expert that every token uses;
* logits: ``c2 * (n * unit(x)) @ head.T``.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List

import torch


def read_model_folder(model_dir: str):
    from safetensors import safe_open
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    weights = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name).to(torch.float64)
    return cfg, weights


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def frequencies(base: float, dims: int, scaling=None) -> torch.Tensor:
    """The angle per position of pair i.  ``scaling``: wavelengths above original/low are
    stretched by ``factor``, those below original/high are kept, in between the two frequencies
    are blended."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims)
    if scaling:
        out = []
        for v in f.tolist():
            wave = 2.0 * math.pi / v
            if wave < scaling["original"] / scaling["high"]:
                out.append(v)
            elif wave > scaling["original"] / scaling["low"]:
                out.append(v / scaling["factor"])
            else:
                s = (scaling["original"] / wave - scaling["low"]) \
                    / (scaling["high"] - scaling["low"])
                out.append((1.0 - s) * v / scaling["factor"] + s * v)
        f = torch.tensor(out, dtype=torch.float64)
    return f


def rotate_front(z, freq, dims: int, first_pos: int = 0):
    """z [S, heads, d]: the first ``dims`` channels of every head are rotated, channel i paired
    with channel i + dims/2; the rest pass."""
    S = z.shape[0]
    half = dims // 2
    ang = (torch.arange(S, dtype=torch.float64) + first_pos)[:, None] * freq[None, :]
    c = torch.cos(ang).to(z.dtype)[:, None, :]
    s = torch.sin(ang).to(z.dtype)[:, None, :]
    u, v = z[..., :half], z[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, z[..., dims:]], dim=-1)


def block_means(rows, P: int):
    """rows [S, ...] -> the means of the complete blocks of P rows [S // P, ...]."""
    n = rows.shape[0] // P
    return rows[:n * P].reshape(n, P, *rows.shape[1:]).mean(dim=1)


def window_and_blocks(S: int, size: int, P: int):
    """(tokens [S, S]: 0 <= i - j < size, blocks [S, S // P]: the block's last token lies
    ``size`` or more behind)."""
    i = torch.arange(S)[:, None]
    j = torch.arange(S)[None, :]
    b = torch.arange(S // P)[None, :]
    return (i - j >= 0) & (i - j < size), b * P + P - 1 <= i - size


def softmax_with_sink(s, visible, sink):
    """Rows of ``s`` over the visible columns, with exp(sink) as one more term of the
    denominator that has no value."""
    s = s.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(dim=-1, keepdim=True).values, sink.expand(s.shape[0], 1))
    e = torch.exp(s - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - m))


def pooled_attention(q, k, v, scale, size, P, sink):
    """q [S, H, d], k [S, G, d], v [S, G, e] -> [S, H, e]."""
    S, H, _ = q.shape
    G = k.shape[1]
    kk, vv = torch.cat([k, block_means(k, P)]), torch.cat([v, block_means(v, P)])
    visible = torch.cat(window_and_blocks(S, size, P), dim=1)
    out = torch.zeros(S, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_with_sink((q[:, h] @ kk[:, g].T) * scale, visible, sink[h]) @ vv[:, g]
    return out


def mixer_attention(h, W, p, m, eps):
    S = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(h @ W[p + "q"].T + W[p + "q.b"], eps) * W[p + "q.norm"]
    k = unit(h @ W[p + "k"].T + W[p + "k.b"], eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(S, G, e)
    freq = frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    q = rotate_front(q.reshape(S, H, d), freq, m["rot"]["dims"])
    k = rotate_front(k.reshape(S, G, d), freq, m["rot"]["dims"])
    o = pooled_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["pool"], W[p + "sink"])
    return o.reshape(S, H * e) @ W[p + "o"].T


def log_sigmoid(z):
    return -torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, max=0.0)


def memory(q, k, v, i, f):
    """q, k [S, H, d], v [S, H, e]; i, f [S, H] the logarithms of the input and the forget gate
    -> o [S, H, e].  Per head a matrix M [d, e], a vector n [d] and a running maximum m, all
    zero at the start."""
    S, H, d = q.shape
    e = v.shape[-1]
    o = torch.zeros(S, H, e, dtype=q.dtype)
    for h in range(H):
        M = torch.zeros(d, e, dtype=q.dtype)
        n = torch.zeros(d, dtype=q.dtype)
        m = torch.zeros((), dtype=q.dtype)
        for t in range(S):
            top = torch.maximum(f[t, h] + m, i[t, h])
            keep, add = torch.exp(f[t, h] + m - top), torch.exp(i[t, h] - top)
            M = keep * M + add * torch.outer(k[t, h], v[t, h])
            n = keep * n + add * k[t, h]
            m = top
            o[t, h] = M.T @ q[t, h] / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return o


def mixer_memory(h, W, p, m, eps):
    S = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W[p + "q"].T).reshape(S, H, d) * d ** -0.5
    k = (h @ W[p + "k"].T).reshape(S, H, d)
    v = (h @ W[p + "v"].T).reshape(S, H, e)
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = unit(memory(q, k, v, i, f), eps).reshape(S, H * e) * W[p + "norm"]
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def mixer_parallel(h, W, p, m, eps):
    return m["left_scale"] * mixer_attention(h, W, p + "left.", m["left"], eps) \
        + m["right_scale"] * mixer_memory(h, W, p + "right.", m["right"], eps)


def gated(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(s, correction, top: int, groups=None):
    """s [E] the scores of one token -> the chosen outputs, best first."""
    c = (s + correction).tolist()
    E = len(c)
    if groups:
        per = E // groups["count"]
        best = [max(c[g * per:(g + 1) * per]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -best[g])[:groups["keep"]]
        c = [v if j // per in kept else -math.inf for j, v in enumerate(c)]
    return sorted(range(E), key=lambda j: -c[j])[:top]


def routed(h, W, p, mlp):
    r = mlp["router"]
    E = r["experts"]
    scores = torch.softmax(h @ W[p + "router"].T, dim=-1)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(scores[t], W[p + "correction"], r["top"], r.get("groups"))
        w = scores[t][ids]
        w = w / (w.sum() + 1e-20)
        for j, a in zip(ids, w):
            y[t] += a * (gated(h[t], W, f"{p}e{j}.") if j < E else h[t])
    if mlp.get("shared"):
        y = y + gated(h, W, p + "shared.")
    return y


def forward(cfg: dict, weights: Dict[str, torch.Tensor], ids: List[int], dtype=torch.float64,
            streams=None) -> torch.Tensor:
    """Logits [S, vocab] of one whole sequence.  ``streams``, a list, receives the residual
    stream after every layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = torch.stack([W["embed"][t] for t in ids]) * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + unit(mixer_parallel(x, W, p + "mix.", layer["mixer"], eps), eps) * W[p + "norm1"]
        if layer.get("mlp") is not None:
            x = x + unit(routed(x, W, p + "mlp.", layer["mlp"]), eps) * W[p + "norm2"]
        if streams is not None:
            streams.append(x.clone())
    return (unit(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt: List[int], n: int, dtype=torch.float64) -> List[int]:
    ids, out = list(prompt), []
    for _ in range(n):
        logits = forward(cfg, weights, ids, dtype)[-1]
        best = int(torch.nonzero(logits == logits.max())[0])
        out.append(best)
        ids.append(best)
    return out
