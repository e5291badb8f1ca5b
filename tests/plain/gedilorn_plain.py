"""Plain, slow implementation of the Gedilorn decoder, used as the test oracle.

One function per mechanism, whole sequences only, no cache, no batching; everything in ``dtype`` (float64 by
default).  It shares no code with ``rocmforge_b200``: tensors come in as a plain {name: tensor} dict and the
configuration as the dict that config.json holds.

Notation: W[name] is stored [out, in] and applied as x @ W.T; rms(x) = x / sqrt(mean(x^2) + eps).
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


# --------------------------------------------------------------------------- tokens to vectors

def pair_rows(tokens, mul_prev: int, mul_cur: int, buckets: int):
    """Row of the bigram table for every token; the first token of a sequence has the row after the last bucket."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * int(mul_prev) + int(cur) * int(mul_cur)) % int(buckets))
    return rows


def embedding(cfg, W, tokens, eps):
    e = cfg.get("embedding") or {}
    x = W["embed"][torch.as_tensor(list(tokens))] * float(e.get("scale", 1.0))
    if e.get("bigram"):
        b = e["bigram"]
        x = x + W["bigram"][torch.tensor(pair_rows(list(tokens), b["mul_prev"], b["mul_cur"], b["buckets"]))]
    return rms_norm(x, W["embed.norm"], eps)


# --------------------------------------------------------------------------- rotation

def stretched_frequencies(dims: int, base: float, scaling):
    """(f [dims/2], magnitude): f_i = base^(-2i/dims); with ``scaling`` a ramp over the pair index blends f_i towards
    f_i / factor, and sine and cosine grow by 0.1 ln(factor) + 1."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def pair_at(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_at(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_at(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def turn_neighbours(x, positions, freqs, magnitude):
    """x [T, ..., dims]: elements 2i and 2i+1 are a pair and turn by position * freqs[i]."""
    ang = positions.to(x.dtype)[:, None] * freqs.to(x.dtype)[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freqs.shape[0],)
    c, s = (torch.cos(ang) * magnitude).view(shape), (torch.sin(ang) * magnitude).view(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


# --------------------------------------------------------------------------- attention over a latent

def causal_softmax(scores):
    T = scores.shape[-1]
    hidden = torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1)
    return torch.softmax(scores.masked_fill(hidden, float("-inf")), dim=-1)


def latent_attention(h, W, pre, m, eps):
    """Keys and values expanded from a normed latent, one rotated key part shared by the heads; with a tensor ``g`` the
    concatenated heads are gated element by element."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ W[pre + "q"].T).view(T, H, D + R)
    down = h @ W[pre + "dkv"].T
    c = rms_norm(down[:, :K], W[pre + "dkv.norm"], eps)
    pos = torch.arange(T)
    qn, qr, kr = q[..., :D], q[..., D:], down[:, K:]
    if R:
        freqs, mag = stretched_frequencies(R, m["rot"]["base"], m["rot"].get("scaling"))
        qr, kr = turn_neighbours(qr, pos, freqs, mag), turn_neighbours(kr, pos, freqs, mag)
    kn = (c @ W[pre + "uk"].T).view(T, H, D)
    v = (c @ W[pre + "uv"].T).view(T, H, V)
    out = []
    for n in range(H):
        s = (qn[:, n] @ kn[:, n].T + qr[:, n] @ kr.T) * m["scale"]
        out.append(causal_softmax(s) @ v[:, n])
    o = torch.stack(out, dim=1).reshape(T, H * V)
    if pre + "g" in W:
        o = o * torch.sigmoid(h @ W[pre + "g"].T)
    return o @ W[pre + "o"].T


# --------------------------------------------------------------------------- feed-forward, streams, the model

def relu_unit(h, W, pre):
    return (torch.relu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def collect(xs, weights):
    """xs [S, T, width] -> sum_s weights[s] xs[s]."""
    return (weights[:, None, None] * xs).sum(dim=0)


def spread(xs, mix, out, y):
    """Every stream anew from all the old ones: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    return torch.einsum("st,snw->tnw", mix, xs) + out[:, None, None] * y[None]


def forward(cfg: dict, W: dict, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) receives the sum of the streams after every layer run."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(cfg, W, tokens, eps)
    S = cfg.get("streams")
    xs = x[None].repeat(S or 1, 1, 1)

    def sublayer(pre, q, fn):
        nonlocal xs
        if not S:
            xs = xs + fn(rms_norm(xs[0], W[f"{pre}norm{q}"], eps))[None]
            return
        u = collect(xs, W[f"{pre}hc{q}.in"])
        xs = spread(xs, W[f"{pre}hc{q}.mix"], W[f"{pre}hc{q}.out"], fn(rms_norm(u, W[f"{pre}norm{q}"], eps)))

    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i if L.get('weights_of') is None else L['weights_of']}."
        sublayer(pre, 1, lambda h: latent_attention(h, W, pre + "mix.", L["mixer"], eps))
        if L.get("mlp") is not None:
            sublayer(pre, 2, lambda h: relu_unit(h, W, pre + "mlp."))
        if trace is not None:
            trace.append(xs.sum(dim=0).clone())
    return rms_norm(xs.sum(dim=0), W["final.norm"], eps) @ W["head"].T * float(cfg.get("logit_scale", 1.0))


class PlainGedilorn:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg, self.W = cfg, tensors

    def logits(self, tokens, trace=None):
        return forward(self.cfg, self.W, list(tokens), trace=trace)
