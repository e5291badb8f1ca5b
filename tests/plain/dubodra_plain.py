"""Plain, slow implementation of the Dubodra decoder, used as the test oracle.

One function per mechanism, whole sequences only, no cache, no batching; everything in ``dtype`` (float64 by
default).  It shares no code with ``rocmforge_b200``: tensors come in as a plain {name: tensor} dict and the
configuration as the dict that config.json holds.

Notation: W[name] is stored [out, in] and applied as x @ W.T; rms(x) = x / sqrt(mean(x^2) + eps).
"""
from __future__ import annotations

import math

import torch


def silu(z):
    return z * torch.sigmoid(z)


def gelu_by_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, W, name, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * W[name] + W[name + ".b"]


def capped(z, cap):
    return z if cap is None else cap * torch.tanh(z / cap)


# --------------------------------------------------------------------------- attention

def turn_pairs(x, positions, dims: int, base: float):
    """x [T, heads, dim]: element i < dims/2 of a head is paired with element i + dims/2 and turns by
    position * base^(-2i/dims); elements from ``dims`` on pass."""
    if dims == 0:
        return x
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v, rest = x[..., : dims // 2], x[..., dims // 2: dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


def capped_attention(q, k, v, scale, cap):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; position i sees j <= i."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = capped((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(~seen, float("-inf"))
        out.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


def attention(h, W, pre, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {}
    dims, base = int(rot.get("dims", 0)), float(rot.get("base", 1.0))
    pos = torch.arange(T)
    q = unit_rms((h @ W[pre + "q"].T).view(T, H, D), eps) * W[pre + "q.norm"]
    k = unit_rms((h @ W[pre + "k"].T).view(T, G, D), eps) * W[pre + "k.norm"]
    v = (h @ W[pre + "v"].T).view(T, G, V)
    o = capped_attention(turn_pairs(q, pos, dims, base), turn_pairs(k, pos, dims, base), v, m["scale"], m.get("softcap"))
    return o.reshape(T, H * V) @ W[pre + "o"].T


# --------------------------------------------------------------------------- lightning attention

def fixed_decay_recurrence(q, k, v, decay, S=None):
    """q, k [T, D], v [T, V], one number ``decay``: S <- decay S + k v^T, o = S^T q."""
    S = q.new_zeros((q.shape[1], v.shape[1])) if S is None else S.clone()
    out = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def lightning(h, W, pre, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[pre + "q"].T).view(T, H, D)
    k = silu(h @ W[pre + "k"].T).view(T, H, D)
    v = silu(h @ W[pre + "v"].T).view(T, H, V)
    o = torch.stack([fixed_decay_recurrence(q[:, n], k[:, n], v[:, n], float(m["decay"][n]))[0] for n in range(H)], dim=1)
    o = unit_rms(o.reshape(T, H * V), eps) * W[pre + "norm"]                # all heads of a token together
    return (o * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


# --------------------------------------------------------------------------- the gated delta rule

def causal_taps(x, w):
    """silu of y_t = sum_j w[:, taps-1-j] x_(t-j): the last column weighs the current token; zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros((taps - 1, C)), x], dim=0)
    return silu(sum(padded[j: j + T] * w[:, j][None, :] for j in range(taps)))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def corrected_recurrence(q, k, v, beta, g, S=None):
    """q, k [T, D], v [T, V], beta [T], g [T]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = q.new_zeros((q.shape[1], v.shape[1])) if S is None else S.clone()
    out = []
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out), S


def delta(h, W, pre, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_taps(h @ W[pre + "q"].T, W[pre + "q.conv"]).view(T, G, D)
    k = causal_taps(h @ W[pre + "k"].T, W[pre + "k.conv"]).view(T, G, D)
    v = causal_taps(h @ W[pre + "v"].T, W[pre + "v.conv"]).view(T, H, V)
    q, k = unit_vector(q) * D ** -0.5, unit_vector(k)
    beta = torch.sigmoid(h @ W[pre + "b"].T)
    g = torch.exp(-torch.exp(W[pre + "A_log"]) * torch.nn.functional.softplus(h @ W[pre + "a"].T + W[pre + "dt_bias"]))
    o = torch.stack([corrected_recurrence(q[:, n // (H // G)], k[:, n // (H // G)], v[:, n], beta[:, n], g[:, n])[0]
                     for n in range(H)], dim=1)
    o = unit_rms(o, eps) * W[pre + "norm"] * silu(h @ W[pre + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ W[pre + "o"].T


# --------------------------------------------------------------------------- feed-forwards

def dense_unit(h, W, pre):
    return (gelu_by_tanh(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def clamped_unit(h, W, pre, limit):
    g = torch.clamp(h @ W[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ W[pre + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[pre + "down"].T


def scores(h, W, pre):
    """(shares [T, E], what the choice ranks by [T, E])."""
    s = torch.softmax(h @ W[pre + "router"].T, dim=-1)
    return s, s + W[pre + "correction"]


def limit_to_groups(c, count: int, keep: int):
    """Choice scores with everything outside the ``keep`` best of ``count`` groups of neighbours at minus infinity; a group
    counts by its largest score."""
    g = c.view(c.shape[0], count, -1)
    best = g.max(dim=-1).values.topk(keep, dim=-1).indices
    open_ = torch.zeros(c.shape[0], count, dtype=torch.bool).scatter_(1, best, True)
    return g.masked_fill(~open_[:, :, None], float("-inf")).reshape(c.shape)


def choice_margin(c, top: int, groups):
    """[T]: how far each token's choice is from being another one: the smaller of the gaps between the last kept and the
    first dropped group and between the last chosen and the first unchosen expert of the kept groups (infinite: no gap)."""
    margin = torch.full((c.shape[0],), float("inf"), dtype=c.dtype)
    if groups and groups["keep"] < groups["count"]:
        g = c.view(c.shape[0], groups["count"], -1).max(dim=-1).values.sort(dim=-1, descending=True).values
        margin = torch.minimum(margin, g[:, groups["keep"] - 1] - g[:, groups["keep"]])
        c = limit_to_groups(c, groups["count"], groups["keep"])
    if top < c.shape[1]:
        e = c.sort(dim=-1, descending=True).values
        margin = torch.minimum(margin, e[:, top - 1] - e[:, top])
    return margin


def mixture(h, W, pre, mlp, forced=None, seen=None):
    """``forced`` [T, top]: the experts to use instead of the chosen ones; ``seen`` (a list) receives the chosen ones with
    their ``choice_margin``."""
    r = mlp["router"]
    s, c = scores(h, W, pre)
    groups = r.get("groups")
    if seen is not None:
        margin = choice_margin(c, r["top"], groups)
    if groups:
        c = limit_to_groups(c, groups["count"], groups["keep"])
    chosen = c.topk(r["top"], dim=-1).indices
    if seen is not None:
        seen.append((chosen, margin))
    if forced is not None:
        chosen = forced
    w = s.gather(1, chosen)
    w = w / (w.sum(dim=-1, keepdim=True) + 1e-20) * r.get("scale", 1.0)
    out = torch.zeros_like(h)
    for e in range(s.shape[1]):
        weight = (w * (chosen == e)).sum(dim=-1)
        rows = (chosen == e).any(dim=-1)
        if rows.any():
            y = clamped_unit(h[rows], W, f"{pre}e{e}.", mlp["expert"]["limit"]) if e < r["experts"] else h[rows]
            out[rows] = out[rows] + weight[rows, None] * y
    if mlp.get("shared"):
        y = clamped_unit(h, W, pre + "shared.", mlp["shared"]["limit"])
        out = out + y * torch.sigmoid(h @ W[pre + "shared.sg"].T)
    return out


# --------------------------------------------------------------------------- the model

def token_side_input(x, e, W, pre, eps):
    """e [T, dim]: the layer's part of the tokens' rows of the second table."""
    g = gelu_by_tanh(x @ W[pre + "side.gate"].T) * e
    return unit_rms(g @ W[pre + "side.proj"].T, eps) * W[pre + "side.norm"]


def forward(cfg: dict, W: dict, tokens, dtype=torch.float64, trace=None, forced=None, seen=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens)
    x = W["embed"][ids] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    mixers = {"attention": attention, "lightning": lightning, "delta": delta}
    forced = list(forced) if forced is not None else None
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + mixers[L["type"]](layer_norm(x, W, pre + "norm1", eps), W, pre + "mix.", L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h = layer_norm(x, W, pre + "norm2", eps)
            if mlp["kind"] == "dense":
                x = x + dense_unit(h, W, pre + "mlp.")
            else:
                x = x + mixture(h, W, pre + "mlp.", mlp, forced.pop(0) if forced is not None else None, seen)
        side = cfg.get("token_side")
        if side:
            d = side["dim"]
            x = x + token_side_input(x, W["side.embed"][ids][:, i * d:(i + 1) * d], W, pre, eps)
        if trace is not None:
            trace.append(x.clone())
    logits = layer_norm(x, W, "final.norm", eps) @ W["head"].T
    return capped(logits, cfg.get("logit_softcap"))


class PlainDubodra:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg, self.W = cfg, tensors

    def logits(self, tokens, trace=None, forced=None, seen=None):
        return forward(self.cfg, self.W, list(tokens), trace=trace, forced=forced, seen=seen)
