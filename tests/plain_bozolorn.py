"""The Bozolorn decoder, plainly: one function per mechanism, float64 throughout, a whole
sequence at a time, token by token where a mechanism is a recurrence, no cache, no batching.
It shares no code with the package; the engine's tests hold the kernels and the step function to it.

Notation: ``x`` [T, W] activations of one sequence (positions 0..T-1), ``w`` a dict of the
model's tensors by name (float64), ``cfg`` the dict of config.json, ``p`` a tensor-name prefix,
``m`` a layer's ``mixer`` entry (or one half of it).
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------------------------

def rotary_frequencies(rot):
    """(f_i, magnitude): f_i = base^(-2i/dims); with ``scaling`` the slow waves are divided by ``factor``, the fast ones stay,
    the ones between are blended by the index of the pair, and cosines and sines carry a magnitude."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(plain, dtype=F), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(index_of(float(sc["fast"]))), 0)
    last = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        part = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(f / factor * part + f * (1.0 - part))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, rot):
    """x [T, heads, d]: elements 2i and 2i + 1 of the first ``dims`` turn together by position * f_i."""
    T, dims = x.shape[0], int(rot["dims"])
    f, magnitude = rotary_frequencies(rot)
    angle = torch.arange(T, dtype=F)[:, None] * f[None, :]
    c, s = (torch.cos(angle) * magnitude)[:, None, :], (torch.sin(angle) * magnitude)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def chunk_mask(T, size):
    """[query, key]: the keys up to the query that lie in its own chunk of ``size`` positions."""
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def causal_mask(T):
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


# ---------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------

def weights_of_scores(s, seen, one_more=False):
    """Softmax over the keys that are seen; ``one_more``: the denominator is one larger."""
    s = s.masked_fill(~seen, float("-inf"))
    top = s.max(dim=-1, keepdim=True).values
    if one_more:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if one_more:
        total = total + torch.exp(-top)
    return e / total


def heads_of_keys(k, heads):
    """[T, G, d] -> [T, heads, d]: query head h reads key head h // (heads / G)."""
    return k.repeat_interleave(heads // k.shape[1], dim=1)


def chunked_attention(h, w, p, m, kv=None):
    """Attention without rotation: a penalty per head linear in the distance, chunks, a gate per output element.  ``kv``:
    another layer's (keys, values) instead of its own.  Returns (y, (keys, values))."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).view(T, H, d)
    if kv is None:
        kv = ((h @ w[p + "k"].T).view(T, G, d), (h @ w[p + "v"].T).view(T, G, dv))
    k, v = heads_of_keys(kv[0], H), heads_of_keys(kv[1], H)
    i = torch.arange(T, dtype=F)
    distance = i[:, None] - i[None, :]
    seen = chunk_mask(T, int(m["mask"]["size"]))
    out = torch.zeros(T, H, dv, dtype=F)
    for a, slope in enumerate(distance_slopes(H)):
        s = (q[:, a] @ k[:, a].T) * float(m["scale"]) - slope * distance
        out[:, a] = weights_of_scores(s, seen) @ v[:, a]
    y = out.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T, kv


def rotary_attention(h, w, p, m, eps):
    """Causal attention with biases, a norm per query and key head, rotation, and a one in the softmax's denominator."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    q = rotate_neighbours(rms(q, eps) * w[p + "q.norm"], m["rot"])
    k = rotate_neighbours(rms(k, eps) * w[p + "k.norm"], m["rot"])
    k, v = heads_of_keys(k, H), heads_of_keys(v, H)
    seen = causal_mask(T)
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        s = (q[:, a] @ k[:, a].T) * float(m["scale"])
        out[:, a] = weights_of_scores(s, seen, one_more=True) @ v[:, a]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------
# the gated delta rule, and the two side by side
# ---------------------------------------------------------------------------------------------

def causal_conv(u, weight):
    """u [T, C], weight [C, taps]: out_t = sum_j weight[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, C = u.shape
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=F), u], dim=0)
    out = torch.zeros(T, C, dtype=F)
    for j in range(taps):
        out = out + padded[j:j + T] * weight[:, j][None, :]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(h, w, p, m, eps):
    """A state per head that forgets by one number a token and is corrected towards what the key should give."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k, v = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d)), v.view(T, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)                                             # [T, H]
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        g = a // (H // G)
        S = torch.zeros(d, dv, dtype=F)
        for t in range(T):
            S = decay[t, a] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            o[t, a] = S.T @ q[t, g]
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left = rotary_attention(h, w, p + "left.", m["left"], eps)
    right = delta_rule(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


# ---------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------

def route(h, w, p, mlp):
    """(ids [T, top], weights [T, top])."""
    r = mlp["router"]
    E, top = int(r["experts"]), int(r["top"])
    s = torch.sigmoid(h @ w[p + "router"].T)
    choice = s + w[p + "correction"]
    groups = r.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        each = choice.view(-1, count, E // count)
        score = torch.sort(each, dim=-1, descending=True).values[..., :2].sum(dim=-1)
        kept = torch.sort(score, dim=-1, descending=True, stable=True).indices[:, :keep]
        allowed = torch.zeros_like(score, dtype=torch.bool).scatter_(1, kept, True)
        choice = each.masked_fill(~allowed[:, :, None], float("-inf")).view(-1, E)
    ids = torch.sort(choice, dim=-1, descending=True, stable=True).indices[:, :top]
    return ids, torch.gather(s, 1, ids)


def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    ids, weights = route(h, w, p, mlp)
    y = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        t, k = torch.nonzero(ids == e, as_tuple=True)
        if len(t):
            y[t] += weights[t, k][:, None] * expert(h[t], w, f"{p}e{e}.", float(mlp["expert"]["limit"]))
    return y


# ---------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------

def token_side(x, w, p, tokens, i, dim, eps):
    """What layer i adds of the token itself: its part of the token's side row, opened by a gate that reads the stream."""
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms(y, eps) * w[p + "side.norm"]


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) takes the residual stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    kept = {}
    for i, entry in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry.get("mlp")
        h = rms(x, eps) * w[p + "norm1"]
        if entry["type"] == "attention":
            source = m.get("kv_from")
            y, kept[i] = chunked_attention(h, w, p + "mix.", m, None if source is None else kept[source])
        elif entry["type"] == "parallel":
            y = parallel(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(entry["type"])
        x = x + rms(y, eps) * w[p + "norm1b"]
        if mlp is not None:
            y = mixture(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", mlp)
            x = x + rms(y, eps) * w[p + "norm2b"]
        side = cfg.get("token_side")
        if side:
            x = x + token_side(x, w, p, tokens, i, int(side["dim"]), eps)
        if streams is not None:
            streams.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
