"""The Zigolix decoder, plainly: one function per mechanism, float64 throughout, a whole
sequence at a time, no cache, no batching.  It shares no code with the package; the engine's
tests hold the kernels and the step function to it.

Notation: ``x`` [T, W] activations of one sequence (positions 0..T-1), ``w`` a dict of the
model's tensors by name (float64), ``cfg`` the dict of config.json, ``p`` a tensor-name prefix,
``m`` a layer's ``mixer`` entry.
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------------
# positions and masks
# ---------------------------------------------------------------------------------------------

def rotary_frequencies(rot):
    """(f_i, magnitude): f_i = base^(-2i/dims); with ``scaling`` the waves that do not fit ``original`` positions ``slow``
    times are divided by ``factor``, those that fit more than ``fast`` times stay, the ones between are blended by the
    index of the pair; cosines and sines then carry the magnitude 0.1 ln(factor) + 1."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F), 1.0
    factor, orig, fast, slow = (float(sc[k]) for k in ("factor", "original", "fast", "slow"))

    def index_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, heads, d]: elements 2i and 2i + 1 of the first ``dims`` turn together by position * f_i."""
    dims = int(rot["dims"])
    f, mag = rotary_frequencies(rot)
    ang = positions.to(F)[:, None] * f[None, :]
    c, s = (torch.cos(ang) * mag)[:, None, :], (torch.sin(ang) * mag)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def visible(T, m):
    """[T, T]: query i sees key j iff 0 <= i - j (and < mask.size, if there is a mask)."""
    pos = torch.arange(T)
    d = pos[:, None] - pos[None, :]
    see = d >= 0
    mask = m.get("mask")
    if mask and mask.get("size"):
        see = see & (d < int(mask["size"]))
    return see


# ---------------------------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------------------------

def softmax_with_sink(s, sink):
    """Rows of scores (-inf: not seen); exp(sink) joins the denominator once."""
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def attention(h, w, p, m, eps):
    """Grouped-query attention whose values are the projected keys; rotation, then a norm without a weight per head; a
    window; a sink per head."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads") or H)
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).view(T, H, d)
    k = (h @ w[p + "k"].T).view(T, G, d)
    v = k
    if m.get("rot"):
        q, k = rotate_pairs(q, pos, m["rot"]), rotate_pairs(k, pos, m["rot"])
    q, k = rms(q, eps), rms(k, eps)
    see = visible(T, m)
    out = torch.zeros(T, H, d, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T * float(m["scale"])).masked_fill(~see, float("-inf"))
        out[:, a] = softmax_with_sink(s, w[p + "sink"][a]) @ v[:, g]
    return out.reshape(T, H * d) @ w[p + "o"].T


def mixing_number(w, p, m):
    """lambda of a differential layer: how much of the second map is taken off the first."""
    a = torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum())
    b = torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum())
    return a - b + float(m["diff"])


def differential_attention(h, w, p, m, eps):
    """Two attention maps per head over the same values, the second taken off the first; capped scores; a window; a norm
    per head; a gate per output element."""
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    G = int(m.get("kv_heads") or H)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, 2, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    see = visible(T, m)
    cap = m.get("softcap")
    lam = mixing_number(w, p, m)
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        g = a // (H // G)
        maps = []
        for j in range(2):
            s = q[:, a, j] @ k[:, g, j].T * float(m["scale"])
            if cap:
                s = float(cap) * torch.tanh(s / float(cap))
            maps.append(torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, g])
        out[:, a] = rms(maps[0] - lam * maps[1], eps) * (1.0 - float(m["diff"]))
    gate = torch.sigmoid(h @ w[p + "g"].T)
    return (out.reshape(T, H * dv) * gate) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------

def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, w, p, mlp):
    """(ids [T, top], weights [T, top]): the largest softmax scores choose, their own sum divides them."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    ids = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :int(mlp["router"]["top"])]
    chosen = torch.gather(s, 1, ids)
    return ids, chosen / (chosen.sum(dim=-1, keepdim=True) + 1e-20)


def mixture(h, w, p, mlp):
    limit = float(mlp["expert"]["limit"])
    ids, weights = route(h, w, p, mlp)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), weights[t]):
            y[t] += wt * expert(h[t:t + 1], w, f"{p}e{e}.", limit)[0]
    if mlp.get("shared"):
        y = y + expert(h, w, p + "shared.", float(mlp["shared"]["limit"]))
    return y


# ---------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------

def layer(x, w, cfg, i):
    """x += mixer(norm1(x)); x += ff(norm2(x))."""
    entry, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    h = rms(x, eps) * w[p + "norm1"]
    if entry["type"] == "attention":
        x = x + attention(h, w, p + "mix.", entry["mixer"], eps)
    elif entry["type"] == "attention_2":
        x = x + differential_attention(h, w, p + "mix.", entry["mixer"], eps)
    else:
        raise ValueError(entry["type"])
    mlp = entry.get("mlp")
    if mlp is not None:
        h = rms(x, eps) * w[p + "norm2"]
        x = x + (dense(h, w, p + "mlp.") if mlp["kind"] == "dense" else mixture(h, w, p + "mlp.", mlp))
    return x


def order(cfg):
    """(layer, pass): the layers as they run; ``pass`` is set on the first layer of a pass through the looped span."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = int(loop["start"]), int(loop["stop"])
    out = [(i, None) for i in range(start)]
    for t in range(int(loop["times"])):
        out += [(i, t if i == start else None) for i in range(start, stop)]
    return out + [(i, None) for i in range(stop, n)]


def enter_pass(x, x0, w, t):
    """The stream of a looped span's pass t: a map of the stream beside the embedding, and the pass's own vector."""
    return torch.cat([x, x0], dim=-1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) takes the residual stream after every layer run."""
    x0 = x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, t in order(cfg):
        if t is not None:
            x = enter_pass(x, x0, w, t)
        x = layer(x, w, cfg, i)
        if streams is not None:
            streams.append(x.clone())
    y = rms(x, float(cfg["norm"]["eps"])) * w["final.norm"]
    return (y @ w["head"].T) * float(cfg.get("logit_scale") or 1.0)
