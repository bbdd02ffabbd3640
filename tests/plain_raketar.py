"""Raketar, stated plainly: a whole sequence at a time, in float64, one function per mechanism.

This is the tests' oracle.  It shares nothing with the engine: it reads the configuration
document and a dict of tensors.  Notation: ``x`` is the residual stream ``[T, width]``, ``x0`` the
embedding's output, ``h`` a layer's normed input, ``p`` a row's position in its sequence (from 0),
``m`` the factor on whatever joins the stream.

A layer is parallel: mixer and feed-forward read the same RMS norm and ``m`` times their sum joins
the stream; behind that a narrow gated pair of the stream and a per-layer piece of a second token
table adds ``m`` times its own norm.  Mixers are differential attention (two softmax maps over the
same values, one subtracted from the other) or a matrix memory with exponential gates; feed-forwards
are dense gated pairs or mixtures whose weights scale the experts' inputs.  A run of layers may
repeat; every pass adds a vector of its own and, from the second on, ``x0``.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
DENOMINATOR_EPS = 1e-6  # added to the matrix memory's denominator


def _w(tensors, name):
    return tensors[name].to(F64)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, tensors, name, eps):
    return unit_rms(x, eps) * _w(tensors, name)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


# --------------------------------------------------------------------------- differential attention


def rotate_neighbours(x, positions, dims, base, factor):
    """Entries ``2i`` and ``2i + 1`` of the first ``dims`` entries of ``x[..., D]`` (rows first) turn by
    ``p * base^(-2i/dims) / factor``; the rest pass."""
    if not dims:
        return x
    i = torch.arange(dims // 2, dtype=F64)
    angle = positions.to(F64)[:, None] * (base ** (-2.0 * i / dims) / factor)[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (dims // 2,)
    cos, sin = torch.cos(angle).view(shape), torch.sin(angle).view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


def causal_softmax(scores):
    T = scores.shape[0]
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    return torch.softmax(scores.masked_fill(hidden, float("-inf")), dim=-1)


def map_weight(tensors, prefix, diff):
    """What the second map's output is multiplied by before it is subtracted: one number per layer."""
    first = torch.exp((_w(tensors, f"{prefix}.lq1") * _w(tensors, f"{prefix}.lk1")).sum())
    second = torch.exp((_w(tensors, f"{prefix}.lq2") * _w(tensors, f"{prefix}.lk2")).sum())
    return first - second + diff


def differential_attention(tensors, prefix, m, h, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    rot = m["rot"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    positions = torch.arange(T)
    q = (h @ _w(tensors, f"{prefix}.q").T).view(T, H, 2, D)
    k = (h @ _w(tensors, f"{prefix}.k").T).view(T, G, 2, D)
    v = (h @ _w(tensors, f"{prefix}.v").T).view(T, G, V)
    q = rotate_neighbours(q, positions, rot["dims"], rot.get("base"), factor)
    k = rotate_neighbours(k, positions, rot["dims"], rot.get("base"), factor)
    second = map_weight(tensors, prefix, m["diff"])
    out = torch.zeros((T, H, V), dtype=F64)
    for a in range(H):
        g = a // (H // G)
        maps = [causal_softmax(q[:, a, i] @ k[:, g, i].T * m["scale"]) @ v[:, g] for i in range(2)]
        out[:, a] = unit_rms(maps[0] - second * maps[1], eps) * (1.0 - m["diff"])
    gated = out.reshape(T, H * V) * torch.sigmoid(h @ _w(tensors, f"{prefix}.g").T)
    return gated @ _w(tensors, f"{prefix}.o").T


# --------------------------------------------------------------------------- matrix memory


def memory(q, k, v, i, f):
    """One head: ``q, k [T, D]``, ``v [T, V]``, log gates ``i, f [T]``; state, normaliser and the running
    maximum start at zero."""
    S, n = torch.zeros((q.shape[1], v.shape[1]), dtype=F64), torch.zeros(q.shape[1], dtype=F64)
    top = torch.zeros((), dtype=F64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + top, i[t])
        keep, add = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        top = new
        out[t] = (S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-top)) + DENOMINATOR_EPS)
    return out


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm(tensors, prefix, m, h, eps):
    H, D, V, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    T = h.shape[0]
    q = (h @ _w(tensors, f"{prefix}.q").T).view(T, H, D) * D**-0.5
    k = (h @ _w(tensors, f"{prefix}.k").T).view(T, H, D)
    v = (h @ _w(tensors, f"{prefix}.v").T).view(T, H, V)
    i = capped(h @ _w(tensors, f"{prefix}.i").T + _w(tensors, f"{prefix}.i.b"), cap)
    f = log_sigmoid(capped(h @ _w(tensors, f"{prefix}.f").T + _w(tensors, f"{prefix}.f.b"), cap))
    out = torch.stack([memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], dim=1)
    out = unit_rms(out, eps).reshape(T, H * V) * _w(tensors, f"{prefix}.norm")
    return (out * torch.sigmoid(h @ _w(tensors, f"{prefix}.g").T)) @ _w(tensors, f"{prefix}.o").T


MIXERS = {"attention": differential_attention, "mlstm": mlstm}


# --------------------------------------------------------------------------- feed-forward


def gated_pair(tensors, prefix, h):
    return (silu(h @ _w(tensors, f"{prefix}.gate").T) * (h @ _w(tensors, f"{prefix}.up").T)) @ _w(tensors, f"{prefix}.down").T


def mixture(tensors, prefix, mlp, h, margins=None):
    """``margins``, a list, gets per row how far the last chosen logit lies above the best one left out."""
    logits, top = h @ _w(tensors, f"{prefix}.router").T, mlp["router"]["top"]
    if margins is not None:
        ranked = torch.sort(logits, dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top] if top < logits.shape[1] else torch.full((h.shape[0],), float("inf"), dtype=F64))
    scores = torch.sigmoid(logits)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in sorted(range(scores.shape[1]), key=lambda e: (-float(scores[t, e]), e))[:top]:
            out[t] += gated_pair(tensors, f"{prefix}.e{e}", scores[t, e] * h[t : t + 1])[0]
    if mlp.get("shared") is not None:
        out = out + gated_pair(tensors, f"{prefix}.shared", h)
    return out


def feed_forward(tensors, prefix, mlp, h, margins=None):
    return gated_pair(tensors, prefix, h) if mlp["kind"] == "dense" else mixture(tensors, prefix, mlp, h, margins)


# --------------------------------------------------------------------------- the model


def token_side(tensors, i, dim, tokens, x, eps):
    piece = tensors["side.embed"][torch.as_tensor(tokens)][:, i * dim : (i + 1) * dim].to(F64)
    y = (gelu_tanh(x @ _w(tensors, f"l{i}.side.gate").T) * piece) @ _w(tensors, f"l{i}.side.proj").T
    return rms_norm(y, tensors, f"l{i}.side.norm", eps)


def run_order(document):
    """``(layer, pass)``: ``pass`` is the number of the pass that begins with this run, or None."""
    n = len(document["layers"])
    loop = document.get("loop")
    if loop is None or loop["start"] == loop["stop"]:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def plain_layers(document, tensors, tokens, hook=None, margins=None):
    """The stream after the last layer; ``hook(run, x)`` sees it after every layer run."""
    eps, factor = document["norm"]["eps"], document.get("residual_mult", 1.0)
    side = document.get("token_side")
    x0 = tensors["embed"][torch.as_tensor(tokens)].to(F64)
    x = x0.clone()
    for run, (i, begins) in enumerate(run_order(document)):
        if begins is not None:
            x = x + (x0 if begins > 0 else 0.0) + _w(tensors, "loop.step")[begins]
        layer = document["layers"][i]
        h = rms_norm(x, tensors, f"l{i}.norm1", eps)
        y = MIXERS[layer["type"]](tensors, f"l{i}.mix", layer["mixer"], h, eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(tensors, f"l{i}.mlp", layer["mlp"], h, margins)
        x = x + factor * y
        if side is not None:
            x = x + factor * token_side(tensors, i, side["dim"], tokens, x, eps)
        if hook is not None:
            hook(run, x)
    return x


def plain_logits(document, tensors, tokens, hook=None, margins=None):
    x = plain_layers(document, tensors, tokens, hook, margins)
    return rms_norm(x, tensors, "final.norm", document["norm"]["eps"]) @ _w(tensors, "head").T
