"""Nodepel, stated plainly: a whole sequence at a time, in float64, one function per mechanism.

This is the tests' oracle.  It shares nothing with the engine: it reads the configuration
document and a dict of tensors.  Notation: ``x`` is the residual stream ``[T, width]``, ``x0`` the
embedding's output, ``h`` a sublayer's normed input, ``p`` a row's position in its sequence (from 0).

A layer is pre-norm with RMS norms whose weights are stored around zero.  Its one kind of mixer,
``parallel``, runs two mixers on the same input - windowed softmax attention with a sink per head
and one norm over all heads together ("left"), and a gated delta rule behind short convolutions
("right") - and halves the sum of their outputs' RMS norms.  The feed-forward is a mixture of
ungated squared-relu experts whose router takes the softmax over the chosen logits only, beside
a shared expert times a sigmoid per token.  A run of layers may repeat; every pass begins with a
projection of the stream and the embedding's output side by side, plus a vector of the pass.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6  # inside the root of the delta rule's unit vectors


def _w(tensors, name):
    return tensors[name].to(F64)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def centred_norm(x, tensors, name, eps):
    """A norm whose weight is stored around zero."""
    return rms_norm(x, 1.0 + _w(tensors, name), eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# --------------------------------------------------------------------------- attention


def rotate_halves(x, positions, dims, base):
    """Entries ``i`` and ``i + dims/2`` of the first ``dims`` entries of ``x[T, heads, D]`` turn by
    ``p * base^(-2i/dims)``; the rest pass."""
    if not dims:
        return x
    i = torch.arange(dims // 2, dtype=F64)
    angle = positions.to(F64)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., : dims // 2], x[..., dims // 2 : dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def in_window(i, j, size):
    return 0 <= i - j < size


def window_hidden(T, size):
    """``[T, T]``, True where the row's position does not see the column's."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d < 0) | (d >= size)


def softmax_with_sink(scores, hidden, sink):
    """Softmax over the keys that are not hidden; the denominator holds ``exp(sink)`` once more."""
    scores = scores.masked_fill(hidden, float("-inf"))
    top = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention(tensors, prefix, m, h, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    positions = torch.arange(T)
    q = rms_norm(h @ _w(tensors, f"{prefix}.q").T, _w(tensors, f"{prefix}.q.norm"), eps)  # over all heads' entries together
    k = rms_norm(h @ _w(tensors, f"{prefix}.k").T, _w(tensors, f"{prefix}.k.norm"), eps)
    v = (h @ _w(tensors, f"{prefix}.v").T).view(T, G, V)
    rot = m["rot"]
    q = rotate_halves(q.view(T, H, D), positions, rot["dims"], rot["base"])
    k = rotate_halves(k.view(T, G, D), positions, rot["dims"], rot["base"])
    sink = _w(tensors, f"{prefix}.sink")
    hidden = window_hidden(T, m["mask"]["size"])
    out = torch.zeros((T, H, V), dtype=F64)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = softmax_with_sink(q[:, a] @ k[:, g].T * m["scale"], hidden, sink[a]) @ v[:, g]
    return out.reshape(T, H * V) @ _w(tensors, f"{prefix}.o").T


# --------------------------------------------------------------------------- the delta rule


def short_convolution(x, taps):
    """``y_t[c] = silu(sum_j taps[c, L-1-j] x_{t-j}[c])``, zeros before the first row."""
    L = taps.shape[1]
    padded = torch.cat([torch.zeros((L - 1, x.shape[1]), dtype=F64), x])
    y = torch.zeros_like(x)
    for j in range(L):
        y += taps[:, j] * padded[j : j + x.shape[0]]
    return silu(y)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_rule(q, k, v, beta, decay):
    """One head: ``q, k [T, D]``, ``v [T, V]``, ``beta, decay [T]``; the state starts at zero."""
    S = torch.zeros((q.shape[1], v.shape[1]), dtype=F64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def gated_delta(tensors, prefix, m, h, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (short_convolution(h @ _w(tensors, f"{prefix}.{n}").T, _w(tensors, f"{prefix}.{n}.conv")) for n in "qkv")
    q = unit_vector(q.view(T, G, D)) * D**-0.5
    k = unit_vector(k.view(T, G, D))
    v = v.view(T, H, V)
    beta = torch.sigmoid(h @ _w(tensors, f"{prefix}.b").T)
    decay = torch.exp(-torch.exp(_w(tensors, f"{prefix}.A_log")) * softplus(h @ _w(tensors, f"{prefix}.a").T + _w(tensors, f"{prefix}.dt_bias")))
    out = torch.zeros((T, H, V), dtype=F64)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = delta_rule(q[:, g], k[:, g], v[:, a], beta[:, a], decay[:, a])
    gate = silu(h @ _w(tensors, f"{prefix}.g").T).view(T, H, V)
    out = rms_norm(out, _w(tensors, f"{prefix}.norm"), eps) * gate
    return out.reshape(T, H * V) @ _w(tensors, f"{prefix}.o").T


def parallel_mixer(tensors, prefix, m, h, eps):
    left = attention(tensors, f"{prefix}.left", m["left"], h, eps)
    right = gated_delta(tensors, f"{prefix}.right", m["right"], h, eps)
    return 0.5 * (rms_norm(left, _w(tensors, f"{prefix}.left.out"), eps) + rms_norm(right, _w(tensors, f"{prefix}.right.out"), eps))


# --------------------------------------------------------------------------- feed-forward


def expert(tensors, prefix, h):
    return torch.relu(h @ _w(tensors, f"{prefix}.up").T) ** 2 @ _w(tensors, f"{prefix}.down").T


def choose(logits, top):
    """One token: the ids of the ``top`` largest logits (the lower id on a tie) and the softmax over them."""
    order = sorted(range(len(logits)), key=lambda e: (-float(logits[e]), e))[:top]
    z = torch.stack([logits[e] for e in order])
    z = torch.exp(z - z.max())
    return order, z / z.sum()


def mixture(tensors, prefix, mlp, h, margins=None):
    """``margins``, a list, gets per row how far the last chosen logit lies above the best one left out."""
    logits = h @ _w(tensors, f"{prefix}.router").T + _w(tensors, f"{prefix}.router.b")
    if margins is not None:
        ranked, top = torch.sort(logits, dim=-1, descending=True).values, mlp["router"]["top"]
        margins.append(ranked[:, top - 1] - ranked[:, top] if top < logits.shape[1] else torch.full((h.shape[0],), float("inf"), dtype=F64))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, weights = choose(logits[t], mlp["router"]["top"])
        for e, w in zip(ids, weights):
            out[t] += w * expert(tensors, f"{prefix}.e{e}", h[t : t + 1])[0]
    if mlp.get("shared") is not None:
        out = out + expert(tensors, f"{prefix}.shared", h) * torch.sigmoid(h @ _w(tensors, f"{prefix}.shared.sg").T)
    return out


# --------------------------------------------------------------------------- the model


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
    eps = document["norm"]["eps"]
    x0 = tensors["embed"][torch.as_tensor(tokens)].to(F64) * (document.get("embedding") or {}).get("scale", 1.0)
    x = x0.clone()
    for run, (i, begins) in enumerate(run_order(document)):
        if begins is not None:
            x = torch.cat([x, x0], dim=-1) @ _w(tensors, "loop.in").T + _w(tensors, "loop.step")[begins]
        layer = document["layers"][i]
        x = x + parallel_mixer(tensors, f"l{i}.mix", layer["mixer"], centred_norm(x, tensors, f"l{i}.norm1", eps), eps)
        if layer.get("mlp") is not None:
            x = x + mixture(tensors, f"l{i}.mlp", layer["mlp"], centred_norm(x, tensors, f"l{i}.norm2", eps), margins)
        if hook is not None:
            hook(run, x)
    return x


def plain_logits(document, tensors, tokens, hook=None, margins=None):
    x = plain_layers(document, tensors, tokens, hook, margins)
    return centred_norm(x, tensors, "final.norm", document["norm"]["eps"]) @ _w(tensors, "head").T
