"""Dogotar restated plainly: float64 torch on the CPU, one function per mechanism, whole sequences at a time, no cache.

Shares no code with the package.  A model is a dict ``config`` in the shape of the design's config.json and a dict of
tensors by checkpoint name; ``forward`` returns the logits of every position (and, on request, the stream after every
layer).

Notation: x is a [tokens, width] stream, positions count from 0, W applies as x @ W.T.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
READOUT_EPS = 1e-6


def weight(w, name):
    return w[name].to(F64)


def project(h, w, name, bias=False):
    y = h @ weight(w, name).T
    return y + weight(w, f"{name}.b") if bias else y


def layer_norm(x, gain, shift, eps):
    """(x - mean) / sqrt(mean of the squared deviations + eps) * gain + shift."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * gain + shift


def rms_norm(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain, the mean over the last axis (``gain`` None: none)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if gain is None else y * gain


def rotate(x, dims, base, factor):
    """x [n, H, d]: elements i and i + dims/2 turn by p * base^(-2i/dims) / factor at position p; the rest stay."""
    half = dims // 2
    freq = base ** (-2.0 * torch.arange(half, dtype=F64) / dims) / factor
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * freq
    c, s = a.cos()[:, None], a.sin()[:, None]
    u, v = x[..., :half], x[..., half: dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def soft_cap(s, cap):
    return s if cap is None else cap * torch.tanh(s / cap)


def in_window(n, size):
    """[n, n] bool: query i sees key j when 0 <= i - j < size (size None: every earlier key)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def in_chunk(n, size):
    """[n, n] bool: query i sees key j <= i of the same run of ``size`` positions (size None: every earlier key)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) if size is None else (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def capped_attention(q, k, v, scale, cap, mask):
    """q [n, H, d], k [n, H, d], v [n, H, dv] -> [n, H, dv]; the scores pass the soft cap before the mask and the softmax."""
    s = soft_cap(torch.einsum("ihd,jhd->hij", q, k) * scale, cap).masked_fill(~mask[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def normed_heads(h, w, name, heads, dim, eps):
    """A projection with a bias, each head divided by its root mean square and multiplied by one gain for all heads."""
    return rms_norm(project(h, w, name, bias=True).view(-1, heads, dim), weight(w, f"{name}.norm"), eps)


def mix_values(v, first, share):
    return (1 - share) * v + share * first


def attention(h, m, w, name, eps, mask, rot=None, v_mix=False, first=None):
    """(concatenated heads, this layer's own values): grouped-query attention with normed queries and keys, positions by
    rotation (or none), a soft cap on the scores; with ``v_mix`` the values are mixed with the first such layer's."""
    H, G, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k = normed_heads(h, w, f"{name}.q", H, dim, eps), normed_heads(h, w, f"{name}.k", G, dim, eps)
    own = project(h, w, f"{name}.v", bias=True).view(-1, G, vdim)
    if rot is not None:
        turn = (int(rot["dims"]), float(rot["base"]), float((rot.get("scaling") or {}).get("factor", 1.0)))
        q, k = rotate(q, *turn), rotate(k, *turn)
    v = mix_values(own, first.view_as(own), weight(w, f"{name}.vmix")) if v_mix and first is not None else own
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    return capped_attention(q, k, v, float(m["scale"]), m.get("softcap"), mask).reshape(h.shape[0], -1), own


def attention_mixer(h, m, w, name, eps, first):
    """Windowed attention with rotation and an output gate; returns (result, own values)."""
    size = (m.get("mask") or {}).get("size")
    o, own = attention(h, m, w, name, eps, in_window(h.shape[0], size), m.get("rot"), bool(m.get("v_mix")), first)
    return project(o * torch.sigmoid(project(h, w, f"{name}.g")), w, f"{name}.o"), own


def matrix_memory(q, k, v, i, f):
    """q, k [n, H, d], v [n, H, dv], log gates i, f [n, H] -> o [n, H, dv]; the state is kept divided by exp(m), m = max(f + m, i)
    from m = 0."""
    n, H, d = q.shape
    S, z, m = torch.zeros(H, d, v.shape[-1], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    out = []
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + write[:, None] * k[t]
        m = new
        norm = torch.maximum((z * q[t]).sum(-1).abs(), torch.exp(-m)) + READOUT_EPS
        out.append(torch.einsum("hd,hdv->hv", q[t], S) / norm[:, None])
    return torch.stack(out)


def matrix_memory_mixer(h, m, w, name, eps):
    """Exponential gating with capped pre-activations around the matrix memory; per-head norm, gain, sigmoid output gate."""
    n, H, dim, vdim, cap = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = project(h, w, f"{name}.q").view(n, H, dim) * dim ** -0.5
    k, v = project(h, w, f"{name}.k").view(n, H, dim), project(h, w, f"{name}.v").view(n, H, vdim)
    i = soft_cap(project(h, w, f"{name}.i", bias=True), cap)
    f = torch.nn.functional.logsigmoid(soft_cap(project(h, w, f"{name}.f", bias=True), cap))
    o = rms_norm(matrix_memory(q, k, v, i, f), None, eps).reshape(n, -1) * weight(w, f"{name}.norm")
    return project(o * torch.sigmoid(project(h, w, f"{name}.g")), w, f"{name}.o")


def parallel_mixer(h, m, w, name, eps):
    """Chunked attention without positions beside the matrix memory, each result times a constant."""
    a = m["left"]
    o, _ = attention(h, a, w, f"{name}.left", eps, in_chunk(h.shape[0], (a.get("mask") or {}).get("size")))
    return (float(m["left_scale"]) * project(o, w, f"{name}.left.o")
            + float(m["right_scale"]) * matrix_memory_mixer(h, m["right"], w, f"{name}.right", eps))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, w, name):
    return project(gelu_tanh(project(h, w, f"{name}.up")), w, f"{name}.down")


def forward(config, w, tokens, *, return_layers=False):
    """tokens: a list of ids of one sequence -> float64 logits [n, vocab] (and the stream after every layer)."""
    eps = float(config["norm"]["eps"])
    norm = lambda x, name: layer_norm(x, weight(w, name), weight(w, f"{name}.b"), eps)
    x = weight(w, "embed")[torch.as_tensor(tokens, dtype=torch.long)]
    after, first = [], None
    for i, layer in enumerate(config["layers"]):
        name, m = f"l{i}", layer["mixer"]
        h = norm(x, f"{name}.norm1")
        if layer["type"] == "attention":
            y, own = attention_mixer(h, m, w, f"{name}.mix", eps, first)
            if m.get("v_mix") and first is None:
                first = own
        else:
            y = parallel_mixer(h, m, w, f"{name}.mix", eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(norm(x, f"{name}.norm2"), w, f"{name}.mlp")
        x = x + y
        after.append(x.clone())
    logits = norm(x, "final.norm") @ weight(w, "embed").T
    return (logits, torch.stack(after)) if return_layers else logits
