"""A plain, slow implementation of the Penopel decoder on the CPU: one function per mechanism, straight from the
equations, whole sequences only, no cache and no batching.  It shares nothing with the package (it reads model
folders with the ``safetensors`` package) and is what the GPU tests compare the engine with.

Notation: ``x`` is the residual stream ``[T, width]``, ``h`` what a sublayer reads, positions count from 0.
"""
import json
import math
import os

import torch


def load_folder(path, dtype=torch.float64):
    from safetensors.torch import load_file
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    W = {k: v.to(dtype) for k, v in load_file(os.path.join(path, "model.safetensors")).items()}
    return cfg, W


def squash(x, W, name):
    """The layers' norm: no statistic of the row, every element on its own through a tanh with a learned slope."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def affine(h, W, name):
    return h @ W[name].T + W[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def frequencies(rot):
    """One frequency per rotated pair.  With ``scaling``, by the pair's wavelength (in positions): short waves keep their
    frequency, long ones are slowed down by ``factor``, the ones between are blended linearly in original / wavelength."""
    n = rot["dims"] // 2
    out = []
    for i in range(n):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            turns = sc["original"] * f / (2.0 * math.pi)          # how often the pair turns over the original length
            if turns < sc["low"]:
                f = f / sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def angles(pos, rot):
    """Angles are formed as the library is asked to form them: a 32-bit product of position and 32-bit frequency."""
    return (pos.to(torch.float32)[:, None] * frequencies(rot).to(torch.float32)[None, :]).to(torch.float64)


def _turn(u, v, a):
    c, s = torch.cos(a).to(u.dtype), torch.sin(a).to(u.dtype)
    while c.dim() < u.dim():
        c, s = c.unsqueeze(1), s.unsqueeze(1)
    return u * c - v * s, v * c + u * s


def rotate_halves(x, pos, rot):
    """x [T, ..., n]: element i of the first ``dims`` paired with element i + dims / 2; the rest passes unchanged."""
    n = rot["dims"] // 2
    out = x.clone()
    out[..., :n], out[..., n:2 * n] = _turn(x[..., :n], x[..., n:2 * n], angles(pos, rot))
    return out


def rotate_neighbours(x, pos, rot):
    """x [T, ..., n]: element 2i of the first ``dims`` paired with element 2i + 1; the rest passes unchanged."""
    d = rot["dims"]
    out = x.clone()
    out[..., 0:d:2], out[..., 1:d:2] = _turn(x[..., 0:d:2], x[..., 1:d:2], angles(pos, rot))
    return out


def weights_beside_a_sink(scores, visible, sink):
    """exp(s_j) / (exp(sink) + sum over the visible keys of exp(s_k)): the sink takes weight and gives no value."""
    s = scores.masked_fill(~visible, -math.inf)
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention_memory(h, W, p, m, pos):
    """What an attention layer keeps per token: rotated keys and values, ``[T, kv_heads, dim | vdim]``."""
    T, G = h.shape[0], m["kv_heads"]
    k = affine(h, W, p + "k").view(T, G, m["dim"])
    v = affine(h, W, p + "v").view(T, G, m["vdim"])
    return (rotate_halves(k, pos, m["rot"]) if m.get("rot") else k), v


def attention(h, W, p, m, pos, memory):
    """Grouped queries over every earlier key of ``memory`` (this layer's own or another's), a sink of score 0."""
    T, H = h.shape[0], m["heads"]
    k, v = memory
    q = affine(h, W, p + "q").view(T, H, m["dim"])
    if m.get("rot"):
        q = rotate_halves(q, pos, m["rot"])
    see = pos[:, None] >= pos[None, :]
    outs = []
    for hh in range(H):
        g = hh // (H // m["kv_heads"])
        outs.append(weights_beside_a_sink(q[:, hh] @ k[:, g].T * m["scale"], see, torch.zeros((), dtype=h.dtype)) @ v[:, g])
    return torch.cat(outs, dim=-1) @ W[p + "o"].T


def latent_attention(h, W, p, m, pos, eps):
    """Keys and values of all heads out of one normed latent per token and one rotated key part that the heads share;
    queries through a normed latent of their own; a window; a learned sink per head; a gate per output element."""
    T, H, D, Dr, Dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T
    q = q.view(T, H, D + Dr)
    down = h @ W[p + "dkv"].T
    c = unit_rms(down[:, :R], eps) * W[p + "dkv.norm"]
    kr, qr = down[:, R:], q[..., D:]
    if m.get("rot"):
        kr, qr = rotate_neighbours(kr, pos, m["rot"]), rotate_neighbours(qr, pos, m["rot"])
    k = (c @ W[p + "uk"].T).view(T, H, D)
    v = (c @ W[p + "uv"].T).view(T, H, Dv)
    back = pos[:, None] - pos[None, :]
    see = back >= 0
    if m.get("mask"):
        see = see & (back < m["mask"]["size"])
    outs = []
    for hh in range(H):
        s = (q[:, hh, :D] @ k[:, hh].T + qr[:, hh] @ kr.T) * m["scale"]
        outs.append(weights_beside_a_sink(s, see, W[p + "sink"][hh]) @ v[:, hh])
    y = torch.cat(outs, dim=-1) * torch.sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, W, p):
    return affine(gelu_tanh(affine(h, W, p + "gate")) * affine(h, W, p + "up"), W, p + "down")


def soft_limit(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, W, tokens, layers_out=None, read=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that takes the stream after every layer.  ``read``: what
    is done to the rows a sublayer reads (a rounding), nothing by default."""
    read = read or (lambda t: t)
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = "l%d." % i, layer["mixer"]
        h = read(squash(x, W, p + "norm1"))
        if layer["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                j = i
                kept[i] = attention_memory(h, W, p + "mix.", m, pos)
            x = x + attention(h, W, p + "mix.", m, pos, kept[j])
        elif layer["type"] == "latent_attention":
            x = x + latent_attention(h, W, p + "mix.", m, pos, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            x = x + feed_forward(read(squash(x, W, p + "norm2")), W, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    z = read(squash(x, W, "final.norm")) @ W["head"].T
    return soft_limit(z, cfg["logit_softcap"]) if cfg.get("logit_softcap") else z
