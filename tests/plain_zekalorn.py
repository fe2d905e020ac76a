"""A plain, slow implementation of the Zekalorn decoder: one function per mechanism, written from the equations, whole
sequences only, float64 on the CPU.  It shares nothing with the package: it reads a configuration as the nested dict of
config.json and weights as a dict ``name -> tensor``.

Notation: ``x [T, W]`` the stream of ONE sequence, ``t`` a position (from 0), ``rms(v) = sqrt(mean(v^2) + eps)``.

    embedding    x_t = s E[id_t] + P[t]
    layer        h = x / rms(x) g ;  x <- x + mixer(h) + ff(h) ;
                 y = Wp (gelu_tanh(Wg x) * e_t), e_t this layer's part of a second table's row id_t ;  x <- x + y / rms(y) n
    delta        q, k, v = silu(conv(W h)), q and k of unit length per head (q also times dim^-1/2);
                 b = sigmoid(Wb h), a = exp(-exp(A) softplus(Wa2 Wa1 h + c)) per head and key channel;
                 S <- diag(a) S,  u = b (v - S^T k),  S <- S + k u^T,  o = S^T q ;  o / rms(o) n sigmoid(Wg2 Wg1 h), Wo
    attention    score_ij = (1 + c ln(floor((i + 1) / m) + 1)) q_i . k_j scale + R[bucket(i - j), head], j <= i, softmax, Wo
    experts      z = Wr h, the largest `top`, weights = softmax of those alone, expert = Wd relu(Wu h)^2
    loop         layers start .. stop-1 run `times` times; x <- x + L[n] ahead of pass n
"""
import json
import math
import os

import torch

F = torch.float64


def load_folder(path):
    from safetensors.torch import load_file
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.to(F) for k, v in load_file(os.path.join(path, "model.safetensors")).items()}


def unit_rms(x, eps):
    x = x.to(F)
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return unit_rms(x, eps) * gain.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(tokens, table, scale, positions):
    return torch.stack([table[tok].to(F) * scale + positions[t].to(F) for t, tok in enumerate(tokens)])


def time_conv(u, taps):
    """``u [T, C]``, ``taps [C, n]``: ``y_t = sum_j taps[:, j] u_(t - n + 1 + j)``, zeros before the start."""
    T, _ = u.shape
    n = taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            y[back:] += taps[:, j].to(F) * u[:T - back]
    return y


def delta_rule(q, k, v, decay, beta):
    """``q, k, decay [T, H, D]``, ``v [T, H, V]``, ``beta [T, H]`` -> ``o [T, H, V]``; every head's state starts at zero."""
    T, H, D = k.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def delta_inputs(x, w, p, m):
    """Everything that enters the recurrence: ``q, k [T, G, D]``, ``v [T, H, V]``, ``decay [T, H, D]``, ``beta [T, H]``."""
    T = x.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = [silu(time_conv(x @ w[p + n].to(F).T, w[p + n + ".conv"])) for n in ("q", "k", "v")]
    q, k, v = q.reshape(T, G, D), k.reshape(T, G, D), v.reshape(T, H, V)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(x @ w[p + "b"].to(F).T)
    z = (x @ w[p + "a1"].to(F).T) @ w[p + "a2"].to(F).T + w[p + "dt_bias"].to(F)
    decay = torch.exp(-torch.exp(w[p + "A_log"].to(F))[None, :, None] * torch.nn.functional.softplus(z).reshape(T, H, D))
    return q, k, v, decay, beta


def channel_delta(x, w, p, m, eps):
    T = x.shape[0]
    H, G, V = m["heads"], m["kv_heads"], m["vdim"]
    q, k, v, decay, beta = delta_inputs(x, w, p, m)
    of_head = [h // (H // G) for h in range(H)]                   # the query/key head each head reads
    o = delta_rule(q[:, of_head], k[:, of_head], v, decay, beta)
    gate = torch.sigmoid((x @ w[p + "g1"].to(F).T) @ w[p + "g2"].to(F).T).reshape(T, H, V)
    y = unit_rms(o, eps) * w[p + "norm"].to(F) * gate
    return y.reshape(T, H * V) @ w[p + "o"].to(F).T


def bucket(n, rows, far):
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def temperature(i, q_temp):
    return 1.0 + q_temp["coef"] * math.log((i + 1) // q_temp["every"] + 1)


def attention(x, w, p, m):
    T = x.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ w[p + "q"].to(F).T).reshape(T, H, D)
    k = (x @ w[p + "k"].to(F).T).reshape(T, G, D)
    v = (x @ w[p + "v"].to(F).T).reshape(T, G, V)
    if m.get("q_temp"):
        q = q * torch.tensor([temperature(i, m["q_temp"]) for i in range(T)], dtype=F)[:, None, None]
    rel = w[p + "rel"].to(F)
    per_distance = rel[[bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)]]      # [T, H]
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = dist >= 0
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * m["scale"] + per_distance[dist.clamp(min=0), h]
        heads.append(torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, g])
    return torch.cat(heads, -1) @ w[p + "o"].to(F).T


def dense_ff(x, w, p):
    return (silu(x @ w[p + "gate"].to(F).T) * (x @ w[p + "up"].to(F).T)) @ w[p + "down"].to(F).T


def choose_experts(z, top):
    """Logits ``z [E]`` -> chosen experts (of equal logits the lower index first) and their weights."""
    ids = sorted(range(z.shape[0]), key=lambda e: (-float(z[e]), e))[:top]
    return ids, torch.softmax(z[ids], 0)


def experts_ff(x, w, p, spec):
    z = x @ w[p + "router"].to(F).T
    out = torch.zeros_like(x)
    per = {e: torch.relu(x @ w[f"{p}e{e}.up"].to(F).T) ** 2 @ w[f"{p}e{e}.down"].to(F).T for e in range(z.shape[1])}
    for t in range(x.shape[0]):
        for e, g in zip(*choose_experts(z[t], spec["router"]["top"])):
            out[t] += g * per[e][t]
    return out


def token_side(x, tokens, w, p, i, dim, eps):
    e = torch.stack([w["side.embed"][tok, i * dim:(i + 1) * dim].to(F) for tok in tokens])
    y = (gelu_tanh(x @ w[p + "side.gate"].to(F).T) * e) @ w[p + "side.proj"].to(F).T
    return rms_norm(y, w[p + "side.norm"], eps)


def run_order(cfg):
    """``(layer, pass)`` in order; ``pass`` is the number of the loop's pass that the run opens, else None."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None, read=None):
    """Logits float64 ``[T, vocab]`` of one sequence; ``layers_out`` (a list) takes the stream after every layer run.
    ``read``: a function applied to what the sublayers read (say, a rounding to 16 bits: how far the result moves under
    it tells how well-conditioned an input is)."""
    eps = cfg["norm"]["eps"]
    read = read or (lambda v: v)
    tokens = list(tokens)
    x = embed(tokens, w["embed"], cfg["embedding"]["scale"], w["pos"])
    for i, opens in run_order(cfg):
        if opens is not None:
            x = x + w["loop.step"][opens].to(F)
        layer, p = cfg["layers"][i], f"l{i}."
        h = read(rms_norm(x, w[p + "norm1"], eps))
        if layer["type"] == "channel_delta":
            a = channel_delta(h, w, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "attention":
            a = attention(h, w, p + "mix.", layer["mixer"])
        else:
            raise ValueError(layer["type"])
        mlp = layer.get("mlp")
        if mlp is not None:
            a = a + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else experts_ff(h, w, p + "mlp.", mlp))
        x = x + a
        if cfg.get("token_side"):
            x = x + token_side(read(x), tokens, w, p, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].to(F).T
