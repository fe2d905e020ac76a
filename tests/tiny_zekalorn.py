"""Small Zekalorn configurations for the tests: they differ in every size and option."""
import functools
import os
import tempfile

import torch

import plain_zekalorn as PZ


def _delta(heads, kv_heads, dim, vdim, conv, ra, rg, mlp):
    return dict(type="channel_delta", mlp=mlp,
                mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, decay_rank=ra, gate_rank=rg))


def _attn(heads, kv_heads, dim, vdim, scale, rows, far, temp, mlp):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, bias_max=far, bias_rows=rows)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    return dict(type="attention", mixer=m, mlp=mlp)


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def _cfg(vocab, width, eps, scale, max_positions, side, loop, layers):
    d = dict(architecture="Zekalorn", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
             max_positions=max_positions, layers=layers)
    if side:
        d["token_side"] = dict(dim=side)
    if loop:
        d["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return d


# attention first, sizes no fast kernel takes, fewer query/key heads than heads, a loop in the middle that runs three times,
# values wider than keys and narrower, a table of 10 distance buckets, a temperature that changes every 13 positions
ZA = _cfg(97, 52, 1e-5, 5.0, 900, 6, (1, 3, 3),
          [_attn(6, 3, 10, 14, 0.3, 10, 50.0, (0.7, 13), _moe(24, 5, 2)),
           _delta(4, 2, 12, 20, 4, 5, 7, _dense(60)),
           _delta(3, 3, 16, 8, 2, 3, 9, _moe(20, 4, 1)),
           _delta(2, 1, 20, 12, 3, 8, 4, None),
           _attn(2, 1, 16, 12, 0.25, 7, 90.0, (0.4, 64), _dense(44))])
ZA_INIT = dict(seed=3, std_matrix=0.14, std_embedding=0.3, std_gain=0.2, std_bias=0.5)

# no loop, no token input, no temperature; heads the chunks do not take (a key size of 6), one tap and five, one expert,
# every expert chosen, one query/key head for all
ZB = _cfg(61, 40, 1e-6, 3.0, 700, None, None,
          [_delta(4, 1, 6, 16, 5, 4, 4, _moe(16, 3, 3)),
           _delta(2, 2, 8, 4, 1, 2, 6, _moe(12, 1, 1)),
           _attn(3, 3, 12, 8, 0.35, 32, 200.0, None, None),
           _delta(1, 1, 24, 40, 4, 6, 3, _dense(52))])
ZB_INIT = dict(seed=8, std_matrix=0.15, std_embedding=0.4, std_gain=0.15, std_bias=0.4)

# sizes the fast products and attention kernels take; head sizes 64 x 64, 32 x 128 (two heads a query/key head), 128 x 32
ZF = _cfg(256, 128, 1e-5, 4.0, 1024, 16, (0, 1, 2),
          [_delta(4, 4, 64, 64, 3, 16, 24, _dense(256)),
           _delta(4, 2, 32, 128, 4, 32, 8, _moe(96, 8, 3)),
           _attn(4, 2, 64, 64, 0.12, 24, 300.0, (0.3, 100), _moe(64, 6, 2)),
           _delta(2, 2, 128, 32, 4, 8, 40, _moe(72, 4, 2))])
ZF_INIT = dict(seed=14, std_matrix=0.08, std_embedding=0.3, std_gain=0.1, std_bias=0.4)

# heads of 128 x 128 with ranks of 128 (one kernel a single-token step, narrow slices in the chunks), attention heads of 128
# in groups of four, all layers twice
ZG = _cfg(300, 256, 1e-5, 2.0, 1100, 32, (0, 3, 2),
          [_delta(2, 1, 128, 128, 4, 128, 128, _moe(128, 8, 2)),
           _attn(4, 1, 128, 128, 0.09, 32, 128.0, (0.5, 256), _dense(512)),
           _delta(2, 2, 64, 128, 2, 64, 32, _moe(136, 4, 2))])
ZG_INIT = dict(seed=23, std_matrix=0.06, std_embedding=0.4, std_gain=0.1, std_bias=0.4)

CONFIGS = {"ZA": (ZA, ZA_INIT), "ZB": (ZB, ZB_INIT), "ZF": (ZF, ZF_INIT), "ZG": (ZG, ZG_INIT)}

_FOLDERS = {}


def folder(name: str) -> str:
    """A model folder with random weights, but for the decays' constants: half of the channels of every head forget next
    to nothing over hundreds of tokens (so that a state that is lost or mixed up shows far behind), the others are spread
    up to a decay that empties its channel within a token or two."""
    if name not in _FOLDERS:
        from safetensors.torch import load_file, save_file
        from synaptix_b200.config import ZekalornConfig
        from synaptix_b200.weights import write_model_folder
        cfg_dict, init = CONFIGS[name]
        init = dict(init)
        path = write_model_folder(ZekalornConfig.from_dict(cfg_dict), tempfile.mkdtemp(prefix=f"sx_{name}_"), init.pop("seed"), **init)
        f = os.path.join(path, "model.safetensors")
        W = load_file(f)
        for i, layer in enumerate(cfg_dict["layers"]):
            if layer["type"] != "channel_delta":
                continue
            H, D = layer["mixer"]["heads"], layer["mixer"]["dim"]
            W[f"l{i}.mix.A_log"] = torch.linspace(-1.0, 1.5, H).to(torch.bfloat16)
            dt = torch.linspace(-2.0, 3.0, D)
            dt[::2] = torch.linspace(-9.0, -5.0, D)[::2]
            W[f"l{i}.mix.dt_bias"] = dt.repeat(H).to(torch.bfloat16).contiguous()
        save_file({k: v.contiguous() for k, v in W.items()}, f)
        _FOLDERS[name] = path
    return _FOLDERS[name]


@functools.lru_cache(maxsize=None)
def oracle(name: str):
    return PZ.load_folder(folder(name))


def _to_bf16(v):
    return v.to(torch.bfloat16).to(torch.float64)


@functools.lru_cache(maxsize=256)
def oracle_logits(name: str, tokens: tuple, dtype: str = "float32") -> torch.Tensor:
    """``dtype="bfloat16"``: the sublayers read what they read rounded to 16 bits, as the library's bfloat16 path has it;
    everything else stays 64-bit."""
    cfg, W = oracle(name)
    return PZ.forward(cfg, W, list(tokens), read=_to_bf16 if dtype == "bfloat16" else None).float()


@functools.lru_cache(maxsize=None)
def _steady_tokens(name: str, n: int, seed: int) -> tuple:
    from tiny import random_tokens
    toks = None
    for attempt in range(6):
        toks = random_tokens(CONFIGS[name][0]["vocab"], n, seed + 1000 * attempt)
        a, b = oracle_logits(name, tuple(toks)), oracle_logits(name, tuple(toks), "bfloat16")
        rel = (a - b).abs().max(dim=1).values / a.abs().max()
        if float(rel.median()) <= 0.01 and float((rel <= 0.03).float().mean()) >= 0.9:
            break
    return tuple(toks)


def tokens(name: str, n: int, seed: int) -> list:
    """``n`` random tokens on which the plain implementation itself moves little when its sublayers read rows rounded to
    16 bits (on some sequences a router's near tie decides differently under any rounding, and every row behind it that
    reads that token's key or state moves: such a sequence measures the tie, not a kernel)."""
    return list(_steady_tokens(name, n, seed))
