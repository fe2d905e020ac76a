"""Small Penopel configurations for the tests: they differ in every size and option."""
import functools
import tempfile

import torch

import plain_penopel as PN


def _attn(heads, kv_heads, dim, vdim, scale, rot, ff, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if rot:
        m["rot"] = rot
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=_dense(ff))


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window, ff):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)
    if base:
        m["rot"] = dict(dims=rot_dim, base=base)
    if window:
        m["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=m, mlp=_dense(ff))


def _dense(ff):
    return None if ff is None else dict(kind="dense", ff=ff)


def _rot(dims, base, bands=None):
    d = dict(dims=dims, base=base)
    if bands:
        d["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return d


def _cfg(vocab, width, eps, scale, cap, layers):
    d = dict(architecture="Penopel", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)
    if cap:
        d["logit_softcap"] = cap
    return d


# a latent layer first, sizes no fast kernel takes, values wider than keys, two layers that read one layer's keys (one of them
# without a feed-forward, both with a scale of their own), windows of 37 and 5
_RA = _rot(6, 9000.0, (3.0, 0.5, 6.0, 60.0))
PA = _cfg(97, 52, 1e-5, 5.0, 4.0,
          [_lat(3, 6, 4, 10, 14, 12, 0.4, 2000.0, 37, 60),
           _attn(6, 3, 10, 14, 0.3, _RA, 44),
           _attn(6, 3, 10, 14, 0.5, _RA, None, kv_from=1),
           _lat(2, 7, 2, 9, 10, 18, 0.5, 300.0, 5, None),
           _attn(6, 3, 10, 14, 0.2, _RA, 52, kv_from=1)])
PA_INIT = dict(seed=3, std_matrix=0.18, std_embedding=0.3, std_gain=0.2, std_bias=0.5)

# no cap, no rotation, no window; one head, as many key/value heads as heads, odd head sizes, a whole head rotated
PB = _cfg(61, 40, 1e-6, 3.0, None,
          [_attn(1, 1, 7, 7, 0.6, _rot(4, 100.0), None),
           _lat(1, 3, 8, 8, 5, 9, 0.4, None, None, 36),
           _attn(4, 4, 12, 12, 0.4, _rot(12, 50.0), 48),
           _attn(2, 1, 9, 16, 0.4, None, None)])
PB_INIT = dict(seed=8, std_matrix=0.3, std_embedding=0.4, std_gain=0.15, std_bias=0.4)

# sizes the fast products and attention kernels take: heads of 64 (a quarter rotated) and 32, latent heads whose keys and
# values have one size (whole prompts form them), windows of 100 and of a page
_RF = _rot(16, 3.0e4, (5.0, 1.0, 3.0, 400.0))
PF = _cfg(256, 128, 1e-5, 4.0, 9.0,
          [_attn(4, 2, 64, 64, 0.2, _RF, 256),
           _lat(3, 40, 24, 64, 40, 48, 0.2, 7.0e3, 100, 192),
           _attn(8, 1, 32, 32, 0.25, _rot(32, 1.0e4), 224),
           _attn(4, 2, 64, 64, 0.15, _RF, 96, kv_from=0),
           _lat(4, 24, 8, 32, 64, 32, 0.3, 500.0, 64, 160)])
PF_INIT = dict(seed=14, std_matrix=0.14, std_embedding=0.3, std_gain=0.1, std_bias=0.4)

# heads of 128 in groups of four, half of a head rotated, an even number of query heads in the layer that has queries only
_RG = _rot(64, 2.0e5, (4.0, 1.0, 8.0, 512.0))
PG = _cfg(300, 256, 1e-5, 2.0, 20.0,
          [_attn(4, 1, 128, 128, 0.1, _RG, 512),
           _attn(4, 1, 128, 128, 0.13, _RG, 256, kv_from=0),
           _lat(2, 96, 32, 128, 96, 64, 0.12, 9.0e3, 200, 320)])
PG_INIT = dict(seed=23, std_matrix=0.1, std_embedding=0.4, std_gain=0.1, std_bias=0.4)

CONFIGS = {"PA": (PA, PA_INIT), "PB": (PB, PB_INIT), "PF": (PF, PF_INIT), "PG": (PG, PG_INIT)}

_FOLDERS = {}


def folder(name: str) -> str:
    """A model folder with random weights, but for the norms' slopes (spread from nearly linear to nearly a step) and the
    latent layers' sinks (spread from one that hardly counts to one that outweighs a window)."""
    if name not in _FOLDERS:
        import os

        from safetensors.torch import load_file, save_file
        from synaptix_b200.config import PenopelConfig
        from synaptix_b200.weights import write_model_folder
        cfg_dict, init = CONFIGS[name]
        init = dict(init)
        path = write_model_folder(PenopelConfig.from_dict(cfg_dict), tempfile.mkdtemp(prefix=f"sx_{name}_"), init.pop("seed"), **init)
        f = os.path.join(path, "model.safetensors")
        W = load_file(f)
        slopes = sorted(k for k in W if k.endswith(".alpha"))
        for i, k in enumerate(slopes):
            W[k] = torch.tensor(0.25 + 0.9 * ((7 * i) % len(slopes)) / len(slopes)).to(torch.bfloat16)
        for k in W:
            if k.endswith(".sink"):
                W[k] = torch.linspace(-2.0, 4.0, W[k].numel()).flip(0).to(torch.bfloat16)
        save_file({k: v.contiguous() for k, v in W.items()}, f)
        _FOLDERS[name] = path
    return _FOLDERS[name]


@functools.lru_cache(maxsize=None)
def oracle(name: str):
    return PN.load_folder(folder(name))


@functools.lru_cache(maxsize=256)
def oracle_logits(name: str, tokens: tuple) -> torch.Tensor:
    cfg, W = oracle(name)
    return PN.forward(cfg, W, list(tokens)).float()


def tokens(name: str, n: int, seed: int) -> list:
    from tiny import random_tokens
    return random_tokens(CONFIGS[name][0]["vocab"], n, seed)
