"""What needs no GPU of the Penopel decoder: its configuration, the model as data (tensor names, cache requests, order of the
runs), how rows and biases are bound, and the plain implementation against other forms of its own equations."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_penopel as PN
from tiny_penopel import CONFIGS

F = torch.float64


def cfg_of(name):
    from synaptix_b200.config import PenopelConfig
    return PenopelConfig.from_dict(CONFIGS[name][0])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_round_trip_and_registry(name):
    from synaptix_b200.config import PenopelConfig, resolve_architecture
    d = CONFIGS[name][0]
    cfg = cfg_of(name)
    assert PenopelConfig.from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == d
    assert resolve_architecture(d).config_cls is PenopelConfig
    assert [l.type for l in cfg.layers] == [l["type"] for l in d["layers"]]


def test_configuration_errors():
    from synaptix_b200.config import ConfigError, PenopelConfig
    base = CONFIGS["PA"][0]

    def broken(change):
        d = copy.deepcopy(base)
        change(d)
        with pytest.raises(ConfigError):
            PenopelConfig.from_dict(d)
    broken(lambda d: d.pop("width"))
    broken(lambda d: d["norm"].pop("eps"))
    broken(lambda d: d["embedding"].pop("scale"))
    broken(lambda d: d.update(logit_softcap=-1.0))
    broken(lambda d: d.update(layers=[]))
    broken(lambda d: d["layers"][0].update(type="other"))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="other"))
    broken(lambda d: d["layers"][0]["mlp"].pop("ff"))
    broken(lambda d: d["layers"][0]["mixer"].pop("kv_rank"))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=6))                   # more than rot_dim
    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5))
    broken(lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("low"))
    broken(lambda d: d["layers"][2]["mixer"].update(kv_from=0))                       # no attention layer
    broken(lambda d: d["layers"][2]["mixer"].update(kv_from=2))                       # itself
    broken(lambda d: d["layers"][4]["mixer"].update(kv_from=2))                       # it has no keys of its own
    broken(lambda d: d["layers"][2]["mixer"].update(heads=3, kv_heads=3))             # other heads than its source
    broken(lambda d: d["layers"][2]["mixer"].update(rot=dict(dims=6, base=8000.0)))   # another rotation than its source


def test_model_as_data():
    from synaptix_b200.cache.store import KVRequest
    from synaptix_b200.models import model_skeleton
    m = model_skeleton(cfg_of("PA"))
    assert [(r.layer, r.cache_entry, r.write_cache) for r in m.schedule] == [
        (0, 0, True), (1, 1, True), (2, 1, False), (3, 2, True), (4, 1, False)]
    assert m.cache_requests() == [KVRequest(1, 16, 37, keys_only=True), KVRequest(3, 10, None, 14), KVRequest(1, 20, 5, keys_only=True)]
    shape = {n: tuple(s.shape) for n, s in m.all_tensor_specs().items()}
    assert shape["l1.mix.k"] == (30, 52) and shape["l1.mix.v.b"] == (42,) and shape["l1.mix.o"] == (52, 84) and "l1.mix.o.b" not in shape
    assert "l2.mix.k" not in shape and "l2.mix.v.b" not in shape and shape["l2.mix.q.b"] == (60,) and "l2.norm2" not in shape
    assert shape["l0.mix.g"] == (30, 52) and shape["l0.mix.sink"] == (3,) and shape["l0.mix.dkv"] == (16, 52) and "l0.mix.dq.b" not in shape
    assert shape["l0.norm1.alpha"] == () and shape["l0.norm2.b"] == (52,) and shape["final.norm.alpha"] == ()
    assert shape["l4.mlp.down.b"] == (52,) and shape["l4.mlp.up.b"] == (52,) and shape["head"] == (97, 52)
    b = model_skeleton(cfg_of("PB"))
    assert b.cache_requests()[1] == KVRequest(1, 17, None, keys_only=True) and b.head.softcap == 0.0


def test_a_partial_rotation_bound_as_a_whole_one():
    """The rows of q and k and their biases are bound in an order in which the pairs (i, i + dim / 2) are the rotated ones
    and pairs of frequency 0: the scores are those of the partial rotation, and the norm gains of a head follow."""
    from synaptix_b200.parts import Attention, RotaryHalf, Runtime
    g = torch.Generator().manual_seed(1)
    W, H, G, D, dims = 12, 4, 2, 10, 4
    w = {n: torch.randn(o, W, generator=g) for n, o in (("q", H * D), ("k", G * D), ("v", G * D))}
    w.update({n + ".b": torch.randn(t.shape[0], generator=g) for n, t in list(w.items())})
    w["o"] = torch.randn(W, H * D, generator=g)
    names = dict(q="q", k="k", v="v", o="o")
    part = Attention("", W, H, G, D, position=RotaryHalf(D, 50.0, rotary_dim=dims), names=names, bias_suffix=".b")
    part.bind_all(w, Runtime(torch.device("cpu"), torch.float32))
    inv, rot = part._rotation()
    assert rot == D and inv.numel() == D // 2 and float(inv[2:].abs().max()) == 0.0
    x, pos = torch.randn(6, W, generator=g), torch.arange(6) * 3
    proj = (x @ part.qkv.weight.T + part.qkv.bias).double()
    qkv = [proj[:, :H * D].view(6, H, D), proj[:, H * D:(H + G) * D].view(6, G, D), proj[:, (H + G) * D:].view(6, G, D)]
    a = (pos[:, None].float() * inv[None, :]).double()[:, None, :]

    def whole(t):
        u, v = t[..., :D // 2], t[..., D // 2:]
        return torch.cat([u * torch.cos(a) - v * torch.sin(a), u * torch.sin(a) + v * torch.cos(a)], -1)
    q, k = whole(qkv[0]), whole(qkv[1])
    r = dict(dims=dims, base=50.0)
    f = lambda n, heads: (x @ w[n].T + w[n + ".b"]).double().view(6, heads, D)
    q2, k2 = PN.rotate_halves(f("q", H), pos, r), PN.rotate_halves(f("k", G), pos, r)
    s = torch.einsum("thd,shd->hts", q, k.repeat_interleave(H // G, 1))
    s2 = torch.einsum("thd,shd->hts", q2, k2.repeat_interleave(H // G, 1))
    assert torch.allclose(s, s2, atol=1e-4) and torch.allclose(qkv[2], f("v", G), atol=1e-5)
    # whole rotations, odd head sizes and no rotation keep the order
    for hd, dims in ((10, 10), (9, 4)):
        p = Attention("", W, H, G, hd, position=RotaryHalf(hd, 50.0, rotary_dim=dims), names=names)
        assert p._order is None and not p.qkv.row_order


def test_frequencies_by_bands_of_wavelengths():
    from synaptix_b200.parts import FrequencyBands, RotaryHalf, RotaryPairs, Runtime
    for dims, base, bands in ((16, 3.0e4, (5.0, 1.0, 3.0, 400.0)), (6, 9000.0, (3.0, 0.5, 6.0, 60.0)), (32, 4.0e6, (6.0, 1.2, 4.5, 90.0)),
                              (8, 10.0, (2.0, 1.5, 1.5, 30.0))):
        rot = dict(dims=dims, base=base, scaling=dict(zip(("factor", "low", "high", "original"), bands)))
        want = PN.frequencies(rot)
        for cls in (RotaryHalf, RotaryPairs):
            p = cls(dims, base, scaling=FrequencyBands(*bands))
            p.bind({}, Runtime(torch.device("cpu"), torch.float32))
            assert torch.equal(p.inv_freq, want.to(torch.float32)) and p.magnitude == 1.0
    # all three branches occur, and the blend meets both ends
    rot = dict(dims=64, base=1.0e4, scaling=dict(factor=4.0, low=1.0, high=4.0, original=256.0))
    f, plain = PN.frequencies(rot).numpy(), PN.frequencies(dict(dims=64, base=1.0e4)).numpy()
    turns = 256.0 * plain / (2 * math.pi)
    assert np.allclose(f[turns > 4], plain[turns > 4]) and np.allclose(f[turns < 1], plain[turns < 1] / 4)
    mid = (turns >= 1) & (turns <= 4)
    assert mid.any() and (turns > 4).any() and (turns < 1).any()
    assert (f[mid] <= plain[mid]).all() and (f[mid] >= plain[mid] / 4).all()
    s = (turns[mid] - 1) / 3
    assert np.allclose(f[mid] / plain[mid], (1 - s) / 4 + s)


def test_sink_as_a_key_with_a_value_of_zero():
    """A sink is an additional key of that score whose value is zero."""
    g = torch.Generator().manual_seed(2)
    s, v = 2 * torch.randn(5, 9, generator=g).double(), torch.randn(9, 3, generator=g).double()
    see = torch.rand(5, 9, generator=g) < 0.6
    see[:, 0] = True
    for sink in (-3.0, 0.0, 5.0):
        got = PN.weights_beside_a_sink(s, see, torch.tensor(sink, dtype=F)) @ v
        more = torch.cat([s.masked_fill(~see, -math.inf), torch.full((5, 1), sink, dtype=F)], 1)
        assert torch.allclose(got, torch.softmax(more, -1) @ torch.cat([v, torch.zeros(1, 3, dtype=F)]))
        e = torch.exp(s) * see
        assert torch.allclose(got, (e / (math.exp(sink) + e.sum(-1, keepdim=True))) @ v)


def test_latent_attention_in_the_latents_space():
    """Keys taken into the query and values applied behind the weights give the same sums as per-head keys and values."""
    g = torch.Generator().manual_seed(3)
    T, width = 11, 16
    m = dict(heads=2, dim=5, rot_dim=4, vdim=6, q_rank=7, kv_rank=8, scale=0.4, rot=dict(dims=4, base=30.0), mask=dict(size=4))
    H, D, Dr, Dv, R = 2, 5, 4, 6, 8
    W = {"dq": (7, width), "uq": (H * (D + Dr), 7), "dkv": (R + Dr, width), "uk": (H * D, R), "uv": (H * Dv, R), "g": (H * Dv, width),
         "o": (width, H * Dv), "dq.norm": (7,), "dkv.norm": (R,), "sink": (H,)}
    W = {n: torch.randn(*s, generator=g).double() for n, s in W.items()}
    h, pos, eps = torch.randn(T, width, generator=g).double(), torch.arange(T), 1e-5
    c = PN.unit_rms((h @ W["dkv"].T)[:, :R], eps) * W["dkv.norm"]
    kr = PN.rotate_neighbours((h @ W["dkv"].T)[:, R:], pos, m["rot"])
    q = ((PN.unit_rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).view(T, H, D + Dr)
    qr = PN.rotate_neighbours(q[..., D:], pos, m["rot"])
    rows = []
    for t in range(T):
        heads = []
        for hh in range(H):
            ql = W["uk"][hh * D:(hh + 1) * D].T @ q[t, hh, :D]
            js = range(max(0, t - 3), t + 1)
            e = torch.stack([torch.exp((ql @ c[j] + qr[t, hh] @ kr[j]) * 0.4) for j in js])
            lat = (e[:, None] * c[list(js)]).sum(0) / (e.sum() + torch.exp(W["sink"][hh]))
            heads.append(W["uv"][hh * Dv:(hh + 1) * Dv] @ lat)
        rows.append(torch.cat(heads) * torch.sigmoid(W["g"] @ h[t]))
    assert torch.allclose(torch.stack(rows) @ W["o"].T, PN.latent_attention(h, W, "", m, pos, eps), atol=1e-10)


def test_norm_and_activation_values():
    W = {"n": torch.tensor([2.0, -1.0, 0.5], dtype=F), "n.b": torch.tensor([0.1, 0.2, 0.3], dtype=F), "n.alpha": torch.tensor(0.5, dtype=F)}
    x = torch.tensor([[0.0, 1.0, -40.0]], dtype=F)
    assert torch.allclose(PN.squash(x, W, "n"), torch.tensor([[0.1, 0.2 - math.tanh(0.5), 0.3 - 0.5]], dtype=F))
    z = torch.linspace(-6, 6, 41, dtype=F)
    assert torch.allclose(PN.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert torch.allclose(PN.soft_limit(z, 3.0), 3.0 * torch.tanh(z / 3.0)) and float(PN.soft_limit(z * 100, 3.0).abs().max()) <= 3.0


def test_a_block_without_a_feed_forward_and_linear_biases_as_data():
    from synaptix_b200.parts import DynamicTanh, GeluGLU, Linear, NoPosition, Attention, PreNormBlock
    a = Attention("m.", 8, 2, 1, 4, position=NoPosition(), own_kv=False, sink_score=0.0)
    assert a.cache_request() is None and [n for n, _ in a.input_parts()] == ["m.q_proj.weight"]
    block = PreNormBlock(DynamicTanh("n", 8), a, None, None)
    assert "n.alpha" in block.all_tensor_specs()
    with pytest.raises(ValueError):
        PreNormBlock(DynamicTanh("n", 8), a, DynamicTanh("n2", 8), None)
    with pytest.raises(ValueError):
        Attention("m.", 8, 2, 1, 4, position=NoPosition(), sinks=True, sink_score=0.0)
    l = Linear(["a", "b"], 4, [3, 2], bias_suffix=".bias")
    assert tuple(l.tensor_specs()["b.bias"].shape) == (2,)
    from synaptix_b200.parts import Runtime
    t = {"a": torch.ones(3, 4), "b": torch.zeros(2, 4), "a.bias": torch.arange(3.0), "b.bias": torch.arange(2.0) + 7}
    l.bind(t, Runtime(torch.device("cpu"), torch.bfloat16))
    assert l.bias.dtype == torch.float32 and l.bias.tolist() == [0, 1, 2, 7, 8]
    assert {"f.gate_proj.weight.b", "f.down_proj.weight.b"} <= set(GeluGLU("f.", 4, 6, bias_suffix=".b").all_tensor_specs())
