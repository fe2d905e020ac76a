"""What needs no GPU of the Zekalorn decoder: its configuration, the model as data (tensor names, cache requests, order of
the runs), the plain implementation against other forms of its own equations, and the limit on positions."""
import copy
import math

import pytest
import torch

import plain_zekalorn as PZ
from tiny_zekalorn import CONFIGS

F = torch.float64


def cfg_of(name):
    from synaptix_b200.config import ZekalornConfig
    return ZekalornConfig.from_dict(CONFIGS[name][0])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_round_trip_and_registry(name):
    from synaptix_b200.config import ZekalornConfig, resolve_architecture
    d = CONFIGS[name][0]
    cfg = cfg_of(name)
    assert ZekalornConfig.from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == d
    assert resolve_architecture(d).config_cls is ZekalornConfig
    assert [l.type for l in cfg.layers] == [l["type"] for l in d["layers"]]
    assert cfg.runs() == PZ.run_order(d)


def test_configuration_errors():
    from synaptix_b200.config import ConfigError, ZekalornConfig
    base = CONFIGS["ZA"][0]

    def broken(change):
        d = copy.deepcopy(base)
        change(d)
        with pytest.raises(ConfigError):
            ZekalornConfig.from_dict(d)
    broken(lambda d: d.pop("max_positions"))
    broken(lambda d: d["embedding"].pop("scale"))
    broken(lambda d: d["layers"][0].update(type="other"))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="other"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mixer"].pop("bias_max"))
    broken(lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=0))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=4))
    broken(lambda d: d["layers"][1]["mixer"].pop("conv"))
    broken(lambda d: d["layers"][1]["mixer"].update(heads=3))                         # over 2 kv heads
    broken(lambda d: d["token_side"].update(dim=0))
    broken(lambda d: d["loop"].update(stop=6))
    broken(lambda d: d["loop"].pop("times"))
    broken(lambda d: d.update(layers=[]))


def test_model_as_data():
    from synaptix_b200.cache.store import KVRequest
    from synaptix_b200.models import Inject, model_skeleton
    m = model_skeleton(cfg_of("ZA"))
    assert [r.layer for r in m.schedule] == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert [s.row for s in m.steps if isinstance(s, Inject)] == [0, 1, 2] and isinstance(m.steps[1], Inject)
    reqs = m.cache_requests()
    assert len(reqs) == 9 and reqs[0] == KVRequest(3, 10, None, 14)
    state, ring = reqs[1].items
    assert tuple(state.shape) == (4, 12, 20) and tuple(ring.shape) == (4, 2 * 2 * 12 + 4 * 20)
    specs = m.all_tensor_specs()
    assert tuple(specs["side.embed"].shape) == (97, 30) and tuple(specs["loop.step"].shape) == (3, 52)
    assert tuple(specs["l1.mix.a2"].shape) == (48, 5) and tuple(specs["l1.mix.g1"].shape) == (7, 52)
    assert tuple(specs["l1.mix.q.conv"].shape) == (24, 4) and tuple(specs["l0.mix.rel"].shape) == (10, 6)
    assert "l0.mlp.e4.up" in specs and "l0.mlp.e0.gate" not in specs and "l3.mlp.gate" not in specs and "l0.norm2" not in specs
    assert tuple(specs["pos"].shape) == (900, 52) and m.max_positions == 900
    b = model_skeleton(cfg_of("ZB"))
    assert "side.embed" not in b.all_tensor_specs() and "loop.step" not in b.all_tensor_specs()


def test_sizes_that_only_the_tensors_give():
    """The ranks and the number of distance buckets may be absent from the configuration: the tensors' own sizes count."""
    from synaptix_b200.config import ZekalornConfig
    from synaptix_b200.models import model_skeleton
    from synaptix_b200.weights.loader import check_tensors
    d = copy.deepcopy(CONFIGS["ZA"][0])
    shapes = {n: tuple(s.shape) for n, s in model_skeleton(ZekalornConfig.from_dict(d)).all_tensor_specs().items()}
    for layer in d["layers"]:
        for key in ("decay_rank", "gate_rank", "bias_rows"):
            layer["mixer"].pop(key, None)
    check_tensors(model_skeleton(ZekalornConfig.from_dict(d)).all_tensor_specs(), shapes)


def test_delta_rule_against_the_product_of_transitions():
    """One step maps ``S`` to ``(I - b k k^T) diag(a) S + b k v^T``: the state after T steps as an explicit sum of products."""
    g = torch.Generator().manual_seed(1)
    T, D, V = 9, 5, 3
    q, k = torch.randn(T, D, generator=g).double(), torch.nn.functional.normalize(torch.randn(T, D, generator=g).double(), dim=-1)
    v, a, b = torch.randn(T, V, generator=g).double(), torch.rand(T, D, generator=g).double(), torch.rand(T, generator=g).double()
    got = PZ.delta_rule(q[:, None], k[:, None], v[:, None], a[:, None], b[:, None])[:, 0]
    M = [(torch.eye(D, dtype=F) - b[t] * torch.outer(k[t], k[t])) @ torch.diag(a[t]) for t in range(T)]
    for t in range(T):
        S = torch.zeros(D, V, dtype=F)
        for j in range(t + 1):
            X = b[j] * torch.outer(k[j], v[j])
            for l in range(j + 1, t + 1):
                X = M[l] @ X
            S += X
        assert torch.allclose(got[t], S.T @ q[t], atol=1e-12)


def test_delta_rule_recalls_what_was_written_last_under_a_key():
    """Step size 1 and no decay: reading with a unit key gives the value written under it last; other keys stay."""
    e = torch.eye(4, dtype=F)
    k = torch.stack([e[0], e[1], e[0], e[2]])[:, None]
    v = torch.arange(12, dtype=F).reshape(4, 1, 3)
    ones, b = torch.ones(4, 1, 4, dtype=F), torch.ones(4, 1, dtype=F)
    q = torch.stack([e[0], e[0], e[0], e[0] + e[1]])[:, None]
    o = PZ.delta_rule(q, k, v, ones, b)[:, 0]
    assert torch.equal(o[0], v[0, 0]) and torch.equal(o[1], v[0, 0]) and torch.equal(o[2], v[2, 0])
    assert torch.equal(o[3], v[2, 0] + v[1, 0])


def test_buckets_and_temperature():
    assert [PZ.bucket(n, 10, 50.0) for n in (0, 4)] == [0, 4]
    assert PZ.bucket(5, 10, 50.0) == 5 and PZ.bucket(50, 10, 50.0) == 9 and PZ.bucket(10 ** 6, 10, 50.0) == 9
    edges = [n for n in range(6, 60) if PZ.bucket(n, 10, 50.0) != PZ.bucket(n - 1, 10, 50.0)]
    assert len(edges) == 4                                                     # five logarithmic buckets: 5, 6, 7, 8, 9
    t = dict(coef=0.5, every=8)
    assert PZ.temperature(6, t) == 1.0 and PZ.temperature(7, t) == pytest.approx(1 + 0.5 * math.log(2))
    assert PZ.temperature(22, t) == PZ.temperature(15, t) != PZ.temperature(23, t)
    from synaptix_b200.parts.scored import distance_columns
    for rows, far in ((10, 50.0), (7, 90.0), (32, 200.0), (24, 300.0)):
        cols = distance_columns(rows, far, None)
        for n in range(2 * int(far)):
            assert int(cols[min(n, len(cols) - 1)]) == PZ.bucket(n, rows, far)


def test_weights_of_the_chosen_experts():
    z = torch.tensor([0.5, 2.0, 2.0, -1.0, 1.0], dtype=F)
    ids, w = PZ.choose_experts(z, 3)
    assert ids == [1, 2, 4] and torch.allclose(w, torch.softmax(z[ids], 0))
    full = torch.softmax(z, 0)
    assert torch.allclose(w, full[ids] / full[ids].sum())                      # the same numbers the other way


def test_generation_stops_at_the_last_position():
    """A session that refuses a step (the model has no further position) ends its longest sequence by capacity."""
    from synaptix_b200.cache.pages import CacheFull
    from synaptix_b200.engine.generate import GenerationOptions, run_generation

    class Session:
        def __init__(self, lens, limit):
            self.lens, self.limit, self.pending, self.in_flight = list(lens), limit, [], 0

        def launch(self, tokens=None):
            if max(self.lens) >= self.limit:
                raise CacheFull("no position is left")
            self.lens = [n + 1 for n in self.lens]
            self.pending.append([1] * len(self.lens))
            self.in_flight += 1

        def collect(self):
            self.in_flight -= 1
            return self.pending.pop(0)

        def drop(self, rows):
            self.lens = [n for i, n in enumerate(self.lens) if i not in set(rows)]

    class Engine:
        max_tokens, max_seqs = 640, 4

        def __init__(self):
            self.next = 0

        def open(self):
            self.next += 1
            return self.next - 1

        def close(self, slot):
            pass

        def step(self, entries, keep=True):
            self.lens = [len(e.tokens) for e in entries]
            return [[0.0]] * len(entries)

        def check_kernels(self):
            pass

        def start_decode(self, rows, sampling=None):
            return Session(self.lens, 10)
    res, _ = run_generation(Engine(), lambda lg, r, s, c: [1] * len(r), [[1] * 6, [1] * 3], GenerationOptions(max_new_tokens=50))
    assert [r.finish_reason for r in res] == ["capacity", "capacity"]
    assert [len(r.tokens) for r in res] == [5, 8]            # prompt + decoded tokens that ran = 10, and one more was sampled
