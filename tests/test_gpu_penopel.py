"""The Penopel decoder on the GPU against the plain implementation: each mechanism's kernels alone, then whole models
through the engine under every way of cutting the work into steps, portions and batches, and greedy generation through the
library's entry point.  Configurations and weights are made here (``tiny_penopel``)."""
import pytest
import torch

import helpers
import plain_penopel as PN
from test_gpu_pidutar import i32, near
from test_gpu_vemedra import portions, step_ctx
from tiny_penopel import CONFIGS, folder, oracle, oracle_logits, tokens

pytestmark = pytest.mark.gpu

NAMES = ["PA", "PB", "PF", "PG"]
DTYPES = ["float32", "bfloat16"]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


def runtime(dtype):
    from synaptix_b200.parts import Runtime
    return Runtime(torch.device("cuda:0"), DT[dtype])


def assert_close(got, ref, dtype, what=""):
    """Logits against the oracle's: 32-bit rows within the shared tolerance; bfloat16 rows within it but for one in twenty
    (which may be off twice as far: scores of these peaky attentions come out of 16-bit queries and keys)."""
    got, ref = got.detach().float().cpu(), ref.detach().float().cpu()
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    rel = (got - ref).abs().max(dim=1).values / ref.abs().max()
    if dtype == "float32":
        assert float(rel.max()) <= helpers.F32_REL, f"{what}: {float(rel.max()):.3e} at row {int(rel.argmax())}"
        return
    within = float((rel <= helpers.BF16_REL).float().mean())
    assert within >= 0.95 and float(rel.max()) <= 2 * helpers.BF16_REL, \
        f"{what}: {within:.3f} of {rel.numel()} rows within {helpers.BF16_REL}, worst {float(rel.max()):.4f} at {int(rel.argmax())}"


class Gathered:
    """Rows of many small steps, compared at once; 32-bit rows are compared as they come."""

    def __init__(self, dtype, what):
        self.dtype, self.what, self.got, self.ref = dtype, what, [], []

    def add(self, got, ref, what=""):
        if self.dtype == "float32":
            return assert_close(got, ref, self.dtype, f"{self.what} {what}")
        self.got.append(got.detach().float().cpu())
        self.ref.append(ref.detach().float().cpu())

    def check(self):
        if self.got:
            assert_close(torch.cat(self.got), torch.cat(self.ref), self.dtype, self.what)


# ---------------------------------------------------------------------------------------------------------------
# each mechanism alone
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width", [(1, 52), (3, 64), (300, 328), (2, 1001), (17, 2560)])
def test_norm_without_statistics(T, width, dtype):
    """Sum into the stream (a branch of either dtype, with and without a bias) and norm; all rows, and picked rows that leave
    the stream alone."""
    from synaptix_b200 import ops
    g = torch.Generator().manual_seed(T + width)
    h = torch.randn(T, width, generator=g) * 3
    w = {"n": 1 + 0.3 * torch.randn(width, generator=g), "n.b": torch.randn(width, generator=g), "n.alpha": torch.tensor(0.7)}
    bias = torch.randn(width, generator=g)
    wd = {k: v.double() for k, v in w.items()}
    for delta_dtype in (None, torch.float32, torch.bfloat16):
        for db in ((None, bias) if delta_dtype is not None else (None,)):
            d = None if delta_dtype is None else torch.randn(T, width, generator=g).to(delta_dtype)
            x = h.double() + (0 if d is None else d.double()) + (0 if db is None else db.double())
            rows = [T - 1, 0, T // 2]
            cuda = lambda t: None if t is None else t.cuda()
            hd = h.cuda()
            args = (0.7, w["n"].cuda(), w["n.b"].cuda(), DT[dtype])
            got = ops.add_dyn_tanh(hd, cuda(d), *args, delta_bias=cuda(db), rows=i32(rows))
            assert torch.equal(hd.cpu(), h)
            near(got.float().cpu(), PN.squash(x, wd, "n")[rows], dtype, f32=2e-6, bf16=6e-3)
            got = ops.add_dyn_tanh(hd, cuda(d), *args, delta_bias=cuda(db))
            near(got.float().cpu(), PN.squash(x, wd, "n"), dtype, f32=2e-6, bf16=6e-3)
            near(hd.cpu(), x, "float32", f32=1e-6)


# rows and sizes that take every product: few rows (mma.sync), weights streamed (tcgen05, one to eight blocks a tile), whole
# tiles, tiles cut over K behind whole ones, few tiles cut, K split with a second kernel, and sizes no fast product takes
PRODUCTS = [(1, 96, 64), (5, 100, 160), (8, 52, 60), (9, 256, 128), (16, 328, 72), (17, 130, 200), (40, 512, 512), (100, 2560, 1024),
            (160, 72, 88), (161, 256, 1024), (200, 100, 136), (300, 97, 52), (512, 2560, 4096), (700, 640, 320), (2048, 2560, 4096),
            (1100, 1024, 256)]


def _product_case(M, N, K, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    x = torch.randn(M, K, generator=g).to(DT[dtype])
    w = (torch.randn(N, K, generator=g) * K ** -0.5).to(DT[dtype])
    return g, x, w, torch.randn(N, generator=g)


def _times(x, w):
    """The product in 64-bit, on the GPU where it is large."""
    if x.shape[0] * w.shape[0] * w.shape[1] > 1 << 26:
        return (x.cuda().double() @ w.cuda().double().T).cpu()
    return x.double() @ w.double().T


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", PRODUCTS)
def test_products_with_biases_and_a_soft_limit(M, N, K, dtype):
    from synaptix_b200 import ops
    g, x, w, b = _product_case(M, N, K, dtype, M + N)
    ref = _times(x, w) + b.double()
    xc, wc, bc = x.cuda(), w.cuda(), b.cuda()
    near(ops.linear(xc, wc, bias=bc).float().cpu(), ref, dtype, f32=2e-5, bf16=8e-3)
    near(ops.linear(xc, wc, out_dtype=torch.float32, bias=bc).cpu(), ref, "float32", f32=2e-5)
    near(ops.linear(xc, wc, out_dtype=torch.float32, bias=bc, cap=1.5).cpu(), PN.soft_limit(ref, 1.5), "float32", f32=2e-5)
    near(ops.linear(xc, wc, out_dtype=torch.float32, cap=2.5).cpu(), PN.soft_limit(ref - b.double(), 2.5), "float32", f32=2e-5)
    if N % 2 == 0:
        with ops.gate_activation(form="gelu_tanh"):
            got = ops.linear(xc, wc, epilogue="silu_mul", bias=bc)
        near(got.float().cpu(), PN.gelu_tanh(ref[:, :N // 2]) * ref[:, N // 2:], dtype, f32=3e-5, bf16=8e-3)
    ops.check_status()


@pytest.mark.parametrize("M,N,K", PRODUCTS)
def test_products_that_end_in_the_stream_and_its_next_norm(M, N, K):
    """The sum into the 32-bit stream happens once per element (cut tiles and split K included), and the rows of the next norm
    are those of the sum; with and without a bias."""
    from synaptix_b200 import ops
    g, x, w, b = _product_case(M, N, K, "bfloat16", M * 3 + N)
    h = torch.randn(M, N, generator=g) * 2
    gain, shift = 1 + 0.3 * torch.randn(N, generator=g), torch.randn(N, generator=g)
    nw = {"n": gain.double(), "n.b": shift.double(), "n.alpha": torch.tensor(0.6, dtype=F)}
    for bias in (None, b):
        ref = h.double() + _times(x, w) + (0 if bias is None else bias.double())
        hd = h.cuda()
        y = ops.linear_into_dyn_tanh(x.cuda(), w.cuda(), None if bias is None else bias.cuda(), hd, 0.6, gain.cuda(), shift.cuda())
        if K % 8:
            assert y is None and torch.equal(hd.cpu(), h)
            continue
        near(hd.cpu(), ref, "float32", f32=2e-5)
        near(y.float().cpu(), PN.squash(ref, nw, "n"), "bfloat16", bf16=6e-3)
    with ops.options(fused_residual=False):
        assert ops.linear_into_dyn_tanh(x.cuda(), w.cuda(), None, h.cuda(), 0.6, gain.cuda(), shift.cuda()) is None
    ops.check_status()


@pytest.mark.parametrize("M", [1, 3, 33, 200, 600])
def test_norm_part_takes_products_fused_and_unfused_alike(M):
    """A branch's unrun product, its materialised form and the form with the option off leave the same stream and rows but
    for the branch's rounding to 16 bits."""
    from synaptix_b200 import ops
    from synaptix_b200.parts import DynamicTanh, PendingLinear
    g, x, w, b = _product_case(M, 128, 96, "bfloat16", M)
    h = torch.randn(M, 128, generator=g)
    n = DynamicTanh("n", 128)
    n.bind({"n": torch.ones(128), "n.b": torch.zeros(128), "n.alpha": torch.tensor(0.5)}, runtime("bfloat16"))
    outs = []
    for form in ("fused", "plain", "materialised"):
        hd, p = h.cuda(), PendingLinear(x.cuda(), w.cuda(), b.cuda())
        if form == "materialised":
            p.materialize()
        with ops.options(fused_residual=form == "fused"):
            outs.append((n.add_forward(hd, p).float().cpu(), hd.cpu()))
    for y, hh in outs[1:]:
        assert float((y - outs[0][0]).abs().max()) <= 1.2e-2 and float((hh - outs[0][1]).abs().max()) <= 2e-2


def _attention_weights(W, H, G, dim, vdim, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    p = "m."
    w = {p + "q": torch.randn(H * dim, W, generator=g) * 0.3, p + "k": torch.randn(G * dim, W, generator=g) * 0.3,
         p + "v": torch.randn(G * vdim, W, generator=g) * 0.3, p + "o": torch.randn(W, H * vdim, generator=g) * 0.3,
         p + "q.b": 0.3 * torch.randn(H * dim, generator=g), p + "k.b": 0.3 * torch.randn(G * dim, generator=g),
         p + "v.b": 0.3 * torch.randn(G * vdim, generator=g)}
    return g, {k: v.to(DT[dtype]) for k, v in w.items()}


ROT = {"none": None, "quarter": dict(base=3.0e3), "bands": dict(base=1.0e4, scaling=dict(factor=4.0, low=1.0, high=5.0, original=150.0))}
SHAPES = [(6, 3, 10, 14, 6, "bands"), (4, 2, 64, 64, 16, "bands"), (4, 1, 128, 128, 128, "quarter"), (4, 4, 128, 128, 64, "bands"),
          (2, 2, 32, 32, 8, "quarter"), (8, 1, 40, 24, 40, "bands"), (3, 3, 7, 5, 4, "quarter"), (5, 5, 16, 16, 0, "none"),
          (2, 1, 64, 64, 64, "quarter"), (1, 1, 48, 48, 2, "quarter")]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,dims,rot", SHAPES)
def test_attention_with_a_sink_of_score_zero_and_another_layers_keys(H, G, dim, vdim, dims, rot, dtype):
    """The whole mixer, and a second one that reads its keys and values with queries and a scale of its own, over portions of
    several sizes with NaN in every page no step wrote.  In one sequence far keys are made to point the way of late queries,
    so that one score stands out among hundreds (position 0, either side of a page's border, just before the query, the query
    itself).  In another, some queries are turned away from every key, so that the sink takes nearly all of the weight."""
    from synaptix_b200.cache.store import KVView
    from synaptix_b200.models.penopel import _position
    from synaptix_b200.config.penopel import RotationSpec
    from synaptix_b200.parts import Attention, RotaryHalf
    W, p = 48, "m."
    g, w = _attention_weights(W, H, G, dim, vdim, dtype, H * dim + dims)
    _, w2 = _attention_weights(W, H, G, dim, vdim, dtype, H * dim + dims + 1)
    lengths = [290, 70, 1]
    xs = [torch.randn(n, W, generator=g) for n in lengths]
    kq = w[p + "k"][:dim].double().T @ w[p + "q"][:dim].double()                  # x_j . (Wk^T Wq) x_i of head 0
    direction = torch.randn(W, generator=g)
    toward = (kq @ direction.double()).float()
    scale = 0.4
    pairs = [(289, 0), (200, 63), (130, 64), (280, 279), (250, 250)]
    for i, j in pairs:
        xs[0][j] = toward * (7.0 / float(toward.norm()))
        if i != j:
            xs[0][i] = direction * (9.0 / (scale * 7.0 * float(toward.norm())))
    # sequence 1: every key of head 0 has a large part that does not depend on the token; queries turned against it
    away = [3, 40, 69] if dims < dim else []
    if away:
        kb = w[p + "k.b"].float()
        kb[dims:dim] = 8.0 * (dim - dims) ** -0.5
        w[p + "k.b"] = kb.to(DT[dtype])
        wq = w[p + "q"][:dim].double()
        back = torch.linalg.lstsq(wq, -torch.cat([torch.zeros(dims), torch.full((dim - dims,), 1.0)]).double().unsqueeze(1)).solution[:, 0]
        if dim > W:                                                               # (as near as the width allows)
            back = -(wq[dims:].sum(0))
            back = back / float((wq[dims:] @ back).abs().mean())
        for i in away:
            xs[1][i] = (back * (10.0 / (scale * 8.0 * (dim - dims) ** 0.5))).float()
    xs = [x.to(DT[dtype]) for x in xs]
    m = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, scale=scale)
    if dims:
        m["rot"] = dict(ROT[rot], dims=dims)
    m2 = dict(m, scale=0.25)
    refs, refs2 = [], []
    for s, x in enumerate(xs):
        pos, wd, wd2 = torch.arange(x.shape[0]), {k: v.double() for k, v in w.items()}, {k: v.double() for k, v in w2.items()}
        mem = PN.attention_memory(x.double(), wd, p, m, pos)
        refs.append(PN.attention(x.double(), wd, p, m, pos, mem))
        refs2.append(PN.attention(x.double(), wd2, p, m2, pos, mem))
    if away and dim <= W:                                                         # the test's own premise
        wd, x = {k: v.double() for k, v in w.items()}, xs[1].double()
        q0 = PN.affine(x, wd, p + "q").view(-1, H, dim)[:, 0]
        k0 = PN.attention_memory(x, wd, p, dict(m, rot=None), torch.arange(70))[0][:, 0]
        s0 = (q0[:, dims:] @ k0[:, dims:].T) * scale                              # what the rotation leaves alone
        assert all(float(torch.exp(s0[i, :i + 1]).sum()) < 0.5 for i in away)
    spec = RotationSpec.from_dict(m["rot"], "rot") if dims else None
    kw = dict(v_head_dim=vdim, sink_score=0.0, bias_suffix=".b", names=dict(q="q", k="k", v="v", o="o"))
    part = Attention(p, W, H, G, dim, position=_position(RotaryHalf, dim, spec), scale=scale, **kw)
    part2 = Attention(p, W, H, G, dim, position=_position(RotaryHalf, dim, spec), scale=0.25, own_kv=False, **kw)
    part.bind_all(w, runtime(dtype))
    part2.bind_all({k: v for k, v in w2.items() if k[2] in "qo"}, runtime(dtype))
    tables = [[1, 2, 3, 4, 5], [6, 7, 0, 0, 0], [8, 0, 0, 0, 0]]
    for cuts in ([300], [1] * 290, [2] * 145, [129, 1, 70, 1, 1, 90], [16, 48, 100, 7, 3, 300]):
        k = torch.full((9, G, 64, dim), float("nan"), dtype=DT[dtype]).cuda()
        v = torch.full((9, G, 64, vdim), float("nan"), dtype=DT[dtype]).cuda()
        view = KVView(k, v, 0, None)
        outs, outs2 = [[] for _ in lengths], [[] for _ in lengths]
        for past, new, who in portions(lengths, cuts):
            ctx = step_ctx(past, new, who, [i32([tables[i] for i in who])], DT[dtype])
            x = torch.cat([xs[i][a:a + n] for i, a, n in zip(who, past, new)]).cuda()
            y, y2 = part.forward(x, ctx, view), part2.forward(x, ctx, view, False)
            at = 0
            for i, n in zip(who, new):
                outs[i].append(y[at:at + n].float().cpu())
                outs2[i].append(y2[at:at + n].float().cpu())
                at += n
        for o, r in zip(outs, refs):            # (scores of 20 and more out of 16-bit queries and keys)
            near(torch.cat(o), r, dtype, f32=2e-4, bf16=5e-2)
        for o, r in zip(outs2, refs2):
            near(torch.cat(o), r, dtype, f32=2e-4, bf16=5e-2)
    with pytest.raises(ValueError):
        part2.forward(x, ctx, view, True)


def _plain_sink_attention(q, k, v, lens, scale, window, sinks):
    """One query a sequence (its last position) over ``lens`` keys in 64-bit: [S, H, hd]."""
    S, H, hd = q.shape
    G = k[0].shape[1]
    out = torch.zeros(S, H, v[0].shape[2], dtype=F)
    for s in range(S):
        lo = 0 if window is None else max(0, lens[s] - window)
        for h in range(H):
            sc = (k[s][lo:, h // (H // G)].double() @ q[s, h].double()) * scale
            see = torch.ones(1, sc.numel(), dtype=torch.bool)
            out[s, h] = (PN.weights_beside_a_sink(sc[None], see, sinks[h].double()) @ v[s][lo:, h // (H // G)].double())[0]
    return out


@pytest.mark.parametrize("H,G,hd", [(8, 2, 128), (6, 2, 64), (4, 4, 32), (16, 1, 64), (16, 1, 128)])
@pytest.mark.parametrize("window", [None, 200])
def test_sinks_in_single_token_attention_over_many_keys(H, G, hd, window):
    """Every form of the single-token kernels (one block a sequence, parts merged in a cluster, parts merged by a second
    kernel, many parts, parts that see nothing of a window): the sink counts exactly once, whether it outweighs the keys or
    vanishes."""
    from synaptix_b200 import ops
    g = torch.Generator().manual_seed(H + hd)
    lens = [1500, 64, 1, 700]
    S, scale = len(lens), 0.5 * hd ** -0.5
    sinks = torch.linspace(-4, 11, H)
    q = torch.randn(S, H, hd, generator=g).to(torch.bfloat16)
    ks = [torch.randn(n, G, hd, generator=g).to(torch.bfloat16) for n in lens]
    vs = [(2 + torch.randn(n, G, hd, generator=g)).to(torch.bfloat16) for n in lens]
    maxp = 24
    n_pages = 1 + sum((n + 63) // 64 for n in lens)
    kp = torch.full((n_pages, G, 64, hd), float("nan"), dtype=torch.bfloat16)
    vp = kp.clone()
    table, nxt = torch.zeros(S, maxp, dtype=torch.int32), 1
    for s, n in enumerate(lens):
        for j in range((n + 63) // 64):
            rows = ks[s][j * 64:(j + 1) * 64]
            kp[nxt, :, :rows.shape[0]] = rows.transpose(0, 1)
            vp[nxt, :, :rows.shape[0]] = vs[s][j * 64:(j + 1) * 64].transpose(0, 1)
            table[s, j] = nxt
            nxt += 1
    kp, vp, bt, sl, qc, sc = kp.cuda(), vp.cuda(), table.cuda(), i32(lens), q.reshape(S, -1).cuda(), sinks.cuda()
    ref = _plain_sink_attention(q, ks, vs, lens, scale, window, sinks).reshape(S, -1)
    none = _plain_sink_attention(q, ks, vs, lens, scale, window, torch.full((H,), -1e30)).reshape(S, -1)
    assert float((ref - none).abs().max()) > 0.3 * float(ref.abs().max())         # the sinks matter here
    for splits in (1, 2, 3, 4, 7, 16, 24):
        got = ops.attn_decode(qc, kp, vp, sl, bt, H, G, hd, scale, window, splits, sinks=sc)
        near(got.float().cpu(), ref, "bfloat16", bf16=1e-2)
        if hd >= 64:
            for cluster in (False, True):
                got = ops.attn_decode_tma(qc, kp, vp, sl, bt, H, G, hd, scale, window, splits, sinks=sc, cluster=cluster)
                near(got.float().cpu(), ref, "bfloat16", bf16=1e-2)
    # heads prepared in the kernel from a projection of the queries alone, against a cache that holds the token
    kw = dict(wq=None, wk=None, inv_freq=None, eps=0.0, write_cache=False, sinks=sc)
    if hd >= 64:
        near(ops.attn_decode_tma(qc, kp, vp, sl, bt, H, G, hd, scale, window, 4, prep=True, **kw).float().cpu(), ref, "bfloat16", bf16=1e-2)
    near(ops.attn_decode_prep(qc, kp, vp, sl, bt, H, G, hd, scale, window, 3, None, None, None, 0.0, False, sinks=sc).float().cpu(),
         ref, "bfloat16", bf16=1e-2)
    ops.check_status()


LATENTS = [(3, 6, 4, 10, 14, 12, 37), (2, 7, 2, 9, 10, 18, 5), (5, 28, 12, 36, 40, 48, 90), (3, 40, 24, 64, 40, 48, 100), (4, 24, 8, 32, 24, 32, 64),
           (2, 96, 32, 128, 64, 64, 200), (1, 3, 8, 8, 5, 9, None), (9, 16, 16, 32, 24, 72, 1), (2, 64, 64, 128, 32, 520, None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,vdim,rq,rk,window", LATENTS)
def test_latent_attention_with_sinks_and_a_gate_per_element(H, dim, rot, vdim, rq, rk, window, dtype):
    """The whole mixer over portions of several sizes (whole prompts of enough tokens form per-head keys and values), NaN in
    every page no step wrote, sinks from one that outweighs everything to one that vanishes.  Keys are made to stand out just
    inside the window of a late query and just outside it, at page borders, and far behind."""
    from synaptix_b200.cache.store import KVView
    from synaptix_b200.parts import LatentAttention, NoPosition, RotaryPairs
    g = torch.Generator().manual_seed(H * dim + rk)
    W, p, base, scale, eps = 56, "m.", 800.0, 0.35, 1e-5
    sizes = {"dq": (rq, W), "uq": (H * (dim + rot), rq), "dkv": (rk + rot, W), "uk": (H * dim, rk), "uv": (H * vdim, rk),
             "g": (H * vdim, W), "o": (W, H * vdim)}
    w = {p + n: torch.randn(*sz, generator=g) * sz[1] ** -0.5 for n, sz in sizes.items()}
    w[p + "dq.norm"], w[p + "dkv.norm"] = 1 + 0.2 * torch.randn(rq, generator=g), 1 + 0.2 * torch.randn(rk, generator=g)
    w[p + "sink"] = torch.linspace(-3.0, 5.0, H) if H > 1 else torch.tensor([1.0])
    w = {k: v.to(DT[dtype]) for k, v in w.items()}
    wd = {k: v.double() for k, v in w.items()}
    lengths = [300, 70, 1]
    xs = [torch.randn(n, W, generator=g) for n in lengths]
    # a latent that head 0 of a certain query scores far above the others': x_j is chosen by the query's own key direction
    win = window or 400
    for i, back in ((299, win - 1), (260, win), (200, min(win - 1, 199)), (190, 1), (150, 150), (128, 64), (127, 63)):
        j = i - back
        if j < 0:
            continue
        x64 = xs[0][i].double()
        q0 = ((PN.unit_rms(x64 @ wd[p + "dq"].T, eps) * wd[p + "dq.norm"]) @ wd[p + "uq"].T)[:dim]
        want = (wd[p + "uk"][:dim].T @ q0) / wd[p + "dkv.norm"].abs().clamp(min=0.1)
        xs[0][j] = (torch.linalg.pinv(wd[p + "dkv"][:rk]) @ want).float()
        xs[0][j] *= W ** 0.5 / float(xs[0][j].norm())
    xs = [x.to(DT[dtype]) for x in xs]
    m = dict(heads=H, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rk, scale=scale)
    if rot != 8:
        m["rot"] = dict(dims=rot, base=base)
    if window:
        m["mask"] = dict(size=window)
    refs = [PN.latent_attention(x.double(), wd, p, m, torch.arange(x.shape[0]), eps) for x in xs]
    part = LatentAttention(p, W, H, dim, rot, vdim, rq, rk, scale=scale, norm_eps=eps, window=window, gated="elements", sinks=True,
                           position=RotaryPairs(rot, base) if rot != 8 else NoPosition())
    part.bind_all(w, runtime(dtype))
    assert (part.ukv is not None) == (dtype == "bfloat16" and dim + rot == vdim and vdim in (32, 64, 128) and rk % 8 == 0)
    tables = [[1, 2, 3, 4, 5], [6, 7, 0, 0, 0], [8, 0, 0, 0, 0]]
    for cuts in ([300], [1] * 300, [2] * 150, [129, 1, 70, 1, 1, 100], [16, 48, 100, 7, 3, 300]):
        pages = torch.full((9, 1, 64, rk + rot), float("nan"), dtype=DT[dtype]).cuda()
        view = KVView(pages, None, 0, window)
        outs = [[] for _ in lengths]
        for past, new, who in portions(lengths, cuts):
            ctx = step_ctx(past, new, who, [i32([tables[i] for i in who])], DT[dtype])
            y = part.forward(torch.cat([xs[i][a:a + n] for i, a, n in zip(who, past, new)]).cuda(), ctx, view)
            at = 0
            for i, n in zip(who, new):
                outs[i].append(y[at:at + n].float().cpu())
                at += n
        for o, r in zip(outs, refs):
            near(torch.cat(o), r, dtype, f32=2e-4, bf16=4e-2)
    y2 = part.forward(xs[2].cuda(), step_ctx([0], [1], [2], [i32([tables[2]])], DT[dtype]), view, defer_output=True)
    near(y2.materialize().float().cpu(), refs[2], dtype, f32=2e-4, bf16=4e-2)


@pytest.mark.parametrize("splits", [1, 2, 5])
def test_the_latents_sink_counts_once_over_parts(splits):
    from synaptix_b200 import ops
    g = torch.Generator().manual_seed(5)
    H, R, Dr, Dv, n = 3, 24, 8, 10, 150
    rows = torch.randn(n, R + Dr, generator=g)
    pages = torch.zeros(4, 1, 64, R + Dr)
    pages[1:, 0] = torch.cat([rows, torch.zeros(192 - n, R + Dr)]).view(3, 64, R + Dr)
    qa = torch.randn(1, H, R + Dr, generator=g)
    sinks, wuv, gate = torch.tensor([-2.0, 3.0, 9.0]), torch.randn(H * Dv, R, generator=g), torch.randn(1, 4 + H * Dv, generator=g)
    ctx = step_ctx([n - 1], [1], [0], None)
    bt = i32([[1, 2, 3]])
    ol = ops.latent_attention(qa.cuda(), pages.cuda(), ctx, bt, H, R, Dr, 0.5, None, splits=splits)
    s = (qa[0].double() @ rows.double().T) * 0.5
    want = torch.stack([PN.weights_beside_a_sink(s[h:h + 1], torch.ones(1, n, dtype=torch.bool), sinks[h].double())[0] @ rows[:, :R].double()
                        for h in range(H)])
    near(ol.merged(sinks.cuda())[0].cpu(), want, "float32")
    got = ops.latent_output(ol, wuv.cuda(), H, Dv, R, gate.cuda(), 4, torch.float32, sinks=sinks.cuda(), gate_elements=True).cpu()
    ref = torch.cat([wuv[h * Dv:(h + 1) * Dv].double() @ want[h] for h in range(H)]) * torch.sigmoid(gate[0, 4:].double())
    near(got[0], ref, "float32")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width,ff", [(1, 52, 44), (9, 128, 96), (70, 256, 320), (300, 96, 200), (600, 256, 512)])
def test_feed_forward_with_biases(T, width, ff, dtype):
    from synaptix_b200.parts import GeluGLU
    g = torch.Generator().manual_seed(T + ff)
    w = {}
    for n, (o, i) in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
        w["f." + n] = torch.randn(o, i, generator=g) * 1.5 * i ** -0.5
        w["f." + n + ".b"] = torch.randn(o, generator=g)
    w = {k: v.to(DT[dtype]) for k, v in w.items()}
    x = torch.randn(T, width, generator=g).to(DT[dtype])
    ref = PN.feed_forward(x.double(), {k: v.double() for k, v in w.items()}, "f.")
    part = GeluGLU("f.", width, ff, names=dict(gate="gate", up="up", down="down"), bias_suffix=".b")
    part.bind_all(w, runtime(dtype))
    near(part.forward(x.cuda(), None).float().cpu(), ref, dtype, f32=2e-4, bf16=2e-2)
    near(part.forward(x.cuda(), None, defer_output=True).materialize().float().cpu(), ref, dtype, f32=2e-4, bf16=2e-2)


# ---------------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def engines():
    from synaptix_b200.engine import Engine
    from synaptix_b200.models import load_model
    made = {}

    def get(name, dtype, max_tokens=2048, max_seqs=None):
        key = (name, dtype, max_tokens, max_seqs)
        if key not in made:
            eng = Engine(load_model(folder(name), dtype=dtype), max_tokens=max_tokens, max_seqs=max_seqs)
            for t in eng.cache._k + eng.cache._v:                 # a place no step wrote shows at once when it is read
                t.fill_(float("nan"))
                t[:, 0] = 0.0                                     # (page 0 stands for pages given back: finite, masked)
            made[key] = eng
        assert made[key].cache.slots.n_live == 0
        return made[key]
    return get


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_every_place(engines, name, dtype):
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    assert type(eng.model.config).__name__ == "PenopelConfig" and eng.use_graphs
    rows = Gathered(dtype, f"{name} {dtype} whole prompts")
    for i, n in enumerate([1, 2, 3, 17, 32, 63, 64, 65, 150, 301, 690]):
        toks = tokens(name, n, 100 + i)
        s = eng.open()
        got = eng.step([Entry(s, toks, list(range(n)))])
        eng.close(s)
        rows.add(got, oracle_logits(name, tuple(toks)), f"n={n}")
    rows.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer(engines, name, fused, dtype):
    """Layer by layer, with the norms finished in the products' epilogues and with every operation a kernel of its own."""
    from synaptix_b200 import ops
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    toks = tokens(name, 190, 4)
    cfg, W = oracle(name)
    ref, seen = [], []
    PN.forward(cfg, W, toks, ref)
    s = eng.open()
    entries = [Entry(s, toks, [0])]
    past, new = eng._check(entries)
    ctx = eng.plan(entries, past, new)
    ctx.observe = lambda n, h, pending: seen.append((h + pending.float()).cpu() if pending is not None else h.cpu().clone())
    with ops.options(fused_residual=fused):
        eng._forward(ctx)
    eng.cache.slots.advance(s, len(toks))
    eng.close(s)
    assert len(seen) == len(ref) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, ref)):
        near(a, b, dtype, f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first_token(engines, name, dtype):
    """Every token a step of its own (captured steps): the first tokens, where the sinks weigh most, and on across page
    borders and windows."""
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    toks = tokens(name, 230, 8)
    s = eng.open()
    got = torch.cat([eng.step([Entry(s, [t], [0])]) for t in toks])
    eng.close(s)
    assert_close(got, oracle_logits(name, tuple(toks)), dtype, f"{name} {dtype} token by token")
    assert any(c.graph is not None for c in eng._captured.values())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("size", [2, 3, 7, 33, 64, 100, 270])
def test_prompts_in_portions(engines, name, dtype, size):
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    toks = tokens(name, 301, 20)
    s = eng.open()
    got = [eng.step([Entry(s, toks[a:a + size], list(range(len(toks[a:a + size]))))]) for a in range(0, len(toks), size)]
    eng.close(s)
    assert_close(torch.cat(got), oracle_logits(name, tuple(toks)), dtype, f"{name} {dtype} portions of {size}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_in_slots_and_pages_used_again(engines, name, dtype):
    """Batches of unequal prompts decoded together, shorter requests ending earlier; the cache holds little more than one
    batch and three slots, so every batch runs in slots and pages that the batch before gave back."""
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype, max_tokens=512, max_seqs=3)
    for b, (lens, decodes) in enumerate([([5, 130, 1], [3, 40, 12]), ([64, 9, 200], [10, 30, 2]), ([2, 3, 100], [25, 1, 70])]):
        seqs = [tokens(name, n + d, 300 + 10 * b + i) for i, (n, d) in enumerate(zip(lens, decodes))]
        refs = [oracle_logits(name, tuple(s)) for s in seqs]
        slots = [eng.open() for _ in seqs]
        rows = Gathered(dtype, f"{name} batch {b}")
        got = eng.step([Entry(s, q[:n], [n - 1]) for s, q, n in zip(slots, seqs, lens)])
        rows.add(got, torch.stack([r[n - 1] for r, n in zip(refs, lens)]), "prompts")
        for j in range(max(decodes)):
            live = [i for i in range(len(seqs)) if j < decodes[i]]
            got = eng.step([Entry(slots[i], [seqs[i][lens[i] + j]], [0]) for i in live])
            rows.add(got, torch.stack([refs[i][lens[i] + j] for i in live]), f"decode {j}")
            for i in live:
                if j == decodes[i] - 1:
                    eng.close(slots[i])
        rows.check()
    assert eng.cache.slots.n_live == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["PF", "PG"])
def test_prompts_and_single_tokens_in_one_step(engines, name, dtype):
    """Portions beside single tokens in one step, and batches of single tokens for which the products of few rows, of dozens
    of rows and of more than those take the step."""
    from synaptix_b200.engine import Entry
    n_seqs = 36
    eng = engines(name, dtype, max_tokens=8192, max_seqs=40)
    seqs = [tokens(name, 80, 500 + i) for i in range(4)]
    refs = [oracle_logits(name, tuple(s)) for s in seqs]
    slots = [eng.open() for _ in range(n_seqs)]
    rows = Gathered(dtype, "mixed")
    at = [0] * n_seqs
    for new in ([30, 1, 17, 2], [1, 1, 1, 40], [5, 30, 1, 1], [30, 30, 30, 20]):
        entries, want = [], []
        for i, s in enumerate(slots):
            n = new[i % 4]
            entries.append(Entry(s, seqs[i % 4][at[i]:at[i] + n], [n - 1]))
            at[i] += n
            want.append(refs[i % 4][at[i] - 1])
        rows.add(eng.step(entries), torch.stack(want), str(new))
    for live in (36, 12, 3, 1):
        entries = [Entry(s, [seqs[i % 4][at[i]]], [0]) for i, s in enumerate(slots[:live])]
        rows.add(eng.step(entries), torch.stack([refs[i % 4][at[i]] for i in range(live)]), f"{live} single tokens")
        at = [a + (1 if i < live else 0) for i, a in enumerate(at)]
    for s in slots:
        eng.close(s)
    rows.check()


@pytest.mark.parametrize("name,dtype", [("PA", "float32"), ("PF", "bfloat16")])
def test_long_decoding(engines, name, dtype):
    """Hundreds of tokens one by one behind a prompt: windows pass over decoded tokens and give pages back, the attention
    layers see every key back to the first (more than a thousand in the second case: parts over the keys)."""
    from synaptix_b200.engine import Entry
    n0, n1 = (90, 500) if name == "PA" else (900, 260)
    eng = engines(name, dtype, max_tokens=2048)
    toks = tokens(name, n0 + n1, 77)
    ref = oracle_logits(name, tuple(toks))
    s = eng.open()
    got = [eng.step([Entry(s, toks[:n0], [n0 - 1])])]
    for t in toks[n0:]:
        got.append(eng.step([Entry(s, [t], [0])]))
    held = [sum(p >= 0 for p in eng.cache.slots.table(s, g)) for g in range(eng.cache.n_block_tables)]
    eng.close(s)
    assert min(held) <= 3 < max(held)                             # windowed groups hold a window's pages
    assert_close(torch.cat(got), ref[n0 - 1:], dtype, f"{name} long decoding")


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_entry_point(name):
    """``LLM.generate`` (scheduler, decode sessions, sampling on the device): greedy tokens of unequal prompts in one
    batch equal the plain implementation's, each computed alone."""
    import synaptix_b200
    llm = synaptix_b200.LLM(folder(name), compute_dtype="float32", max_tokens=1024)
    prompts = [tokens(name, n, 900 + n) for n in (3, 41, 1, 18)]
    out = llm.generate(prompts, max_new_tokens=12, temperature=0.0)
    cfg, W = oracle(name)
    for p, new in zip(prompts, out):
        seq = list(p)
        for tok in new:
            lg = PN.forward(cfg, W, seq)[-1]
            top2 = lg.topk(2).values
            if float(top2[0] - top2[1]) > 1e-3 * float(lg.abs().max()):       # a near tie may fall either way
                assert tok == int(lg.argmax()), f"{name}: token {len(seq) - len(p)} of prompt of {len(p)}"
            seq.append(tok)
        assert len(new) == 12
    assert llm.generate(prompts, max_new_tokens=12, temperature=0.0, prefill_batch=5) == out


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_program_with_a_batch_whose_requests_end_at_different_times(tmp_path, dtype):
    """``bin/trace_run`` as a user drives it (a subprocess fed JSON lines): three requests of unequal lengths begin in one
    step, go on one token a step, the shorter ones end earlier, and a fourth runs afterwards in what they gave back."""
    from test_gpu_trace_run import Replay
    name = "PA"
    seqs = {f"q{i}": tokens(name, n, 800 + i) for i, n in enumerate([31, 75, 12, 50])}
    refs = {k: oracle_logits(name, tuple(v)) for k, v in seqs.items()}
    r = Replay(folder(name), dtype, str(tmp_path), 192)
    heads = {"q0": 20, "q1": 60, "q2": 11}
    rows = Gathered(dtype, "replay")
    got = r.step([{"id": k, "tokens": seqs[k][:h], "want": [0, h - 1]} for k, h in heads.items()])
    rows.add(got, torch.stack([refs[k][j] for k, h in heads.items() for j in (0, h - 1)]), "prompts")
    at = dict(heads)
    while at:
        live = list(at)
        ends = [k for k in live if at[k] + 1 == len(seqs[k])]
        got = r.step([{"id": k, "tokens": [seqs[k][at[k]]], "want": [0]} for k in live], end=ends)
        rows.add(got, torch.stack([refs[k][at[k]] for k in live]), f"decode {sorted(at.values())}")
        for k in live:
            at[k] += 1
            if k in ends:
                del at[k]
    got = r.step([{"id": "q3", "tokens": seqs["q3"], "want": [45, 46, 47, 48, 49]}], end=["q3"])
    rows.add(got, refs["q3"][45:50], "afterwards")
    rows.check()
    r.finish()


def test_command_line_run_and_inspect(tmp_path):
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "PB"
    cfg, W = oracle(name)
    prompt = tokens(name, 9, 1300)
    env = dict(os.environ, PYTHONPATH=root)
    r = subprocess.run([sys.executable, "-m", "synaptix_b200", "run", folder(name), ",".join(map(str, prompt)),
                        "--max-tokens", "6", "--temperature", "0", "--compute-dtype", "f32", "--stop-ids", "", "--json"],
                       capture_output=True, text=True, env=env, cwd=str(tmp_path))
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    seq = list(prompt)
    for tok in out["outputs"][0]["tokens"]:
        lg = PN.forward(cfg, W, seq)[-1]
        top2 = lg.topk(2).values
        if float(top2[0] - top2[1]) > 1e-3 * float(lg.abs().max()):
            assert tok == int(lg.argmax())
        seq.append(tok)
    assert out["prompt_tokens"] == 9 and out["new_tokens"] == 6
    r = subprocess.run([sys.executable, "-m", "synaptix_b200", "inspect", folder(name)], capture_output=True, text=True, env=env)
    assert r.returncode == 0 and "architecture: Penopel" in r.stdout, r.stdout + r.stderr
