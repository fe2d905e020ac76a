"""The Zekalorn decoder on the GPU against the plain implementation: each mechanism's kernels alone, then whole models
through the engine under every way of cutting the work into steps, portions and batches, and greedy generation through the
library's entry point.  Configurations and weights are made here (``tiny_zekalorn``)."""
import pytest
import torch

import helpers
import plain_zekalorn as PZ
from test_gpu_pidutar import i32, near
from test_gpu_vemedra import portions, step_ctx
from tiny_zekalorn import CONFIGS, folder, oracle, oracle_logits, tokens

pytestmark = pytest.mark.gpu

NAMES = ["ZA", "ZB", "ZF", "ZG"]
DTYPES = ["float32", "bfloat16"]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


def assert_close(got, ref, dtype, what=""):
    """Logits against the oracle's.  32-bit: every row within the shared tolerance.  bfloat16: a row that hangs on a
    router's near tie is off by more than rounding, and so, a little, is every later row that reads its key or state; the
    comparison is a statistic over rows (the median within half the shared tolerance, three rows in four within it; the
    worst seen over these models and schedules: 0.010 and 0.82, in the narrowest model with its nine layer runs)."""
    got, ref = got.detach().float().cpu(), ref.detach().float().cpu()
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    rel = (got - ref).abs().max(dim=1).values / ref.abs().max()
    if dtype == "float32":
        assert float(rel.max()) <= helpers.F32_REL, f"{what}: {float(rel.max()):.3e} at row {int(rel.argmax())}"
        return
    within = float((rel <= helpers.BF16_REL).float().mean())
    median = float(rel.median())
    assert within >= 0.75 and (rel.numel() < 8 or median <= helpers.BF16_REL / 2), \
        f"{what}: {within:.2f} of {rel.numel()} rows are within {helpers.BF16_REL}, median error {median:.4f}"


class Gathered:
    """Rows of many small steps, compared at once (see ``assert_close``); 32-bit rows are compared as they come."""

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
class DeltaCase:
    """Random projections (other columns before and behind) and constants for sequences of ``lengths``, and the oracle's
    result for them with weights that pick those columns.  ``change(case)`` may rewrite the inputs first."""

    def __init__(self, heads, kv_heads, dim, vdim, taps, lengths, seed, dtype, change=None, ranks=(5, 9)):
        g = self.g = torch.Generator().manual_seed(seed)
        self.H, self.G, self.D, self.V, self.taps, self.lengths, self.dtype = heads, kv_heads, dim, vdim, taps, lengths, dtype
        GD, HV, HD = kv_heads * dim, heads * vdim, heads * dim
        self.C, self.col = 2 * GD + HV, 4
        self.b_col = self.col + self.C
        self.lr_col = self.b_col + heads
        self.ra, self.rg = ranks
        self.row = self.lr_col + self.ra + self.rg + 3
        n = sum(lengths)
        self.x = torch.randn(n, self.row, generator=g)
        self.conv = 0.6 * torch.randn(self.C, taps, generator=g)
        self.a2 = 0.4 * torch.randn(HD, self.ra, generator=g)
        self.g2 = 0.4 * torch.randn(HV, self.rg, generator=g)
        self.a_log = torch.linspace(-1.0, 1.0, heads)
        dt = torch.linspace(-2.0, 2.0, dim)
        dt[::2] = torch.linspace(-9.0, -5.0, dim)[::2]
        self.dt_bias = dt.repeat(heads)
        self.gain = 1 + 0.2 * torch.randn(vdim, generator=g)
        if change:
            change(self)
        # what the kernels read: the projection and the low-rank matrices in the compute dtype
        self.x, self.a2, self.g2 = (t.to(DT[dtype]) for t in (self.x, self.a2, self.g2))
        off = [0]
        for m in lengths:
            off.append(off[-1] + m)
        self.xs = [self.x[a:b] for a, b in zip(off, off[1:])]
        self.refs = [self.reference(x.double()) for x in self.xs]

    def z(self, x):
        """The pre-activations of decays and output gates."""
        x = x.double()
        return torch.cat([x[:, self.lr_col:self.lr_col + self.ra] @ self.a2.double().T,
                          x[:, self.lr_col + self.ra:self.lr_col + self.ra + self.rg] @ self.g2.double().T], 1)

    def reference(self, x):
        T, (H, G, D, V) = x.shape[0], (self.H, self.G, self.D, self.V)
        u = PZ.silu(PZ.time_conv(x[:, self.col:self.col + self.C], self.conv.double()))
        q, k, v = u[:, :G * D].reshape(T, G, D), u[:, G * D:2 * G * D].reshape(T, G, D), u[:, 2 * G * D:].reshape(T, H, V)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        z = self.z(x)
        beta = torch.sigmoid(x[:, self.b_col:self.b_col + H])
        sp = torch.nn.functional.softplus(z[:, :H * D] + self.dt_bias.double()).reshape(T, H, D)
        decay = torch.exp(-torch.exp(self.a_log.double())[None, :, None] * sp)
        rep = [h // (H // G) for h in range(H)]
        o = PZ.delta_rule(q[:, rep], k[:, rep], v, decay, beta)
        y = PZ.unit_rms(o, 1e-5) * self.gain.double() * torch.sigmoid(z[:, H * D:]).reshape(T, H, V)
        return y.reshape(T, H * V)

    def run(self, slots, cuts, low_rank=False, n_slots=None):
        """The kernels over the steps that ``cuts`` makes; every slot that no sequence has holds NaN."""
        from synaptix_b200 import ops
        n_slots = n_slots or max(slots) + 2
        S = torch.full((n_slots, self.H, self.D, self.V), float("nan")).cuda()
        ring = torch.full((n_slots, self.taps, self.C), float("nan")).cuda()
        S[slots], ring[slots] = 0.0, 0.0
        f = lambda t: t.float().contiguous().cuda()
        w = ops.DeltaWeights(f(self.conv), f(self.a_log), f(self.dt_bias), f(self.gain))
        lr = torch.zeros(self.H * (self.D + self.V), self.ra + self.rg, dtype=DT[self.dtype])
        lr[:self.H * self.D, :self.ra], lr[self.H * self.D:, self.ra:] = self.a2, self.g2
        lr = lr.cuda()
        outs = [[] for _ in self.lengths]
        for past, new, who in portions(self.lengths, cuts):
            ctx = step_ctx(past, new, [slots[i] for i in who], None, DT[self.dtype])
            x = torch.cat([self.xs[i][p:p + n] for i, p, n in zip(who, past, new)])
            kw = dict(z=self.z(x).float().contiguous().cuda())
            single = ctx.all_single and low_rank and ops.delta_step_fits(self.D, self.V, self.ra, self.rg)
            if single:
                kw = dict(low_rank=lr, ra=self.ra, rg=self.rg, lr_col=self.lr_col)
            proj = x.cuda() if not (single and self.dtype == "bfloat16") else x.float().cuda()
            y = ops.delta_rule(proj, self.col, self.b_col, self.H, self.G, self.D, self.V, w, self.D ** -0.5, 1e-6, 1e-5, S, ring,
                               ctx, DT[self.dtype], **kw)
            at = 0
            for i, n in zip(who, new):
                outs[i].append(y[at:at + n].float().cpu())
                at += n
        free = [s for s in range(n_slots) if s not in slots]
        assert torch.isnan(S[free]).all() and torch.isnan(ring[free]).all()
        self.last_state = S[slots].cpu()
        return [torch.cat(o) for o in outs]


SHAPES = [(4, 2, 12, 20, 4), (2, 1, 64, 64, 3), (3, 3, 128, 128, 4), (4, 4, 64, 32, 2), (2, 2, 32, 256, 4), (6, 3, 6, 8, 5),
          (2, 1, 256, 64, 1), (1, 1, 8, 1, 4), (4, 1, 20, 36, 3), (1, 1, 1, 4, 2), (2, 2, 100, 16, 6),
          # as many (sequence, head) pairs as give the scan wide and middle slices of the state, with one tile of it and two
          (40, 40, 16, 32, 2), (20, 10, 16, 36, 3), (30, 30, 132, 16, 2), (15, 5, 136, 32, 4)]
CUTS = [[200], [1] * 200, [2] * 100, [3, 1, 2, 64, 7, 1, 1, 150], [17, 15, 33, 1, 31, 32, 90], [100, 1, 1, 1, 1, 1, 100]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", SHAPES)
def test_delta_rule_over_portions(heads, kv_heads, dim, vdim, taps, dtype):
    """State and convolution ring carried over portions of many sizes (chunks, token walks, single tokens with and without
    the low-rank products inside, portions shorter than the taps reach back), in batches of unequal sequences."""
    lengths, slots = [150, 9, 77, 1], [2, 0, 5, 3]
    case = DeltaCase(heads, kv_heads, dim, vdim, taps, lengths, heads * dim + taps, dtype)
    for cuts in (CUTS if heads < 10 else CUTS[:1] + CUTS[3:5]):
        for low_rank in ((False, True) if 1 in cuts else (False,)):
            for o, r in zip(case.run(slots, cuts, low_rank), case.refs):
                near(o, r, dtype, f32=2e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_with_ranks_of_whole_vectors(dtype):
    """Ranks whose rows are read 16 bytes at a time, and a batch in one step."""
    lengths = [40, 40, 40, 40, 40, 3]
    case = DeltaCase(2, 2, 64, 128, 4, lengths, 5, dtype, ranks=(64, 32))
    for cuts in ([1] * 40, [20] + [1] * 20):
        for o, r in zip(case.run([0, 1, 2, 3, 4, 6], cuts, True), case.refs):
            near(o, r, dtype, f32=2e-4, bf16=3e-2)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(2, 1, 64, 64), (2, 2, 12, 20), (1, 1, 128, 128), (1, 1, 6, 8)])
def test_decays_of_every_strength(heads, kv_heads, dim, vdim):
    """Channels that empty within a token (logarithms of -1,000 and below: any factor with a positive exponent overflows),
    channels that keep everything, and channels that change from one to the other every few tokens."""
    def change(c):
        c.a_log = torch.linspace(2.0, 6.5, c.H)
        dt = torch.full((c.D,), -30.0)
        dt[1::3] = 2.0
        dt[2::3] = -3.0
        c.dt_bias = dt.repeat(c.H)
        c.a2 *= 6.0
    lengths = [150, 70]
    case = DeltaCase(heads, kv_heads, dim, vdim, 2, lengths, 31, "float32", change)
    for cuts in CUTS:
        for o, r in zip(case.run([1, 0], cuts, True), case.refs):
            assert torch.isfinite(o).all()
            # where hardly any state is left and q and k are nearly orthogonal, the output norm magnifies the last bits
            rel = (o.double() - r).abs().max(dim=1).values / float(r.abs().max())
            assert float((rel <= 2e-4).float().mean()) >= 0.97 and float(rel.max()) <= 3e-3, float(rel.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim", [(64, 64), (12, 20), (128, 32)])
def test_a_value_written_far_back_is_recalled(dim, vdim, dtype):
    """One token's key is a direction no other key has, its step size is 1 and nothing decays: any later query along that
    direction returns its value.  Written at the first token, at chunk borders (15, 16, 31, 32), read at once, at the
    borders of chunks and portions, and far behind, in prompts and single tokens."""
    writes = [0, 15, 16, 31, 32, 63]
    reads = {0: [0, 1, 31, 32, 149], 15: [15, 16, 17, 148], 16: [16, 32, 33, 147], 31: [31, 32, 63, 146], 32: [32, 63, 64, 145], 63: [64, 96, 128, 144]}
    n = 150
    lengths = [n] * len(writes)

    def change(c):
        c.conv.zero_()
        c.conv[:, -1] = 1.0
        c.dt_bias = torch.full((c.H * c.D,), -40.0)                      # no decay
        c.a2.zero_()
        c.g2.zero_()                                                     # gates of 1/2
        c.gain.fill_(2.0)
        GD = c.G * c.D
        half = c.D // 2
        for s, j in enumerate(writes):
            rows = c.x[s * n:(s + 1) * n]
            kcols, qcols = rows[:, c.col + GD:c.col + 2 * GD], rows[:, c.col:c.col + GD]
            kcols[:, half:] = -60.0                                      # silu of it is 0: other keys live in the first half
            direction = torch.full((c.D - half,), -60.0)
            direction[s % (c.D - half)] = 6.0
            kcols[j, :half] = -60.0
            kcols[j, half:] = direction
            rows[j, c.b_col] = 60.0                                      # step size 1
            for i in reads[j]:
                if i < n:
                    qcols[i, :half] = -60.0
                    qcols[i, half:] = direction
    case = DeltaCase(1, 1, dim, vdim, 1, lengths, 77, dtype, change)
    # the test's own premise: the oracle returns the normed value at every read
    for s, j in enumerate(writes):
        v = PZ.silu(case.xs[s][j, case.col + 2 * dim:case.col + 2 * dim + vdim].double())
        for i in reads[j]:
            assert torch.allclose(case.refs[s][i], PZ.unit_rms(v * dim ** -0.5, 1e-5), atol=2e-2), (j, i)
    for cuts in ([n], [1] * n, [2] * 75, [31, 1, 1, 31, 64, 50], [16, 16, 1, 1, 200]):
        for o, r in zip(case.run(list(range(len(writes))), cuts, True), case.refs):
            near(o, r, dtype, f32=3e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_state_slots_used_again(dtype):
    """The state that a run leaves equals the state the same tokens leave under another cut; a slot that is zeroed and
    used again for another sequence gives what a fresh one gives."""
    case = DeltaCase(4, 2, 32, 64, 4, [90], 9, dtype)
    case.run([0], [90])
    whole = case.last_state
    case.run([3], [33, 1, 1, 20, 35])
    assert torch.allclose(case.last_state, whole, atol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,rows,far,temp", [(6, 3, 10, 14, 10, 50.0, (0.7, 13)), (4, 2, 64, 64, 24, 300.0, (0.3, 100)),
                                                        (4, 1, 128, 128, 32, 128.0, (0.5, 64)), (2, 2, 32, 32, 7, 40.0, None),
                                                        (8, 1, 40, 24, 16, 60.0, (0.25, 1)), (3, 3, 16, 48, 5, 33.0, (1.5, 7))])
def test_attention_with_distance_bias_and_query_temperature(H, G, dim, vdim, rows, far, temp, dtype):
    """The whole mixer over portions of several sizes with NaN in every page no step wrote.  In one sequence a far key is
    made to point the way of a late query, so that its score stands out among hundreds (and with it the bias of its
    distance and the temperature of its position): a key at position 0, at a page's border, and just before the query."""
    from synaptix_b200.cache.store import KVView
    from synaptix_b200.parts import Runtime, ScoredAttention
    g = torch.Generator().manual_seed(H * dim + rows)
    W = 48
    p = "m."
    w = {p + "q": torch.randn(H * dim, W, generator=g) * 0.3, p + "k": torch.randn(G * dim, W, generator=g) * 0.3,
         p + "v": torch.randn(G * vdim, W, generator=g) * 0.3, p + "o": torch.randn(W, H * vdim, generator=g) * 0.3,
         p + "rel": torch.randn(rows, H, generator=g)}
    w = {k: v.to(DT[dtype]) for k, v in w.items()}
    lengths = [290, 70, 1]
    xs = [torch.randn(n, W, generator=g) for n in lengths]
    direction = torch.randn(W, generator=g)
    kq = w[p + "k"][:dim].double().T @ w[p + "q"][:dim].double()               # x_j . (Wk^T Wq) x_i
    toward = (kq @ direction.double()).float()
    for i, j in ((289, 0), (200, 63), (130, 64), (280, 279)):                  # a key of the usual size, a scaled score of 9
        xs[0][j] = toward * (7.0 / float(toward.norm()))
        xs[0][i] = direction * (9.0 / (0.4 * 7.0 * float(toward.norm())))
    xs = [x.to(DT[dtype]) for x in xs]
    scale = 0.4
    m = dict(heads=H, kv_heads=G, dim=dim, vdim=vdim, scale=scale, bias_max=far)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    refs = [PZ.attention(x.double(), {k: v.double() for k, v in w.items()}, p, m) for x in xs]
    part = ScoredAttention(p, W, H, G, dim, vdim, scale=scale, weights="softmax", distance_bias=(rows, far), q_temp=temp)
    part.bind_all(w, Runtime(torch.device("cuda:0"), DT[dtype]))
    tables = [[1, 2, 3, 4, 5], [6, 7, 0, 0, 0], [8, 0, 0, 0, 0]]
    for cuts in ([300], [1] * 290, [2] * 145, [129, 1, 70, 1, 1, 90], [16, 48, 100, 7, 3, 300]):
        k = torch.full((9, G, 64, dim), float("nan"), dtype=DT[dtype]).cuda()
        v = torch.full((9, G, 64, vdim), float("nan"), dtype=DT[dtype]).cuda()
        view = KVView(k, v, 0, None)
        outs = [[] for _ in lengths]
        for past, new, who in portions(lengths, cuts):
            bt = i32([tables[i] for i in who])
            ctx = step_ctx(past, new, who, [bt], DT[dtype])
            y = part.forward(torch.cat([xs[i][a:a + n] for i, a, n in zip(who, past, new)]).cuda(), ctx, view)
            at = 0
            for i, n in zip(who, new):
                outs[i].append(y[at:at + n].float().cpu())
                at += n
        for o, r in zip(outs, refs):            # (scores of 20 and more out of 16-bit queries and keys)
            near(torch.cat(o), r, dtype, f32=2e-4, bf16=5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,experts,top,ff,width", [(1, 5, 2, 24, 52), (3, 1, 1, 16, 40), (9, 4, 4, 40, 328), (70, 9, 3, 40, 64),
                                                    (300, 16, 4, 104, 136), (700, 6, 2, 200, 328), (600, 8, 1, 264, 128)])
def test_experts_without_a_gate(T, experts, top, ff, width, dtype):
    """Router and experts of two matrices with relu^2 over the FFMA product, the mma.sync product of few rows and (from 512
    rows in bfloat16) the tcgen05 product; the weights are the softmax over the chosen logits alone."""
    from synaptix_b200.parts import MixtureOfExperts, Runtime
    g = torch.Generator().manual_seed(T * experts + ff)
    p = "f."
    W = {p + "router": torch.randn(experts, width, generator=g) * 0.4}
    for e in range(experts):
        W[f"{p}e{e}.up"] = torch.randn(ff, width, generator=g) * 0.15
        W[f"{p}e{e}.down"] = torch.randn(width, ff, generator=g) * 0.2
    W = {k: v.to(DT[dtype]) for k, v in W.items()}
    x = torch.randn(T, width, generator=g).to(DT[dtype])
    Wd = {k: v.double() for k, v in W.items()}
    ref = PZ.experts_ff(x.double(), Wd, p, dict(router=dict(top=top, experts=experts)))
    part = MixtureOfExperts(p, width, ff, experts, top, gated=False)
    part.bind(W, Runtime(torch.device("cuda:0"), DT[dtype]))
    ctx = step_ctx([0], [T], [0], None, DT[dtype])
    got = part.forward(x.cuda(), ctx).float().cpu()
    # a choice that hangs on a near tie may fall either way
    z = (x.double() @ Wd[p + "router"].T).sort(-1, descending=True).values
    clear = (z[:, top - 1] - z[:, top] > 1e-3) if top < experts else torch.ones(T, dtype=torch.bool)
    near(got[clear], ref[clear], dtype, f32=2e-4, bf16=2e-2)
    assert float(clear.float().mean()) > 0.9 or T < 10
    rows = part.forward(x.cuda(), ctx, defer_combine=True)
    near(rows.materialize().float().cpu()[clear], ref[clear], dtype, f32=2e-4, bf16=2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width,dim", [(1, 52, 6), (7, 256, 32), (40, 128, 16), (300, 320, 24), (2, 1000, 256)])
def test_token_input_of_a_layer(T, width, dim, dtype):
    """Sum of the branches into the 32-bit stream (one of them a mixture's unformed weighted sum), gate, product and the
    branch's norm; the layer's own columns of the table and no others."""
    from synaptix_b200 import ops
    from synaptix_b200.parts import Runtime, TokenSide
    g = torch.Generator().manual_seed(T + width)
    V, n, i, eps = 37, 3, 1, 1e-5
    w = {"side.embed": torch.randn(V, n * dim, generator=g), "l.side.gate": torch.randn(dim, width, generator=g) * 0.1,
         "l.side.proj": torch.randn(width, dim, generator=g) * 0.3, "l.side.norm": 1 + 0.2 * torch.randn(width, generator=g)}
    w = {k: v.to(DT[dtype]) for k, v in w.items()}
    part = TokenSide("l.side.", "side.embed", V, width, dim, i, n, eps)
    part.bind_all(w, Runtime(torch.device("cuda:0"), DT[dtype]))
    h, a = torch.randn(T, width, generator=g) * 3, torch.randn(T, width, generator=g).to(DT[dtype])
    rows, place = torch.randn(T * 2, width, generator=g), torch.randperm(2 * T, generator=g).to(torch.int32)
    wts = torch.rand(T, 2, generator=g)
    mix = torch.stack([sum(wts[t, k].double() * rows[int(place[t * 2 + k])].double() for k in range(2)) for t in range(T)])
    toks = [int(v) for v in torch.randint(0, V, (T,), generator=g)]
    ctx = step_ctx([0], [T], [0], None, DT[dtype])
    ctx.token_ids = i32(toks)
    Wd = {k: v.double() for k, v in w.items()}
    read = (lambda v: v) if dtype == "float32" else (lambda v: v.to(torch.bfloat16).double())
    for b, extra in ((None, 0.0), (ops.WeightedRows(rows.cuda(), place.cuda(), wts.cuda(), DT[dtype]), mix)):
        ref_h = h.double() + a.double() + extra
        ref_y = PZ.token_side(read(ref_h), toks, Wd, "l.", i, dim, eps)
        hd = h.cuda()
        d = part.forward(hd, [(a.cuda(), None)] + ([(b, None)] if b is not None else []), ctx)
        near(hd.cpu(), ref_h, "float32", f32=2e-6)
        near(d.materialize().cpu(), ref_y, dtype, f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_learned_positions(dtype):
    from synaptix_b200 import ops
    g = torch.Generator().manual_seed(4)
    table, pos = torch.randn(50, 24, generator=g).to(DT[dtype]), torch.randn(33, 24, generator=g).to(DT[dtype])
    ids, at = [3, 49, 0, 7], [0, 32, 5, 5]
    got = ops.embed_gather(table.cuda(), i32(ids), scale=2.5, pos_table=pos.cuda(), positions=i32(at)).cpu().double()
    assert torch.allclose(got, table[ids].double() * 2.5 + pos[at].double(), atol=1e-5)


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
            for t in eng.cache._k + eng.cache._v + eng.cache._state:      # a place no step wrote shows at once when it is read
                t.fill_(float("nan"))
            made[key] = eng
        assert made[key].cache.slots.n_live == 0
        return made[key]
    return get


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_every_place(engines, name, dtype):
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    assert type(eng.model.config).__name__ == "ZekalornConfig" and eng.use_graphs
    rows = Gathered(dtype, f"{name} {dtype} whole prompts")
    for i, n in enumerate([1, 2, 3, 17, 32, 33, 64, 65, 150, 301, 690]):
        toks = tokens(name, n, 100 + i)
        s = eng.open()
        got = eng.step([Entry(s, toks, list(range(n)))])
        eng.close(s)
        rows.add(got, oracle_logits(name, tuple(toks), dtype), f"n={n}")
    rows.check()


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer_run(engines, name):
    from synaptix_b200.engine import Entry
    eng = engines(name, "float32")
    toks = tokens(name, 90, 4)
    cfg, W = oracle(name)
    ref = []
    PZ.forward(cfg, W, toks, ref)
    seen = []
    s = eng.open()
    entries = [Entry(s, toks, [0])]
    past, new = eng._check(entries)
    ctx = eng.plan(entries, past, new)
    ctx.observe = lambda n, h, pending: seen.append((h + pending.float()).cpu() if pending is not None else h.cpu().clone())
    eng._forward(ctx)
    eng.cache.slots.advance(s, len(toks))
    eng.close(s)
    assert len(seen) == len(ref)
    for i, (a, b) in enumerate(zip(seen, ref)):
        assert torch.allclose(a.double(), b, atol=1e-4 * float(b.abs().max())), f"{name}: layer run {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first_token(engines, name, dtype):
    """Every token a step of its own (captured steps): the first tokens of a sequence, whose states and rings begin from
    zeros, and on across page borders."""
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    toks = tokens(name, 150, 8)
    s = eng.open()
    got = torch.cat([eng.step([Entry(s, [t], [0])]) for t in toks])
    eng.close(s)
    assert_close(got, oracle_logits(name, tuple(toks), dtype), dtype, f"{name} {dtype} token by token")
    assert any(c.graph is not None for c in eng._captured.values())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ZA", "ZG"])
def test_branches_on_two_streams_change_no_bit(name, dtype):
    from synaptix_b200 import ops
    from synaptix_b200.engine import Engine, Entry
    from synaptix_b200.models import load_model
    toks = [tokens(name, n, 60 + n) for n in (90, 37, 64)]

    def run(eng):
        slots = [eng.open() for _ in toks]
        out = [eng.step([Entry(s, t[:20], [19]) for s, t in zip(slots, toks)])]
        for j in range(20, 37):
            out.append(eng.step([Entry(s, [t[j]], [0]) for s, t in zip(slots, toks)]))
        for j in range(37, 64):                                  # the shorter requests end earlier
            out.append(eng.step([Entry(s, [t[j]], [0]) for s, t in zip(slots[::2], toks[::2])]))
        for s in slots:
            eng.close(s)
        return torch.cat(out).cpu()
    with ops.options(branch_streams=False):
        ref = run(Engine(load_model(folder(name), dtype=dtype), max_tokens=1024, max_seqs=3))
    eng = Engine(load_model(folder(name), dtype=dtype), max_tokens=1024, max_seqs=3)
    first, second = run(eng), run(eng)
    assert any(c.graph is not None for c in eng._captured.values())
    assert torch.equal(first, ref) and torch.equal(second, ref)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("size", [2, 3, 7, 33, 64, 100])
def test_prompts_in_portions(engines, name, dtype, size):
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype)
    toks = tokens(name, 277, 20)
    s = eng.open()
    got = [eng.step([Entry(s, toks[a:a + size], list(range(len(toks[a:a + size]))))]) for a in range(0, len(toks), size)]
    eng.close(s)
    assert_close(torch.cat(got), oracle_logits(name, tuple(toks), dtype), dtype, f"{name} {dtype} portions of {size}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_in_slots_and_pages_used_again(engines, name, dtype):
    """Batches of unequal prompts decoded together, shorter requests ending earlier; the cache holds little more than one
    batch and three slots, so every batch runs in slots, states, rings and pages that the batch before gave back."""
    from synaptix_b200.engine import Entry
    eng = engines(name, dtype, max_tokens=512, max_seqs=3)
    for b, (lens, decodes) in enumerate([([5, 130, 1], [3, 40, 12]), ([64, 9, 200], [10, 30, 2]), ([2, 3, 100], [25, 1, 70])]):
        seqs = [tokens(name, n + d, 300 + 10 * b + i) for i, (n, d) in enumerate(zip(lens, decodes))]
        refs = [oracle_logits(name, tuple(s), dtype) for s in seqs]
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
def test_prompts_and_single_tokens_in_one_step(engines, dtype):
    """Portions beside single tokens in one step, and a batch of more sequences than the low-rank products run inside the
    single-token kernel for."""
    from synaptix_b200.engine import Entry
    eng = engines("ZF", dtype, max_tokens=4096, max_seqs=24)
    seqs = [tokens("ZF", 60, 500 + i) for i in range(4)]
    refs = [oracle_logits("ZF", tuple(s), dtype) for s in seqs]
    slots = [eng.open() for _ in range(20)]
    rows = Gathered(dtype, "mixed")
    at = [0] * 20
    for new in ([30, 1, 17, 2], [1, 1, 1, 40], [5, 30, 1, 1]):
        entries, want = [], []
        for i, s in enumerate(slots):
            n = new[i % 4]
            entries.append(Entry(s, seqs[i % 4][at[i]:at[i] + n], [n - 1]))
            at[i] += n
            want.append(refs[i % 4][at[i] - 1])
        rows.add(eng.step(entries), torch.stack(want), str(new))
    for _ in range(10):
        entries = [Entry(s, [seqs[i % 4][at[i]]], [0]) for i, s in enumerate(slots)]
        rows.add(eng.step(entries), torch.stack([refs[i % 4][at[i]] for i in range(20)]), "20 single tokens")
        at = [a + 1 for a in at]
    for s in slots:
        eng.close(s)
    rows.check()


def test_long_decoding(engines):
    """500 tokens one by one behind a prompt: the states run on, the attention layers see every key back to the first."""
    from synaptix_b200.engine import Entry
    eng = engines("ZA", "float32", max_tokens=1024)
    toks = tokens("ZA", 90 + 500, 77)
    ref = oracle_logits("ZA", tuple(toks))
    s = eng.open()
    got = [eng.step([Entry(s, toks[:90], [89])])]
    for t in toks[90:]:
        got.append(eng.step([Entry(s, [t], [0])]))
    eng.close(s)
    assert_close(torch.cat(got), ref[89:], "float32", "ZA long decoding")


def test_no_position_beyond_the_table(engines):
    """A step that would pass the last learned position is refused and leaves the sequence as it was; the last position
    itself runs; generation ends there by capacity."""
    import synaptix_b200
    from synaptix_b200.engine import Entry
    from synaptix_b200.engine.step import StepError
    limit = CONFIGS["ZB"][0]["max_positions"]
    eng = engines("ZB", "float32")
    toks = tokens("ZB", limit, 6)
    ref = oracle_logits("ZB", tuple(toks))
    s = eng.open()
    eng.step([Entry(s, toks[:limit - 3], [])])
    with pytest.raises(StepError):
        eng.step([Entry(s, toks[limit - 3:] + [1], [0])])
    got = [eng.step([Entry(s, toks[limit - 3:limit - 1], [0, 1])]), eng.step([Entry(s, toks[limit - 1:], [0])])]
    assert_close(torch.cat(got), ref[limit - 3:], "float32", "the last positions")
    with pytest.raises(StepError):
        eng.step([Entry(s, [0], [0])])
    eng.close(s)
    llm = synaptix_b200.LLM(folder("ZB"), compute_dtype="float32", max_tokens=2048)
    out = llm.generate([toks[:limit - 4], toks[:9]], max_new_tokens=20, temperature=0.0, eos_token_ids=[])
    assert len(out[0]) == 5 and len(out[1]) == 20             # four more tokens run, and one is sampled behind the last


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
            lg = PZ.forward(cfg, W, seq)[-1]
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
    name = "ZA"
    seqs = {f"q{i}": tokens(name, n, 800 + i) for i, n in enumerate([31, 75, 12, 50])}
    refs = {k: oracle_logits(name, tuple(v), dtype) for k, v in seqs.items()}
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
    name = "ZB"
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
        lg = PZ.forward(cfg, W, seq)[-1]
        top2 = lg.topk(2).values
        if float(top2[0] - top2[1]) > 1e-3 * float(lg.abs().max()):
            assert tok == int(lg.argmax())
        seq.append(tok)
    assert out["prompt_tokens"] == 9 and out["new_tokens"] == 6
    r = subprocess.run([sys.executable, "-m", "synaptix_b200", "inspect", folder(name)], capture_output=True, text=True, env=env)
    assert r.returncode == 0 and "architecture: Zekalorn" in r.stdout, r.stdout + r.stderr
