"""The kernels and kernel options that the Pirozen design adds, each alone against its plain PyTorch version
(tests/ref_ops.py), in 32-bit and in bfloat16: two norms of one stream in one kernel; a second pending term; the few-rows products
with a bias and with a 32-bit addend, behind norms and on long rows; the activation times a table's rows by token id; the gate
that leaves the padding of heads out; experts chosen apart from their scores, identities, and the combine onto the residual
stream; a single token's whole attention with a stretched rotation, and the attention part as a whole with planted keys at the
window's edges."""
import pytest
import torch

import plain_pirozen as P
import ref_ops
from test_gpu_kernels import make_step
from test_gpu_zikevik_kernels import expert_tensors
from zig_ai_b200.cache.manager import CacheView
from zig_ai_b200.parts import PartSpec, make_part
from zig_ai_b200.parts.base import LazyNorm, Residual

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def ops():
    from zig_ai_b200.kernels import ops as o
    o.require(extra=("attention", "attention_mma", "attention_tma", "attention_tc", "qkv_prepare", "moe", "gemm_tc"))
    return o


def tol(dtype):
    return dict(atol=3e-5, rtol=3e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,H", [(5, 96), (3, 1000), (17, 2048), (1, 66), (70, 1024), (2, 4096), (4, 5000), (3, 37), (200, 4)])
def test_two_norms_of_one_stream(dtype, N, H):
    o = ops()
    g = torch.Generator().manual_seed(2)
    h = torch.randn(N, H, generator=g).cuda() * 3
    d = torch.randn(N, H, generator=g).to(dtype).cuda()
    wa, wb, wd = ((1 + 0.3 * torch.randn(H, generator=g)).cuda() for _ in range(3))
    for delta, gamma in ((None, None), (d, None), (d, wd)):
        ha, hb = h.clone(), h.clone()
        a = o.add_rmsnorm_pair(ha, delta, wa, wb, 1e-5, dtype, gamma, 1e-3)
        b = ref_ops.add_rmsnorm_pair(hb, delta, wa, wb, 1e-5, dtype, gamma, 1e-3)
        assert torch.allclose(ha, hb, atol=2e-6, rtol=2e-6)
        for i in range(2):
            assert a[i].dtype == dtype and torch.allclose(a[i].float(), b[i].float(), **tol(dtype))
        # one norm alone gives the same rows
        hc = h.clone()
        one = o.add_rmsnorm(hc, delta, wb, 1e-5, dtype, gamma, 1e-3)
        assert torch.allclose(one.float(), a[1].float(), **tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,H", [(5, 96), (3, 1000), (1, 66), (70, 1024), (3, 37)])
def test_a_second_pending_term(dtype, N, H):
    o = ops()
    g = torch.Generator().manual_seed(3)
    h = torch.randn(N, H, generator=g).cuda() * 3
    d1, d2 = (torch.randn(N, H, generator=g).to(dtype).cuda() for _ in range(2))
    w = (1 + 0.3 * torch.randn(H, generator=g)).cuda()
    for gamma in (None, w):
        ha, hb = h.clone(), h.clone()
        a = o.add_cast(ha, d1, dtype, gamma, 1e-5, delta2=d2)
        b = ref_ops.add_cast(hb, d1, dtype, gamma, 1e-5, delta2=d2)
        assert torch.allclose(ha, hb, atol=2e-6, rtol=2e-6) and torch.allclose(a.float(), b.float(), **tol(dtype))


@pytest.mark.parametrize("M", [1, 3, 8, 13, 16, 40])
@pytest.mark.parametrize("K,O", [(256, 512), (1024, 1528), (2048, 320), (192, 100), (64, 33), (3072, 256), (8192, 64)])
def test_products_with_a_bias_and_an_addend(M, K, O):
    """bfloat16: plain rows (short and long: other kernels), and behind the two norms; the addend is 32-bit and so is its sum."""
    o = ops()
    g = torch.Generator().manual_seed(4)
    dt = torch.bfloat16
    x = torch.randn(M, K, generator=g).to(dt).cuda()
    w = (torch.randn(O, K, generator=g) * K ** -0.5).to(dt).cuda()
    b = (3 * torch.randn(O, generator=g)).to(dt).cuda()
    add = (100 * torch.randn(M, O, generator=g)).cuda()
    exact = x.double() @ w.double().T
    assert torch.allclose(o.linear(x, w, bias=b).double(), exact + b.double(), atol=3e-2, rtol=6e-3)
    got = o.linear_add(x, w, add)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), exact + add.double(), atol=1e-4, rtol=1e-6)
    if M <= 16 and K <= 2048:
        h = (torch.randn(M, K, generator=g) * 2 + 0.7).cuda()
        delta = torch.randn(M, K, generator=g).to(dt).cuda()
        gamma, beta = (1 + 0.2 * torch.randn(K, generator=g)).cuda(), (0.5 * torch.randn(K, generator=g)).cuda()
        for bt in (None, beta):
            hr = h.clone()
            xr = ref_ops.add_rmsnorm(hr, delta, gamma, 1e-5, dt) if bt is None else ref_ops.add_layernorm(hr, delta, gamma, bt, 1e-5, dt)
            res = Residual(h.clone())
            y = o.linear(LazyNorm(res, delta, gamma, 1e-5, dt, beta=bt), w, bias=b)
            assert torch.allclose(y.float(), ref_ops.linear(xr, w, bias=b).float(), atol=3e-2, rtol=3e-2)
            assert torch.allclose(res.data, hr, atol=1e-6, rtol=0)


@pytest.mark.parametrize("M", [1, 16, 70])
def test_the_addend_in_32_bit(M):
    o = ops()
    g = torch.Generator().manual_seed(5)
    x, w, add = torch.randn(M, 66, generator=g).cuda(), torch.randn(50, 66, generator=g).cuda(), torch.randn(M, 50, generator=g).cuda()
    assert torch.allclose(o.linear_add(x, w, add).double(), x.double() @ w.double().T + add.double(), atol=1e-4, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 7, 16, 50])
@pytest.mark.parametrize("K,O,at,cols", [(256, 24, 48, 96), (64, 7, 3, 11), (1024, 256, 256, 1024), (1600, 16, 0, 16), (40, 1, 4, 5)])
def test_the_activation_times_a_tables_rows(dtype, M, K, O, at, cols):
    o = ops()
    g = torch.Generator().manual_seed(6)
    x, w = torch.randn(M, K, generator=g).to(dtype).cuda(), (torch.randn(O, K, generator=g) * K ** -0.5 * 2).to(dtype).cuda()
    table = torch.randn(90, cols, generator=g).to(dtype).cuda()
    ids = torch.randint(0, 90, (M,), generator=g).to(torch.int32).cuda()
    a, b = o.linear_side(x, w, table, ids, at), ref_ops.linear_side(x, w, table, ids, at)
    assert a.shape == (M, O) and torch.allclose(a.float(), b.float(), **tol(dtype))
    assert o.read_status() == 0
    bad = ids.clone()
    bad[0] = 90
    o.linear_side(x, w, table, bad, at)                  # an id outside the table: the kernels read row 0 and raise the status
    assert o.read_status() == 2
    zero = ids.clone()
    zero[0] = 0
    bad[0] = -1
    assert torch.equal(o.linear_side(x, w, table, bad, at), o.linear_side(x, w, table, zero, at)) and o.read_status() == 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,Dv,Dp", [(4, 64, 128), (3, 24, 24), (5, 10, 16), (2, 8, 40), (16, 128, 128), (1, 1, 3)])
def test_the_gate_leaves_the_padding_out(dtype, H, Dv, Dp):
    o = ops()
    g = torch.Generator().manual_seed(7)
    for N in (1, 37, 600):
        x = torch.randn(N, H * Dp, generator=g).to(dtype).cuda()
        wide = (3 * torch.randn(N, H + 9, generator=g)).to(dtype).cuda()
        gate = wide[:, 5:5 + H]
        a = o.sigmoid_gate(x, gate, H, Dv, True, row_dim=Dp)
        b = ref_ops.sigmoid_gate(x, gate, H, Dv, True, row_dim=Dp)
        assert a.shape == (N, H * Dv) and torch.allclose(a.float(), b.float(), **tol(dtype))
        full = (3 * torch.randn(N, H * Dp, generator=g)).to(dtype).cuda()
        assert torch.allclose(o.sigmoid_gate(x, full, H, Dp, False).float(), ref_ops.sigmoid_gate(x, full, H, Dp, False).float(), **tol(dtype))


def margins(x, w_router, correction, groups, top):
    """Per row: the distance of the choice from another one (see `plain_pirozen.margin`)."""
    s = torch.softmax(x.double() @ w_router.double().t(), dim=-1)
    router = {"top": top, "groups": None if groups is None else {"count": groups[0], "keep": groups[1]}}
    corr = correction.double().tolist() if correction is not None else [0.0] * s.shape[1]
    return torch.tensor([P.margin(row.tolist(), corr, router) for row in s])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,W,F,E,I,top,groups,scale", [
    (1, 64, 24, 5, 3, 2, (4, 2), 2.0), (7, 40, 20, 9, 0, 1, (3, 1), 0.5), (33, 66, 16, 3, 5, 8, None, 1.0), (70, 128, 64, 8, 4, 3, (3, 2), 1.7),
    (300, 192, 96, 6, 2, 2, (8, 5), 1.0), (600, 256, 136, 4, 12, 4, (4, 4), 2.5), (5, 50, 12, 1, 1, 1, (2, 1), 3.0), (40, 320, 128, 1, 1, 2, (1, 1), 1.0),
    (130, 96, 40, 40, 24, 6, (16, 3), 1.3), (1500, 128, 72, 12, 4, 2, (4, 2), 2.0), (900, 200, 328, 2, 2, 2, None, 0.7), (520, 64, 24, 300, 100, 5, (20, 4), 1.0)])
def test_experts_chosen_apart_from_their_scores(dtype, N, W, F, E, I, top, groups, scale):
    o = ops()
    g = torch.Generator().manual_seed(17)
    w_router, _, _ = expert_tensors(g, E + I, F, W, dtype)
    _, w_gate_up, w_down = expert_tensors(g, E, F, W, dtype)
    correction = (torch.randn(E + I, generator=g) * 0.3 - 0.2).cuda()
    wide = torch.randn(N, W + 16, generator=g).to(dtype).cuda()
    x = wide[:, 8:8 + W]
    unit, other = (torch.randn(N, W, generator=g).to(dtype).cuda() for _ in range(2))
    kw = dict(score="softmax", correction=correction, groups=groups, identities=I, weight_scale=scale)
    a = o.routed_experts(x, w_router, w_gate_up, w_down, top, True, "output", unit=unit, **kw)
    b = ref_ops.routed_experts(x, w_router, w_gate_up, w_down, top, True, "output", unit=unit, **kw)
    sure = (margins(x.cpu(), w_router.cpu(), correction.cpu(), groups, top) > 1e-5).cuda()      # (the rest may be chosen the other way round)
    assert int(sure.sum()) >= N - max(2, N // 50)
    assert torch.allclose(a.float()[sure], b.float()[sure], **tol(dtype))
    # onto the residual stream: the same sums, not rounded on their way, and the rows beside them
    h = torch.randn(N, W, generator=g).cuda() * 2
    for rows in (other, None):
        ha, hb = h.clone(), h.clone()
        ca = o.routed_experts(x, w_router, w_gate_up, w_down, top, True, "output", unit=unit, onto=(ha, rows, True), **kw)
        cb = ref_ops.routed_experts(x, w_router, w_gate_up, w_down, top, True, "output", unit=unit, onto=(hb, rows, True), **kw)
        assert torch.allclose(ha[sure], hb[sure], **tol(dtype)) and torch.equal(ca, ha.to(dtype))
        assert torch.allclose(ca.float()[sure], cb.float()[sure], **tol(dtype))
        hc = h.clone()
        assert o.routed_experts(x, w_router, w_gate_up, w_down, top, True, "output", unit=unit, onto=(hc, rows, False), **kw) is None
        assert torch.equal(hc, ha)
    # sigmoid scores and weights on the experts' inputs take the same options
    kw["score"] = "sigmoid"
    s = torch.sigmoid(x.float() @ w_router.t())
    a = o.routed_experts(x, w_router, w_gate_up, w_down, top, False, "input", **kw)
    b = ref_ops.routed_experts(x, w_router, w_gate_up, w_down, top, False, "input", **kw)
    ok = (a.float() - b.float()).abs().amax(dim=-1) < 3 * tol(dtype)["atol"] * (1 + b.float().abs().amax(dim=-1))
    assert int(ok.sum()) >= N - max(2, N // 50) and s.shape == (N, E + I)
    assert o.read_status() == 0


def test_the_choice_with_known_scores():
    """Scores made so that the choice is known: groups by their best choice value, not by their sum; corrections decide the choice
    but not the weights; all choice values negative; the lower index of equals; identities give the row times its weight."""
    o = ops()
    W, F, E, I = 32, 8, 4, 4
    x = torch.zeros(3, W).cuda()
    x[:, 0] = 1.0
    x[:, 2] = torch.tensor([1.0, -2.0, 3.0]).cuda()
    logits = torch.tensor([0.3, 0.1, 0.2, 0.15, 0.25, 0.05, 0.1, 0.2])
    w_router = torch.zeros(E + I, W).cuda()
    w_router[:, 0] = logits.cuda()
    s = torch.softmax(logits.double(), dim=0)
    w_gate_up = torch.zeros(E, 2 * F, W).cuda()
    w_down = torch.zeros(E, W, F).cuda()                       # experts give zeros: only identities show

    def identity_weight(correction, groups, top, renorm=True, scale=1.0):
        c = torch.tensor(correction, dtype=torch.float32).cuda()
        y = o.routed_experts(x, w_router, w_gate_up, w_down, top, renorm, "output", score="softmax", correction=c, groups=groups, identities=I,
                             weight_scale=scale)
        assert torch.allclose(y[:, 2] / x[:, 2], y[0, 2].expand(3), atol=1e-6) and bool((y[:, 3:] == 0).all())
        return float(y[0, 2])
    zero = [0.0] * 8
    close = lambda a, b: abs(a - float(b)) < 1e-6
    # experts 0 and 4 (an identity) have the largest scores
    assert close(identity_weight(zero, None, 2), s[4] / (s[0] + s[4]))
    assert close(identity_weight(zero, None, 2, False, 3.0), 3 * s[4])
    assert close(identity_weight(zero, None, 2, True, 3.0), 3 * s[4] / (s[0] + s[4]))
    # the correction brings in 5 and 7; their weights go by the scores
    c = [0.0, 0.0, 0.0, 0.0, 0.0, 1.0, 0.0, 0.5]
    assert close(identity_weight(c, None, 2), 1.0) and close(identity_weight(c, None, 2, False), s[5] + s[7])
    assert close(identity_weight(c, None, 1, False), s[5])
    # groups of two: {0,1} wins by expert 0 although {2,3} has the larger sum with these corrections
    c = [0.0, -9.0, -0.001, -0.002, -9.0, -9.0, -9.0, -9.0]
    assert close(identity_weight(c, (4, 1), 1), 0.0)
    # all negative: a group left out counts as less than any of them
    c = [-5.0] * 4 + [-6.0] * 4
    assert close(identity_weight(c, (2, 1), 4), 0.0)
    c = [-6.0] * 4 + [-5.0] * 4
    assert close(identity_weight(c, (2, 1), 4), 1.0) and close(identity_weight(c, (2, 1), 2, False), s[4] + s[7])
    # equal choice values: the lower index; equal groups: the lower group
    flat = [(1.0 - float(v)) for v in s]
    w_router.zero_()
    assert close(identity_weight(zero, (2, 1), 4), 0.0) and close(identity_weight(zero, (8, 5), 5), 1 / 5) and len(flat) == 8


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_rows_experts_do_not_depend_on_the_other_rows(dtype, monkeypatch):
    o = ops()
    g = torch.Generator().manual_seed(19)
    W, F, E, I, top = 128, 64, 8, 4, 3
    w_router, _, _ = expert_tensors(g, E + I, F, W, dtype)
    _, w_gate_up, w_down = expert_tensors(g, E, F, W, dtype)
    kw = dict(score="softmax", correction=(torch.randn(E + I, generator=g) * 0.2).cuda(), groups=(3, 2), identities=I, weight_scale=2.0)
    x = torch.randn(900, W, generator=g).to(dtype).cuda()
    run = lambda rows: o.routed_experts(rows.contiguous(), w_router, w_gate_up, w_down, top, True, "output", **kw)
    many = run(x)
    perm = torch.randperm(900, generator=g).cuda()
    assert torch.equal(run(x[perm]), many[perm])
    monkeypatch.setattr(o, "USE_MOE_GROUPED_TC", False)
    all_rows = run(x)
    assert torch.allclose(all_rows.float(), many.float(), **tol(dtype))
    for rows in ([0], [3, 4, 5], list(range(100, 140)), list(range(690, 700)) + list(range(10))):
        assert torch.equal(run(x[rows]), all_rows[rows]), rows[:3]


STRETCH = (4.0, 60.0, 8.0, 0.5)


@pytest.mark.parametrize("H,G,D,rot,ps,window", [(8, 2, 64, 32, 16, 33), (4, 1, 128, 128, 64, 100), (6, 3, 32, 16, 8, 9), (4, 4, 96, 96, 16, 1), (3, 1, 80, 0, 32, 500),
                                                (8, 1, 48, 24, 8, None)])
def test_a_single_tokens_attention_with_a_stretched_rotation(H, G, D, rot, ps, window):
    """The one kernel (rows with a gate's columns behind them) against preparing the rows and attending to the pages."""
    o = ops()
    g = torch.Generator().manual_seed(9)
    dt = torch.bfloat16
    ctx = [0, 1, ps - 1, ps, 3 * ps + 5, 200, 33]
    step = make_step(o, dt, ctx, [1] * len(ctx), ps, 256, 4)
    y = torch.randn(len(ctx), (H + 2 * G) * D + H + 5, generator=g).to(dt).cuda()
    qw, kw = ((1 + 0.2 * torch.randn(D, generator=g)).cuda() for _ in range(2))
    pages = (torch.randn(256, 2, G, ps, D, generator=g)).to(dt).cuda()
    va, vb = (CacheView(0, pages.clone(), step.block_tables[0], ps) for _ in range(2))
    a = o.decode_attention_fused(y, qw, kw, 1e-5, rot, 300.0, step, va, H, G, D, 0.2, window, True, scaling=STRETCH)
    table = ref_ops.rope_table(make_step(ref_ops, dt, ctx, [1] * len(ctx), ps, 256, 4, device="cpu"), rot, 300.0, None, STRETCH).cuda() if rot else None
    q = ref_ops.qkv_prepare(y, qw, kw, 1e-5, 1, table, rot, step, vb, H, G, D, D, D)
    b = ref_ops.paged_attention(q, step, vb, H, G, D, 0.2, window)
    assert torch.allclose(a.float(), b.float(), **tol(dt)) and torch.allclose(va.pages.float(), vb.pages.float(), **tol(dt))
    # with a gate per head from the rows' last columns, and the first values of every head alone
    V = max(D // 2, 1)
    gate = y[:, (H + 2 * G) * D + 3:(H + 2 * G) * D + 3 + H]
    c = o.decode_attention_fused(y, qw, kw, 1e-5, rot, 300.0, step, va, H, G, D, 0.2, window, True, scaling=STRETCH,
                                 gate_at=(H + 2 * G) * D + 3, value_dim=V)
    assert c.shape == (len(ctx), H * V) and torch.allclose(c.float(), ref_ops.sigmoid_gate(b, gate, H, V, True, row_dim=D).float(), **tol(dt))


@pytest.mark.parametrize("H,G,D,Dv,rot,scope", [(8, 2, 64, 64, 32, 1), (3, 1, 128, 64, 128, 1), (4, 4, 96, 96, 48, 1), (2, 1, 8, 24, 0, 1), (5, 5, 16, 8, 16, 0),
                                                (6, 2, 24, 40, 16, 1), (2, 2, 200, 256, 64, 1), (1, 1, 80, 80, 80, 0), (6, 3, 40, 40, 24, 1)])
def test_rows_prepared_for_attention(H, G, D, Dv, rot, scope):
    """bfloat16 rows whose heads are multiples of eight values: the kernel that keeps a head in registers (and, at a rotation
    whose halves are none, the other one), with every option that goes with a norm per head."""
    o = ops()
    g = torch.Generator().manual_seed(5)
    dt, Dp, ps, num_pages = torch.bfloat16, max(D, Dv), 8, 64
    ctx, q_lens = [0, 7, 30, 3], [9, 1, 20, 1]
    step = make_step(o, dt, ctx, q_lens, ps, num_pages, 6)
    N = sum(q_lens)
    y = torch.randn(N, -(-((H + G) * D + G * Dv + H) // 8) * 8, generator=g).to(dt).cuda()
    first, lam = torch.randn(N, G * Dv, generator=g).to(dt).cuda(), torch.tensor([0.3]).cuda()
    qw, kw = ((1 + 0.2 * torch.randn(D, generator=g)).cuda() if scope else None for _ in range(2))
    table = o.rope_table(step, rot, 10000.0, y.device, STRETCH) if rot else None
    for more in ({}, {"temp": (0.2, 3)}, {"v_first": first, "v_lambda": lam}):
        pages_a = torch.full((num_pages, 2, G, ps, Dp), 7.0, dtype=dt, device="cuda")
        pages_b = pages_a.clone()
        va, vb = CacheView(0, pages_a, step.block_tables[0], ps), CacheView(0, pages_b, step.block_tables[0], ps)
        a = o.qkv_prepare(y, qw, kw, 1e-5, scope, table, rot, step, va, H, G, D, Dv, Dp, True, **more)
        b = ref_ops.qkv_prepare(y, qw, kw, 1e-5, scope, table, rot, step, vb, H, G, D, Dv, Dp, True, **more)
        assert torch.allclose(a.float(), b.float(), atol=2e-2, rtol=1e-2) and torch.allclose(pages_a.float(), pages_b.float(), atol=2e-2, rtol=1e-2)
        keep = pages_a.clone()
        o.qkv_prepare(y * 2, qw, kw, 1e-5, scope, table, rot, step, va, H, G, D, Dv, Dp, False, **more)
        assert torch.equal(pages_a, keep)
    assert o.read_status() == 0


def attention_part(H, G, D, V, window, dims, scale, g, hidden):
    position = PartSpec("rotary_half_split", dict(head_dim=D, theta=500.0, rotary_dim=dims,
                                                  scaling=dict(factor=4.0, original=60, fast=8.0, slow=0.5))) if dims else PartSpec("none", {})
    part = make_part("mixer", PartSpec("attention", dict(
        hidden=hidden, heads=H, kv_heads=G, head_dim=D, value_dim=V, qk_norm=True, eps=1e-5, position=position, window=window, scale=scale,
        bias=True, out_bias=True, gate="head")))
    nm, t = part.names, {}
    for k, n in (("q", H * D), ("k", G * D), ("v", G * V), ("g", H)):
        t[nm[k]] = torch.randn(n, hidden, generator=g) * hidden ** -0.5
    t[nm["o"]] = torch.randn(hidden, H * V, generator=g) * (H * V) ** -0.5
    for k, n in (("q_bias", H * D), ("k_bias", G * D), ("v_bias", G * V), ("o_bias", hidden)):
        t[nm[k]] = (torch.randn(n, generator=g) * 0.5).to(torch.bfloat16).float()
    for k in ("q_norm", "k_norm"):
        t[nm[k]] = 1 + 0.2 * torch.randn(D, generator=g)
    m = dict(heads=H, kv_heads=G, dim=D, vdim=V, scale=scale, mask={"size": window},
             rot={"base": 500.0, "dims": dims, "scaling": {"factor": 4.0, "original": 60, "fast": 8.0, "slow": 0.5}})
    return part, t, m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,window,dims", [(6, 2, 32, 32, 24, 16), (2, 1, 16, 24, 5, 16), (3, 3, 8, 40, 70, 0), (4, 1, 64, 64, 33, 32),
                                                 (8, 2, 128, 64, 40, 64), (2, 2, 20, 12, 1, 10), (6, 2, 64, 48, 1000, 64), (4, 2, 96, 96, 13, 24)])
def test_attention_part_with_planted_keys(dtype, H, G, D, V, window, dims):
    """The part over cached pages against the formula, with one row whose key stands out in every score: just inside and just
    outside the window, at a page border, far away, for a row of a span and for a single token.  A key that the last row sees
    takes the weight; one that it does not see changes nothing."""
    o = ops()
    g = torch.Generator().manual_seed(11)
    hidden, ps, T = 64, 8, 150
    part, t, m = attention_part(H, G, D, V, window, dims, 3.0 * D ** -0.5, g, hidden)
    cuda = {k: (v.to(dtype) if v.dim() == 2 else v).cuda() for k, v in t.items()}
    part.bind(cuda, dtype)
    need = part.cache_need()
    stored = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
              "q_norm": "q.norm", "k_norm": "k.norm"}
    w64 = {"m." + n: cuda[part.names[k]].double().cpu() for k, n in stored.items()}
    base = torch.randn(T, hidden, generator=g).to(dtype)
    plain_base = P.attention(m, w64, "m.", base.double(), 1e-5, torch.float64)
    for place in sorted({T - 1, max(T - window, 0), max(T - window - 1, 0), 7, 8, 64, 0}):
        seen = T - 1 - place < window
        x = base.clone()
        x[place] = (base[place].float() * 6.0).to(dtype)
        want = P.attention(m, w64, "m.", x.double(), 1e-5, torch.float64)
        if place != T - 1:
            assert bool((want[-1] - plain_base[-1]).abs().max() > 1e-4) == seen     # the formula itself: the edge counts
        for cuts in ([T], [60, 90], [T - 1, 1], [10, 2, 52, 22, 63, 1]):
            pages = torch.zeros(40, 2, need.kv_heads, ps, need.head_dim, dtype=dtype).cuda()
            at, got = 0, []
            for c in cuts:
                step = make_step(o, dtype, [at], [c], ps, 40, 3)
                got.append(part.forward(x[at:at + c].cuda().contiguous(), step, CacheView(0, pages, step.block_tables[0], ps)))
                at += c
            err = (torch.cat(got).double().cpu() - want).abs().max(dim=-1).values / want.abs().max()
            assert float(err.max()) < (1e-5 if dtype == torch.float32 else 2.5e-2), (place, cuts, int(err.argmax()), float(err.max()))
    assert o.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_and_the_embedding_merged(dtype):
    """The block that replaces the stream by a product of the stream and the embedding's output, several times in one step (the
    embedding's share is made once), behind each kind of pending term."""
    from zig_ai_b200.parts.base import NormedTerm
    o = ops()
    g = torch.Generator().manual_seed(21)
    for N, W in ((1, 40), (9, 128), (200, 66)):
        block = make_part("block", PartSpec("stream_merge", dict(hidden=W, weight="in")))
        w = (torch.randn(W, 2 * W, generator=g) * (2 * W) ** -0.5).to(dtype).cuda()
        block.bind({"in": w}, dtype)
        step = make_step(o, dtype, [0], [N], 8, 64, 3)
        x0 = torch.randn(N, W, generator=g).to(dtype).cuda()
        step.scratch["embedding"] = x0
        h = torch.randn(N, W, generator=g).cuda() * 4
        res, plain = Residual(h.clone()), h.double()
        delta, gamma = torch.randn(N, W, generator=g).to(dtype).cuda(), (1 + 0.2 * torch.randn(W, generator=g)).cuda()
        for pending in (None, delta, NormedTerm(delta, gamma, 1e-5)):
            if isinstance(pending, NormedTerm):
                plain = plain + P.rms(delta.double(), 1e-5) * gamma.double()
            elif pending is not None:
                plain = plain + delta.double()
            plain = torch.cat([plain, x0.double()], dim=-1) @ w.double().T
            res, left = block.forward(res, pending, step, [])
            assert left is None and res.data.dtype == torch.float32
            assert float((res.data.double() - plain).abs().max()) < (1e-4 if dtype == torch.float32 else 6e-2)
