"""The kernels and kernel options that the Sogenex design adds, each alone against its plain PyTorch version
(tests/ref_ops.py), in 32-bit and in bfloat16: embedding rows with sinusoidal position vectors; the state-space recurrence
(walked, in chunks on the tensor cores and as one kernel for single tokens; spans beside single tokens, later steps that
continue from earlier ones' state, chunk borders, decays near one and near zero, a far token that stands out); the
difference of the two maps of differential attention, and the part as a whole with planted keys at the window's edges in
each map; experts without a gate chosen by their logits, with a bias and a gated unit beside them; relu squared as the
few-rows product's epilogue."""
import pytest
import torch

import plain_sogenex as P
import ref_ops
from test_gpu_kernels import make_step
from test_gpu_recurrent_kernels import MANY_SINGLES, STEPS
from zig_ai_b200.cache.manager import CacheView
from zig_ai_b200.parts import PartSpec, make_part

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def ops():
    from zig_ai_b200.kernels import ops as o
    o.require(extra=("attention", "attention_mma", "attention_tma", "attention_tc", "attention_difference", "mamba2", "causal_conv", "moe",
                     "gemm_tc"))
    return o


def tol(dtype):
    return dict(atol=3e-5, rtol=3e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 40, 67, 1024, 1])
def test_embedding_with_position_vectors(dtype, width):
    o = ops()
    g = torch.Generator().manual_seed(1)
    table = torch.randn(50, width, generator=g).to(dtype).cuda()
    ids = torch.randint(0, 50, (37,), generator=g).to(torch.int32).cuda()
    pos = torch.randint(0, 1 << 20, (37,), generator=g).to(torch.int32).cuda()
    pos[:4] = torch.tensor([0, 1, 2, 9999], dtype=torch.int32)
    for scale, base in ((1.0, 10000.0), (0.5, 300.0)):
        a = o.embed(ids, table, scale, pos, base)
        b = ref_ops.embed(ids, table, scale, pos, base)
        assert a.dtype == torch.float32 and torch.allclose(a, b, atol=2e-6, rtol=0)
    vec = P.positions(3, width, torch.float64, first=5)
    got = o.embed(torch.zeros(3, dtype=torch.int32).cuda(), torch.zeros_like(table), 1.0, torch.tensor([5, 6, 7], dtype=torch.int32).cuda())
    assert torch.allclose(got.cpu().double(), vec, atol=1e-6)
    bad = torch.tensor([3, 99], dtype=torch.int32).cuda()
    o.embed(bad, table, 1.0, pos[:2].contiguous())
    assert o.read_status() == 2


SIZES = [(2, 64, 1, 32, 1, 4), (3, 20, 3, 10, 3, 2), (4, 64, 2, 128, 4, 4), (2, 40, 1, 33, 1, 3), (6, 16, 2, 12, 2, 1), (1, 130, 1, 64, 1, 5),
         (4, 32, 4, 16, 8, 4), (2, 96, 2, 200, 1, 4), (3, 7, 1, 5, 1, 4), (8, 128, 4, 256, 2, 4)]


def columns(I, ch, H):
    """First columns of z, x | B | C and dt in rows whose parts start on multiples of eight columns."""
    up = lambda n: -(-n // 8) * 8
    return (0, up(I), up(I) + up(ch)), up(I) + up(ch) + up(H)


def make_mamba(g, H, V, G, Ns, L, slots, dt_shift=-2.0):
    I, ch = H * V, H * V + 2 * G * Ns
    w = dict(conv_w=(torch.randn(ch, L, generator=g) * 0.5).cuda(), conv_b=(torch.randn(ch, generator=g) * 0.2).cuda(),
             dt_bias=(torch.randn(H, generator=g) + dt_shift).cuda(), a_log=(torch.randn(H, generator=g) * 0.7).cuda(),
             d_skip=torch.randn(H, generator=g).cuda(), norm_w=(1 + 0.2 * torch.randn(I, generator=g)).cuda())
    state = torch.zeros(slots, H, Ns, V).cuda()
    hist = torch.zeros(slots, max(L - 1, 1), ch).cuda()
    return w, state, hist, I, ch


def run_mamba(o, y, at, w, parts, state, hist, step, H, G, Ns, V, write=True, **kw):
    return o.mamba2(y, at, w["conv_w"], w["conv_b"], w["dt_bias"], w["a_log"], w["d_skip"], w["norm_w"], 1e-5, parts, state, hist, step,
                    H, G, Ns, V, write, **kw)


@pytest.mark.parametrize("impl", [None, "walk", "chunks"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V,G,Ns,parts,L", SIZES)
def test_state_space_recurrence(dtype, H, V, G, Ns, parts, L, impl):
    """Every way through the rows against the recurrence in 64-bit; the state and the convolution's history go on from step
    to step."""
    o = ops()
    g = torch.Generator().manual_seed(4)
    w, sa, ha, I, ch = make_mamba(g, H, V, G, Ns, L, 22)
    at, cols = columns(I, ch, H)
    sb, hb = sa.clone(), ha.clone()
    for q_lens in STEPS + (MANY_SINGLES,):
        step = make_step(o, dtype, [3] * len(q_lens), q_lens, 8, 256, 5)
        y = torch.randn(sum(q_lens), cols, generator=g).to(dtype).cuda()
        a = run_mamba(o, y, at, w, parts, sa, ha, step, H, G, Ns, V, impl=impl)
        b = run_mamba(ref_ops, y, at, w, parts, sb, hb, step, H, G, Ns, V, precision=torch.float64)
        limit = dict(atol=1e-4, rtol=1e-4) if dtype == torch.float32 else tol(dtype)
        assert torch.allclose(a.float(), b.float(), **limit), (q_lens, float((a.float() - b.float()).abs().max()))
        # bfloat16: the convolution's output may round the other way in the two versions, so a state may differ by that much
        close = dict(atol=1e-5, rtol=1e-4) if dtype == torch.float32 else dict(atol=5e-3, rtol=5e-3)
        assert torch.allclose(sa, sb, **close), (q_lens, float((sa - sb).abs().max()))
        assert torch.allclose(ha, hb, atol=1e-6), q_lens
    keep_s, keep_h = sa.clone(), ha.clone()
    for q_lens in (STEPS[4], [1] * 5):
        step = make_step(o, dtype, [3] * 5, q_lens, 8, 256, 5)
        y = torch.randn(sum(q_lens), cols, generator=g).to(dtype).cuda()
        run_mamba(o, y, at, w, parts, sa, ha, step, H, G, Ns, V, write=False, impl=impl)           # write_state off: it stays
        assert torch.equal(sa, keep_s) and torch.equal(ha, keep_h)
    assert o.read_status() == 0


@pytest.mark.parametrize("impl", ["walk", "chunks"])
@pytest.mark.parametrize("decay", ["near one", "middling", "near zero", "mixed"])
def test_recurrence_holds_32_bits(decay, impl):
    """bfloat16 rows: the state after hundreds of rows against the recurrence in 64-bit over the very numbers that the
    convolution's kernel gave, whatever the decays; the read-outs of the two ways agree but for their rounding to bfloat16."""
    o = ops()
    g = torch.Generator().manual_seed(6)
    H, V, G, Ns, L = 4, 64, 2, 128, 4
    w, sa, ha, I, ch = make_mamba(g, H, V, G, Ns, L, 8)
    w["a_log"].copy_({"near one": torch.tensor([-8.0, -6.0, -7.0, -9.0]), "middling": torch.tensor([1.0, 2.0, 1.5, 0.0]),
                      "near zero": torch.tensor([4.0, 5.0, 3.0, 6.0]), "mixed": torch.tensor([-9.0, -1.0, 2.0, 5.0])}[decay].cuda())
    at, cols = columns(I, ch, H)
    hb, hc, sc = ha.clone(), ha.clone(), sa.clone()
    exact = torch.zeros(8, H, Ns, V, dtype=torch.float64)
    for q_lens in ([300, 64, 1, 65, 127], [128, 2, 700, 63, 33]):
        step = make_step(o, torch.bfloat16, [0] * 5, q_lens, 8, 512, 5)
        y = torch.randn(sum(q_lens), cols, generator=g).to(torch.bfloat16).cuda()
        a = run_mamba(o, y, at, w, 4, sa, ha, step, H, G, Ns, V, impl=impl)
        other = run_mamba(o, y, at, w, 4, sc, hc, step, H, G, Ns, V, impl="walk" if impl == "chunks" else "chunks")
        assert torch.allclose(a.float(), other.float(), atol=4e-3, rtol=8e-3)
        u = o.causal_conv(y[:, at[1]:at[1] + ch], w["conv_w"], w["conv_b"], hb, step, True, True).double().cpu()
        d = torch.nn.functional.softplus(y[:, at[2]:at[2] + H].double().cpu() + w["dt_bias"].double().cpu())
        keep = torch.exp(-torch.exp(w["a_log"].double().cpu()) * d)
        for s, (lo, hi) in enumerate(zip(step.cu_q.tolist()[:-1], step.cu_q.tolist()[1:])):
            S = exact[int(step.slot_ids[s])]
            for t in range(lo, hi):
                B = u[t, I:I + G * Ns].reshape(G, Ns).repeat_interleave(H // G, dim=0)
                S = keep[t][:, None, None] * S + d[t][:, None, None] * B[:, :, None] * u[t, :I].reshape(H, 1, V)
            exact[int(step.slot_ids[s])] = S
        err = ((sa.double().cpu() - exact).abs().amax(dim=(0, 2, 3)) / exact.abs().amax(dim=(0, 2, 3)))
        assert float(err.max()) < (1e-5 if impl == "walk" else 4e-6), err.tolist()      # (800 roundings, one after the other)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_stands_out_of_the_state(dtype):
    """Decays of nearly one and one token with a large step: its value is read out hundreds of rows later by the one row whose C
    is its B, whether the rows between come as one span, as spans cut next to chunk borders, or one by one."""
    o = ops()
    g = torch.Generator().manual_seed(7)
    H, V, G, Ns, L = 2, 32, 1, 64, 1
    w, s0, h0, I, ch = make_mamba(g, H, V, G, Ns, L, 3)
    w["conv_w"].fill_(1.0)
    w["conv_b"].zero_()
    w["a_log"].fill_(-12.0)
    w["dt_bias"].fill_(-8.0)
    w["d_skip"].zero_()
    w["norm_w"].fill_(1.0)
    at, cols = columns(I, ch, H)
    n = 330
    y = torch.zeros(n, cols)
    y[:, at[0]:at[0] + I] = 4.0
    y[:, at[1]:at[1] + I] = torch.randn(n, I, generator=g) * 0.3
    key = (torch.randn(Ns, generator=g) > 0).float() * 4.0
    y[5, at[1] + I:at[1] + I + Ns] = key                      # B of row 5
    y[5, at[2]:at[2] + H] = 12.0                              # ... with a step of 4 where the others have e^-8
    y[5, at[1]:at[1] + I] = torch.arange(I).float() % 7 + 1.0
    y[n - 1, at[1] + I + Ns:at[1] + I + 2 * Ns] = key         # C of the last row
    y = y.to(dtype).cuda()
    want = torch.nn.functional.silu(torch.arange(I).float() % 7 + 1.0).reshape(H, V)
    want = (want / want.reshape(1, -1).pow(2).mean().sqrt()).reshape(-1)
    for cuts in ([330], [64, 64, 65, 63, 74], [3, 2, 190, 135], [300] + [1] * 30, [1] * 330):
        state, hist = s0.clone(), h0.clone()
        at_row = 0
        for c in cuts:
            step = make_step(o, dtype, [at_row], [c], 8, 128, 5)
            out = run_mamba(o, y[at_row:at_row + c].contiguous(), at, w, 1, state, hist, step, H, G, Ns, V)
            at_row += c
        assert torch.allclose(out[-1].float().cpu(), want, atol=3e-2, rtol=2e-2), cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V,Dp", [(1, 8, 8), (3, 12, 20), (8, 128, 128), (2, 300, 300), (5, 64, 64)])
def test_difference_of_two_maps(dtype, H, V, Dp):
    o = ops()
    g = torch.Generator().manual_seed(9)
    x = torch.randn(41, 2 * H * Dp, generator=g).to(dtype).cuda()
    for lam, factor in ((0.7, 0.4), (-0.3, 1.0), (1.0, 0.2)):
        a = o.attention_difference(x, H, V, Dp, lam, factor, 1e-5)
        b = ref_ops.attention_difference(x, H, V, Dp, lam, factor, 1e-5)
        assert torch.allclose(a.float(), b.float(), **tol(dtype)), (lam, factor)


def differential_part(H, G, D, V, window, scale, diff, g, hidden=64):
    part = make_part("mixer", PartSpec("attention", dict(
        hidden=hidden, heads=H, kv_heads=G, head_dim=D, value_dim=V, qk_norm=False, eps=1e-5, position=PartSpec("none", {}), window=window,
        scale=scale, differential={"diff": diff})))
    nm = part.names
    t = {nm["q"]: torch.randn(H * 2 * D, hidden, generator=g) * hidden ** -0.5, nm["k"]: torch.randn(G * 2 * D, hidden, generator=g) * hidden ** -0.5,
         nm["v"]: torch.randn(G * V, hidden, generator=g) * hidden ** -0.5, nm["o"]: torch.eye(hidden)[:, :1].repeat(1, H * V) * 0}
    t[nm["o"]] = torch.randn(hidden, H * V, generator=g) * (H * V) ** -0.5
    for k in ("lq1", "lk1", "lq2", "lk2"):
        t[nm[k]] = torch.randn(D, generator=g) * 0.3
    return part, t


def cancellation(m, w, h):
    """Per row: the largest ratio over the heads of the maps' sizes to their difference's, at least 1."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["m." + n].T for n in "qkv")
    lam = P.mixing(w, "m.", m["diff"], torch.float64)
    v = v.reshape(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    maps = [P.one_map(q.reshape(T, H, 2, D)[:, :, i].permute(1, 0, 2), k.reshape(T, G, 2, D)[:, :, i].permute(1, 0, 2)
                      .repeat_interleave(H // G, dim=0), v, m["scale"], m["mask"]["size"]) for i in range(2)]
    ratio = (maps[0].norm(dim=-1) + lam.abs() * maps[1].norm(dim=-1)) / (maps[0] - lam * maps[1]).norm(dim=-1)
    return ratio.max(dim=0).values.clamp(min=1.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,window", [(6, 2, 32, 64, 24), (2, 1, 16, 24, 5), (3, 3, 8, 40, 70), (4, 1, 64, 128, 33), (2, 2, 20, 40, 1),
                                            (6, 2, 24, 16, 1000)])
def test_differential_attention_with_planted_keys(dtype, H, G, D, V, window):
    """The part over cached pages against the formula, with one key made to match the last row's query in one of the two maps: just
    inside and just outside the window, at a page border, far away, for a row of a span and for a single token.  A key that
    the row sees takes that map's weight; one that it does not see changes nothing."""
    o = ops()
    g = torch.Generator().manual_seed(11)
    hidden, ps = 64, 8
    part, t = differential_part(H, G, D, V, window, D ** -0.5, 0.4, g, hidden)
    cuda = {k: (v.to(dtype) if v.dim() == 2 else v).cuda() for k, v in t.items()}
    part.bind(cuda, dtype)
    need = part.cache_need()
    T = 150
    w64 = {"m." + n: cuda[part.names[n]].double().cpu() for n in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")}
    m = dict(heads=H, kv_heads=G, dim=D, vdim=V, scale=D ** -0.5, mask={"size": window}, diff=0.4)
    base = (torch.randn(T, hidden, generator=g)).to(dtype)
    plain_base = P.attention(m, w64, "m.", base.double(), 1e-5, torch.float64)
    for place in sorted({T - 1, max(T - window, 0), max(T - window - 1, 0), 7, 8, 64, 0}):
        seen = T - 1 - place < window
        x = base.clone()
        x[place] = (base[place].float() * 12.0).to(dtype)                # a row that stands out in every score
        want = P.attention(m, w64, "m.", x.double(), 1e-5, torch.float64)
        if place != T - 1:
            assert bool((want[-1] - plain_base[-1]).abs().max() > 1e-3) == seen     # the formula itself: the edge counts
        # where the two maps nearly cancel, their rounding grows with the norm behind the difference
        grown = cancellation(m, w64, x.double())
        for cuts in ([T], [60, 90], [T - 1, 1], [10, 2, 52, 22, 63, 1]):
            pages = torch.zeros(40, 2, need.kv_heads, ps, need.head_dim, dtype=dtype).cuda()
            at, got = 0, []
            for c in cuts:
                step = make_step(o, dtype, [at], [c], ps, 40, 3)
                got.append(part.forward(x[at:at + c].cuda().contiguous(), step, CacheView(0, pages, step.block_tables[0], ps)))
                at += c
            err = (torch.cat(got).double().cpu() - want).abs().max(dim=-1).values / want.abs().max()
            limit = (1e-5 if dtype == torch.float32 else 1.5e-2) * grown
            assert bool((err < limit).all()), (place, cuts, int((err / limit).argmax()), float((err / limit).max()))
    assert o.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,W,F,E,top", [(1, 64, 32, 4, 2), (7, 48, 24, 5, 5), (40, 128, 96, 8, 4), (300, 128, 64, 8, 2), (700, 256, 128, 8, 4),
                                         (16, 66, 20, 3, 1), (2000, 128, 128, 4, 2), (33, 72, 40, 40, 6), (600, 64, 40, 17, 3)])
def test_experts_without_a_gate(dtype, N, W, F, E, top):
    o = ops()
    g = torch.Generator().manual_seed(17)
    w_router = (torch.randn(E + 1, W, generator=g) * 0.3).cuda()
    bias = torch.randn(E, generator=g).cuda()
    w_up, w_dn = (torch.randn(E, F, W, generator=g) * W ** -0.5).to(dtype).cuda(), (torch.randn(E, W, F, generator=g) * F ** -0.5).to(dtype).cuda()
    x, unit = torch.randn(N, W, generator=g).to(dtype).cuda(), torch.randn(N, W, generator=g).to(dtype).cuda()
    z = (x.float() @ w_router[:E].t() + bias).sort(dim=-1, descending=True).values
    sure = torch.ones(N, dtype=torch.bool, device="cuda") if top == E else (z[:, top - 1] - z[:, top]) > 1e-3
    assert int(sure.sum()) >= N - max(3, N // 50)
    for kw in (dict(router_bias=bias, unit=unit, unit_gated=True), dict(router_bias=bias), dict(unit=unit), {}):
        r = w_router if kw.get("unit_gated") else w_router[:E].contiguous()
        a = o.routed_experts(x, r, w_up, w_dn, top, False, "output", score="chosen", act="relu2", **kw)
        b = ref_ops.routed_experts(x, r, w_up, w_dn, top, False, "output", score="chosen", act="relu2", **kw)
        if kw.get("router_bias") is not None:
            assert torch.allclose(a.float()[sure], b.float()[sure], **tol(dtype)), sorted(kw)
        else:
            bad = ~torch.isclose(a.float(), b.float(), **tol(dtype)).all(dim=-1)
            assert int(bad.sum()) <= max(3, N // 50), sorted(kw)
    plain = ref_ops.routed_experts(x, w_router[:E].contiguous(), w_up, w_dn, top, False, "output", score="chosen", act="relu2", unit=unit)
    full = ref_ops.routed_experts(x, w_router, w_up, w_dn, top, False, "output", score="chosen", act="relu2", router_bias=bias, unit=unit,
                                  unit_gated=True)
    assert (plain.float() - full.float()).abs().max() > 0.05              # bias and gate count
    assert o.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_large_bias_and_equal_logits(dtype):
    """Logits far from zero (a bias of a thousand) give the softmax over the chosen all the same; equal logits go to the lower index."""
    o = ops()
    g = torch.Generator().manual_seed(19)
    E, W, F, top = 6, 32, 16, 3
    w_up, w_dn = torch.randn(E, F, W, generator=g).to(dtype).cuda() * 0.2, torch.randn(E, W, F, generator=g).to(dtype).cuda() * 0.2
    x = torch.randn(20, W, generator=g).to(dtype).cuda()
    zero = torch.zeros(E, W).cuda()
    for bias in (torch.tensor([1000.0, 999.0, -1000.0, 998.5, 5.0, 6.0]), torch.tensor([-900.0, -901.0, -900.5, -1000.0, -950.0, -902.0]),
                 torch.zeros(E)):
        a = o.routed_experts(x, zero, w_up, w_dn, top, False, "output", score="chosen", act="relu2", router_bias=bias.cuda())
        order = sorted(range(E), key=lambda e: (-float(bias[e]), e))[:top]
        wts = torch.softmax(bias[order], dim=0)
        want = sum(float(wts[i]) * ((torch.relu(x.float() @ w_up[e].float().t()) ** 2).to(dtype).float() @ w_dn[e].float().t())
                   for i, e in enumerate(order))
        assert torch.allclose(a.float(), want, **tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
def test_relu_squared(dtype):
    o = ops()
    g = torch.Generator().manual_seed(23)
    x = torch.randn(37, 72, generator=g).to(dtype).cuda()
    assert torch.allclose(o.activation(x, "relu2").float(), ref_ops.activation(x, "relu2").float(), **tol(dtype))
    for rows, K, F in ((37, 40, 72), (5, 256, 128), (16, 2048, 384), (1, 128, 70), (8, 4096, 256)):   # (few rows in bfloat16: the product's epilogue)
        x = torch.randn(rows, K, generator=g).to(dtype).cuda()
        w = (torch.randn(F, K, generator=g) * K ** -0.5).to(dtype).cuda()
        assert torch.allclose(o.linear_activation(x, w, "relu2").float(), ref_ops.linear_activation(x, w, "relu2").float(), **tol(dtype)), (rows, K, F)
