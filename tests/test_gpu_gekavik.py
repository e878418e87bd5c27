"""Gekavik on the GPU against the plain float64 restatement in ``oracle/gekavik.py`` (no code shared with the package).

Kernel level: every new or extended mechanism alone, with inputs built so that a fault shows (one key that takes the whole
softmax, just inside / just outside a window, among the kept first keys and just behind them, at page borders, far among
hundreds; clamps that bite; experts that only their group keeps out; a residual stream whose low bits matter).  Engine level,
through ``CausalLMEngine`` and its scheduler: whole prompts, token-by-token decoding, portions, mixed batches, reuse of pages
and slots, long decoding across pages and windows, loops, odd sizes, greedy generation, CUDA graphs against eager.  The float32
engine is the sharp comparison; bfloat16 is checked against its rounding noise."""
import json

import pytest
import torch

from oracle import gekavik as O
from tests.test_gekavik_config import sharpened
from tests.lm_util import DEV, Lay, cuts_of, make_engine, nerr, nerr_rows, rel, replay, tokens_for

pytestmark = pytest.mark.gpu
F64 = torch.float64
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


@pytest.fixture(scope="module")
def nat():
    import nano_qwen3tts_vllm_b200._native as n
    n.lib()
    return n


def norm_of(cols, g, alpha=0.9):
    """(w, b, alpha) of a dynamic tanh on the GPU, and the same in float64 under the plain code's names."""
    w, b, a = torch.randn(cols, generator=g), torch.randn(cols, generator=g) * 0.5, torch.tensor([alpha])
    return tuple(t.to(DEV) for t in (w, b, a)), {"n": w.double(), "n.b": b.double(), "n.alpha": a.double()}


# ------------------------------------------------------------------------------------------------ per-row kernels
@BOTH
@pytest.mark.parametrize("n,cols,top", [(5, 24, 2), (3, 257, 1), (9, 1000, 4), (4500, 512, 3), (1, 8, 7)])
def test_dynamic_tanh_around_a_sublayer(nat, dtype, n, cols, top):
    g = torch.Generator().manual_seed(cols)
    d = lambda t: t.to(DEV)
    (post, post64), (pre, pre64) = norm_of(cols, g, -1.3), norm_of(cols, g, 0.6)
    x0 = torch.randn(n, cols, generator=g) * 2
    a = (torch.randn(n, cols, generator=g) * 4).to(dtype)                       # well into saturation and around zero
    z, zw = torch.randn(n * top, cols, generator=g).to(dtype), torch.rand(n, top, generator=g)
    moe = (zw.double()[:, :, None] * z.double().view(n, top, cols)).sum(1)
    for kw, y in ((dict(a=d(a)), a.double()), (dict(z=d(z), zw=d(zw)), moe), (dict(a=d(a), z=d(z), zw=d(zw)), a.double() + moe)):
        x = d(x0.clone())
        h = nat.tanh_residual(x, post=post, mult=0.3, pre=pre, **kw)
        want = x0.double() + 0.3 * O.dyt(y, post64, "n")
        assert rel(x, want) < 2e-6 and rel(h, O.dyt(want, pre64, "n")) < TOL[dtype]
        x = d(x0.clone())
        assert nat.tanh_residual(x, post=post, mult=0.3, **kw) is None and rel(x, want) < 2e-6
    # no sublayer: the norm alone, the stream untouched
    x = d(x0.clone())
    h = nat.tanh_residual(x, pre=pre, dtype=dtype)
    assert torch.equal(x.cpu(), x0) and rel(h, O.dyt(x0.double(), pre64, "n")) < TOL[dtype]
    # an embedding row per token, whatever the stream held; ids outside the table read as row 0
    table, ids = torch.randn(11, cols, generator=g).to(dtype), torch.randint(0, 11, (n,), generator=g)
    x = d(torch.full((n, cols), 1e9))
    h = nat.tanh_residual(x, table=d(table), index=d(ids.int()), init=True, pre=pre)
    assert torch.equal(x.cpu(), table.float()[ids]) and rel(h, O.dyt(table.double()[ids], pre64, "n")) < TOL[dtype]
    x = torch.empty(n, cols, device=DEV)
    nat.tanh_residual(x, table=d(table), index=d(torch.full((n,), 99, dtype=torch.int32)), init=True)
    assert torch.equal(x.cpu(), table.float()[:1].expand(n, cols))
    # gathered rows
    rows = torch.randint(0, n, (7,), generator=g)
    got = nat.tanh_gather(d(x0), d(rows.int()), pre, dtype)
    assert rel(got, O.dyt(x0.double()[rows], pre64, "n")) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("n,width", [(5, 24), (7, 128), (130, 192), (600, 256), (1, 72)])
def test_projection_in_front_of_a_pass_keeps_the_streams_low_bits(nat, dtype, n, width):
    """W [x; x0] + step with a stream that is 1 plus a part 2^-9 as large: rounding it to 8 bits would lose that part, which the
    weights of this case single out (their rows sum to zero, so the ones cancel)."""
    from nano_qwen3tts_vllm_b200.layers.pass_input import PassInput
    g = torch.Generator().manual_seed(width)
    table, ids = (torch.randn(13, width, generator=g) * 2.0 ** -9).to(dtype), torch.randint(0, 13, (n,), generator=g)
    x0 = 1.0 + torch.randn(n, width, generator=g) * 2.0 ** -9
    half = torch.randn(width, width // 2, generator=g)
    W = torch.cat([half, -half, torch.randn(width, width, generator=g)], 1).to(torch.bfloat16)
    step = (torch.randn(3, width, generator=g) * 2.0 ** -9).to(torch.bfloat16)
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        layer = PassInput(width, 3).to(DEV)
    finally:
        torch.set_default_dtype(prev)
    layer.weight.data.copy_(layer.expand(W))
    layer.step.data.copy_(step)
    matmul = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        x = x0.to(DEV)
        cat = nat.tanh_residual(x, table=table.to(DEV), index=ids.int().to(DEV), want_cat=True)
        assert cat.shape == (n, (3 if dtype == torch.bfloat16 else 2) * width) and torch.equal(x.cpu(), x0)
        layer(x, cat, 2)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = matmul
    want = torch.cat([x0.double(), table.double()[ids]], 1) @ W.double().T + step.double()[2]
    rounded = torch.cat([x0.to(torch.bfloat16).double(), table.double()[ids]], 1) @ W.double().T + step.double()[2]
    assert rel(x, want) < (5e-4 if dtype == torch.float32 else 1e-2)
    assert rel(rounded, want) > 0.1                                            # what one bf16 number per coordinate would give


@pytest.mark.parametrize("m,n,k", [(1, 128, 64), (64, 384, 192), (130, 256, 128), (700, 256, 128), (5, 100, 60), (0, 128, 64)])
def test_float_output_of_a_bf16_product(nat, m, n, k):
    from nano_qwen3tts_vllm_b200.layers.linear import linear_float
    g = torch.Generator().manual_seed(m + n)
    x, w, b = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((m, k), (n, k), (n,)))
    dx, dw, db = (t.to(DEV) for t in (x, w, b))
    want = x.double() @ w.double().T
    for bias in (None, b):
        ref = want if bias is None else want + b.double()
        got = linear_float(dx, dw, None if bias is None else db)
        assert got.dtype == torch.float32 and got.shape == (m, n)
        if m:
            assert rel(got, ref) < 3e-6


# ------------------------------------------------------------------------------------------------ experts
def expert64(x, gate_up, limit):
    ff = gate_up.shape[0] // 2
    u = x.double() @ gate_up.double().T
    gt, up = u[:, :ff].clamp(max=limit), u[:, ff:].clamp(-limit, limit)
    return gt * torch.sigmoid(1.702 * gt) * (up + 1)


@BOTH
@pytest.mark.parametrize("m,ff,k", [(1, 64, 64), (40, 192, 128), (130, 64, 192), (600, 128, 64), (6, 10, 24), (3, 33, 50)])
@pytest.mark.parametrize("limit", [0.7, 3.0])
def test_clamped_gate_in_the_gemm_and_alone(nat, dtype, m, ff, k, limit):
    """Pre-activations of standard deviation 3 reach past both limits on both sides."""
    from nano_qwen3tts_vllm_b200.layers.linear import linear_clamped_gate
    g = torch.Generator().manual_seed(m + ff)
    x = torch.randn(m, k, generator=g).to(dtype)
    w = (3 * k ** -0.5 * torch.randn(2 * ff, k, generator=g)).to(dtype)
    pre = x.double() @ w.double().T
    assert (pre[:, :ff] > limit).any() and (pre[:, ff:] > limit).any() and (pre[:, ff:] < -limit).any() and (pre[:, :ff] < -limit).any()
    got = linear_clamped_gate(x.to(DEV), w.to(DEV), limit)
    assert rel(got, expert64(x, w, limit)) < TOL[dtype]
    gu = pre.to(dtype)
    ref = expert64(gu, torch.eye(2 * ff), limit)
    assert rel(nat.clamped_gate_mul(gu.to(DEV), limit), ref) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("n,E,top,ff,k", [(1, 4, 2, 8, 16), (7, 5, 3, 24, 40), (300, 6, 2, 72, 64), (500, 3, 1, 136, 128), (9, 4, 2, 10, 24),
                                          (64, 16, 4, 200, 96)])
def test_grouped_clamped_experts(nat, dtype, n, E, top, ff, k):
    g = torch.Generator().manual_seed(n * ff)
    h = torch.randn(n, k, generator=g).to(dtype)
    w = (2 * k ** -0.5 * torch.randn(E, 2 * ff, k, generator=g)).to(dtype)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)])
    if E > 3:
        idx[idx == 1] = 0                                                      # an expert without a token
    pairs = idx.reshape(-1)
    order = torch.argsort(pairs, stable=True)
    offsets = torch.tensor([(pairs < e).sum() for e in range(E + 1)], dtype=torch.int32)
    c = torch.full((n * top, ff), 7.0, dtype=dtype, device=DEV)
    nat.grouped_gemm_gated(h.to(DEV), w.to(DEV), c, offsets.to(DEV), order.int().to(DEV), n * top, top, 1.1)
    want = torch.stack([expert64(h[p // top][None], w[pairs[p]], 1.1)[0] for p in order.tolist()])
    assert rel(c, want) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("E,top,count,keep", [(6, 3, 3, 2), (6, 2, 3, 2), (16, 4, 4, 1), (64, 6, 8, 3), (8, 3, 1, 1), (12, 5, 12, 7), (9, 4, 3, 2), (256, 8, 64, 9)])
def test_group_limited_routing(nat, dtype, E, top, count, keep):
    g = torch.Generator().manual_seed(E + top)
    n, cols = 37, 48
    h, r = torch.randn(n, cols, generator=g).to(dtype), torch.randn(E, cols, generator=g) * 0.5
    ti, tw = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
    off, sp = torch.empty(E + 1, dtype=torch.int32, device=DEV), torch.empty(n * top, dtype=torch.int32, device=DEV)
    nat.moe_route(h.to(DEV), r.to(DEV), ti, tw, off, sp, top, 1.0, mode=nat.ROUTE_SOFTMAX_ALL, groups=count, groups_keep=keep)
    idx, w = O.route(h.double(), r.double(), top, {"count": count, "keep": keep})
    assert torch.equal(ti.cpu().long(), idx) and rel(tw, w) < 1e-5
    if keep < min(top, count) and E // count > 1:                              # the groups do keep experts out
        assert not torch.equal(idx.sort(-1).values, O.route(h.double(), r.double(), top)[0].sort(-1).values)
    flat = ti.cpu().reshape(-1)
    assert off.cpu().tolist() == [int((flat < e).sum()) for e in range(E + 1)]
    assert flat[sp.cpu().long()].tolist() == sorted(flat.tolist())


def test_group_limited_routing_rejects_impossible_choices(nat):
    e = lambda *s: torch.empty(*s, device=DEV)
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=DEV)
    for kw in (dict(groups=4), dict(groups=3, groups_keep=4), dict(groups=3, groups_keep=1)):      # 6 experts, top 3
        with pytest.raises(RuntimeError):
            nat.moe_route(e(2, 8), e(6, 8), i(2, 3), e(2, 3), i(7), i(6), 3, 1.0, mode=nat.ROUTE_SOFTMAX_ALL, **kw)


# ------------------------------------------------------------------------------------------------ attention
@BOTH
@pytest.mark.parametrize("H,G,d,dv,rot,interleaved", [(4, 2, 12, 8, 8, True), (3, 1, 10, 7, 6, True), (4, 2, 64, 64, 64, True), (2, 2, 96, 48, 32, True),
                                                      (2, 1, 200, 128, 100, True), (2, 1, 16, 32, 0, True), (6, 3, 20, 20, 12, False), (2, 1, 4, 4, 2, True),
                                                      (1, 1, 1, 3, 0, True)])
def test_preparation_with_head_norms_before_the_rotation(nat, dtype, H, G, d, dv, rot, interleaved):
    from nano_qwen3tts_vllm_b200.layers.attention import SinkSoftmaxAttention
    from nano_qwen3tts_vllm_b200.layers.rotary_embedding import HalfRotaryTable, PairRotaryTable
    from nano_qwen3tts_vllm_b200.utils.context import reset_context, set_context
    g = torch.Generator().manual_seed(d + dv)
    page, base, eps = 16, 77.0, 1e-2
    big = d == 64                                                              # enough rows for the runs of several tokens per lane group
    lay = Lay([(5, 9, [2, 0]), (0, 3, [1]), (0, 0, [4])] + ([(0, 151, list(range(5 + 10 * i, 15 + 10 * i))) for i in range(40)] if big else []),
              page, 10 if big else 2)
    n, pages = lay.n_tokens, 410 if big else 5
    sizes = [H * d, G * d, G * dv]
    bias = [torch.randn(s, generator=g) for s in sizes]
    u = torch.cat([torch.randn(n, s, generator=g) for s in sizes] + [torch.zeros(n, 5)], 1).to(dtype)
    attn = SinkSoftmaxAttention(H, G, d, dv, "window", 8, 1.0, bias=True, sink="none", eps=eps, head_norm=True,
                                rotary=(PairRotaryTable if interleaved else HalfRotaryTable)(rot, base) if rot else None).to(DEV)
    qw, kw = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    for p, v in zip((attn.q_bias, attn.k_bias, attn.v_bias, attn.q_norm, attn.k_norm), bias + [qw, kw]):
        p.data.copy_(v)
    attn.k_cache = torch.full((pages, page, G * d), 5.0, dtype=dtype, device=DEV)
    attn.v_cache = torch.full((pages, page, G * dv), 5.0, dtype=dtype, device=DEV)
    if rot:
        attn.rotary.fill(lay.positions)
    set_context(False, step_layout=lay)
    try:
        q = attn.prepare(u.to(DEV), 0, sizes[0], sizes[0] + sizes[1])
    finally:
        reset_context()
    pos = lay.positions.cpu()
    part = [u[:, sum(sizes[:i]):sum(sizes[:i + 1])].double() + bias[i].double() for i in range(3)]

    def turn(v):
        if not rot or interleaved:
            return O.rotate_pairs(v, pos, rot, base)
        pair = torch.stack([v[..., :rot // 2], v[..., rot // 2:rot]], -1).flatten(-2)      # halves side by side, then back
        t = O.rotate_pairs(pair, pos, rot, base)
        return torch.cat([t[..., 0::2], t[..., 1::2], v[..., rot:]], -1)

    want_q = turn(O.unit_rms(part[0].view(n, H, d), eps, qw.double())).reshape(n, -1)
    want_k = turn(O.unit_rms(part[1].view(n, G, d), eps, kw.double())).reshape(n, -1)
    live = lay.slot_mapping.cpu() >= 0
    rows = lay.slot_mapping[live.to(DEV)].long()
    assert rel(q[live.to(DEV)], want_q[live]) < TOL[dtype]
    assert rel(attn.k_cache.view(-1, G * d)[rows], want_k[live]) < TOL[dtype]
    assert rel(attn.v_cache.view(-1, G * dv)[rows], part[2][live]) < TOL[dtype]
    others = torch.ones(pages * page, dtype=torch.bool)
    others[rows.cpu()] = False
    assert (attn.k_cache.view(-1, G * d).cpu()[others] == 5.0).all() and (attn.v_cache.view(-1, G * dv).cpu()[others] == 5.0).all()


def attention_case(nat, H, G, d, dv, window, keep, seqs, dtype, spike=None, page=16, seed=0):
    """Keys and values in shuffled pages; ``spike`` (sequence, key position): the last query of that sequence and that key
    point the same way, so the key takes the softmax when it is visible and must not when it is hidden."""
    from nano_qwen3tts_vllm_b200.layers.attention import SinkSoftmaxAttention
    from nano_qwen3tts_vllm_b200.utils.context import reset_context, set_context
    g = torch.Generator().manual_seed(seed)
    scale = (6.0 if spike else 1.0) * d ** -0.5
    nb = [(p + n + page - 1) // page for p, n in seqs]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    kc = torch.full((len(perm), page, G * d), 7.0, dtype=dtype)
    vc = torch.full((len(perm), page, G * dv), 7.0, dtype=dtype)
    lay_seqs, Q, want, gates, o = [], [], [], [], 0
    for s, (p0, n) in enumerate(seqs):
        bt = perm[o:o + nb[s]]
        o += nb[s]
        T = p0 + n
        unit = lambda *shape: O.unit_rms(torch.randn(*shape, generator=g), 1e-6)
        q, k, v = unit(T, H, d), unit(T, G, d), unit(T, G, dv)
        if spike and spike[0] == s:
            for h in range(H):
                q[T - 1, h] = k[spike[1], h // (H // G)]
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        gate = (2 * torch.randn(T, H * dv, generator=g)).to(dtype)
        for p in range(T):
            kc[bt[p // page], p % page], vc[bt[p // page], p % page] = k[p].reshape(-1), v[p].reshape(-1)
        mask = O.visible(T, window, keep)
        ref = O.softmax_attention(q.double(), k.double(), v.double(), scale, mask).reshape(T, -1) * torch.sigmoid(gate.double())
        if spike and spike[0] == s:                                          # the case shows what it is meant to show
            other = mask.clone()
            other[T - 1, spike[1]] = not other[T - 1, spike[1]]
            alt = O.softmax_attention(q.double(), k.double(), v.double(), scale, other).reshape(T, -1) * torch.sigmoid(gate.double())
            assert T == 1 or rel(alt[T - 1], ref[T - 1]) > 0.1
        lay_seqs.append((p0, n, bt)), Q.append(q[p0:].reshape(n, -1)), want.append(ref[p0:]), gates.append(gate[p0:])
    lay = Lay(lay_seqs, page, max(nb))
    attn = SinkSoftmaxAttention(H, G, d, dv, "window", window, scale, sink="none", keep_first=keep, element_gate=True).to(DEV)
    attn.k_cache, attn.v_cache = kc.to(DEV), vc.to(DEV)
    lead = 2 if seed % 2 else 3                                              # gate columns on and off a pair boundary
    wide = torch.cat([torch.zeros(lay.n_tokens, lead, dtype=dtype), torch.cat(gates), torch.zeros(lay.n_tokens, lead % 2, dtype=dtype)], 1).to(DEV)
    set_context(False, step_layout=lay)
    try:
        out = attn(torch.cat(Q).to(DEV), wide[:, lead:lead + H * dv])
    finally:
        reset_context()
    return rel(out, torch.cat(want))


@BOTH
@pytest.mark.parametrize("H,G,d,dv", [(3, 3, 10, 6), (4, 2, 96, 64), (2, 1, 128, 128), (6, 2, 64, 64), (4, 4, 32, 48), (4, 1, 32, 32)])
def test_gated_window_attention_with_kept_first_keys(nat, dtype, H, G, d, dv):
    tol = TOL[dtype]
    W, F = 24, 5
    for window, keep in ((W, F), (W, 0), (1, 1), (0, 0), (500, 3)):
        assert attention_case(nat, H, G, d, dv, window, keep, [(0, 1), (0, 70), (3, 2), (64, 1), (40, 31), (129, 1), (0, 2)], dtype, seed=window) < tol
    mixed = [(310, 40), (349, 1), (0, 350), (348, 2)]
    i = 349                                                                  # the position of every last query
    for s in range(len(mixed)):
        # kept keys and the first one behind them, both sides of the window's edge and of page borders, far, itself
        for key in (0, F - 1, F, F + 1, i - W - 1, i - W, i - W + 1, 335, 336, 200, i - 1, i):
            assert attention_case(nat, H, G, d, dv, W, F, mixed, dtype, spike=(s, key), seed=key) < tol, (s, key)


# ------------------------------------------------------------------------------------------------ latent attention
def latent_case(H, R, window, seqs, dtype, spike=None, page=16, seed=0):
    """Attention over cached latents without a rotated part, queries given in the latent's coordinates."""
    from nano_qwen3tts_vllm_b200.layers.attention import LatentSinkAttention
    from nano_qwen3tts_vllm_b200.layers.rotary_embedding import PairRotary
    from nano_qwen3tts_vllm_b200.utils.context import reset_context, set_context
    g = torch.Generator().manual_seed(seed)
    scale = (6.0 if spike else 1.0) * R ** -0.5
    nb = [(p + n + page - 1) // page for p, n in seqs]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    cache = torch.full((len(perm), page, R), 7.0, dtype=dtype)
    lay_seqs, Q, want, o = [], [], [], 0
    for s, (p0, n) in enumerate(seqs):
        bt = perm[o:o + nb[s]]
        o += nb[s]
        T = p0 + n
        c, q = O.unit_rms(torch.randn(T, R, generator=g), 1e-6), O.unit_rms(torch.randn(T, H, R, generator=g), 1e-6)
        if spike and spike[0] == s:
            q[T - 1] = c[spike[1]]
        c, q = c.to(dtype), q.to(dtype)
        for p in range(T):
            cache[bt[p // page], p % page] = c[p]
        ref = O.softmax_attention(q.double(), c.double()[:, None], c.double()[:, None], scale, O.visible(T, window))
        lay_seqs.append((p0, n, bt)), Q.append(q[p0:]), want.append(ref[p0:])
    lay = Lay(lay_seqs, page, max(nb))
    attn = LatentSinkAttention(H, R, 0, window, scale, PairRotary(0, 1.0)).to(DEV)
    attn.sink = None
    ql = torch.cat(Q).transpose(0, 1).contiguous().to(DEV)
    qr = torch.empty(ql.shape[1], 0, dtype=dtype, device=DEV)
    set_context(False, step_layout=lay)
    try:
        out = attn(ql, qr, (0, 0), cache.to(DEV))
    finally:
        reset_context()
    return rel(out.transpose(0, 1), torch.cat(want))


@BOTH
@pytest.mark.parametrize("H,R", [(3, 12), (4, 64), (2, 96), (16, 128), (20, 256), (1, 512), (5, 40)])
def test_latent_attention_without_positions(nat, dtype, H, R):
    tol = TOL[dtype]
    W = 20
    for window in (W, 1, 0):
        assert latent_case(H, R, window, [(0, 1), (0, 70), (3, 2), (64, 1), (40, 31), (129, 1), (0, 2)], dtype, seed=window) < tol
        assert latent_case(H, R, window, [(200, 1), (40, 1), (0, 1)], dtype, seed=window) < tol            # a decode step
    mixed = [(310, 40), (349, 1), (0, 350), (348, 2)]
    for s in range(len(mixed)):
        for key in (0, 349 - W - 1, 349 - W, 349 - W + 1, 335, 336, 200, 349):
            assert latent_case(H, R, W, mixed, dtype, spike=(s, key), seed=key) < tol, (s, key)
    assert nat.latent_attn_timeouts() == 0


@BOTH
@pytest.mark.parametrize("n,H,dv", [(5, 3, 7), (64, 16, 64), (1, 1, 1)])
def test_one_gate_per_head(nat, dtype, n, H, dv):
    g = torch.Generator().manual_seed(n)
    v, gate = torch.randn(H, n, dv, generator=g).to(dtype), torch.randn(n, H + 2, generator=g).to(dtype)
    out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
    nat.gate_heads(v.to(DEV), (dv, n * dv), gate.to(DEV)[:, 2:], out, H, dv, per_head=True)
    want = v.double().transpose(0, 1) * torch.sigmoid(gate.double()[:, 2:])[:, :, None]
    assert rel(out, want.reshape(n, -1)) < TOL[dtype]


# ------------------------------------------------------------------------------------------------ the engine
def engine_for(cfg, sd, **kw):
    from nano_qwen3tts_vllm_b200.config import GekavikConfig
    return make_engine(GekavikConfig.from_dict(cfg), sd, **kw)


CONFIGS = {
    "loop_from_the_first_layer": dict(),
    "looped_middle": dict(loop=(1, 3, 3), types=("latent_attention", "attention", "latent_attention", "attention")),
    "loop_of_everything_once": dict(loop=(0, 3, 1), ff=("moe", None)),
    "loop_of_one_layer_at_the_end": dict(loop=(2, 3, 2), ff=(None, "moe", "moe")),
    "no_loop_no_feed_forward": dict(loop=None, ff=(None,)),
    "latent_only": dict(types=("latent_attention", "latent_attention"), loop=(0, 1, 2)),
    "attention_only": dict(types=("attention", "attention"), loop=(1, 2, 2), residual_mult=1.0),
    "all_ones": dict(attention=dict(heads=1, kv_heads=1, dim=4, vdim=4, scale=1.0, rot={"dims": 4, "base": 50.0}, mask={"size": 1, "keep_first": 1}),
                     latent=dict(heads=1, dim=4, vdim=4, kv_rank=4, q_rank=4, scale=1.0, mask={"size": 1}), residual_mult=1.0,
                     moe=dict(expert={"ff": 1, "limit": 1.0}, router={"experts": 1, "top": 1, "groups": {"count": 1, "keep": 1}},
                              shared={"ff": 1, "limit": 1.0}), loop=(0, 1, 1)),
    "no_kept_keys_no_rotation_no_shared": dict(attention=dict(mask={"size": 7}, rot=None), moe=dict(shared=None)),
    "every_key_seen": dict(attention=dict(mask=None), latent=dict(mask=None), moe=dict(router={"experts": 5, "top": 3})),
    "odd_sizes": dict(width=21, vocab=53, attention=dict(heads=3, kv_heads=3, dim=7, vdim=11, rot={"dims": 2, "base": 9.0}),
                      latent=dict(heads=5, dim=3, vdim=9, kv_rank=13, q_rank=5), moe=dict(expert={"ff": 3, "limit": 0.3}, shared={"ff": 5, "limit": 0.4}),
                      eps=1e-2),
    "two_rotations_many_groups": dict(types=("attention", "attention"), moe=dict(router={"experts": 20, "top": 5, "groups": {"count": 10, "keep": 3}})),
    "vector_width_shapes": dict(width=128, vocab=256, attention=dict(heads=6, kv_heads=2, dim=64, vdim=64, scale=0.2, rot={"dims": 32, "base": 1e4},
                                                                    mask={"size": 30, "keep_first": 3}),
                                latent=dict(heads=4, dim=32, vdim=32, kv_rank=64, q_rank=64, scale=0.2, mask={"size": 50}),
                                moe=dict(expert={"ff": 32, "limit": 1.2}, router={"experts": 12, "top": 4, "groups": {"count": 6, "keep": 3}},
                                         shared={"ff": 64, "limit": 0.9})),
    "wide_heads": dict(width=64, vocab=100, attention=dict(heads=2, kv_heads=2, dim=128, vdim=128, rot={"dims": 128, "base": 1e3}),
                       latent=dict(heads=18, dim=16, vdim=24, kv_rank=96, q_rank=40)),
}


def config_named(name):
    cfg = O.random_config(**CONFIGS[name])
    if name == "two_rotations_many_groups":
        cfg["layers"][1]["mixer"]["rot"] = {"dims": 10, "base": 40.0}
    return cfg


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_decode_and_portions_match_plain_model(name):
    cfg = config_named(name)
    sd = sharpened(cfg, O.random_weights(cfg, seed=len(name)))
    toks = tokens_for(cfg, 90, 1)
    ref = O.forward(cfg, sd, toks)
    eng = engine_for(cfg, sd, page=16, pages=20, max_len=96)
    try:
        whole = replay(eng, {"a": toks}, [[("a", 90)]])["a"]
        decode = replay(eng, {"b": toks}, [[("b", 5)]] + [[("b", 1)] for _ in range(85)])["b"]
        parts = replay(eng, {"c": toks}, [[("c", n)] for n in cuts_of(90)])["c"]
        pairs = replay(eng, {"d": toks}, [[("d", 2)] for _ in range(45)])["d"]
    finally:
        eng.exit()
    for got in (whole, decode, parts, pairs):
        assert nerr(got, ref) < 5e-5


@pytest.mark.parametrize("name", ["loop_from_the_first_layer", "looped_middle", "no_loop_no_feed_forward"])
def test_residual_stream_after_every_layer_run(name):
    cfg = config_named(name)
    sd = O.random_weights(cfg, seed=3)
    toks = tokens_for(cfg, 40, 2)
    trace = []
    O.forward(cfg, sd, toks, trace)
    eng = engine_for(cfg, sd, page=16, pages=8, max_len=64)
    try:
        plain = replay(eng, {"a": toks}, [[("a", 40)]])["a"]
        eng.model_runner.model.trace_layers = got = []
        traced = replay(eng, {"b": toks}, [[("b", 40)]])["b"]
    finally:
        eng.exit()
    assert len(got) == len(trace) == len(O.layer_runs(cfg))
    for i, (g, t) in enumerate(zip(got, trace)):
        assert rel(g, t) < 2e-5, i
    assert nerr(traced, plain) < 1e-6                      # looking at the stream does not change it


def test_every_pass_has_its_own_cache_and_vector():
    cfg = O.random_config(loop=(1, 3, 2))
    sd = O.random_weights(cfg, seed=4)
    toks = tokens_for(cfg, 30, 5)
    eng = engine_for(cfg, sd, page=16, pages=8, max_len=64)
    try:
        got = replay(eng, {"a": toks}, [[("a", 10)]] + [[("a", 1)] for _ in range(20)])["a"]
        r = eng.model_runner
        ptrs = [t.data_ptr() for run in range(5) for t in r.kv_cache[run]]
        assert len(r.kv_cache) == 5 and len(set(ptrs)) == len(ptrs) == 8
    finally:
        eng.exit()
    assert nerr(got, O.forward(cfg, sd, toks)) < 5e-5
    assert nerr(got, O.forward(cfg, {**sd, "loop.step": sd["loop.step"].flip(0)}, toks)) > 1e-2


def test_unequal_batch_matches_each_alone_and_reuses_pages_and_slots():
    """Five requests over four live slots and a pool smaller than their sum: portions of some beside single tokens of
    others; the fifth request takes over the pages and the slot of the first one that ends."""
    cfg = O.random_config()
    sd = sharpened(cfg, O.random_weights(cfg, seed=7))
    reqs = {i: tokens_for(cfg, n, 10 + k) for k, (i, n) in enumerate([("a", 70), ("b", 33), ("c", 100), ("d", 17), ("e", 64)])}
    refs = {i: O.forward(cfg, sd, t) for i, t in reqs.items()}
    sched = [[("a", 40), ("b", 2)], [("a", 1), ("b", 20), ("c", 64)], [("b", 1), ("c", 3), ("d", 17)], [("a", 29), ("b", 10), ("c", 1)],
             [("e", 5), ("c", 32)], [("e", 1)], [("e", 58)]]
    eng = engine_for(cfg, sd, pages=18, page=16, seqs=4, slots=4, max_len=128)
    try:
        got = replay(eng, reqs, sched)
        for i in reqs:
            assert nerr(got[i], refs[i]) < 5e-5, i
        alone = replay(eng, {"c2": reqs["c"]}, [[("c2", 100)]])["c2"]
        assert nerr(alone, got["c"]) < 2e-5
    finally:
        eng.exit()


def test_long_decode_over_pages_and_windows_graph_equals_eager():
    cfg = O.random_config(latent=dict(mask={"size": 37}))
    sd = sharpened(cfg, O.random_weights(cfg, seed=11))
    toks = tokens_for(cfg, 150, 2)
    ref = O.forward(cfg, sd, toks)
    sched = [[("a", 9)]] + [[("a", 1)] for _ in range(141)]
    outs = []
    for eager in (True, False):
        eng = engine_for(cfg, sd, page=16, pages=12, eager=eager, max_len=160)
        try:
            outs.append(replay(eng, {"a": toks}, sched)["a"])
        finally:
            eng.exit()
    assert nerr(outs[0], ref) < 5e-5 and nerr(outs[1], ref) < 5e-5
    assert nerr(outs[1], outs[0]) < 1e-6


@pytest.mark.parametrize("name", ["loop_from_the_first_layer", "vector_width_shapes", "wide_heads"])
def test_bfloat16_serving_precision_and_cut_independence(name):
    cfg = config_named(name)
    sd = O.random_weights(cfg, seed=13)
    toks = tokens_for(cfg, 150, 3)
    ref = O.forward(cfg, sd, toks)
    eng = engine_for(cfg, sd, dtype="bfloat16", page=16, pages=24, max_len=160)
    try:
        whole = replay(eng, {"a": toks}, [[("a", 150)]])["a"]
        parts = replay(eng, {"b": toks}, [[("b", n)] for n in cuts_of(150)])["b"]
        other = tokens_for(cfg, 120, 4)
        mixed = replay(eng, {"c": toks, "x": other}, [[("c", 30), ("x", 1)]] + [[("c", 1), ("x", 1)] for _ in range(119)] + [[("c", 1)]])["c"]
    finally:
        eng.exit()
    for got in (whole, parts, mixed):
        e = nerr_rows(got, ref[:got.shape[0]])
        assert e.median().item() < 0.03, name                # a token near a routing tie may choose another expert
        assert (e > 0.1).double().mean().item() < 0.05, name


def test_greedy_generation_through_the_scheduler():
    """``generate``: chunked prompts beside decoding sequences under a small token budget, greedy sampling by the
    package's sampler; the completions are the plain model's greedy continuations (ties aside: margins are checked)."""
    from nano_qwen3tts_vllm_b200.sampling_params import SamplingParams
    cfg = O.random_config()
    sd = O.random_weights(cfg, seed=17)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (5, 37, 18)]
    eng = engine_for(cfg, sd, page=16, pages=16, seqs=3, budget=64, max_len=64)
    try:
        outs = eng.generate(prompts, SamplingParams(temperature=1.0, max_tokens=12, ignore_eos=True, top_k=1))
    finally:
        eng.exit()
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o["token_ids"]:
            lg = O.forward(cfg, sd, seq)[-1]
            top = torch.topk(lg, 2).values
            if (top[0] - top[1]).item() > 1e-3:
                assert tok == int(lg.argmax()), (len(seq), tok)
            seq.append(tok)
        assert len(o["token_ids"]) == 12


def test_checkpoint_folder_through_the_registry(tmp_path):
    from safetensors.torch import save_file
    from nano_qwen3tts_vllm_b200.llm import LLM
    cfg = config_named("two_rotations_many_groups")
    sd = {k: v.to(torch.bfloat16) for k, v in O.random_weights(cfg, seed=19).items()}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(sd, str(tmp_path / "model.safetensors"))
    toks = tokens_for(cfg, 20, 1)
    eng = LLM(str(tmp_path), dtype="float32", kvcache_block_size=16, num_kvcache_blocks=4, max_num_seqs=2, max_model_len=64,
              max_num_batched_tokens=128, enforce_eager=True, device=DEV)
    try:
        got = replay(eng, {"a": toks}, [[("a", 20)]])["a"]
    finally:
        eng.exit()
    assert nerr(got, O.forward(cfg, {k: v.double() for k, v in sd.items()}, toks)) < 5e-5
