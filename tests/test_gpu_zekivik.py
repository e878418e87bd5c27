"""Zekivik on the GPU against the plain float64 restatement in ``oracle/zekivik.py`` (no code shared with the package).

Kernel level: every new or extended mechanism alone, with inputs built so that a fault shows (one key that takes the whole
softmax far back, at a page border, at the sequence's first token; a retained token hundreds of steps back that one query
asks for; convolution taps and recurrent state carried over portions of 1, 2, 3 tokens through slots another sequence used;
portions around the edges of a chunk; decays of zero and one).
Engine level, through ``CausalLMEngine`` and its scheduler: whole prompts, token-by-token decoding, portions, mixed
batches, reuse of pages and state slots, long decoding across pages, looped layers, odd sizes, greedy generation, CUDA
graphs against eager.  The float32 engine is the sharp comparison; bfloat16 is checked against its rounding noise."""
import json

import pytest
import torch

from oracle import zekivik as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def nat():
    import nano_qwen3tts_vllm_b200._native as n
    n.lib()
    return n


class Lay:
    """A hand-made step layout for kernel tests: sequences [(pos0, n_new, slot, block_table)]."""

    def __init__(self, seqs, page=16, max_blocks=1):
        tok_seq, pos, slots, start = [], [], [], []
        o = 0
        for b, (p0, n, _, bt) in enumerate(seqs):
            start.append(o)
            for t in range(n):
                p = p0 + t
                tok_seq.append(b), pos.append(p), slots.append(bt[p // page] * page + p % page if bt else 0)
            o += n
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        self.tok_seq, self.positions, self.slot_mapping = i32(tok_seq), i32(pos), i32(slots)
        self.seq_start, self.seq_pos0 = i32(start), i32([s[0] for s in seqs])
        self.seq_len, self.seq_slot = i32([s[1] for s in seqs]), i32([s[2] for s in seqs])
        bt = torch.zeros(len(seqs), max_blocks, dtype=torch.int32)
        for b, s in enumerate(seqs):
            bt[b, :len(s[3])] = torch.tensor(s[3], dtype=torch.int32)
        self.block_tables = bt.to(DEV)
        self.n_tokens, self.n_seqs, self.max_new = o, len(seqs), max(s[1] for s in seqs)


def rel(a, b):
    return ((a.double().cpu() - b.double().cpu()).abs().max() / b.double().abs().max().clamp_min(1e-30)).item()


TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def freq_of(dims, base):
    from nano_qwen3tts_vllm_b200.layers.rotary_embedding import HalfRotary
    return HalfRotary(dims, base).freq.to(DEV)


# ------------------------------------------------------------------------------------------------ per-row kernels
@BOTH
@pytest.mark.parametrize("cols", [21, 260, 2048, 4104])
def test_gated_residual_with_what_a_pass_adds_and_the_next_norm(nat, dtype, cols):
    g = torch.Generator().manual_seed(cols)
    n, eps, tol = 7, 1e-3, TOL[dtype]
    d = lambda t: t.to(DEV)
    x0 = torch.randn(n, cols, generator=g)
    y = torch.randn(n, cols, generator=g).to(dtype)
    wide = (torch.randn(n, cols + 9, generator=g) * 2).to(dtype)             # the gate is a column slice of a merged projection
    zb, add, w = torch.randn(cols, generator=g), torch.randn(cols, generator=g), torch.rand(cols, generator=g) + 0.5
    table = torch.randn(11, cols, generator=g).to(dtype)
    ids = torch.randint(0, 11, (n,), generator=g)
    want0 = x0.double() + y.double() * torch.sigmoid(wide.double()[:, 4:4 + cols] + zb.double())
    norm = lambda v: O.unit_rms(v, eps) * w.double()
    for extra in ({}, {"add": add}, {"table": table, "index": ids.int()}, {"add": add, "table": table, "index": ids.int()}):
        want = want0 + (table.double()[ids] if "table" in extra else 0) + (add.double() if "add" in extra else 0)
        kw = {k: d(v) for k, v in extra.items()}
        x = d(x0.clone())
        h = nat.gated_residual(x, y=d(y), z=d(wide)[:, 4:4 + cols], zb=d(zb), w=d(w), eps=eps, **kw)
        assert h.dtype == dtype and rel(x, want) < 1e-5 and rel(h, norm(want)) < tol
        x = d(x0.clone())
        assert nat.gated_residual(x, y=d(y), z=d(wide)[:, 4:4 + cols], zb=d(zb), **kw) is None and rel(x, want) < 1e-5
    # no gate; only the additions; the embedding into a dirty stream
    x = d(x0.clone())
    nat.gated_residual(x, y=d(y))
    assert rel(x, x0.double() + y.double()) < 1e-5
    x = d(x0.clone())
    h = nat.gated_residual(x, add=d(add), w=d(w), eps=eps, dtype=dtype)
    assert rel(x, x0.double() + add.double()) < 1e-6 and rel(h, norm(x0.double() + add.double())) < tol
    x = d(torch.full((n, cols), 1e9))
    h = nat.gated_residual(x, table=d(table), index=d(ids.int()), add=d(add), init=True, w=d(w), eps=eps)
    want = table.double()[ids] + add.double()
    assert rel(x, want) < 1e-6 and rel(h, norm(want)) < tol


@BOTH
@pytest.mark.parametrize("rows,ff,width", [(3, 64, 128), (70, 192, 64), (300, 320, 192), (5, 27, 20), (700, 64, 64)])
def test_gelu_gated_product_in_the_gemm_and_beside_it(nat, dtype, rows, ff, width):
    from nano_qwen3tts_vllm_b200.layers.linear import linear_gelu_mul
    g = torch.Generator().manual_seed(ff)
    h = torch.randn(rows, width, generator=g).to(dtype)
    w = (torch.randn(2 * ff, width, generator=g) * 2 * width ** -0.5).to(dtype)
    gu = h.double() @ w.double().T
    want = O.gelu_tanh(gu[:, :ff]) * gu[:, ff:]
    prev = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        assert rel(linear_gelu_mul(h.to(DEV), w.to(DEV)), want) < TOL[dtype]
    finally:
        torch.backends.cuda.matmul.allow_tf32 = prev
    assert rel(nat.gelu_mul(gu.to(dtype).to(DEV)), O.gelu_tanh(gu.to(dtype).double()[:, :ff]) * gu.to(dtype).double()[:, ff:]) < TOL[dtype]


def test_rotation_table_at_near_and_far_positions(nat):
    from nano_qwen3tts_vllm_b200.layers.rotary_embedding import HalfRotaryTable
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4095, 20000], dtype=torch.int32)
    for dims, base in ((2, 10.0), (24, 1e4), (128, 5e5)):
        r = HalfRotaryTable(dims, base).to(DEV)
        r.fill(pos.to(DEV))
        ang = pos.double()[:, None] * r.freq.double().cpu()
        assert r.table.shape == (8, dims)
        # the angle is a float: half a unit in its last place is what a correct table may be off by
        bound = 4e-7 + ang.abs() * 2.0 ** -24
        assert ((r.table[:, :dims // 2].double().cpu() - torch.cos(ang)).abs() <= bound).all()
        assert ((r.table[:, dims // 2:].double().cpu() - torch.sin(ang)).abs() <= bound).all()


# ------------------------------------------------------------------------------------------------ convolution, rotation, norms
@BOTH
@pytest.mark.parametrize("H,G,d,dv,taps,rot", [(3, 1, 7, 5, 3, 4), (4, 2, 16, 12, 4, 16), (2, 2, 64, 128, 4, 32), (2, 1, 160, 200, 2, 24),
                                               (1, 1, 24, 24, 1, 0), (2, 1, 12, 8, 5, 8), (2, 2, 10, 6, 11, 2), (6, 2, 128, 64, 3, 120)])
def test_convolved_rotated_unit_normed_heads_in_portions_through_reused_slots(nat, dtype, H, G, d, dv, taps, rot):
    """Three sequences advance side by side and alone in portions down to one token; slots and pages hold another owner's
    values at the start; a portion can be shorter than the convolution."""
    g = torch.Generator().manual_seed(d * taps)
    page, base, eps, T = 16, 90.0, 1e-3, [41, 22, 3]
    C = H * d + G * (d + dv)
    w = torch.randn(C, taps, generator=g) * 0.6
    us = [torch.randn(n, C, generator=g).to(dtype) for n in T]
    want = []
    for n, u in zip(T, us):
        y, pos = O.causal_conv(u.double(), w.double()), torch.arange(n)
        q, k, v = y[:, :H * d].view(n, H, d), y[:, H * d:(H + G) * d].view(n, G, d), y[:, (H + G) * d:].view(n, G, dv)
        if rot:
            q, k = O.rotate_halves(q, pos, rot, base), O.rotate_halves(k, pos, rot, base)
        want.append([O.unit_rms(t, eps).reshape(n, -1) for t in (q, k, v)])
    R = max(taps - 1, 1)
    state = torch.full((4, R, C), 3.0, dtype=dtype, device=DEV)
    kc = torch.full((9, page, G * d), 5.0, dtype=dtype, device=DEV)
    vc = torch.full((9, page, G * dv), 5.0, dtype=dtype, device=DEV)
    tables = [[4, 0, 7], [2, 8], [5]]
    freq = freq_of(rot, base) if rot else None
    got_q, at = [[], [], []], [0, 0, 0]
    for cuts in [(1, 2, 0), (2, 1, 1), (1, 0, 2), (17, 2, 0), (1, 1, 0), (19, 16, 0)]:
        live = [s for s, n in enumerate(cuts) if n]
        lay = Lay([(at[s], cuts[s], 3 - s, tables[s]) for s in live], page, 3)
        u = torch.cat([us[s][at[s]:at[s] + cuts[s]] for s in live])
        u = torch.cat([u, torch.full((u.shape[0], 8), 9.0, dtype=dtype)], 1).to(DEV)          # more columns behind q | k | v
        q = torch.empty(lay.n_tokens, H * d, dtype=dtype, device=DEV)
        nat.conv_headnorm_kvwrite(u, w.to(DEV), state if taps > 1 else None, lay, None, None, q, kc, vc, H, G, d, dv, taps, eps,
                                  rot=nat.rotary_table(lay.positions, freq) if rot else None, flags=nat.CONV_UNIT_V)
        o = 0
        for s in live:
            got_q[s].append(q[o:o + cuts[s]].cpu())
            o += cuts[s]
            at[s] += cuts[s]
    assert at == T
    for s, n in enumerate(T):
        rows = torch.tensor([tables[s][p // page] * page + p % page for p in range(n)], device=DEV)
        assert rel(torch.cat(got_q[s]), want[s][0]) < TOL[dtype], s
        assert rel(kc.view(-1, G * d)[rows], want[s][1]) < TOL[dtype] and rel(vc.view(-1, G * dv)[rows], want[s][2]) < TOL[dtype], s
        if taps > 1:
            last = torch.cat([torch.zeros(R, C, dtype=dtype), us[s]])[-R:]
            if n >= R:
                assert torch.equal(state[3 - s].cpu(), last)


# ------------------------------------------------------------------------------------------------ attention
def attention_case(nat, H, G, d, dv, seqs, dtype, spike=None, page=16, seed=0):
    """Unit-normed keys and values in shuffled pages; ``spike`` (sequence, key position): the last query of that sequence
    and that key point the same way, so the key takes the softmax."""
    from nano_qwen3tts_vllm_b200.layers.attention import SinkSoftmaxAttention
    from nano_qwen3tts_vllm_b200.utils.context import reset_context, set_context
    g = torch.Generator().manual_seed(seed)
    scale, eps = (4.0 if spike else 1.0) * d ** -0.5, 1e-5
    nb = [(p + n + page - 1) // page for p, n in seqs]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    kc = torch.full((len(perm), page, G * d), 7.0, dtype=dtype)
    vc = torch.full((len(perm), page, G * dv), 7.0, dtype=dtype)
    lay_seqs, Q, want, gates, o = [], [], [], [], 0
    for s, (p0, n) in enumerate(seqs):
        bt = perm[o:o + nb[s]]
        o += nb[s]
        T = p0 + n
        unit = lambda *shape: O.unit_rms(torch.randn(*shape, generator=g), eps)
        q, k, v = unit(T, H, d), unit(T, G, d), unit(T, G, dv)
        if spike and spike[0] == s:
            for h in range(H):
                q[T - 1, h] = k[spike[1], h // (H // G)]
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        gate = torch.randn(T, H, generator=g).to(dtype)
        for p in range(T):
            kc[bt[p // page], p % page], vc[bt[p // page], p % page] = k[p].reshape(-1), v[p].reshape(-1)
        ref = O.softmax_attention(q.double(), k.double(), v.double(), scale) * torch.sigmoid(gate.double())[:, :, None]
        if spike and spike[0] == s:                                          # the case shows what it is meant to show
            row = (q.double()[T - 1, 0] @ k.double()[:, 0].T * scale).softmax(-1)
            assert row[spike[1]] > 0.5
        lay_seqs.append((p0, n, s, bt)), Q.append(q[p0:].reshape(n, -1)), want.append(ref[p0:].reshape(n, -1)), gates.append(gate[p0:])
    lay = Lay(lay_seqs, page, max(nb))
    attn = SinkSoftmaxAttention(H, G, d, dv, "window", 0, scale, sink="none", eps=eps).to(DEV)
    attn.k_cache, attn.v_cache = kc.to(DEV), vc.to(DEV)
    wide = torch.cat([torch.zeros(lay.n_tokens, 3, dtype=dtype), torch.cat(gates)], 1).to(DEV)
    set_context(False, step_layout=lay)
    try:
        out = attn(torch.cat(Q).to(DEV), wide[:, 3:])
    finally:
        reset_context()
    return rel(out, torch.cat(want))


@BOTH
@pytest.mark.parametrize("H,G,d,dv", [(3, 3, 10, 6), (4, 2, 96, 64), (2, 1, 128, 128), (6, 2, 64, 64), (4, 4, 32, 48), (4, 1, 48, 128)])
def test_causal_attention_far_keys_page_borders_first_tokens(nat, dtype, H, G, d, dv):
    tol = TOL[dtype]
    assert attention_case(nat, H, G, d, dv, [(0, 1), (0, 70), (3, 2), (64, 1), (40, 31), (129, 1), (0, 2)], dtype) < tol
    mixed = [(310, 40), (349, 1), (0, 350), (348, 2)]
    for s, (p0, n) in enumerate(mixed):
        for key in (0, 1, 15, 16, 31, 32, 200, 348, 349):                    # first tokens, both sides of page borders, far, itself
            assert attention_case(nat, H, G, d, dv, mixed, dtype, spike=(s, key), seed=key) < tol, (s, key)


# ------------------------------------------------------------------------------------------------ retention
def retention_reference(q, k, v, gate, m, rot, base, eps):
    """Whole sequence: rotated, scaled, from a zero state -> normed and gated rows, and the final state."""
    n, (H, d, dv) = q.shape[0], m
    pos = torch.arange(n)
    q, k, v = q.double().view(n, H, d), k.double().view(n, H, d), v.double().view(n, H, dv)
    if rot:
        q, k = O.rotate_halves(q, pos, rot, base), O.rotate_halves(k, pos, rot, base)
    return q, k * d ** -0.5, v, O.silu(gate.double())


def run_retention(nat, dtype, H, d, dv, rot, decay, seqs_T, schedule, path=0, spike=None, seed=0):
    """Returns (worst relative error of the outputs, worst of the final states).  ``schedule``: new tokens per sequence and
    step.  ``spike`` (sequence, early token, late token): the late query asks for what the early key wrote."""
    g = torch.Generator().manual_seed(seed)
    eps, base = 1e-4, 70.0
    ins, refs, finals = [], [], []
    for s, n in enumerate(seqs_T):
        q, k = (torch.randn(n, H * d, generator=g) for _ in range(2))
        v, gate = torch.randn(n, H * dv, generator=g), torch.randn(n, H * dv, generator=g)
        if spike and spike[0] == s:
            early, late = spike[1:]
            k[early] *= 30.0
            q[late] = k[early]
            if rot:                                                          # undo the rotation between the two positions
                r = O.rotate_halves(k[early].double().view(1, H, d), torch.tensor([float(early - late)]), rot, base)
                q[late] = r.reshape(-1).float()
        q, k, v, gate = (t.to(dtype) for t in (q, k, v, gate))
        qr, kr, vr, gr = retention_reference(q, k, v, gate, (H, d, dv), rot, base, eps)
        o = O.unit_rms(O.retention(qr, kr, vr, decay), eps).reshape(n, -1) * gr
        if spike and spike[0] == s:                                          # without the early token the row is another one
            k0 = kr.clone()
            k0[spike[1]] = 0
            other = O.unit_rms(O.retention(qr, k0, vr, decay), eps).reshape(n, -1) * gr
            assert rel(other[late], o[late]) > 0.2
        S = torch.zeros(H, d, dv, dtype=F64)
        for t in range(n):
            S = torch.tensor(decay, dtype=F64)[:, None, None] * S + kr[t][:, :, None] * vr[t][:, None, :]
        ins.append((q, k, v, gate)), refs.append(o), finals.append(S)
    state = torch.full((len(seqs_T) + 1, H, d, dv), 7.0, device=DEV)         # dirty slots
    freq = freq_of(rot, base) if rot else None
    dec = torch.tensor(decay, dtype=torch.float32, device=DEV)
    got, at = [[] for _ in seqs_T], [0] * len(seqs_T)
    for cuts in schedule:
        live = [s for s, n in enumerate(cuts) if n]
        lay = Lay([(at[s], cuts[s], len(seqs_T) - s, []) for s in live])
        u = torch.cat([torch.cat([t[at[s]:at[s] + cuts[s]] for t in ins[s]], 1) for s in live]).to(DEV)      # [q | k | v | gate]
        out = torch.empty(lay.n_tokens, H * dv, dtype=dtype, device=DEV)
        c = [0, H * d, 2 * H * d, 2 * H * d + H * dv, u.shape[1]]
        q, k, v, gate = (u[:, c[i]:c[i + 1]] for i in range(4))
        nat.retention(q, k, v, nat.rotary_table(lay.positions, freq) if rot else None, dec, d ** -0.5, state, gate, out, lay, H, d, dv, eps, path)
        o = 0
        for s in live:
            got[s].append(out[o:o + cuts[s]].cpu())
            o += cuts[s]
            at[s] += cuts[s]
    assert at == list(seqs_T)
    return (max(rel(torch.cat(a), b) for a, b in zip(got, refs)),
            max(rel(state[len(seqs_T) - s], f) for s, f in enumerate(finals)))


SHAPES = [(2, 5, 7, 4), (3, 32, 32, 32), (2, 64, 64, 16), (1, 128, 128, 128), (2, 96, 32, 48), (1, 130, 16, 130), (2, 32, 96, 0),
          (2, 64, 100, 24), (1, 32, 64, 12)]


@BOTH
@pytest.mark.parametrize("H,d,dv,rot", SHAPES)
def test_retention_in_portions_through_reused_slots(nat, dtype, H, d, dv, rot):
    """Portions of 1, 2, 3, ... tokens and around a chunk's edge, side by side and alone, in every kernel the shape has; the
    state is as exact in bfloat16 as in float32: only its inputs are rounded."""
    decay = [0.9, 0.999, 0.5][:H]
    schedule = [(1, 2, 0), (2, 1, 0), (3, 0, 2), (1, 1, 1), (63, 17, 0), (64, 2, 0), (65, 1, 0), (1, 0, 0), (2, 66, 0)]
    T = [sum(c[s] for c in schedule) for s in range(3)]
    paths = [nat.RETENTION_AUTO, nat.RETENTION_SCAN]
    for path in paths:
        eo, es = run_retention(nat, dtype, H, d, dv, rot, decay, T, schedule, path=path, seed=d)
        assert eo < (5e-5 if dtype == torch.float32 else 8e-3) and es < 5e-5, (path, eo, es)


@pytest.mark.parametrize("n", [2, 3, 15, 16, 17, 63, 64, 65, 127, 128, 129, 200])
@pytest.mark.parametrize("H,d,dv,rot", [(2, 32, 64, 32), (1, 128, 32, 64), (1, 96, 128, 96), (2, 64, 64, 0)])
def test_retention_chunks_of_every_length_on_the_tensor_cores(nat, n, H, d, dv, rot):
    eo, es = run_retention(nat, torch.bfloat16, H, d, dv, rot, [0.97, 0.9995][:H], [n, 1, n + 5], [(n, 1, 5), (0, 0, n)],
                           path=nat.RETENTION_AUTO, seed=n)
    assert eo < 8e-3 and es < 5e-5
    eo, es = run_retention(nat, torch.bfloat16, H, d, dv, rot, [0.97, 0.9995][:H], [n], [(n,)], path=nat.RETENTION_TENSOR, seed=n)
    assert eo < 8e-3 and es < 5e-5


@BOTH
@pytest.mark.parametrize("H,d,dv,rot", [(2, 6, 8, 4), (2, 64, 64, 64), (1, 128, 128, 32)])
def test_retention_of_a_far_token_and_extreme_decays(nat, dtype, H, d, dv, rot):
    tol = 1e-4 if dtype == torch.float32 else 1e-2
    for late, sched in ((299, [(300,)]), (299, [(299,), (1,)]), (299, [(150,), (148,), (2,)]), (64, [(300,)]), (63, [(60,), (240,)])):
        for early in (0, 1, 63 if late > 63 else 40, late - 1):
            eo, _ = run_retention(nat, dtype, H, d, dv, rot, [0.9995] * H, [300], sched, spike=(0, early, late), seed=late)
            assert eo < tol, (late, early)
    for dec in (0.0, 1.0):                                                   # nothing is kept; nothing is lost
        eo, es = run_retention(nat, dtype, H, d, dv, rot, [dec] * H, [150], [(100,), (1,), (49,)], seed=3)
        assert eo < tol and es < 5e-5, dec


# ------------------------------------------------------------------------------------------------ the engine
def make_engine(cfg: dict, sd: dict, dtype="float32", pages=12, page=64, seqs=4, slots=None, eager=True, budget=None, max_len=256):
    from nano_qwen3tts_vllm_b200.config import ZekivikConfig
    from nano_qwen3tts_vllm_b200.engine.llm_engine.lm_engine import CausalLMEngine
    c = ZekivikConfig.from_dict(cfg)
    return CausalLMEngine(c, state_dict={k: v.to(torch.bfloat16) for k, v in sd.items()}, dtype=dtype, kvcache_block_size=page,
                          num_kvcache_blocks=pages, max_num_seqs=seqs, max_state_slots=slots or seqs, max_model_len=max_len,
                          max_num_batched_tokens=budget or seqs * max_len, enforce_eager=eager, device=DEV)


def replay(engine, requests: dict, schedule: list):
    """Feed ``schedule`` = [[(id, count), ...], ...] through engine.step as held sequences; logits of every position."""
    at = {i: 0 for i in requests}
    live, got = set(), {i: [] for i in requests}
    for step in schedule:
        want = {}
        for i, n in step:
            toks = requests[i][at[i]:at[i] + n]
            if i in live:
                engine.feed(i, toks)
            else:
                engine.add_request(toks, request_id=i, hold=True)
                live.add(i)
            want[i] = list(range(n))
            at[i] += n
        out = engine.step(want=want)
        assert out.scheduled == {i: n for i, n in step}
        o = 0
        for i, n in step:
            got[i].append(out.logits[o:o + n].double().cpu())
            o += n
        for i, _ in step:
            if at[i] == len(requests[i]):
                engine.clear_request(i)
                live.discard(i)
    return {i: torch.cat(v) for i, v in got.items() if v}


def nerr_rows(got, ref):
    """Per-position error: rms over the vocabulary of the mean-free difference, relative to the rms of the logits."""
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()


def nerr(got, ref):
    return nerr_rows(got, ref).max().item()


def tokens_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def cuts_of(T, sizes=(2, 3, 1, 17, 2, 1, 1, 30, 2)):
    cuts, left = [], T
    for n in sizes:
        n = min(n, left)
        if n:
            cuts.append(n)
            left -= n
    return cuts + [1] * left


CONFIGS = {
    "looped_middle": dict(),
    "loop_from_the_first_layer": dict(loop=(0, 2, 3), types=("attention", "retention", "retention")),
    "loop_of_everything_once": dict(loop=(0, 3, 1), types=("retention", "attention", "attention"), ff=(16, None)),
    "loop_of_one_layer_at_the_end": dict(loop=(2, 3, 2), types=("attention", "retention", "attention"), ff=(None, 16, 24)),
    "no_loop_attention_only": dict(loop=None, types=("attention", "attention"), ff=(None,)),
    "retention_only": dict(types=("retention", "retention", "retention"), ff=(12, None, 20), loop=(1, 2, 2)),
    "all_ones": dict(attention=dict(heads=1, kv_heads=1, dim=4, vdim=4, conv=1, scale=1.0, rot={"dims": 4, "base": 50.0}),
                     retention=dict(heads=1, dim=4, vdim=4, decay=[0.95], rot={"dims": 4, "base": 50.0}), loop=(1, 2, 1)),
    "two_rotations_long_filter": dict(attention=dict(heads=6, kv_heads=3, dim=12, vdim=8, conv=7, rot={"dims": 12, "base": 40.0}),
                                      retention=dict(heads=2, dim=10, vdim=12, decay=[1.0, 0.2], rot={"dims": 2, "base": 9.0}), eps=1e-2),
    "vector_width_shapes": dict(width=128, vocab=128, ff=(256, None), loop=(1, 3, 2),
                                attention=dict(heads=4, kv_heads=2, dim=64, vdim=64, conv=4, scale=0.2, rot={"dims": 32, "base": 1e4}),
                                retention=dict(heads=2, dim=64, vdim=32, decay=[0.98, 0.999], rot={"dims": 64, "base": 1e4})),
    "equal_heads_wide_values": dict(width=64, vocab=100, ff=(64,), attention=dict(heads=2, kv_heads=2, dim=32, vdim=128, conv=2,
                                                                                  rot={"dims": 32, "base": 1e3}),
                                    retention=dict(heads=3, dim=32, vdim=96, decay=[0.9, 0.99, 0.9999], rot={"dims": 16, "base": 1e3})),
}


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_decode_and_portions_match_plain_model(name):
    cfg = O.random_config(**CONFIGS[name])
    sd = O.random_weights(cfg, seed=len(name))
    toks = tokens_for(cfg, 90, 1)
    ref = O.forward(cfg, sd, toks)
    eng = make_engine(cfg, sd, page=16, pages=20, max_len=96)
    try:
        whole = replay(eng, {"a": toks}, [[("a", 90)]])["a"]
        decode = replay(eng, {"b": toks}, [[("b", 5)]] + [[("b", 1)] for _ in range(85)])["b"]
        parts = replay(eng, {"c": toks}, [[("c", n)] for n in cuts_of(90)])["c"]
        pairs = replay(eng, {"d": toks}, [[("d", 2)] for _ in range(45)])["d"]
    finally:
        eng.exit()
    for got in (whole, decode, parts, pairs):
        assert nerr(got, ref) < 5e-5


@pytest.mark.parametrize("name", ["looped_middle", "loop_from_the_first_layer", "no_loop_attention_only"])
def test_residual_stream_after_every_layer_run(name):
    cfg = O.random_config(**CONFIGS[name])
    sd = O.random_weights(cfg, seed=3)
    toks = tokens_for(cfg, 40, 2)
    trace = []
    O.forward(cfg, sd, toks, trace)
    eng = make_engine(cfg, sd, page=16, pages=8, max_len=64)
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


def test_every_pass_has_its_own_cache_state_and_vector():
    """The passes' tensors are separate, and the passes are told apart: exchanging the passes' vectors changes the logits."""
    cfg = O.random_config(loop=(1, 3, 2))
    sd = O.random_weights(cfg, seed=4)
    toks = tokens_for(cfg, 30, 5)
    eng = make_engine(cfg, sd, page=16, pages=8, max_len=64)
    try:
        got = replay(eng, {"a": toks}, [[("a", 10)]] + [[("a", 1)] for _ in range(20)])["a"]
        r = eng.model_runner
        ptrs = [t.data_ptr() for run in range(6) for t in r.kv_cache[run] + r.seq_state[run]]
        assert len(r.kv_cache) == 6 and len(set(ptrs)) == len(ptrs)
    finally:
        eng.exit()
    assert nerr(got, O.forward(cfg, sd, toks)) < 5e-5
    assert nerr(got, O.forward(cfg, {**sd, "loop.step": sd["loop.step"].flip(0)}, toks)) > 1e-2


def test_unequal_batch_matches_each_alone_and_reuses_pages_and_slots():
    """Five requests over four live slots and a pool smaller than their sum: portions of some beside single tokens of
    others; the fifth request takes over the pages and the slot of the first one that ends."""
    cfg = O.random_config()
    sd = O.random_weights(cfg, seed=7)
    reqs = {i: tokens_for(cfg, n, 10 + k) for k, (i, n) in enumerate([("a", 70), ("b", 33), ("c", 100), ("d", 17), ("e", 64)])}
    refs = {i: O.forward(cfg, sd, t) for i, t in reqs.items()}
    sched = [[("a", 40), ("b", 2)], [("a", 1), ("b", 20), ("c", 64)], [("b", 1), ("c", 3), ("d", 17)], [("a", 29), ("b", 10), ("c", 1)],
             [("e", 5), ("c", 32)], [("e", 1)], [("e", 58)]]
    eng = make_engine(cfg, sd, pages=18, page=16, seqs=4, slots=4, max_len=128)
    try:
        got = replay(eng, reqs, sched)
        for i in reqs:
            assert nerr(got[i], refs[i]) < 5e-5, i
        alone = replay(eng, {"c2": reqs["c"]}, [[("c2", 100)]])["c2"]
        assert nerr(alone, got["c"]) < 2e-5
    finally:
        eng.exit()


def test_long_decode_over_pages_graph_equals_eager():
    cfg = O.random_config(retention=dict(decay=[0.99, 0.9995, 0.9]))
    sd = O.random_weights(cfg, seed=11)
    toks = tokens_for(cfg, 150, 2)
    ref = O.forward(cfg, sd, toks)
    sched = [[("a", 9)]] + [[("a", 1)] for _ in range(141)]
    outs = []
    for eager in (True, False):
        eng = make_engine(cfg, sd, page=16, pages=12, eager=eager, max_len=160)
        try:
            outs.append(replay(eng, {"a": toks}, sched)["a"])
        finally:
            eng.exit()
    assert nerr(outs[0], ref) < 5e-5
    assert nerr(outs[1], ref) < 5e-5
    assert nerr(outs[1], outs[0]) < 1e-6


@pytest.mark.parametrize("name", ["looped_middle", "vector_width_shapes", "equal_heads_wide_values"])
def test_bfloat16_serving_precision_and_cut_independence(name):
    cfg = O.random_config(**CONFIGS[name])
    sd = O.random_weights(cfg, seed=13)
    toks = tokens_for(cfg, 150, 3)
    ref = O.forward(cfg, sd, toks)
    eng = make_engine(cfg, sd, dtype="bfloat16", page=16, pages=24, max_len=160)
    try:
        whole = replay(eng, {"a": toks}, [[("a", 150)]])["a"]
        parts = replay(eng, {"b": toks}, [[("b", n)] for n in cuts_of(150)])["b"]
        other = tokens_for(cfg, 120, 4)
        mixed = replay(eng, {"c": toks, "x": other}, [[("c", 30), ("x", 1)]] + [[("c", 1), ("x", 1)] for _ in range(119)] + [[("c", 1)]])["c"]
    finally:
        eng.exit()
    for got in (whole, parts, mixed):
        e = nerr_rows(got, ref[:got.shape[0]])
        assert e.median().item() < 0.02 and e.max().item() < 0.08
    assert nerr(parts, whole) < 0.08 and nerr(mixed, whole[:mixed.shape[0]]) < 0.08


def test_greedy_generation_through_the_scheduler():
    """``generate``: chunked prompts beside decoding sequences under a small token budget, greedy sampling by the
    package's sampler; the completions are the plain model's greedy continuations (ties aside: margins are checked)."""
    from nano_qwen3tts_vllm_b200.sampling_params import SamplingParams
    cfg = O.random_config()
    sd = O.random_weights(cfg, seed=17)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (5, 37, 18)]
    eng = make_engine(cfg, sd, page=16, pages=16, seqs=3, budget=64, max_len=64)
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
    cfg = O.random_config(**CONFIGS["two_rotations_long_filter"])
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
