"""Gekavik: a decoder-only token model over one 32-bit residual stream whose sublayers are normed on the way in and on the
way out by dynamic tanh, D(v) = tanh(alpha v) * w + b, some of its layers looped.

    x = x0 = embed[token]
    layer:  x <- x + m D_1b(mixer(D_1(x)));   x <- x + m D_2b(ff(D_2(x)))                     (the second line optional)
    mixers: "attention"         biased rotary attention: every q and k head RMS-normed in front of the pair rotation, sliding
                                window with kept first keys, an element-wise sigmoid gate on the output
            "latent_attention"  queries through a normed latent, keys and values expanded from one normed latent per token, no
                                positions, sliding window, a sigmoid gate per head
    ff:     a softmax-routed, group-limited mixture of clamped gated experts beside a shared one, or absent
    loop:   a range of layers runs several times in a row with the same weights; in front of pass t
            x <- W [x; x0] + step[t]
    logits = head D_f(x)

Every layer carries its own sizes (``config.GekavikLayerSpec``); every layer RUN has a cache of its own.  One forward runs a
whole engine step: prompt portions and single decoded tokens side by side, described by the step layout in the global Context.
Launches per attention layer run: ONE input GEMM for q, k, v and the gate, preparation (biases, head norms, rotation, cache
write), attention (its gate inside), output GEMM, ONE elementwise launch for norm, residual update and the next norm; then
routing and grouping, the experts' gate / up product with its activation, their down product, the shared expert's two GEMMs
(activation in the first) and the same residual launch, which takes the weighted sum over experts.  In front of a pass the
residual launch writes the operand of the pass's projection instead of a norm.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _native as nat
from ..config import GekavikConfig, GekavikLayerSpec, SinkAttentionSpec
from ..layers.attention import SinkSoftmaxAttention
from ..layers.layernorm import DynamicTanh, TanhSandwich
from ..layers.linear import MergedColumnParallelLinear, RowParallelLinear, linear_float
from ..layers.moe import SharedClampedMoE
from ..layers.pass_input import PassInput
from ..layers.rotary_embedding import PairRotaryTable
from .checkpoint import load_targets
from .teberax import LatentMixer

GEMM_ROWS = 128          # the native GEMM's output tile: merged input projections are padded to whole tiles


class GatedAttentionMixer(nn.Module):
    """q | k | v | gate behind one merged projection; attention over the paged cache with its gate inside; output projection."""

    PARTS = ("q", "k", "v", "g")

    def __init__(self, width: int, spec: SinkAttentionSpec, eps: float, rotary: PairRotaryTable | None):
        super().__init__()
        m = self.spec = spec
        sizes = [m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim, m.heads * m.vdim]
        self.in_proj = MergedColumnParallelLinear(width, sizes, pad_to=GEMM_ROWS)
        self.offs = [sum(sizes[:i]) for i in range(5)]
        self.attn = SinkSoftmaxAttention(m.heads, m.kv_heads, m.dim, m.vdim, m.mask_kind, m.mask_size, m.scale, bias=m.bias, rotary=rotary,
                                         eps=eps, sink=m.sink, keep_first=m.keep_first, head_norm=m.head_norm, element_gate=m.element_gate)
        self.o_proj = RowParallelLinear(m.heads * m.vdim, width)

    def cache_plan(self):
        m = self.spec
        return {"paged": [m.kv_heads * m.dim, m.kv_heads * m.vdim], "state": []}

    def bind(self, paged, state):
        self.attn.k_cache, self.attn.v_cache = paged

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        u, (q, k, v, g, end) = self.in_proj(h), self.offs
        return self.o_proj(self.attn(self.attn.prepare(u, q, k, v), u[:, g:end]))


class GekavikLayer(nn.Module):
    def __init__(self, width: int, spec: GekavikLayerSpec, eps: float, mult: float, rotary: PairRotaryTable | None):
        super().__init__()
        self.norm1 = TanhSandwich(width, mult)
        self.mix = GatedAttentionMixer(width, spec.mixer, eps, rotary) if spec.type == "attention" else LatentMixer(width, spec.mixer, eps)
        self.mlp = self.norm2 = None
        if (f := spec.mlp) is not None:
            self.norm2 = TanhSandwich(width, mult)
            self.mlp = SharedClampedMoE(width, f.ff, f.experts, f.top, f.limit, f.groups, f.groups_keep,
                                        *((f.shared.ff, f.shared.limit) if f.shared is not None else ()))

    def forward(self, x: torch.Tensor, h: torch.Tensor, nxt: DynamicTanh | None, cat_with: tuple | None = None):
        """x [n, width] float, updated in place; h = norm1.pre(x).  Returns what comes next (see ``TanhSandwich.add``)."""
        if self.mlp is None:
            return self.norm1.add(x, nxt, a=self.mix(h), cat_with=cat_with)
        h = self.norm1.add(x, self.norm2.pre, a=self.mix(h))
        z, zw, shared = self.mlp(h)
        return self.norm2.add(x, nxt, a=shared, z=z, zw=zw, cat_with=cat_with)


class GekavikForCausalLM(nn.Module):
    def __init__(self, config: GekavikConfig):
        super().__init__()
        self.config = c = config
        self.embed = nn.Parameter(torch.empty(c.vocab, c.width), requires_grad=False)
        self.head = nn.Parameter(torch.empty(c.vocab, c.width), requires_grad=False)
        self.pass_in = PassInput(c.width, c.loop["times"]) if c.loop else None
        rotaries: dict = {}                    # layers with the same frequencies share the step's table
        for spec in c.layers:
            r = spec.mixer.rot if spec.type == "attention" else None
            if r is not None and (r.dims, r.base) not in rotaries:
                rotaries[r.dims, r.base] = PairRotaryTable(r.dims, r.base)
        self.rotaries = nn.ModuleList(rotaries.values())
        pick = lambda spec: rotaries[spec.mixer.rot.dims, spec.mixer.rot.base] if spec.type == "attention" and spec.mixer.rot is not None else None
        self.layers = nn.ModuleList([GekavikLayer(c.width, spec, c.norm_eps, c.residual_mult, pick(spec)) for spec in c.layers])
        self.final_norm = DynamicTanh(c.width)
        self.runs = c.runs()
        self.caches: list = [None] * len(self.runs)          # per layer RUN: (paged tensors, state tensors)
        self.trace_layers = None               # a list: forward() appends a copy of the residual stream after every layer run

    @property
    def dtype(self) -> torch.dtype:
        return self.head.dtype

    def forward(self, tokens: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """One engine step over the packed tokens of the batch -> the residual stream [n, width] (float)."""
        for r in self.rotaries:
            r.fill(positions)
        runs, rows = self.runs, (self.embed, tokens)
        norm_of = lambda run: self.layers[runs[run][0]].norm1.pre if run < len(runs) else None
        opens = lambda run: run < len(runs) and runs[run][1] is not None         # a pass starts right in front of the run
        x = torch.empty(tokens.shape[0], self.config.width, dtype=torch.float32, device=tokens.device)
        first = norm_of(0)
        h = nat.tanh_residual(x, table=self.embed, index=tokens, init=True, want_cat=opens(0),
                              pre=first.args() if first is not None and not opens(0) else None)
        for run, (li, t) in enumerate(runs):
            layer = self.layers[li]
            if t is not None:                  # h is the operand of the pass's projection
                self.pass_in(x, h, t)
                h = nat.tanh_residual(x, pre=layer.norm1.pre.args(), dtype=self.dtype)
            layer.mix.bind(*self.caches[run])
            ahead = opens(run + 1)
            h = layer(x, h, None if ahead else norm_of(run + 1), cat_with=rows if ahead else None)
            if self.trace_layers is not None:
                self.trace_layers.append(x.clone())
        return x

    def compute_logits(self, x: torch.Tensor, rows: torch.Tensor | None) -> torch.Tensor:
        return linear_float(self.final_norm(x, self.dtype, rows), self.head)

    # ------------------------------------------------------------------ cache and state
    def cache_plan(self) -> list[dict]:
        """Per layer run: widths of its paged tensors; no layer carries state."""
        return [self.layers[li].mix.cache_plan() for li, _ in self.runs]

    def bind_cache(self, run: int, paged: list, state: list):
        self.caches[run] = (paged, state)

    # ------------------------------------------------------------------ weights
    def _targets(self) -> dict:
        """Checkpoint name -> (parameter, shard of a merged weight or None, transform of the stored tensor or None)."""
        t = {"embed": (self.embed, None, None), "head": (self.head, None, None)}

        def norm(name, module):
            t[name], t[name + ".b"], t[name + ".alpha"] = (module.weight, None, None), (module.bias, None, None), (module.alpha, None, None)

        norm("final.norm", self.final_norm)
        if self.pass_in is not None:
            t["loop.in"], t["loop.step"] = (self.pass_in.weight, None, self.pass_in.expand), (self.pass_in.step, None, None)
        for i, (layer, spec) in enumerate(zip(self.layers, self.config.layers)):
            p, mix = f"l{i}.", layer.mix
            M = p + "mix."
            norm(p + "norm1", layer.norm1.pre), norm(p + "norm1b", layer.norm1.post)
            if spec.type == "attention":
                a = mix.attn
                for shard, name in enumerate(mix.PARTS):
                    t[M + name] = (mix.in_proj.weight, shard, None)
                t[M + "q.b"], t[M + "k.b"], t[M + "v.b"] = (a.q_bias, None, None), (a.k_bias, None, None), (a.v_bias, None, None)
                t[M + "q.norm"], t[M + "k.norm"] = (a.q_norm, None, None), (a.k_norm, None, None)
                t[M + "o"] = (mix.o_proj.weight, None, None)
            else:
                c = mix.core
                t[M + "dq"], t[M + "dkv"], t[M + "g"] = ((c.in_proj.weight, shard, None) for shard in range(3))
                t[M + "dq.norm"], t[M + "dkv.norm"], t[M + "uq"] = (c.q_norm, None, None), (c.kv_norm, None, None), (c.uq.weight, None, None)
                t[M + "uk"], t[M + "uv"], t[M + "o"] = (c.uk, None, None), (c.uv, None, None), (c.o_proj.weight, None, None)
            if (e := layer.mlp) is None:
                continue
            norm(p + "norm2", layer.norm2.pre), norm(p + "norm2b", layer.norm2.post)
            F = p + "mlp."
            t[F + "router"] = (e.router, None, None)
            for j in range(e.experts):
                t[f"{F}e{j}.gate"], t[f"{F}e{j}.up"] = (e.up[j, :e.ff], None, None), (e.up[j, e.ff:], None, None)
                t[f"{F}e{j}.down"] = (e.down[j], None, None)
            if e.shared is not None:
                t[F + "shared.gate"], t[F + "shared.up"] = (e.shared.gate_up.weight, 0, None), (e.shared.gate_up.weight, 1, None)
                t[F + "shared.down"] = (e.shared.down.weight, None, None)
        return t

    def checkpoint_names(self) -> list[str]:
        return sorted(self._targets())

    def load_state_dict(self, state_dict, strict=True):
        """Checkpoint names: ``embed``, ``head``, ``loop.in``, ``loop.step``, norms (``final.norm``, ``l<i>.norm1|norm1b|norm2|norm2b``)
        with ``.b`` and ``.alpha``, the mixer's tensors under ``l<i>.mix.`` and the feed-forward's under ``l<i>.mlp.`` (experts
        ``.e<j>.``, the shared one ``.shared.``)."""
        return load_targets(self._targets(), state_dict, strict)


def checkpoint_shapes(config: GekavikConfig) -> dict:
    """Checkpoint name -> shape, from the configuration alone."""
    D = config.width
    sh = {"embed": (config.vocab, D), "head": (config.vocab, D)}

    def norm(name):
        sh[name], sh[name + ".b"], sh[name + ".alpha"] = (D,), (D,), ()

    norm("final.norm")
    if config.loop:
        sh["loop.in"], sh["loop.step"] = (D, 2 * D), (config.loop["times"], D)
    for i, spec in enumerate(config.layers):
        p, m = f"l{i}.", spec.mixer
        M = p + "mix."
        norm(p + "norm1"), norm(p + "norm1b")
        if spec.type == "attention":
            for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                sh[M + n], sh[M + n + ".b"] = (rows, D), (rows,)
            sh[M + "q.norm"] = sh[M + "k.norm"] = (m.dim,)
            sh[M + "g"] = (m.heads * m.vdim, D)
        else:
            sh[M + "dq"], sh[M + "dq.norm"], sh[M + "uq"] = (m.q_rank, D), (m.q_rank,), (m.heads * m.dim, m.q_rank)
            sh[M + "dkv"], sh[M + "dkv.norm"] = (m.kv_rank, D), (m.kv_rank,)
            sh[M + "uk"], sh[M + "uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
            sh[M + "g"] = (m.heads, D)
        sh[M + "o"] = (D, m.heads * m.vdim)
        f = spec.mlp
        if f is None:
            continue
        norm(p + "norm2"), norm(p + "norm2b")
        F = p + "mlp."
        sh[F + "router"] = (f.experts, D)
        for n, ff in [(f"e{j}", f.ff) for j in range(f.experts)] + ([("shared", f.shared.ff)] if f.shared is not None else []):
            sh[f"{F}{n}.gate"], sh[f"{F}{n}.up"], sh[f"{F}{n}.down"] = (ff, D), (ff, D), (D, ff)
    return sh


def random_state_dict(config: GekavikConfig, seed: int = 0) -> dict:
    """Random bfloat16 tensors under the checkpoint's names (benchmarks, tests and smoke runs; no trained weights exist)."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in sorted(checkpoint_shapes(config).items()):
        leaf = name.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=g)
        if leaf == "alpha":
            t = 0.8 + 0.1 * t
        elif leaf in ("b", "step"):
            t = 0.2 * t
        elif len(shape) == 1:
            t = 1.0 + 0.1 * t                                     # norm weights
        elif leaf != "embed":
            t = t * shape[1] ** -0.5
        sd[name] = t.to(torch.bfloat16)
    return sd
