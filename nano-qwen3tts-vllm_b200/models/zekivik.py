"""Zekivik: a decoder-only token model over one 32-bit residual stream with gated sublayers, some of its layers looped.

    x = x0 = embed[token]
    layer:  x <- x + sigmoid(W_1 h + b_1) * mixer(h),  h = n_1(x);   x <- x + sigmoid(W_2 h + b_2) * ff(h),  h = n_2(x)
            (the second line optional);  n(v) = v / sqrt(mean(v^2) + eps) * (1 + w)
    mixers: "attention"   causal softmax attention: short convolutions on q, k and v, half-split rotation of q and k, then q, k
                          and v heads divided by their root mean square; one sigmoid gate per head on the output
            "retention"   linear attention with a fixed decay per head over rotated q and k; unit-normed read-outs, SiLU gate
    ff:     W_down (gelu_tanh(W_gate h) * W_up h), or absent
    loop:   a range of layers runs several times in a row with the same weights; in front of pass t the stream gets
            step[t], and x0 before that when t > 0
    logits = head n_f(x)

Every layer carries its own sizes (``config.ZekivikLayerSpec``); every layer RUN has a cache or state of its own.  One
forward runs a whole engine step: prompt portions and single decoded tokens side by side, described by the step layout in
the global Context.  Launches per layer run: ONE input GEMM for the mixer's projections and its residual gate, convolution +
rotation + norms + cache write, attention (its head gate inside) - or the recurrence (rotation inside; in a step of single
tokens also norm and gate) -, output GEMM, ONE launch for the gated residual update, what a pass adds and the next norm; then the
feed-forward's merged GEMM with its activation, the gate's GEMM, the down GEMM and the same residual launch.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _native as nat
from ..config import RetentionSpec, SinkAttentionSpec, ZekivikConfig, ZekivikLayerSpec
from ..layers.attention import SinkSoftmaxAttention
from ..layers.layernorm import GatedResidual, OffsetRMSNorm
from ..layers.linear import ColumnParallelLinear, MergedColumnParallelLinear, RowParallelLinear, linear, linear_gelu_mul
from ..layers.recurrent import Retention
from ..layers.rotary_embedding import HalfRotaryTable
from ..layers.short_conv import ShortConvRotaryQKV
from .checkpoint import load_targets

GEMM_ROWS = 128          # the native GEMM's output tile: merged input projections are padded to whole tiles


class _MergedInput(nn.Module):
    """The mixer's projections and the residual gate's ("rg", width columns) behind one weight."""

    def __init__(self, width: int, parts: list):
        super().__init__()
        self.width = width
        # a number per head ("g" of the attention) goes last: everything in front of it starts on vector boundaries
        self.parts = parts[:-1] + [("rg", width), parts[-1]]
        self.in_proj = MergedColumnParallelLinear(width, [w for _, w in self.parts], pad_to=GEMM_ROWS)
        self.cols, off = {}, 0
        for name, w in self.parts:
            self.cols[name] = off
            off += w

    def shard(self, name: str) -> int:
        return [n for n, _ in self.parts].index(name)

    def residual_gate(self, u: torch.Tensor) -> torch.Tensor:
        return u[:, self.cols["rg"]:self.cols["rg"] + self.width]


class ConvAttentionMixer(_MergedInput):
    def __init__(self, width: int, spec: SinkAttentionSpec, eps: float, rotary: HalfRotaryTable | None):
        m = spec
        super().__init__(width, [("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim), ("g", m.heads)])
        self.spec = m
        self.conv = ShortConvRotaryQKV(m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, rotary)
        self.attn = SinkSoftmaxAttention(m.heads, m.kv_heads, m.dim, m.vdim, m.mask_kind, m.mask_size, m.scale, sink=m.sink, eps=eps)
        self.o_proj = RowParallelLinear(m.heads * m.vdim, width)

    def cache_plan(self):
        m = self.spec
        return {"paged": [m.kv_heads * m.dim, m.kv_heads * m.vdim], "state": [self.conv.state_plan()]}

    def bind(self, paged, state):
        self.attn.k_cache, self.attn.v_cache = paged
        (self.conv.state,) = state

    def forward(self, h: torch.Tensor):
        u = self.in_proj(h)
        q = self.conv(u, self.attn.k_cache, self.attn.v_cache)
        g = self.cols["g"]
        return self.o_proj(self.attn(q, u[:, g:g + self.spec.heads])), self.residual_gate(u)


class RetentionMixer(_MergedInput):
    def __init__(self, width: int, spec: RetentionSpec, eps: float, rotary: HalfRotaryTable | None):
        core = Retention(spec, eps, rotary)
        super().__init__(width, core.proj_parts())
        self.spec, self.core = spec, core
        self.o_proj = RowParallelLinear(spec.heads * spec.vdim, width)

    def cache_plan(self):
        return {"paged": [], "state": self.core.state_plan()}

    def bind(self, paged, state):
        self.core.bind(state)

    def forward(self, h: torch.Tensor):
        u = self.in_proj(h)
        return self.o_proj(self.core(u, self.cols)), self.residual_gate(u)


class GatedGeluFF(nn.Module):
    """W_down (gelu_tanh(W_gate h) * W_up h) over a merged [gate; up] weight, beside the residual gate's projection."""

    def __init__(self, width: int, ff: int):
        super().__init__()
        self.gate_up = MergedColumnParallelLinear(width, [ff, ff])
        self.rg = ColumnParallelLinear(width, width)
        self.down = RowParallelLinear(ff, width)

    def forward(self, h: torch.Tensor):
        return self.down(linear_gelu_mul(h, self.gate_up.weight)), self.rg(h)


class ZekivikLayer(nn.Module):
    def __init__(self, width: int, spec: ZekivikLayerSpec, eps: float, rotary: HalfRotaryTable | None):
        super().__init__()
        self.norm1, self.res1 = OffsetRMSNorm(width, eps), GatedResidual(width)
        mixer = ConvAttentionMixer if spec.type == "attention" else RetentionMixer
        self.mix = mixer(width, spec.mixer, eps, rotary)
        self.mlp = self.norm2 = self.res2 = None
        if spec.mlp is not None:
            self.norm2, self.res2, self.mlp = OffsetRMSNorm(width, eps), GatedResidual(width), GatedGeluFF(width, spec.mlp.ff)

    def forward(self, x: torch.Tensor, h: torch.Tensor, nxt: OffsetRMSNorm | None, **ahead):
        """x [n, width] float, updated in place; h = norm1(x).  ``ahead``: what the stream gets behind this layer (see
        ``GatedResidual``).  Returns ``nxt(x)`` (None without ``nxt``)."""
        y, z = self.mix(h)
        if self.mlp is None:
            return self.res1(x, y, z, nxt, **ahead)
        h = self.res1(x, y, z, self.norm2)
        y, z = self.mlp(h)
        return self.res2(x, y, z, nxt, **ahead)


class ZekivikForCausalLM(nn.Module):
    def __init__(self, config: ZekivikConfig):
        super().__init__()
        self.config = c = config
        self.embed = nn.Parameter(torch.empty(c.vocab, c.width), requires_grad=False)
        self.head = nn.Parameter(torch.empty(c.vocab, c.width), requires_grad=False)
        self.step = nn.Parameter(torch.zeros(c.loop["times"], c.width, dtype=torch.float32), requires_grad=False) if c.loop else None
        rotaries: dict = {}                    # layers with the same frequencies share the step's table
        for spec in c.layers:
            r = spec.mixer.rot
            if r is not None and (r.dims, r.base) not in rotaries:
                rotaries[r.dims, r.base] = HalfRotaryTable(r.dims, r.base)
        self.rotaries = nn.ModuleList(rotaries.values())
        pick = lambda r: rotaries[r.dims, r.base] if r is not None else None
        self.layers = nn.ModuleList([ZekivikLayer(c.width, spec, c.norm_eps, pick(spec.mixer.rot)) for spec in c.layers])
        self.final_norm = OffsetRMSNorm(c.width, c.norm_eps)
        self.runs = c.runs()
        self.caches: list = [None] * len(self.runs)          # per layer RUN: (paged tensors, state tensors)
        self.trace_layers = None               # a list: forward() appends a copy of the residual stream after every layer run

    @property
    def dtype(self) -> torch.dtype:
        return self.head.dtype

    def _ahead(self, run: int, tokens: torch.Tensor) -> dict:
        """What joins the stream right in front of layer run ``run``."""
        t = self.runs[run][1] if run < len(self.runs) else None
        if t is None:
            return {}
        return {"add": self.step[t], **({"table": self.embed, "index": tokens} if t > 0 else {})}

    def forward(self, tokens: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """One engine step over the packed tokens of the batch -> the residual stream [n, width] (float)."""
        for r in self.rotaries:
            r.fill(positions)
        eps = self.config.norm_eps
        norm_of = lambda run: self.layers[self.runs[run][0]].norm1 if run < len(self.runs) else None
        x = torch.empty(tokens.shape[0], self.config.width, dtype=torch.float32, device=tokens.device)
        first = norm_of(0)
        h = nat.gated_residual(x, table=self.embed, index=tokens, init=True, add=self._ahead(0, tokens).get("add"),
                               w=first.weight if first is not None else None, eps=eps)
        for run, (li, _) in enumerate(self.runs):
            layer, nxt = self.layers[li], norm_of(run + 1)
            layer.mix.bind(*self.caches[run])
            if self.trace_layers is None:
                h = layer(x, h, nxt, **self._ahead(run + 1, tokens))
            else:                              # the stream is looked at between the layer and what a pass adds
                layer(x, h, None)
                self.trace_layers.append(x.clone())
                if nxt is not None:
                    h = nat.gated_residual(x, w=nxt.weight, eps=eps, dtype=self.dtype, **self._ahead(run + 1, tokens))
        return x

    def compute_logits(self, x: torch.Tensor, rows: torch.Tensor | None) -> torch.Tensor:
        return linear(self.final_norm(x, self.dtype, rows), self.head).float()

    # ------------------------------------------------------------------ cache and state
    def cache_plan(self) -> list[dict]:
        """Per layer run: widths of its paged tensors and shapes (after the slot axis) / dtypes of its state tensors."""
        return [self.layers[li].mix.cache_plan() for li, _ in self.runs]

    def bind_cache(self, run: int, paged: list, state: list):
        self.caches[run] = (paged, state)

    # ------------------------------------------------------------------ weights
    def _targets(self) -> dict:
        """Checkpoint name -> (parameter, shard of a merged weight or None, transform of the stored tensor or None)."""
        one_plus = OffsetRMSNorm.from_stored
        t = {"embed": (self.embed, None, None), "head": (self.head, None, None), "final.norm": (self.final_norm.weight, None, one_plus)}
        if self.step is not None:
            t["loop.step"] = (self.step, None, None)
        for i, (layer, spec) in enumerate(zip(self.layers, self.config.layers)):
            p, mix, m = f"l{i}.", layer.mix, spec.mixer
            t[p + "norm1"] = (layer.norm1.weight, None, one_plus)
            t[p + "rg1"], t[p + "rg1.b"] = (mix.in_proj.weight, mix.shard("rg"), None), (layer.res1.bias, None, None)
            for name, _ in mix.parts:
                if name != "rg":
                    t[f"{p}mix.{name}"] = (mix.in_proj.weight, mix.shard(name), None)
            t[p + "mix.o"] = (mix.o_proj.weight, None, None)
            if spec.type == "attention":
                off = 0
                for name, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                    t[f"{p}mix.{name}.conv"] = (mix.conv.weight[off:off + rows], None, None)
                    off += rows
            if layer.mlp is not None:
                f = layer.mlp
                t[p + "norm2"] = (layer.norm2.weight, None, one_plus)
                t[p + "rg2"], t[p + "rg2.b"] = (f.rg.weight, None, None), (layer.res2.bias, None, None)
                t[p + "mlp.gate"], t[p + "mlp.up"] = (f.gate_up.weight, 0, None), (f.gate_up.weight, 1, None)
                t[p + "mlp.down"] = (f.down.weight, None, None)
        return t

    def checkpoint_names(self) -> list[str]:
        return sorted(self._targets())

    def load_state_dict(self, state_dict, strict=True):
        """Checkpoint names: ``embed``, ``head``, ``final.norm``, ``loop.step``, per layer ``l<i>.norm1|norm2``,
        ``l<i>.rg1|rg2`` with ``.b``, the mixer's tensors under ``l<i>.mix.`` and the feed-forward's under ``l<i>.mlp.``.
        Tensors are bfloat16 in the file; what the kernels keep in float (norm weights plus one, gate biases, filters, the
        passes' vectors) is widened exactly."""
        return load_targets(self._targets(), state_dict, strict)


def checkpoint_shapes(config: ZekivikConfig) -> dict:
    """Checkpoint name -> shape, from the configuration alone."""
    D = config.width
    sh = {"embed": (config.vocab, D), "head": (config.vocab, D), "final.norm": (D,)}
    if config.loop:
        sh["loop.step"] = (config.loop["times"], D)
    for i, spec in enumerate(config.layers):
        p, m = f"l{i}.", spec.mixer
        attention = spec.type == "attention"
        G = m.kv_heads if attention else m.heads
        sh[p + "norm1"], sh[p + "rg1"], sh[p + "rg1.b"] = (D,), (D, D), (D,)
        for name, rows in (("q", m.heads * m.dim), ("k", G * m.dim), ("v", G * m.vdim)):
            sh[f"{p}mix.{name}"] = (rows, D)
            if attention:
                sh[f"{p}mix.{name}.conv"] = (rows, m.conv)
        sh[p + "mix.g"] = (m.heads if attention else m.heads * m.vdim, D)
        sh[p + "mix.o"] = (D, m.heads * m.vdim)
        if spec.mlp is not None:
            f = spec.mlp.ff
            sh[p + "norm2"], sh[p + "rg2"], sh[p + "rg2.b"] = (D,), (D, D), (D,)
            sh[p + "mlp.gate"], sh[p + "mlp.up"], sh[p + "mlp.down"] = (f, D), (f, D), (D, f)
    return sh


def random_state_dict(config: ZekivikConfig, seed: int = 0) -> dict:
    """Random bfloat16 tensors under the checkpoint's names (benchmarks, tests and smoke runs; no trained weights exist)."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in sorted(checkpoint_shapes(config).items()):
        t = torch.randn(shape, generator=g)
        if name.endswith(".conv"):
            t = 0.5 * t
        elif len(shape) == 1:
            t = 0.1 * t                                           # norm weights (around zero), gate biases
        elif name not in ("embed", "loop.step"):
            t = t * shape[1] ** -0.5
        sd[name] = t.to(torch.bfloat16)
    return sd
