"""Plain, slow restatement of the Zekivik decoder (test infrastructure only: nothing in the package imports it).

One function per mechanism, whole sequences at a time, no cache, no carried state and no batching: attention looks at
the full prefix, the convolution at the whole projected sequence, and the retention walks the sequence from a zero
state, so the engine's paged K/V, state slots, portions and mixed batches have something independent to be compared with.
Arithmetic is done in the dtype of the tensors handed in (float64 in the tests).

Notation: x [T, D] the residual stream, H query heads over G key/value heads, d / dv the key and value size per head.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def unit_rms(v, eps):
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def rotate_halves(v, positions, dims, base):
    """v [T, heads, d]: coordinates i and i + dims/2 (i < dims/2) of every head are turned by the angle
    position * base^(-2i/dims); coordinates from ``dims`` on pass."""
    half = dims // 2
    if half == 0:
        return v
    i = torch.arange(half, dtype=v.dtype)
    ang = positions.to(v.dtype)[:, None] * (torch.tensor(float(base), dtype=v.dtype) ** (-2.0 * i / dims))
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., dims:]], -1)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + w[:, j] * pad[j:j + T]
    return y


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ mixers
def retention(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H]: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    a = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    o = []
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        o.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(o)


def retention_mixer(h, w, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w["q"].T).view(T, H, d)
    k = (h @ w["k"].T).view(T, H, d)
    v = (h @ w["v"].T).view(T, H, dv)
    r = m["rot"]
    q, k = rotate_halves(q, pos, r["dims"], r["base"]), rotate_halves(k, pos, r["dims"], r["base"]) * d ** -0.5
    o = unit_rms(retention(q, k, v, m["decay"]), eps).reshape(T, H * dv)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def softmax_attention(q, k, v, scale):
    """Causal; q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~mask, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def attention_mixer(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = causal_conv(h @ w["q"].T, w["q.conv"]).view(T, H, d)
    k = causal_conv(h @ w["k"].T, w["k.conv"]).view(T, G, d)
    v = causal_conv(h @ w["v"].T, w["v.conv"]).view(T, G, dv)
    r = m["rot"]
    q = unit_rms(rotate_halves(q, pos, r["dims"], r["base"]), eps)
    k = unit_rms(rotate_halves(k, pos, r["dims"], r["base"]), eps)
    o = softmax_attention(q, k, unit_rms(v, eps), m["scale"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------------------------ the rest of a layer
def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def gated(y, h, w, b):
    """A sublayer's result y times sigmoid(W h + b), h being the sublayer's input."""
    return y * torch.sigmoid(h @ w.T + b)


def sub(sd, prefix):
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


def layer_runs(cfg):
    """[(layer, pass that starts right before it or None)] in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b, times = lp["start"], lp["stop"], lp["times"]
    runs = [(i, None) for i in range(a)]
    for t in range(times):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg: dict, sd: dict, tokens, trace=None):
    """tokens: a list of ids -> logits [T, vocab].  ``sd``: checkpoint names -> tensors (already in the working dtype).
    ``trace``: a list that receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = sd["embed"][torch.tensor(tokens)]
    x = x0
    for i, t in layer_runs(cfg):
        layer, w = cfg["layers"][i], sub(sd, f"l{i}.")
        if t is not None:
            x = (x + x0 if t > 0 else x) + sd["loop.step"][t]
        h = offset_norm(x, w["norm1"], eps)
        mix = {"attention": attention_mixer, "retention": retention_mixer}[layer["type"]]
        x = x + gated(mix(h, sub(w, "mix."), layer["mixer"], eps), h, w["rg1"], w["rg1.b"])
        if layer.get("mlp") is not None:
            h = offset_norm(x, w["norm2"], eps)
            x = x + gated(dense_ff(h, sub(w, "mlp.")), h, w["rg2"], w["rg2.b"])
        if trace is not None:
            trace.append(x.clone())
    return offset_norm(x, sd["final.norm"], eps) @ sd["head"].T


# ------------------------------------------------------------------------------------------------ small random models
def random_config(vocab=59, width=20, types=("retention", "attention", "retention", "attention"), ff=(None, 28), eps=1e-5,
                  loop=(1, 3, 2), attention=None, retention=None) -> dict:
    """A small configuration in the checkpoint's format.  ``types``: the mixers in order; ``ff``: inner sizes of the
    feed-forwards, taken in turn (None: none); ``loop``: (start, stop, times) or None; the dicts override fields of
    every mixer of that kind."""
    att = dict(heads=4, kv_heads=2, dim=10, vdim=6, conv=3, scale=0.4, rot={"dims": 6, "base": 300.0})
    att.update(attention or {})
    ret = dict(heads=3, dim=8, vdim=5, decay=[0.6, 0.9, 0.995], rot={"dims": 4, "base": 120.0})
    ret.update(retention or {})
    layers = []
    for i, kind in enumerate(types):
        f = ff[i % len(ff)]
        layers.append({"type": kind, "mixer": dict(att if kind == "attention" else ret),
                       "mlp": None if f is None else {"kind": "dense", "ff": f}})
    out = {"architecture": "Zekivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def tensor_shapes(cfg: dict) -> dict:
    D = cfg["width"]
    sh = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    if cfg.get("loop"):
        sh["loop.step"] = (cfg["loop"]["times"], D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        sh[p + "norm1"], sh[p + "rg1"], sh[p + "rg1.b"] = (D,), (D, D), (D,)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        sh[p + "mix.q"], sh[p + "mix.k"], sh[p + "mix.v"], sh[p + "mix.o"] = (H * d, D), (G * d, D), (G * dv, D), (D, H * dv)
        if layer["type"] == "attention":
            sh[p + "mix.q.conv"], sh[p + "mix.k.conv"], sh[p + "mix.v.conv"] = (H * d, m["conv"]), (G * d, m["conv"]), (G * dv, m["conv"])
            sh[p + "mix.g"] = (H, D)
        else:
            sh[p + "mix.g"] = (H * dv, D)
        if layer.get("mlp") is not None:
            f = layer["mlp"]["ff"]
            sh[p + "norm2"], sh[p + "rg2"], sh[p + "rg2.b"] = (D,), (D, D), (D,)
            sh[p + "mlp.gate"], sh[p + "mlp.up"], sh[p + "mlp.down"] = (f, D), (f, D), (D, f)
    return sh


def random_weights(cfg: dict, seed: int = 0) -> dict:
    """Random tensors under the checkpoint's names, rounded to bfloat16 (what a file would hold), returned as float64."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        t = torch.randn(shape, generator=g)
        if name.endswith(".conv"):
            t = 0.5 * t
        elif name in ("embed", "loop.step"):
            t = 0.7 * t
        elif len(shape) == 2:
            t = t * shape[1] ** -0.5
        else:
            t = 0.3 * t                                          # norm weights (around zero), gate biases
        sd[name] = t.to(torch.bfloat16).double()
    return sd
