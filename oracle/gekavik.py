"""Plain, slow restatement of the Gekavik decoder (test infrastructure only: nothing in the package imports it).

One function per mechanism, whole sequences at a time, no cache, no carried state and no batching: every token looks at
the full prefix under its mask and walks its experts one by one, so the engine's paged keys, values and latents, its
portions and its mixed batches have something independent to be compared with.  Arithmetic is done in the dtype of the
tensors handed in (float64 in the tests).

Notation: x [T, D] the residual stream, H query heads over G key/value heads, d / dv the key and value size per head,
W a window length, F kept first tokens.
"""
from __future__ import annotations

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def unit_rms(v, eps, weight=None):
    """v / sqrt(mean(v^2) + eps) over the last axis, times a weight vector."""
    y = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def dyt(x, w, name):
    """Dynamic tanh: tanh(alpha x) w + b with the tensors ``name``, ``name.b`` and ``name.alpha`` of ``w``."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rotate_pairs(v, positions, dims, base):
    """v [T, heads, d]: coordinates 2i and 2i+1 (i < dims/2) of every head are turned by the angle
    position * base^(-2i/dims); coordinates from ``dims`` on pass."""
    if not dims:
        return v
    i = torch.arange(dims // 2, dtype=v.dtype)
    ang = positions.to(v.dtype)[:, None] * (torch.tensor(float(base), dtype=v.dtype) ** (-2.0 * i / dims))
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    return torch.cat([torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2), v[..., dims:]], -1)


def visible(T, window=None, keep_first=0):
    """[T, T] bool: i sees j when j <= i and (no window, or i - j < window, or j < keep_first)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    if window:
        ok = ok & ((i - j < window) | (j < keep_first))
    return ok


def softmax_attention(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~mask, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


# ------------------------------------------------------------------------------------------------ mixers
def attention_mixer(h, w, m, eps):
    """Biased projections, per-head RMS norm of q and k with one weight for all heads, then the rotation; window with kept
    first tokens; the concatenated heads times sigmoid(W_g h), element by element."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = unit_rms((h @ w["q"].T + w["q.b"]).view(T, H, d), eps, w["q.norm"])
    k = unit_rms((h @ w["k"].T + w["k.b"]).view(T, G, d), eps, w["k.norm"])
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    r = m.get("rot")
    if r:
        q, k = rotate_pairs(q, pos, r["dims"], r["base"]), rotate_pairs(k, pos, r["dims"], r["base"])
    mc = m.get("mask") or {}
    o = softmax_attention(q, k, v, m["scale"], visible(T, mc.get("size"), mc.get("keep_first", 0)))
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def latent_attention_mixer(h, w, m, eps):
    """Queries expanded from a normed query latent, keys and values from one normed latent per token; no positions; each
    head's output times its own sigmoid(W_g h)."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (unit_rms(h @ w["dq"].T, eps, w["dq.norm"]) @ w["uq"].T).view(T, H, d)
    c = unit_rms(h @ w["dkv"].T, eps, w["dkv.norm"])
    k = (c @ w["uk"].T).view(T, H, d)
    v = (c @ w["uv"].T).view(T, H, dv)
    mc = m.get("mask") or {}
    o = softmax_attention(q, k, v, m["scale"], visible(T, mc.get("size")))
    return (o * torch.sigmoid(h @ w["g"].T)[:, :, None]).reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_expert(h, w, name, limit):
    """g = min(gate, limit), u = clamp(up, -limit, limit), W_down (g sigmoid(1.702 g) (u + 1))."""
    p = name + "."
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, top, groups=None):
    """Softmax over all experts; the best ``keep`` of ``count`` equal groups of neighbours (by their largest score) stay
    eligible; of those the ``top`` largest scores.  -> (experts [T, top], their scores as they are)."""
    s = torch.softmax(h @ router.T, -1)
    pick = s.clone()
    if groups:
        T, E = s.shape
        best = s.view(T, groups["count"], E // groups["count"]).amax(-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, torch.topk(best, groups["keep"], dim=-1).indices, True)
        pick[~kept.repeat_interleave(E // groups["count"], 1)] = -1.0
    idx = torch.topk(pick, top, dim=-1).indices
    return idx, torch.gather(s, 1, idx)


def moe_ff(h, w, f):
    r = f["router"]
    idx, wt = route(h, w["router"], r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(idx[t].tolist(), wt[t]):
            out[t] += p * clamped_expert(h[t], w, f"e{e}", f["expert"]["limit"])
    if f.get("shared"):
        out = out + clamped_expert(h, w, "shared", f["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------------------ the model
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
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = sd["embed"][torch.tensor(tokens)]
    x = x0
    for i, t in layer_runs(cfg):
        layer, w = cfg["layers"][i], sub(sd, f"l{i}.")
        if t is not None:
            x = torch.cat([x, x0], 1) @ sd["loop.in"].T + sd["loop.step"][t]
        mix = {"attention": attention_mixer, "latent_attention": latent_attention_mixer}[layer["type"]]
        x = x + mult * dyt(mix(dyt(x, w, "norm1"), sub(w, "mix."), layer["mixer"], eps), w, "norm1b")
        if layer.get("mlp") is not None:
            x = x + mult * dyt(moe_ff(dyt(x, w, "norm2"), sub(w, "mlp."), layer["mlp"]), w, "norm2b")
        if trace is not None:
            trace.append(x.clone())
    return dyt(x, sd, "final.norm") @ sd["head"].T


# ------------------------------------------------------------------------------------------------ small random models
def random_config(vocab=61, width=24, types=("attention", "latent_attention", "attention"), ff=("moe",), eps=1e-5,
                  residual_mult=0.7, loop=(0, 2, 2), attention=None, latent=None, moe=None) -> dict:
    """A small configuration in the checkpoint's format.  ``types``: the mixers in order; ``ff``: "moe" or None, taken in
    turn; ``loop``: (start, stop, times) or None; the dicts override fields of every mixer / feed-forward of that kind."""
    att = dict(heads=4, kv_heads=2, dim=10, vdim=6, scale=0.4, rot={"dims": 6, "base": 300.0}, mask={"size": 9, "keep_first": 2})
    att.update(attention or {})
    lat = dict(heads=3, dim=6, vdim=5, kv_rank=12, q_rank=7, scale=0.35, mask={"size": 11})
    lat.update(latent or {})
    me = dict(kind="moe", expert={"ff": 10, "limit": 0.8}, router={"experts": 8, "top": 3, "groups": {"count": 4, "keep": 2}},
              shared={"ff": 9, "limit": 1.5})
    me.update(moe or {})
    layers = [{"type": kind, "mixer": dict(att if kind == "attention" else lat), "mlp": None if ff[i % len(ff)] is None else dict(me)}
              for i, kind in enumerate(types)]
    out = {"architecture": "Gekavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult, "layers": layers}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def tensor_shapes(cfg: dict) -> dict:
    D = cfg["width"]
    sh = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D)}

    def norm(name):
        sh[name], sh[name + ".b"], sh[name + ".alpha"] = (D,), (D,), ()

    norm("final.norm")
    if cfg.get("loop"):
        sh["loop.in"], sh["loop.step"] = (D, 2 * D), (cfg["loop"]["times"], D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1"), norm(p + "norm1b")
        M, H, d, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            for n, rows in (("q", H * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * dv)):
                sh[M + n], sh[M + n + ".b"] = (rows, D), (rows,)
            sh[M + "q.norm"] = sh[M + "k.norm"] = (d,)
            sh[M + "g"] = (H * dv, D)
        else:
            qr, kr = m["q_rank"], m["kv_rank"]
            sh[M + "dq"], sh[M + "dq.norm"], sh[M + "uq"] = (qr, D), (qr,), (H * d, qr)
            sh[M + "dkv"], sh[M + "dkv.norm"], sh[M + "uk"], sh[M + "uv"] = (kr, D), (kr,), (H * d, kr), (H * dv, kr)
            sh[M + "g"] = (H, D)
        sh[M + "o"] = (D, H * dv)
        f = layer.get("mlp")
        if f is None:
            continue
        norm(p + "norm2"), norm(p + "norm2b")
        F = p + "mlp."
        sh[F + "router"] = (f["router"]["experts"], D)
        experts = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else [])
        for n, ff in experts:
            sh[f"{F}{n}.gate"], sh[f"{F}{n}.up"], sh[f"{F}{n}.down"] = (ff, D), (ff, D), (D, ff)
    return sh


def random_weights(cfg: dict, seed: int = 0) -> dict:
    """Random tensors under the checkpoint's names, rounded to bfloat16 (what a file would hold), returned as float64."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        leaf = name.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=g)
        if leaf == "alpha":
            t = 0.8 + 0.2 * t
        elif leaf == "b":
            t = 0.2 * t
        elif len(shape) == 1:
            t = 1.0 + 0.2 * t                                    # norm weights
        elif leaf == "step":
            t = 0.5 * t
        elif leaf == "router":
            t = 1.5 * t * shape[1] ** -0.5
        elif leaf != "embed":
            t = t * shape[1] ** -0.5
        sd[name] = t.to(torch.bfloat16).double()
    return sd
