"""CPU: the Gekavik configuration, checkpoint names and shapes, layer runs of a loop and merged-weight layout, the equations of
the plain restatement on hand-made numbers."""
import json

import pytest
import torch

from oracle import gekavik as O
from tests.lm_util import nerr, tokens_for


def config_of(cfg):
    from nano_qwen3tts_vllm_b200.config import GekavikConfig
    return GekavikConfig.from_dict(cfg)


def test_configuration_round_trip_shapes_and_names():
    from nano_qwen3tts_vllm_b200.models.gekavik import GekavikForCausalLM, checkpoint_shapes, random_state_dict
    from nano_qwen3tts_vllm_b200.models.registry import resolve, resolve_config_object
    for over in (dict(), dict(loop=None, ff=("moe", None)), dict(loop=(1, 3, 3), types=("latent_attention",) * 4),
                 dict(attention=dict(rot=None, mask=None), latent=dict(mask=None), moe=dict(shared=None))):
        cfg = O.random_config(**over)
        assert resolve(cfg).name == "Gekavik"
        c = config_of(cfg)
        assert resolve_config_object(c).name == "Gekavik" and c.to_dict() == cfg
        assert {k: tuple(v) for k, v in checkpoint_shapes(c).items()} == O.tensor_shapes(cfg)
        assert c.runs() == O.layer_runs(cfg)
        with torch.device("meta"):
            model = GekavikForCausalLM(c)
        assert model.checkpoint_names() == sorted(O.tensor_shapes(cfg))
        assert {k: tuple(v.shape) for k, v in random_state_dict(c, 3).items()} == O.tensor_shapes(cfg)
        plan = model.cache_plan()
        assert len(plan) == len(c.runs())
        for (li, _), p in zip(c.runs(), plan):
            m = c.layers[li].mixer
            want = [m.kv_heads * m.dim, m.kv_heads * m.vdim] if c.layers[li].type == "attention" else [m.kv_rank]
            assert p == {"paged": want, "state": []}


def test_every_constant_comes_from_the_configuration():
    c = config_of(O.random_config(residual_mult=0.3, eps=2e-3, attention=dict(mask={"size": 5}, scale=0.11),
                                  moe=dict(expert={"ff": 4, "limit": 0.25}, shared={"ff": 6, "limit": 3.0},
                                           router={"experts": 8, "top": 3, "groups": {"count": 4, "keep": 3}})))
    a, l, f = c.layers[0].mixer, c.layers[1].mixer, c.layers[0].mlp
    assert (c.residual_mult, c.norm_eps, a.mask_size, a.keep_first, a.scale) == (0.3, 2e-3, 5, 0, 0.11)
    assert (l.q_rank, l.kv_rank, l.window, l.rot_dim, l.head_gate) == (7, 12, 11, 0, True)
    assert (f.ff, f.limit, f.experts, f.top, f.groups, f.groups_keep) == (4, 0.25, 8, 3, 4, 3)
    assert (f.shared.ff, f.shared.limit) == (6, 3.0)
    one = config_of(O.random_config(moe=dict(router={"experts": 3, "top": 2}))).layers[0].mlp
    assert (one.groups, one.groups_keep) == (1, 1)


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].update(heads=3),                                  # 3 heads over 2 key/value heads
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12),                           # more rotated coordinates than the head has
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3),                            # an odd number of them
    lambda c: c["layers"][1]["mixer"].update(rot_dim=4),                                # no rotated part in this family
    lambda c: c["layers"][1]["mlp"].update(kind="other"),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3),                # 8 experts in 3 groups
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=5),                            # two groups of two hold four experts
    lambda c: c["loop"].update(stop=5),
    lambda c: c["loop"].update(start=2),
    lambda c: c["loop"].update(times=0),
])
def test_configuration_errors(bad):
    cfg = json.loads(json.dumps(O.random_config()))
    bad(cfg)
    with pytest.raises(ValueError):
        config_of(cfg)


@pytest.mark.parametrize("dtype,parts", [(torch.bfloat16, 3), (torch.float32, 2)])
def test_loading_is_strict_and_fills_merged_padded_and_pass_weights(dtype, parts):
    from nano_qwen3tts_vllm_b200.models.gekavik import GekavikForCausalLM
    cfg = O.random_config()
    sd = {k: v.to(torch.bfloat16) for k, v in O.random_weights(cfg, 1).items()}
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        model = GekavikForCausalLM(config_of(cfg))
    finally:
        torch.set_default_dtype(prev)
    assert model.load_state_dict(sd) == set(sd)
    D, m = cfg["width"], cfg["layers"][0]["mixer"]
    w = model.layers[0].mix.in_proj.weight
    q, k, v, g, end = model.layers[0].mix.offs
    assert w.shape[0] % 128 == 0 and not w[end:].any()
    for name, off in (("q", q), ("k", k), ("v", v), ("g", g)):
        assert torch.equal(w[off:off + sd["l0.mix." + name].shape[0]].float(), sd["l0.mix." + name].float())
    assert end == m["heads"] * (m["dim"] + m["vdim"]) + m["kv_heads"] * (m["dim"] + m["vdim"])
    core, lat = model.layers[1].mix.core, cfg["layers"][1]["mixer"]
    rows = torch.cat([sd["l1.mix." + n] for n in ("dq", "dkv", "g")]).float()
    assert torch.equal(core.in_proj.weight[:rows.shape[0]].float(), rows) and not core.in_proj.weight[rows.shape[0]:].any()
    assert torch.equal(core.uk.float().reshape(-1, lat["kv_rank"]), sd["l1.mix.uk"].float()) and core.attn.sink is None
    # the pass projection: the stream's columns once per part of the stream, then the embedding's
    W = sd["loop.in"].float()
    assert model.pass_in.weight.shape == (D, parts * D)
    assert torch.equal(model.pass_in.weight.float(), torch.cat([W[:, :D]] * (parts - 1) + [W[:, D:]], 1))
    e = model.layers[2].mlp
    assert torch.equal(e.up[3, :e.ff].float(), sd["l2.mlp.e3.gate"].float()) and torch.equal(e.up[3, e.ff:].float(), sd["l2.mlp.e3.up"].float())
    assert torch.equal(e.shared.gate_up.weight[cfg["layers"][2]["mlp"]["shared"]["ff"]:].float(), sd["l2.mlp.shared.up"].float())
    for broken in (dict(sd, extra=sd["embed"]), {k: v for k, v in sd.items() if k != "l1.norm2b.alpha"}):
        with pytest.raises(KeyError):
            model.load_state_dict(broken)
    with pytest.raises(ValueError):
        model.load_state_dict(dict(sd, embed=sd["embed"][:-1]))


# ------------------------------------------------------------------------------------------------ the plain restatement
def test_plain_routing_drops_experts_of_weak_groups():
    logits = torch.tensor([[5.0, 0.0, 3.0, 2.9, 4.0, 1.0]], dtype=torch.float64)         # groups {0, 1}, {2, 3}, {4, 5}
    idx, w = O.route(logits, torch.eye(6, dtype=torch.float64), 3, {"count": 3, "keep": 2})
    assert sorted(idx[0].tolist()) == [0, 4, 5]                                          # 2 and 3 are larger than 5, their group is not
    s = torch.softmax(logits, -1)
    assert torch.allclose(w, s[0, idx[0]][None]) and w.sum() < 1
    assert sorted(O.route(logits, torch.eye(6, dtype=torch.float64), 3)[0][0].tolist()) == [0, 2, 4]


def test_plain_expert_clamps_the_gate_above_and_the_up_part_on_both_sides():
    w = {"e.gate": torch.eye(1, dtype=torch.float64), "e.up": torch.eye(1, dtype=torch.float64), "e.down": torch.eye(1, dtype=torch.float64)}
    f = lambda v: O.clamped_expert(torch.tensor([[v]], dtype=torch.float64), w, "e", 2.0).item()
    sig = lambda z: 1.0 / (1.0 + torch.exp(torch.tensor(-1.702 * z, dtype=torch.float64)).item())
    assert abs(f(9.0) - 2 * sig(2) * 3) < 1e-12 and abs(f(1.0) - sig(1) * 2) < 1e-12
    assert abs(f(-5.0) - (-5 * sig(-5) * -1)) < 1e-12


def test_plain_mask_keeps_first_tokens():
    ok = O.visible(9, 3, 2)
    assert ok[8].tolist() == [True, True, False, False, False, False, True, True, True]
    assert ok[1].tolist() == [True, True] + [False] * 7 and O.visible(4).tolist() == torch.ones(4, 4).tril().bool().tolist()


def sharpened(cfg, sd, by=4.0):
    """Norm weights of the queries scaled up (by a power of two: they stay bfloat16 numbers): a few keys take each softmax, so a key that is seen or missed by mistake shows."""
    return {k: v * by if k.endswith(("q.norm", "dq.norm")) else v for k, v in sd.items()}


def test_mechanisms_show_in_the_logits():
    """The engine tests above could pass with a mechanism missing on both sides only; each of these changes moves the logits of
    the plain model by far more than the tolerance."""
    cfg = O.random_config()
    sd = sharpened(cfg, O.random_weights(cfg, seed=25))
    toks = tokens_for(cfg, 40, 1)
    ref = O.forward(cfg, sd, toks)

    def other(edit):
        c = json.loads(json.dumps(cfg))
        for layer in c["layers"]:
            edit(c, layer)
        return nerr(O.forward(c, sd, toks), ref)

    def field(kind, path, value):
        def edit(c, layer):
            d = layer["mixer"] if kind == layer["type"] else layer["mlp"] if kind == "mlp" else {}
            for k in path[:-1]:
                d = d.get(k, {})
            if d:
                d[path[-1]] = value
        return edit

    for edit in (field("attention", ("mask", "size"), 10), field("attention", ("mask", "keep_first"), 1), field("attention", ("mask", "keep_first"), 3),
                 field("latent_attention", ("mask", "size"), 10), field("attention", ("rot", "dims"), 4), field("attention", ("rot", "base"), 310.0),
                 field("mlp", ("expert", "limit"), 0.9), field("mlp", ("shared", "limit"), 1.4), field("mlp", ("router", "groups", "keep"), 3),
                 field("mlp", ("router", "top"), 2), field("mlp", ("shared",), None), lambda c, l: c.update(residual_mult=0.69)):
        assert other(edit) > 1e-3
