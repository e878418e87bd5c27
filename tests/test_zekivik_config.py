"""CPU: the Zekivik configuration, checkpoint names and shapes, layer runs of a loop and merged-weight layout - against
``oracle/zekivik.py``."""
import json

import pytest
import torch

from oracle import zekivik as O


def test_configuration_round_trip_shapes_and_names():
    from nano_qwen3tts_vllm_b200.config import ZekivikConfig
    from nano_qwen3tts_vllm_b200.models.registry import resolve, resolve_config_object
    from nano_qwen3tts_vllm_b200.models.zekivik import ZekivikForCausalLM, checkpoint_shapes, random_state_dict
    for over in (dict(), dict(loop=None, ff=(None,)), dict(loop=(0, 4, 3), types=("attention",) * 4, ff=(8, 9))):
        cfg = O.random_config(**over)
        assert resolve(cfg).name == "Zekivik"
        c = ZekivikConfig.from_dict(cfg)
        assert resolve_config_object(c).name == "Zekivik" and c.to_dict() == cfg
        assert {k: tuple(v) for k, v in checkpoint_shapes(c).items()} == O.tensor_shapes(cfg)
        assert c.runs() == O.layer_runs(cfg)
        with torch.device("meta"):
            model = ZekivikForCausalLM(c)
        assert model.checkpoint_names() == sorted(O.tensor_shapes(cfg))
        assert {k: tuple(v.shape) for k, v in random_state_dict(c, 3).items()} == O.tensor_shapes(cfg)
        plan = model.cache_plan()
        assert len(plan) == len(c.runs())
        for (li, _), p in zip(c.runs(), plan):
            m = c.layers[li].mixer
            if c.layers[li].type == "attention":
                assert p["paged"] == [m.kv_heads * m.dim, m.kv_heads * m.vdim]
                assert p["state"] == [((m.conv - 1, m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)), None)]
            else:
                assert p["paged"] == [] and p["state"] == [((m.heads, m.dim, m.vdim), torch.float32)]


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][1]["mixer"].update(heads=3),                   # 3 heads over 2 key/value heads
    lambda c: c["layers"][1]["mixer"].update(conv=0),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12),            # more rotated coordinates than the head has
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3),             # an odd number of them
    lambda c: c["layers"][0]["mixer"].update(decay=[0.5]),               # one decay for three heads
    lambda c: c["layers"][1]["mlp"].update(kind="other"),
    lambda c: c["loop"].update(stop=5),
    lambda c: c["loop"].update(start=3),
    lambda c: c["loop"].update(times=0),
])
def test_configuration_errors(bad):
    from nano_qwen3tts_vllm_b200.config import ZekivikConfig
    cfg = json.loads(json.dumps(O.random_config()))
    bad(cfg)
    with pytest.raises(ValueError):
        ZekivikConfig.from_dict(cfg)


def test_loading_is_strict_and_fills_merged_and_offset_weights():
    from nano_qwen3tts_vllm_b200.config import ZekivikConfig
    from nano_qwen3tts_vllm_b200.models.zekivik import ZekivikForCausalLM
    cfg = O.random_config()
    sd = {k: v.to(torch.bfloat16) for k, v in O.random_weights(cfg, seed=1).items()}
    prev = torch.get_default_dtype()
    torch.set_default_dtype(torch.bfloat16)
    try:
        model = ZekivikForCausalLM(ZekivikConfig.from_dict(cfg))
    finally:
        torch.set_default_dtype(prev)
    model.load_state_dict(sd)
    for i, layer in enumerate(model.layers):
        w = layer.mix.in_proj.weight
        names = {"rg": f"l{i}.rg1", **{n: f"l{i}.mix.{n}" for n, _ in layer.mix.parts if n != "rg"}}
        for n, rows in layer.mix.parts:
            assert torch.equal(w[layer.mix.cols[n]:layer.mix.cols[n] + rows], sd[names[n]])
        used = sum(rows for _, rows in layer.mix.parts)
        assert w.shape[0] % 128 == 0 and w.shape[0] - used < 128 and not w[used:].any()
        assert layer.norm1.weight.dtype == torch.float32 and torch.equal(layer.norm1.weight, 1.0 + sd[f"l{i}.norm1"].float())
    assert torch.equal(model.layers[1].mix.conv.weight, torch.cat([sd[f"l1.mix.{n}.conv"] for n in "qkv"]).float())
    with pytest.raises(KeyError, match="missing"):
        model.load_state_dict({k: v for k, v in sd.items() if k != "loop.step"})
    with pytest.raises(KeyError, match="unexpected"):
        model.load_state_dict({**sd, "l0.mix.extra": sd["embed"]})
    with pytest.raises(ValueError, match="shape"):
        model.load_state_dict({**sd, "l0.rg1.b": sd["l0.rg1.b"][:-1]})
