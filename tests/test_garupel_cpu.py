"""Host side of the Garupel model: configuration, registry, checkpoint files, packing of a step, and the plain
implementation against closed forms."""
import math

import pytest
import torch

import garupel_models as gm
from oracle import garupel_ref as ref


def test_configuration_is_read_and_checked():
    from pace_b200.llm.models.garupel import GarupelConfig
    c = GarupelConfig.from_dict(gm.CONFIGS["mixed"])
    assert (c.vocab_size, c.hidden_size, c.eps) == (61, 72, 1e-4)
    assert [i for i, _ in c.runs()] == [0] + [1, 2, 3] * 3 + [4] and c.num_hidden_layers == 11
    assert [n for n, (_, again) in enumerate(c.runs()) if again] == [4, 7]
    assert c.layers[1].ff is None and c.layers[0].ff == 50
    assert c.layers[4].mixer.temp_every == 5.0 and c.layers[4].mixer.scale == 1 / math.sqrt(40)
    assert [r for r, _ in GarupelConfig.from_dict(gm.CONFIGS["ones"]).runs()] == [0, 1, 2]     # no loop
    for change in ({"layers": [gm.layer("mamba", {})]}, {"loop": {"start": 2, "stop": 9, "times": 2}},
                   {"layers": [{"type": "rglru", "mixer": gm.lru(10, 2, 2), "mlp": {"kind": "moe", "ff": 4}}]},
                   {"layers": [gm.layer("rglru", gm.lru(10, 3, 2))]}, {"layers": [gm.layer("attention", gm.att(3, 2, 4, 4))]},
                   {"layers": [gm.layer("lightning", gm.lin(2, 4, 4, [0.5]))]}):
        with pytest.raises(ValueError):
            GarupelConfig.from_dict({**gm.CONFIGS["mixed"], **change})


def test_registry_finds_architectures():
    import pace_b200.llm.models  # noqa: F401
    from pace_b200.llm.registry import UnsupportedDtype, build_model, model_registry
    assert {"Garupel", "LlamaForCausalLM"} <= set(model_registry.architectures())
    assert model_registry.find({"architectures": ["X", "LlamaForCausalLM"]}).dtypes == (torch.bfloat16,)
    with pytest.raises(ValueError, match="no model for architecture"):
        model_registry.find({"architecture": "Unheard"})
    with pytest.raises(UnsupportedDtype):
        build_model({"architectures": ["LlamaForCausalLM"]}, torch.float32, "cpu")


def test_checkpoint_round_trip_and_loading(tmp_path):
    from pace_b200.llm.models.garupel import GarupelConfig, GarupelForCausalLM
    from pace_b200.llm.weights import read_safetensors, write_safetensors
    cfg = gm.CONFIGS["mixed"]
    w = gm.weights(cfg, 3)
    w["l0.table"] = torch.arange(7, dtype=torch.int32)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, w)
    back = read_safetensors(path)
    assert set(back) == set(w) and all(torch.equal(back[k], w[k]) and back[k].dtype == w[k].dtype for k in w)
    model = GarupelForCausalLM(GarupelConfig.from_dict(cfg), torch.float32)
    with pytest.raises(ValueError, match="l0.table"):
        model.load_weights(back)
    del back["l0.table"]
    model.load_weights(back)
    lay = model.model.layers[1].mix
    assert torch.equal(lay.qkvg[:144], w["l1.mix.q"].float()) and torch.equal(lay.bias[144:216], w["l1.mix.k.b"].float())
    assert float(lay.bias[lay.nq + lay.nk + lay.nv:].abs().max()) == 0.0
    lru = model.model.layers[2].mix
    assert torch.equal(lru.gate_w[:, 1], w["l2.mix.ri"].float())
    torch.testing.assert_close(lru.decay_base, -8 * torch.nn.functional.softplus(w["l2.mix.lam"].float()))
    with pytest.raises(KeyError, match="head"):
        model.load_weights({k: v for k, v in back.items() if k != "head"})
    with pytest.raises(ValueError, match="shape"):
        model.load_weights({**back, "head": back["head"][:-1]})
    raw = open(path, "rb").read()                   # a header of odd length, a truncated file
    n = int.from_bytes(raw[:8], "little")
    odd = str(tmp_path / "odd.safetensors")
    open(odd, "wb").write((n + 1).to_bytes(8, "little") + raw[8:8 + n] + b" " + raw[8 + n:])
    assert torch.equal(read_safetensors(odd)["embed"], w["embed"])
    open(odd, "wb").write(raw[:-10])
    with pytest.raises(ValueError, match="extent"):
        read_safetensors(odd)


def test_step_packs_decode_entries_first():
    from pace_b200.llm.step import Step
    toks = torch.arange(10, 21)
    s = Step([3, 1, 0, 5, 1, 1], [7, 100, 4, 0, 0, 63], [5, 4, 3, 2, 1, 0], toks, 50, "cpu")
    assert s.rows == [1, 4, 5, 0, 3] and s.n_decode == 3 and s.max_count == 5 and not s.decode_only
    assert s.token.tolist() == [13, 19, 20, 10, 11, 12, 14, 15, 16, 17, 18]
    assert s.tok_pos.tolist() == [100, 0, 63, 7, 8, 9, 0, 1, 2, 3, 4]
    assert s.q_row.tolist() == [0, 1, 2, 3, 4, 5, 8, 9, 10, 11, 12] and s.staging_rows == 13
    assert s.cu.tolist() == [0, 1, 2, 3, 6, 11] and s.start.tolist() == [100, 0, 63, 7, 0]
    assert s.slot.tolist() == [4, 1, 0, 5, 2] and s.first_row == {1: 0, 4: 1, 5: 2, 0: 3, 3: 6}
    with pytest.raises(ValueError, match="token ids"):
        Step([1], [0], [0], torch.tensor([50]), 50, "cpu")
    with pytest.raises(ValueError):
        Step([0, 0], [0, 0], [0, 1], torch.tensor([], dtype=torch.long), 50, "cpu")


def test_plain_recurrences_match_closed_forms():
    g = torch.Generator().manual_seed(1)
    n, H, d, v = 9, 2, 3, 4
    q, k, val = (torch.rand(n, H, x, generator=g, dtype=torch.float64) for x in (d, d, v))
    decay = torch.tensor([0.5, 0.9], dtype=torch.float64)
    S = torch.zeros(H, d, v, dtype=torch.float64)
    for t in range(n):
        S, o = ref.lightning_step(S, q[t], k[t], val[t], decay)
        want = sum((decay ** (t - j))[:, None] * (q[t] * k[j]).sum(-1, keepdim=True) * val[j] for j in range(t + 1))
        torch.testing.assert_close(o, want)
    # a recurrence with r = i = 1 everywhere has a geometric weight per step
    lam = torch.tensor([-3.0], dtype=torch.float64)
    a = math.exp(-8 * math.log1p(math.exp(-3.0)))
    s, one = torch.zeros(1, dtype=torch.float64), torch.ones(1, dtype=torch.float64)
    for t in range(5):
        s = ref.rglru_step(s, one * (t + 1), one, one, lam)
    assert abs(float(s) - sum(a ** (4 - t) * math.sqrt(1 - a * a) * (t + 1) for t in range(5))) < 1e-12
    past = []
    taps = torch.tensor([[1.0, 10.0, 100.0]])
    outs = [float(ref.causal_conv_token(torch.tensor([x]), taps, torch.tensor([0.5]), past)) for x in (1.0, 2.0, 3.0, 4.0)]
    assert outs == [100.5, 210.5, 321.5, 432.5]
    assert ref.query_temperature(14, 0.3, 16) == 1.0 and ref.query_temperature(15, 0.3, 16) == 1 + 0.3 * math.log(2)


def test_llama_checkpoints_load_through_the_registry(tmp_path):
    """The attention-only decoder takes the same road: config.json, safetensors, plain MLP names, tied head."""
    import json
    from pace_b200.llm.registry import load_model
    from pace_b200.llm.weights import write_safetensors
    cfg = {"architectures": ["LlamaForCausalLM"], "hidden_size": 128, "intermediate_size": 96, "num_hidden_layers": 1,
           "num_attention_heads": 2, "num_key_value_heads": 1, "vocab_size": 40, "max_position_embeddings": 64,
           "rms_norm_eps": 1e-5}
    g = torch.Generator().manual_seed(0)
    names = {"model.embed_tokens.weight": (40, 128), "model.norm.weight": (128,)}
    pre = "model.layers.0."
    names.update({pre + "input_layernorm.weight": (128,), pre + "post_attention_layernorm.weight": (128,),
                  pre + "self_attn.q_proj.weight": (128, 128), pre + "self_attn.k_proj.weight": (64, 128),
                  pre + "self_attn.v_proj.weight": (64, 128), pre + "self_attn.o_proj.weight": (128, 128),
                  pre + "mlp.gate_proj.weight": (96, 128), pre + "mlp.up_proj.weight": (96, 128),
                  pre + "mlp.down_proj.weight": (128, 96)})
    w = {k: torch.randn(*s, generator=g).bfloat16() for k, s in names.items()}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    m = load_model(str(tmp_path), torch.bfloat16, "cpu")
    assert torch.equal(m.model.layers[0].mlp.gate_proj.linear.weight, w[pre + "mlp.gate_proj.weight"])
    assert torch.equal(m.lm_head.weight, w["model.embed_tokens.weight"])
