"""Host side of the Gekupel model: configuration, registry, checkpoints, rotation tables, key lists of a step, and the
plain implementation against closed forms."""
import math

import pytest
import torch

import gekupel_models as gk
from oracle import gekupel_ref as ref


def test_configuration_is_read_and_checked():
    from pace_b200.llm.models.gekupel import AttentionConfig, DenseConfig, GekupelConfig, MoeConfig
    c = GekupelConfig.from_dict(gk.CONFIGS["mixed"])
    assert (c.vocab_size, c.hidden_size, c.eps, c.embedding_scale, c.num_hidden_layers) == (59, 88, 1e-3, 3.5, 6)
    assert [lay.weights_of for lay in c.layers] == [None, None, None, 1, None, 0]
    first, second, third = c.layers[:3]
    assert first.mixer.sink and first.mixer.yarn.factor == 4.0 and first.mixer.window == 21 and first.mlp == DenseConfig(72)
    assert second.mixer == AttentionConfig(6, 2, 40, 24, 1 / math.sqrt(40), 50) and second.mlp == MoeConfig(24, 5, 2)
    assert not third.mixer.sink and third.mixer.yarn is None and third.mixer.rot_base == 5e5 and third.mlp is None
    ok = gk.layer(gk.A, gk.att(2, 1, 8, 8, 4), gk.moe(8, 4, 2))
    for layers in ([gk.layer("mamba", {})], [gk.layer(gk.A, gk.att(3, 2, 4, 4, 4))], [{**ok, "mlp": {"kind": "sparse"}}],
                   [gk.layer(gk.A, gk.att(2, 1, 8, 8, 0))], [{**ok, "mlp": gk.moe(8, 2, 3)}], [{**ok, "weights_of": 0}],
                   [ok, {**ok, "weights_of": 2}], [ok, {**ok, "mixer": gk.att(2, 1, 8, 8, 5), "weights_of": 0}],
                   [{**ok, "weights_of": 1}, {**ok, "weights_of": 0}], [gk.layer(gk.L1, gk.lat(2, 8, 3, 8, 8, 8, 4))]):
        with pytest.raises(ValueError):
            GekupelConfig.from_dict(gk.config(layers, 16))
    chain = GekupelConfig.from_dict(gk.config([ok, {**ok, "weights_of": 0}, {**ok, "weights_of": 1}], 16))
    assert chain.layers[2].weights_of == 0


def test_registry_and_checkpoint(tmp_path):
    from pace_b200.llm.models.gekupel import GekupelForCausalLM
    from pace_b200.llm.registry import build_model, model_registry
    from pace_b200.llm.weights import read_safetensors, write_safetensors
    cfg = gk.CONFIGS["mixed"]
    w = gk.weights(cfg, 3)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, w)
    back = read_safetensors(path)
    model = build_model(cfg, torch.float32, "cpu")
    assert isinstance(model, GekupelForCausalLM) and "Gekupel" in model_registry.architectures()
    model.load_weights(back)
    m = model.model.layers
    assert m[3] is m[1] and m[5] is m[0] and m[2] is not m[4]
    assert torch.equal(m[1].mix.qkv[240:320], w["l1.mix.k"].float()) and torch.equal(m[1].mlp.down[4], w["l1.mlp.e4.down"].float())
    assert torch.equal(m[1].mlp.gate_up[2, 24:], w["l1.mlp.e2.up"].float())
    assert torch.equal(m[0].mix.down[56:], w["l0.mix.dkv"].float()) and torch.equal(m[0].mix.ukv[96:], w["l0.mix.uv"].float())
    assert len(model.model.cache_specs()) == 6 and not hasattr(m[2].mix, "sink")
    for change in ({"l3.norm1": w["l1.norm1"]}, {"l2.mix.sink": w["l0.mix.sink"]}):        # tensors without a place
        with pytest.raises(ValueError, match="without a place"):
            model.load_weights({**back, **change})
    with pytest.raises(KeyError, match="l4.mlp.e6.up"):
        model.load_weights({k: v for k, v in back.items() if k != "l4.mlp.e6.up"})
    with pytest.raises(ValueError, match="shape"):
        model.load_weights({**back, "l0.mix.uq": back["l0.mix.uq"][:-1]})


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, None), (2, 3e5, None), (64, 1e5, gk.yarn(8.0, 1024, 32.0, 1.0)),
                                               (24, 500.0, gk.yarn(3.0, 100, 4.0, 0.5)), (8, 1e4, gk.yarn(1.0))])
def test_rotation_tables(dims, base, scaling):
    from pace_b200.ops import RotaryEmbedding
    kind = {"rope_type": "precise"} if scaling is None else {
        "rope_type": "yarn", "factor": scaling["factor"], "original_max_position_embeddings": scaling["original"],
        "beta_fast": scaling["fast"], "beta_slow": scaling["slow"]}
    rope = RotaryEmbedding(kind, dims, 70000, base, is_neox_style=False)
    freq, mult = ref.rotation_frequencies(dims, base, scaling)
    for p in (0, 1, 777, 69999):
        for i, f in enumerate(freq):
            assert abs(float(rope.cos_cache[p, i]) - math.cos(p * f) * mult) < 2e-7
            assert abs(float(rope.sin_cache[p, i]) - math.sin(p * f) * mult) < 2e-7


def test_key_rows_of_a_step():
    from pace_b200.llm.step import Step
    toks = torch.zeros(12, dtype=torch.long)
    s = Step([1, 5, 0, 6], [9, 0, 4, 7], [3, 2, 1, 0], toks, 5, "cpu")
    k = s.key_rows(4, s.n_decode)                       # entries: row 1 (positions 0..4) and row 3 (7..12)
    assert k.cu.tolist() == [0, 5, 14] and k.first_pos.tolist() == [0, 4] and k.total == 14
    assert k.pos.tolist() == [0, 1, 2, 3, 4] + list(range(4, 13)) and k.slot.tolist() == [2] * 5 + [0] * 9
    assert s.key_rows(4, s.n_decode) is k and s.key_rows(None, 0).total == 10 + 5 + 13 and s.max_keys == 13


def test_which_form_latents_take():
    """Long prompts expand, short portions over many cached keys do not, sizes the prompt kernel refuses never do."""
    from pace_b200.llm.step import Step
    from pace_b200.ops.hybrid import expand_pays
    toks = torch.zeros(600, dtype=torch.long)
    prompt, portion = Step([600], [0], [0], toks, 1, "cpu"), Step([2], [5000], [0], toks, 1, "cpu")
    args = (8, 128, 64, 128, 512)
    assert expand_pays(prompt, torch.bfloat16, *args, 4096) and not expand_pays(portion, torch.bfloat16, *args, 4096)
    assert not expand_pays(prompt, torch.float32, *args, 4096)
    assert not expand_pays(prompt, torch.bfloat16, 8, 128, 60, 128, 512, 4096)
    assert not expand_pays(prompt, torch.bfloat16, 8, 128, 64, 136, 512, 4096)


def test_plain_mechanisms_match_closed_forms():
    assert ref.window_mask(4, 2).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert ref.chunk_mask(5, 2).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    assert ref.distance_slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8] and ref.distance_slopes(3)[0] == 2.0 ** (-8 / 3)
    p = ref.masked_softmax(torch.log(torch.tensor([[1.0, 2.0, 5.0]])).double(), torch.tensor([[True, True, False]]), torch.tensor(0.0))
    torch.testing.assert_close(p, torch.tensor([[0.25, 0.5, 0.0]]).double())
    x = torch.randn(6, 2, 8, dtype=torch.float64)
    freq, mult = ref.rotation_frequencies(4, 100.0)
    assert freq == [1.0, 0.1] and mult == 1.0
    r = ref.rotate_pairs(x, 4, freq, 1.0)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])
    z = torch.view_as_complex(x[..., :4].reshape(6, 2, 2, 2).contiguous()) * torch.exp(1j * torch.arange(6)[:, None, None] * torch.tensor(freq, dtype=torch.float64))
    torch.testing.assert_close(r[..., :4].reshape(6, 2, 2, 2), torch.view_as_real(z))
    f2, m2 = ref.rotation_frequencies(8, 1e4, gk.yarn(4.0, 256, 16.0, 2.0))
    plain = ref.rotation_frequencies(8, 1e4)[0]
    assert f2[0] == plain[0] and abs(f2[3] - plain[3] / 4) < 1e-12 and abs(m2 - (0.1 * math.log(4.0) + 1)) < 1e-12
    h = torch.eye(3, dtype=torch.float64)
    chosen, wt = ref.route(h, torch.tensor([[0.0, 2, 0], [1, 0, 0], [0, 1, 0.1]]).double(), torch.tensor([0.1, 0.0, 0.5]).double(), 2)
    sig = lambda v: 1 / (1 + math.exp(-v))      # noqa: E731
    assert [sorted(r) for r in chosen.tolist()] == [[1, 2], [0, 2], [0, 2]]
    assert abs(float(wt[1][chosen[1] == 0]) - sig(2)) < 1e-12 and abs(float(wt[1][chosen[1] == 2]) - sig(1)) < 1e-12
