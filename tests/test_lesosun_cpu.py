"""Host side of the Lesosun model: configuration, registry, checkpoints, caches of layers that remember several things, and the
plain implementation against closed forms."""
import math

import pytest
import torch

import lesosun_models as lm
from oracle import lesosun_ref as ref


def test_configuration_is_read_and_checked():
    from pace_b200.llm.models.lesosun import DeltaConfig, DenseConfig, LesosunConfig, MoeConfig
    c = LesosunConfig.from_dict(lm.CONFIGS["mixed"])
    assert (c.vocab_size, c.hidden_size, c.eps, c.residual_mult, c.logit_softcap, c.num_hidden_layers) == (67, 88, 1e-3, 0.7, 9.0, 5)
    first, second, third, fourth, last = c.layers
    assert (first.mixer.left.softcap, first.mixer.left.rot_dims, first.mixer.right.norm_groups, first.mixer.left_scale) == (5.0, 16, 2, 1.3)
    assert first.mlp == MoeConfig(24, 5, 2, 3, 1.7, 40) and last.mlp == MoeConfig(40, 6, 1, 2, 1.7, None)
    assert second.mixer == DeltaConfig(6, 2, 24, 40, 3) and second.mlp == DenseConfig(56) and third.mlp is None
    assert fourth.mixer.right_scale == -1.1 and fourth.mixer.left.rot_base == 5e5
    a, r = lm.left(2, 1, 8, 8, 4, 4), lm.right(2, 1, 8, 8, 4, 1)
    ok = lm.layer(lm.P, lm.par(a, r), lm.moe(8, 4, 2))
    for bad in (lm.layer("mamba", {}), lm.layer(lm.P, lm.par({**a, "heads": 3, "kv_heads": 2}, r)),
                lm.layer(lm.P, lm.par(a, {**r, "groups": 3})), lm.layer(lm.P, lm.par(a, {**r, "norm_groups": 3})),
                lm.layer(lm.P, lm.par(lm.left(2, 1, 8, 8, 4, 3), r)), lm.layer(lm.P, lm.par(lm.left(2, 1, 8, 8, 4, 10), r)),
                lm.layer(lm.P, lm.par({**a, "softcap": 0.0}, r)), lm.layer(lm.P, lm.par({**a, "conv": 0}, r)),
                lm.layer(lm.D, lm.cd(3, 2, 8, 8, 4)), lm.layer(lm.D, lm.cd(2, 2, 8, 8, 0)), {**ok, "mlp": {"kind": "sparse"}},
                {**ok, "mlp": lm.moe(8, 2, 4, 1)}):
        with pytest.raises(ValueError):
            LesosunConfig.from_dict(lm.config([bad], 16))
    with pytest.raises(ValueError):
        LesosunConfig.from_dict(lm.config([ok], 16, cap=0.0))
    LesosunConfig.from_dict(lm.config([{**ok, "mlp": lm.moe(8, 2, 4, 2)}], 16))


def test_registry_and_checkpoint(tmp_path):
    from pace_b200.llm.models.lesosun import LesosunForCausalLM
    from pace_b200.llm.registry import build_model, model_registry
    from pace_b200.llm.weights import read_safetensors, write_safetensors
    cfg = lm.CONFIGS["mixed"]
    w = lm.weights(cfg, 3)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, w)
    back = read_safetensors(path)
    model = build_model(cfg, torch.float32, "cpu")
    assert isinstance(model, LesosunForCausalLM) and "Lesosun" in model_registry.architectures()
    model.load_weights(back)
    assert model.lm_head.weight is model.model.embed and torch.equal(model.model.embed_norm, w["embed.norm"].float())
    m = model.model.layers
    mix = m[0].mix                                  # q 240, k 80, v 48 | x 96, B 72, C 72 | z 96 | dt 6
    assert torch.equal(mix.proj[240:320], w["l0.mix.left.k"].float()) and torch.equal(mix.bias[320:368], w["l0.mix.left.v.b"].float())
    win = w["l0.mix.right.in"].float()
    assert torch.equal(mix.proj[368:608], win[96:336]) and torch.equal(mix.proj[608:704], win[:96]) and torch.equal(mix.proj[704:710], win[336:])
    assert float(mix.proj[710:].abs().max()) == 0 and float(mix.bias[368:].abs().max()) == 0
    assert torch.equal(mix.left_taps[2, 240:320], w["l0.mix.left.k.conv"].float()[:, 2])
    torch.testing.assert_close(mix.norm, w["l0.mix.right.norm"].float() * 0.6)
    torch.testing.assert_close(mix.out_bias, w["l0.mix.left.o.b"].float() * 1.3)
    torch.testing.assert_close(mix.neg_a, -w["l0.mix.right.A_log"].float().exp())
    assert torch.equal(m[0].out[:, :144], w["l0.mix.left.o"].float()) and torch.equal(m[0].out[:, 144:240], w["l0.mix.right.o"].float())
    assert torch.equal(m[0].out[:, 240:], w["l0.mlp.shared.down"].float()) and torch.equal(m[0].mlp.up[3], w["l0.mlp.e3.up"].float())
    delta = m[1].mix                                # ranks come from the checkpoint: 10 and 19, padded to 16 and 24
    assert delta.ranks == (10, 19) and delta.up.shape == (144 + 240, 40)
    assert torch.equal(delta.up[:144, :10], w["l1.mix.a2"].float()) and torch.equal(delta.up[144:, 16:35], w["l1.mix.g2"].float())
    assert float(delta.up[:144, 10:].abs().max()) == 0 and m[2].mlp is None and m[2].norm2 is None
    assert torch.equal(m[1].out[:, 240:], w["l1.mlp.down"].float())
    for change in ({"l2.norm2": w["l1.norm2"]}, {"head": w["embed"]}, {"l4.mlp.shared.up": w["l0.mlp.shared.up"]}):
        with pytest.raises(ValueError, match="without a place"):
            model.load_weights({**back, **change})
    for name in ("l1.mix.a1", "l4.mlp.e5.up", "embed.norm"):
        with pytest.raises(KeyError, match=name):
            model.load_weights({k: v for k, v in back.items() if k != name})
    with pytest.raises(ValueError, match="shape"):
        model.load_weights({**back, "l0.mix.right.in": back["l0.mix.right.in"][:-1]})


def test_what_layers_remember():
    from pace_b200.llm.hybrid_cache import JointSpec, StateSpec
    from pace_b200.llm.registry import build_model
    model = build_model(lm.CONFIGS["mixed"], torch.bfloat16, "cpu")
    specs = model.model.cache_specs()
    assert [type(s) for s in specs] == [JointSpec, StateSpec, StateSpec, JointSpec, StateSpec]
    kv, state = specs[0].parts
    assert (kv.kv_heads, kv.dim, kv.vdim) == (2, 40, 24)
    assert state.shapes == (("S", (6, 24, 16)), ("conv", (4, 368 + 240)))       # the longer one of the two convolutions
    assert specs[2].shapes == (("S", (3, 48, 16)), ("conv", (5, 3 * 48 * 2 + 48)))


def test_plain_mechanisms_match_closed_forms():
    x = torch.arange(1.0, 7.0, dtype=torch.float64)[:, None]
    assert ref.short_conv(x, torch.tensor([[100.0, 10, 1]]).double())[:, 0].tolist() == [1, 12, 123, 234, 345, 456]
    assert ref.short_conv(x[:2], torch.tensor([[5.0]]).double(), torch.tensor([1.0]).double())[:, 0].tolist() == [6, 11]
    z = torch.tensor([-40.0, -1.0, 0.0, 3.0, 50.0]).double()
    torch.testing.assert_close(ref.softplus(z), torch.nn.functional.softplus(z, threshold=1e9), rtol=1e-12, atol=0)
    torch.testing.assert_close(ref.gelu_erf(z), torch.nn.functional.gelu(z))
    assert float(ref.soft_cap(torch.tensor(1e9).double(), 3.0)) == 3.0 and abs(float(ref.soft_cap(torch.tensor(1e-3).double(), 3.0)) - 1e-3) < 1e-9
    r = ref.rotate_pairs(torch.randn(5, 2, 8).double(), 4, 100.0)
    h = torch.randn(5, 2, 8).double()
    r = ref.rotate_pairs(h, 4, 100.0)
    want = torch.view_as_complex(h[..., :4].reshape(5, 2, 2, 2).contiguous()) * torch.exp(
        1j * torch.arange(5)[:, None, None] * torch.tensor([1.0, 0.1]).double())
    torch.testing.assert_close(r[..., :4].reshape(5, 2, 2, 2), torch.view_as_real(want))
    assert torch.equal(r[..., 4:], h[..., 4:])
    # state space: a constant decay is a geometric sum
    n = 6
    one = torch.ones(n, 1, 1).double()
    y = ref.ssd_scan(one, one, one, one[:, :, 0] * 0.5, torch.tensor([0.3]).double(), torch.tensor([2.0]).double())[:, 0, 0]
    f = math.exp(-math.exp(0.3) * 0.5)
    torch.testing.assert_close(y, torch.tensor([2 + 0.5 * (1 - f ** (t + 1)) / (1 - f) for t in range(n)]).double())
    # delta rule: writing the same key again replaces its value (beta 1), half of it (beta 1/2)
    k = torch.zeros(3, 1, 4).double()
    k[:, 0, 2] = 1
    v = torch.tensor([3.0, 7.0, 5.0]).double().view(3, 1, 1)
    g = torch.ones(3, 1, 4).double()
    assert ref.delta_scan(k, k, v, g, torch.ones(3, 1).double())[:, 0, 0].tolist() == [3, 7, 5]
    assert ref.delta_scan(k, k, v, g, torch.full((3, 1), 0.5).double())[:, 0, 0].tolist() == [1.5, 4.25, 4.625]
    g[:, 0, 2] = 0.5                                          # the decay comes in front of the read-out
    assert ref.delta_scan(k, k, v, g, torch.zeros(3, 1).double() + torch.tensor([[1.0], [0.0], [0.0]]).double())[:, 0, 0].tolist() == [3, 1.5, 0.75]
    # routing: softmax scores, the correction only chooses, weights sum to the scale
    h = torch.eye(2, dtype=torch.float64)
    router = torch.log(torch.tensor([[1.0, 4.0], [2.0, 4.0], [5.0, 2.0]])).double()
    chosen, wt = ref.route(h, router, torch.tensor([0.6, 0.0, 0.0]).double(), 2, 1.5)
    assert chosen.tolist() == [[0, 2], [0, 1]]
    torch.testing.assert_close(wt, torch.tensor([[1.5 / 6, 7.5 / 6], [0.75, 0.75]]).double())
    y = ref.gated_group_norm(torch.tensor([[3.0, 4.0, 1.0, 1.0]]).double(), torch.full((1, 4), 50.0).double(), torch.ones(4).double(), 2, 0.0)
    torch.testing.assert_close(y, torch.tensor([[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 1.0, 1.0]]).double())
