"""Host side of the Kibotar model: configuration, registry, checkpoints, what layers remember, rotation tables, and the plain
implementation against closed forms."""
import math

import pytest
import torch

import kibotar_models as km
from oracle import kibotar_ref as ref


def test_configuration_is_read_and_checked():
    from pace_b200.llm.models.kibotar import AttentionConfig, GlaConfig, KibotarConfig, LatentConfig, ScalingConfig
    c = KibotarConfig.from_dict(km.CONFIGS["mixed"])
    assert (c.vocab_size, c.hidden_size, c.eps, c.embedding_scale, c.num_hidden_layers) == (67, 88, 1e-3, 3.0, 11)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur, c.loop) == (31, 7, 11, (1, 4, 3))
    first, second, third, fourth, last = c.layers
    assert first.mixer == AttentionConfig(6, 2, 40, 24, 1 / math.sqrt(40), 37, 5, 24, 1e4, ScalingConfig(8.0, 1.0, 4.0, 40.0))
    assert second.mixer == GlaConfig(3, 24, 40, 4.0) and third.mixer == LatentConfig(5, 24, 40, 48, 1 / math.sqrt(24))
    assert (first.ff, third.ff, fourth.mixer.scaling, fourth.mixer.rot_base, last.mixer.tau) == (56, None, None, 5e5, 16.0)
    assert c.runs() == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (1, 2), (2, None), (3, None), (4, None)]
    assert c.runs() == ref.runs(km.CONFIGS["mixed"])
    plain = KibotarConfig.from_dict(km.config([km.layer(km.G, km.gla(2, 8, 8))], 16, bigram=None))
    assert plain.bigram is None and plain.loop is None and plain.runs() == [(0, None)]
    a = km.att(2, 1, 8, 8, 4, 2, 4)
    for bad in (km.layer("rwkv", {}), km.layer(km.A, {**a, "heads": 3, "kv_heads": 2}), km.layer(km.A, km.att(2, 1, 8, 8, 4, 2, 3)),
                km.layer(km.A, km.att(2, 1, 8, 8, 4, 2, 10)), km.layer(km.A, {**a, "mask": {"size": 0, "pool": 2}}),
                km.layer(km.A, {**a, "mask": {"size": 4, "pool": 0}}), km.layer(km.G, km.gla(2, 8, 8, 0.0)),
                {**km.layer(km.A, a), "mlp": {"kind": "moe"}}):
        with pytest.raises(ValueError):
            KibotarConfig.from_dict(km.config([bad], 16))
    for loop in ((0, 2, 1), (1, 1, 2), (0, 1, 0)):
        with pytest.raises(ValueError, match="loop"):
            KibotarConfig.from_dict(km.config([km.layer(km.A, a)], 16, loop=loop))
    with pytest.raises(ValueError, match="bucket"):
        KibotarConfig.from_dict(km.config([km.layer(km.A, a)], 16, bigram=(0, 1, 1)))


def test_registry_and_checkpoint(tmp_path):
    from pace_b200.llm.models.kibotar import KibotarForCausalLM
    from pace_b200.llm.registry import build_model, model_registry
    from pace_b200.llm.weights import read_safetensors, write_safetensors
    cfg = km.CONFIGS["mixed"]
    w = km.weights(cfg, 3)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, w)
    back = read_safetensors(path)
    model = build_model(cfg, torch.float32, "cpu")
    assert isinstance(model, KibotarForCausalLM) and "Kibotar" in model_registry.architectures()
    model.load_weights(back)
    m = model.model
    assert model.lm_head.weight is m.embed and torch.equal(m.bigram, w["bigram"].float()) and torch.equal(m.steps, w["loop.step"].float())
    a = m.layers[0].mix                             # q 240, k 80, v 48 | gate 144
    assert torch.equal(a.qkvg[240:320], w["l0.mix.k"].float()) and torch.equal(a.bias[320:368], w["l0.mix.v.b"].float())
    assert torch.equal(a.qkvg[368:], w["l0.mix.g"].float()) and float(a.bias[368:].abs().max()) == 0
    assert torch.equal(a.talk, w["l0.mix.talk"].float()) and torch.equal(a.out_bias, w["l0.mix.o.b"].float())
    r = m.layers[1].mix                             # q 72, k 72, v 120 | gate 120 | a1 10 of 16
    assert r.rank == 10 and r.proj.shape == (400, 88) and torch.equal(r.proj[264:384], w["l1.mix.g"].float())
    assert torch.equal(r.proj[384:394], w["l1.mix.a1"].float()) and float(r.proj[394:].abs().max()) == 0
    assert torch.equal(r.up[:, :10], w["l1.mix.a2"].float()) and float(r.up[:, 10:].abs().max()) == 0
    t = m.layers[2].mix                             # q 120 | latent 48 | gate 5 of 8
    assert torch.equal(t.proj[168:173], w["l2.mix.g"].float()) and torch.equal(t.ukv[120:], w["l2.mix.uv"].float())
    assert m.layers[2].ff is None and torch.equal(m.layers[2].shift, w["l2.shift"].float())
    for change in ({"l2.norm2": w["l1.norm2"]}, {"head": w["embed"]}, {"l1.mix.q.b": w["l0.mix.q.b"]}):
        with pytest.raises(ValueError, match="without a place"):
            model.load_weights({**back, **change})
    for name in ("l1.mix.a1", "l0.mix.talk", "bigram", "loop.step", "l4.shift"):
        with pytest.raises(KeyError, match=name):
            model.load_weights({k: v for k, v in back.items() if k != name})
    with pytest.raises(ValueError, match="shape"):
        model.load_weights({**back, "bigram": back["bigram"][:-1]})


def test_what_layers_remember():
    from pace_b200.llm.hybrid_cache import BlockSpec, JointSpec, KVSpec, LatentSpec, StateSpec
    from pace_b200.llm.registry import build_model
    specs = build_model(km.CONFIGS["mixed"], torch.bfloat16, "cpu").model.cache_specs()
    assert len(specs) == 12
    assert specs[0] == JointSpec((KVSpec(2, 40, 24), BlockSpec(2, 40, 24, 5)))
    assert specs[1] == StateSpec((("S", (3, 24, 40)),)) == specs[4] == specs[7] and specs[2] == LatentSpec(48, 0)
    assert specs[11] == JointSpec((StateSpec((("h", (11, 88)), ("next", (11, 88)))), StateSpec((("token", ()),), torch.int32)))


def test_pages_of_blocks_are_counted_in_tokens():
    """A pool with a row per 5 tokens: pages of 64 rows cover 320 tokens."""
    import ctypes as C
    from pace_b200 import _C
    pb, mb = C.c_uint64(), C.c_uint64()

    def size(**kw):
        geom = dict(n_layers=2, n_kv_heads=3, head_dim=64, page_tokens=320, n_pages=4, max_seqs=2, max_pages_per_seq=3, row_tokens=5)
        rc = _C.lib.pace_kv_pool_bytes(C.byref(_C.KVPoolStruct(**{**geom, **kw})), C.byref(pb), C.byref(mb))
        return pb.value if rc == _C.PACE_OK else None
    assert size() == 2 * 2 * 4 * 3 * 64 * 64 * 2
    assert size(row_tokens=0, page_tokens=64) == size() == size(row_tokens=1, page_tokens=64)
    assert size(row_tokens=3) is None and size(row_tokens=-1) is None and size(row_format=_C.ROWS_SHARED) is None


@pytest.mark.parametrize("scaling", [None, km.SCALING, {"factor": 4.0, "low": 2.0, "high": 3.0, "original": 500}])
def test_rotation_tables(scaling):
    from pace_b200.ops import RotaryEmbedding
    kind = {"rope_type": "precise"} if scaling is None else {
        "rope_type": "llama3_precise", "factor": scaling["factor"], "low_freq_factor": scaling["low"], "high_freq_factor": scaling["high"],
        "original_max_position_embeddings": scaling["original"]}
    rope = RotaryEmbedding(kind, 24, 5000, 3e4)
    a = torch.arange(5000, dtype=torch.float64)[:, None] * ref.frequencies(24, 3e4, scaling)
    torch.testing.assert_close(rope.cos_cache.double(), a.cos(), rtol=0, atol=1e-7)
    torch.testing.assert_close(rope.sin_cache.double(), a.sin(), rtol=0, atol=1e-7)
    if scaling is not None:                         # both bands and the blend are there
        wavelength = 2 * math.pi / ref.frequencies(24, 3e4)
        ratio = ref.frequencies(24, 3e4, scaling) / ref.frequencies(24, 3e4)
        assert float(ratio.max()) == 1.0 and abs(float(ratio.min()) * scaling["factor"] - 1) < 1e-12
        inside = (wavelength > scaling["original"] / scaling["high"]) & (wavelength < scaling["original"] / scaling["low"])
        assert bool(inside.any()) or scaling["original"] == 500


# ---- the plain implementation against closed forms -----------------------------------------------------------------------
def test_bigram_rows():
    assert ref.bigram_rows([5, 2, 2, 9], 10, 3, 4) == [10, 3, 4, 2]
    assert ref.bigram_rows([7], 1, 1, 1) == [1]


def test_what_a_position_sees():
    m = ref.pooled_mask(12, 4, 3)
    seen = [[j for j in range(12) if m[i, j]] + [("b", b) for b in range(4) if m[i, 12 + b]] for i in range(12)]
    assert seen[3] == [0, 1, 2, 3] and seen[5] == [2, 3, 4, 5] and seen[6] == [3, 4, 5, 6, ("b", 0)]
    assert seen[8] == [5, 6, 7, 8, ("b", 0)] and seen[9] == [6, 7, 8, 9, ("b", 0), ("b", 1)] and seen[11][4:] == [("b", 0), ("b", 1)]
    m = ref.pooled_mask(3, 1, 1)                     # the token itself, and every earlier one as a block of its own
    assert m.tolist() == [[True, False, False] + [False] * 3, [False, True, False, True, False, False], [False, False, True, True, True, False]]


def test_softmax_with_one_in_the_denominator():
    s = torch.tensor([[0.0, -math.inf], [1000.0, 999.0], [-1000.0, -1000.0]], dtype=torch.float64)
    p = ref.softmax_plus_one(s)
    assert p[0].tolist() == [0.5, 0.0] and abs(float(p[1].sum()) - 1) < 1e-12 and float(p[2].sum()) == 0.0


def test_rotation_and_shift_and_recurrence():
    x = torch.randn(6, 1, 7, generator=torch.Generator().manual_seed(0)).double()
    y = ref.rotate_half(x, 4, 100.0)
    a = 3 * 100.0 ** (-2.0 / 4)
    assert abs(float(y[3, 0, 1] - (x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a)))) < 1e-12
    assert abs(float(y[3, 0, 3] - (x[3, 0, 3] * math.cos(a) + x[3, 0, 1] * math.sin(a)))) < 1e-12 and torch.equal(y[..., 4:], x[..., 4:])
    h = torch.tensor([[1.0, 2.0], [3.0, 5.0]], dtype=torch.float64)
    assert ref.token_shift(h, torch.tensor([0.0, 0.25]).double()).tolist() == [[1.0, 1.5], [3.0, 4.25]]
    n = 5
    q, k, v = (torch.randn(n, 1, 2, generator=torch.Generator().manual_seed(s)).double() for s in (1, 2, 3))
    al = torch.full((n, 1, 2), 0.5).double()
    want = sum(0.5 ** (n - 1 - j) * float(q[-1, 0] @ k[j, 0]) * v[j, 0] for j in range(n))
    torch.testing.assert_close(ref.gla_scan(q, k, v, al)[-1, 0], want)


def test_mixing_identity_and_permutation():
    g = torch.Generator().manual_seed(4)
    q, k, v = torch.randn(9, 4, 6, generator=g).double(), torch.randn(9, 2, 6, generator=g).double(), torch.randn(9, 2, 3, generator=g).double()
    p = ref.pooled_weights(q, k, 0.5, 4, 2)
    own = ref.mixed_heads(p, v, torch.eye(4).double(), 2)
    perm = [2, 0, 3, 1]
    mixed = ref.mixed_heads(p, v, torch.eye(4).double()[perm], 2)
    values = torch.cat([v, ref.block_means(v, 2)])
    for h in range(4):
        torch.testing.assert_close(own[:, h], p[h] @ values[:, h // 2])
        torch.testing.assert_close(mixed[:, h], p[perm[h]] @ values[:, h // 2])
