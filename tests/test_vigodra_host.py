"""Vigodra on the host: configuration and its errors, tensor names, cache needs (filters' inputs beside keys and values, kept
first positions, an owner that holds its latents as long as the farthest-seeing reader needs them), the cache manager's and
the scheduler's side of kept positions, distance buckets, and the plain implementation against closed forms."""
import copy
import math

import pytest
import torch

import plain_vigodra as pv
from vigodra_util import VIG_A, VIG_B, VIG_C, VIG_D


def test_configuration_round_trip_and_spec():
    from tiny_llm_b200.config import VigodraConfig, config_from_dict
    for cfg in (VIG_A, VIG_B, VIG_C, VIG_D):
        c = config_from_dict(cfg)
        assert isinstance(c, VigodraConfig) and config_from_dict(c.to_dict()) == c
        spec = c.model_spec()
        assert spec.vocab_size == cfg["vocab"] and spec.hidden_size == cfg["width"] and len(spec.layers) == len(cfg["layers"])
        assert spec.embedding_scale == cfg["embedding"]["scale"] and spec.depth_average == "dwa"
        for layer, src, call in zip(spec.layers, cfg["layers"], spec.order):
            assert layer.block == "post_norm" and layer.stream_scale == cfg["postln_alpha"]
            assert (layer.ffn is None) == (src["mlp"] is None) == (layer.norm2 is None)
            assert call.reads_cache_of == src["mixer"].get("kv_from")
            assert layer.mixer.kind == {"attention": "sink_attention", "latent_attention": "latent_attention"}[src["type"]]
            if layer.ffn is not None:
                assert layer.ffn.params["act"] == "clamped" and layer.ffn.params["limit"] == src["mlp"]["limit"]
    att = config_from_dict(VIG_A).model_spec().layers[0].mixer.params
    assert att["window"] == 20 and att["keep_first"] == 5 and att["conv"] == 4 and att["bias_max"] == 37.0 and att["qk_norm"] == "whole"
    assert config_from_dict(VIG_B).model_spec().layers[3].mixer.params["window"] is None


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(bias_max=0.5), "bias_max"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=2), "keeps no first"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "keeps no latents"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=16), "kv_rank"),
    (lambda c: c["layers"][3]["mixer"].update(rot={"dims": 16, "base": 50.0}), "rot"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown kind"),
    (lambda c: c["layers"][1]["mlp"].update(limit=0), "limit"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_errors_name_the_key(edit, word):
    from tiny_llm_b200.config import ConfigError, config_from_dict
    cfg = copy.deepcopy(VIG_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


def test_tensor_names_and_cache_needs():
    from tiny_llm_b200.cache import KVNeed, StateNeed
    from tiny_llm_b200.config import config_from_dict
    from tiny_llm_b200.parts import DecoderModel
    model = DecoderModel(config_from_dict(VIG_A).model_spec())
    names = model.weight_specs()
    for n in ("embed", "head", "final.norm", "final.norm.b", "l0.norm1", "l0.norm1.b", "l0.norm2", "l0.norm2.b", "l0.mix.q.b",
              "l0.mix.o.b", "l0.mix.q.conv", "l0.mix.v.conv", "l0.mix.k.norm", "l0.mix.rel", "l0.mix.sink", "l1.mix.dkv",
              "l1.mix.dkv.norm", "l1.mix.g", "l3.mix.uk", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down", "l0.dwa", "l3.dwa"):
        assert n in names, n
    for n in ("l3.mix.dkv", "l3.mix.dkv.norm", "l2.norm2", "l2.norm2.b", "l2.mlp.up", "l1.mix.q.b", "l1.mix.sink", "l1.mix.o.b", "l0.mix.g"):
        assert n not in names, n
    assert names["l0.mix.q.norm"].shape == (64,) and names["l0.mix.k.norm"].shape == (32,) and names["l0.mix.v.conv"].shape == (64, 4)
    assert names["l0.mix.rel"].shape == (None, 4) and names["l3.dwa"].shape == (5,) and names["l1.mix.g"].shape == (96, 64)
    needs = model.cache_needs()
    assert needs[0] == (KVNeed(2, 16, 20, value_dim=32, keep_first=5), StateNeed((3, 64 + 32 + 64)))
    assert needs[1] == KVNeed(1, 48, 50, value_dim=32)         # held for the reader, whose window is the longer one
    assert needs[2] == (KVNeed(1, 32, 33, value_dim=16, keep_first=40), StateNeed((2, 128 + 32 + 16))) and needs[3] is None
    assert model.graph_safe
    b = DecoderModel(config_from_dict(VIG_B).model_spec()).cache_needs()
    assert b[0] == KVNeed(1, 28, None, value_dim=18) and b[2] is None
    assert b[3] == KVNeed(2, 12, None, value_dim=14)           # one tap keeps no inputs; no window keeps every key anyway
    assert b[4][0].keep_first == 0
    d = DecoderModel(config_from_dict(VIG_D).model_spec()).cache_needs()
    assert d[1] == KVNeed(1, 80, None, value_dim=64) and d[4] == KVNeed(1, 80, 200, value_dim=48)


def test_a_reader_widens_what_its_owner_holds():
    from tiny_llm_b200.cache import KVNeed
    a = KVNeed(1, 8, 10)
    assert a.reaching(KVNeed(2, 4, 30)).window == 30 and a.reaching(KVNeed(1, 8, 3)) == a
    assert a.reaching(KVNeed(1, 8)) == KVNeed(1, 8) and KVNeed(1, 8).reaching(a) == KVNeed(1, 8)
    assert KVNeed(1, 8, 10, keep_first=4).reaching(KVNeed(1, 8, 5, keep_first=9)).keep_first == 9
    assert KVNeed(1, 8, 10, keep_first=4).reaching(KVNeed(1, 8)).keep_first == 0
    assert KVNeed(1, 8, chunk=16).reaching(KVNeed(1, 8, chunk=16)).chunk == 16
    assert KVNeed(1, 8, chunk=16).reaching(KVNeed(1, 8, chunk=8)).chunk is None


def test_pages_of_kept_positions_stay_until_the_request_ends():
    from tiny_llm_b200.cache import CacheManager, KVNeed
    with pytest.raises(ValueError, match="window"):
        CacheManager([KVNeed(1, 8, keep_first=3)], 64, 4, 2)
    for keep, kept in ((0, 0), (1, 1), (4, 1), (5, 2), (11, 3)):
        cache = CacheManager([KVNeed(1, 8, 6, keep_first=keep)], 64, 4, 2)
        cache.add_request("a")
        for _ in range(10):
            assert cache.reserve("a", 5)
            cache.commit("a", 5)
            cache.check()
            table, n = cache.block_table(0, "a"), cache.kv_len["a"]
            first = max(0, n - 6 + 1) // 4
            assert [i for i, p in enumerate(table) if p >= 0] == sorted(set(range(min(kept, len(table)))) | set(range(first, len(table)))), (keep, n)
        cache.free_request("a")
        cache.check()
        assert all(g.pool.num_used == 0 for g in cache.groups)


def test_the_scheduler_counts_the_kept_pages():
    from tiny_llm_b200.cache import CacheManager, KVNeed
    from tiny_llm_b200.engine.scheduler import Request, RequestRefused, Scheduler
    from tiny_llm_b200.sampling import SamplingParams

    def scheduler(tokens):
        cache = CacheManager([KVNeed(1, 8, 8, keep_first=9)], tokens, 4, 2)
        return Scheduler(cache, 1000, max_tokens_per_step=16, max_requests_per_step=2, chunk=4)
    params = SamplingParams(max_new_tokens=100, do_sample=False)
    # 8 of the window, two pages for its edges, three pages of kept positions
    scheduler(8 + 8 + 12).add(Request("a", [1] * 50, params))
    with pytest.raises(RequestRefused):
        scheduler(8 + 8 + 12 - 4).add(Request("a", [1] * 50, params))


def test_distance_buckets():
    from tiny_llm_b200.parts import distance_buckets
    for buckets, far in [(2, 2), (2, 50), (8, 5), (16, 100), (32, 128), (32, 20.5), (6, 1000), (7, 90), (64, 33)]:
        rows = distance_buckets(buckets, far)
        assert rows[:buckets // 2] == list(range(buckets // 2)) and rows[-1] == buckets - 1
        assert all(b - a in range(0, buckets) for a, b in zip(rows, rows[1:])) and rows == sorted(rows)
        for n in range(3 * int(far) + 5):
            assert rows[min(n, len(rows) - 1)] == pv.distance_bucket(n, buckets, far), (buckets, far, n)
        assert len(rows) <= math.ceil(far) + 1 and (len(rows) == 1 or rows[-2] < buckets - 1)
    # powers: with 8 buckets and a largest distance of 64, distance 4 * 16^(k / 4) = 4, 8, 16, 32, 64
    assert [pv.distance_bucket(n, 8, 64) for n in (3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    for buckets, far in [(1, 10), (8, 4), (8, 3.9)]:
        with pytest.raises(ValueError, match="distance bias"):
            distance_buckets(buckets, far)


def test_parts_refuse_what_they_do_not_have():
    from tiny_llm_b200.config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
    from tiny_llm_b200.parts import DecoderModel, LatentAttention, SinkAttention, SwiGLU
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, key_dim=8, value_dim=8, scale=1.0, eps=1e-5)
    with pytest.raises(ValueError, match="norms per head"):
        SinkAttention(**base, conv=3)
    with pytest.raises(ValueError, match="stretched queries"):
        SinkAttention(**base, qk_norm="whole", stretch_coef=0.5, stretch_every=4)
    with pytest.raises(ValueError, match="mixed scores"):
        SinkAttention(**base, talk=True, bias_max=10.0)
    with pytest.raises(ValueError, match="query/key norm"):
        SinkAttention(**base, qk_norm="row")
    with pytest.raises(ValueError, match="gate"):
        LatentAttention(16, 2, 4, 4, 8, 8, 1.0, 1e-5, gate="row")
    with pytest.raises(ValueError, match="limit"):
        SwiGLU(16, 32, act="clamped")
    norm, mix = PartSpec("layer_norm", {"size": 16, "eps": 1e-5}), PartSpec("sink_attention", base)
    layer = LayerSpec("l0.", norm, mix, block="post_norm")
    spec = dict(architecture="x", vocab_size=8, hidden_size=16, max_positions=8, final_norm=norm, depth_average="dwa")
    with pytest.raises(ValueError, match="depth average"):
        DecoderModel(ModelSpec(layers=[layer], order=[LayerCall(0), LayerCall(0)], **spec))
    with pytest.raises(ValueError, match="post_norm"):
        DecoderModel(ModelSpec(layers=[LayerSpec("l0.", norm, mix, norm2=norm, block="post_norm")], order=[LayerCall(0)], **spec))


def test_plain_pieces_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(3, 10, generator=g, dtype=torch.float64)
    y = pv.layer_norm(x, torch.full((10,), 2.0), torch.full((10,), -1.0), 0.0)
    assert torch.allclose(y.mean(-1), torch.full((3,), -1.0, dtype=torch.float64)) and torch.allclose(y.var(-1, unbiased=False), torch.full((3,), 4.0, dtype=torch.float64))
    assert torch.allclose(pv.layer_norm(x + 7.0, torch.ones(10), torch.zeros(10), 0.0), pv.layer_norm(x, torch.ones(10), torch.zeros(10), 0.0))
    a = [torch.full((2, 2), float(i)) for i in (1, 10, 100)]
    assert torch.equal(pv.depth_average(a, torch.tensor([3.0, 2.0, 1.0])), torch.full((2, 2), 123.0))
    assert pv.short_conv(torch.tensor([[1.0], [2.0], [3.0]]), torch.tensor([[10.0, 1.0]])).flatten().tolist() == [1.0, 12.0, 23.0]
    # a window of 3 that keeps the first two positions
    assert pv.visible(7, 3, 2)[6].tolist() == [True, True, False, False, True, True, True]
    assert pv.visible(7, 3, 2)[3].tolist() == [True, True, True, True, False, False, False]
    assert pv.visible(4, None, 5)[1].tolist() == [True, True, False, False]
    # biases by distance: the same along every diagonal
    rel = torch.randn(4, 2, generator=g)
    b = pv.distance_bias(rel, 9, 6)
    assert torch.equal(b[:, 5, 4], rel[1]) and torch.equal(b[:, 8, 0], rel[3]) and torch.equal(b[:, 3, 3], rel[0]) and torch.equal(b[:, 8, 6], b[:, 4, 2])
    # a sink alone halves a lone key's weight at score 0
    v = torch.ones(1, 1, 1, dtype=torch.float64)
    assert float(pv.masked_softmax_attention(torch.zeros(1, 1, 1, dtype=torch.float64), v, pv.visible(1), torch.zeros(1, dtype=torch.float64))) == pytest.approx(0.5)
    # the rotation keeps lengths, and scores depend on the distance alone
    q, k = torch.randn(1, 1, 12, generator=g, dtype=torch.float64), torch.randn(1, 1, 12, generator=g, dtype=torch.float64)

    def turned(z, p):
        return pv.rotate_halves(z, torch.tensor([p]), 8, 100.0)
    assert torch.allclose(turned(q, 40).norm(), q.norm()) and torch.equal(turned(q, 40)[..., 8:], q[..., 8:])
    assert torch.allclose((turned(q, 40) * turned(k, 33)).sum(), (turned(q, 107) * turned(k, 100)).sum())
    assert torch.allclose(turned(q, 1)[..., 0], q[..., 0] * math.cos(1.0) - q[..., 4] * math.sin(1.0))
    # the clamped gate: linear in u inside the limits, flat outside, the gate side bounded above only
    assert float(pv.clamped_glu(torch.tensor(100.0), torch.tensor(-100.0), 2.0)) == pytest.approx(2.0 / (1 + math.exp(-3.404)) * -1.0)
    assert float(pv.clamped_glu(torch.tensor(-3.0), torch.tensor(0.5), 2.0)) == pytest.approx(-3.0 / (1 + math.exp(5.106)) * 1.5)
