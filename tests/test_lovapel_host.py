"""Lovapel on the host: configuration and its errors, the run order of a repeated span, tensor names, cache needs, what the
parts refuse, the norm handed ahead, and the plain implementation against closed forms."""
import copy
import math
from types import SimpleNamespace

import pytest
import torch

import plain_lovapel as pl
from lovapel_util import LOV_A, LOV_B, LOV_C, LOV_D, separate_corrections


def test_configuration_round_trip_and_spec():
    from tiny_llm_b200.config import LovapelConfig, config_from_dict
    for cfg in (LOV_A, LOV_B, LOV_C, LOV_D):
        c = config_from_dict(cfg)
        assert isinstance(c, LovapelConfig) and config_from_dict(c.to_dict()) == c
        spec = c.model_spec()
        assert spec.vocab_size == cfg["vocab"] and spec.hidden_size == cfg["width"] and len(spec.layers) == len(cfg["layers"])
        assert spec.tie_word_embeddings and spec.embedding_scale == 1.0
        assert [call.layer for call in spec.order] == pl.layer_order(cfg)
        assert all(call.reads_cache_of is None and not call.add_embedding for call in spec.order)
        for layer, src in zip(spec.layers, cfg["layers"]):
            assert layer.block == "sandwich_norm" and (layer.ffn is None) == (src["mlp"] is None) == (layer.norm2 is None)
            p, m = layer.mixer.params, src["mixer"]
            assert layer.mixer.kind == "sink_attention" and p["qk_norm"] == "whole" and p["sink"] and not p["bias"] and not p["gate"]
            assert p["window"] == (m.get("mask") or {}).get("size") and p["rot_dims"] == (m.get("rot") or {}).get("dims", 0)
            if src["mlp"] is not None and src["mlp"]["kind"] == "dense":
                assert layer.ffn.params["act"] == "gelu_tanh"
    a = config_from_dict(LOV_A).model_spec()
    assert a.on_logits.params == {"scale": 1.5, "cap": 8.0} and config_from_dict(LOV_C).model_spec().on_logits is None
    assert config_from_dict(LOV_D).model_spec().on_logits.params == {"scale": 1.0, "cap": 20.0}
    r = a.layers[1].ffn.params
    assert (r["num_experts"], r["identity"], r["groups"], r["keep"], r["top"], r["shared_size"], r["renorm"]) == (10, 2, 3, 2, 3, 24, True)
    assert config_from_dict(LOV_B).model_spec().layers[0].ffn.params["groups"] == 1
    nulls = copy.deepcopy(LOV_C)     # null switches a mechanism off just as leaving the key out does
    nulls.update(loop=None, logit_scale=None, logit_softcap=None)
    nulls["layers"][0]["mixer"].update(mask=None, rot=None)
    nulls["layers"][1]["mlp"].update(shared=None)
    nulls["layers"][1]["mlp"]["router"].update(groups=None)
    assert config_from_dict(nulls).model_spec() == config_from_dict(LOV_C).model_spec()


def test_a_repeated_span_runs_in_order():
    from tiny_llm_b200.config import config_from_dict
    assert [c.layer for c in config_from_dict(LOV_A).run_order()] == [0, 1, 2, 1, 2]
    assert [c.layer for c in config_from_dict(LOV_B).run_order()] == [0, 1, 2, 2, 2]
    assert [c.layer for c in config_from_dict(LOV_C).run_order()] == [0, 1, 2]
    assert [c.layer for c in config_from_dict(LOV_D).run_order()] == [0, 1, 0, 1, 2, 3]


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=-1), "base"),
    (lambda c: c["layers"][1]["mlp"].update(kind="soft"), "unknown kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=3), "divide"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "ff"),
    (lambda c: c["loop"].update(stop=4), "span"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c.update(logit_scale="big"), "logit_scale"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_errors_name_the_key(edit, word):
    from tiny_llm_b200.config import ConfigError, config_from_dict
    cfg = copy.deepcopy(LOV_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


def test_tensor_names_and_cache_needs():
    from tiny_llm_b200.cache import KVNeed
    from tiny_llm_b200.config import config_from_dict
    from tiny_llm_b200.parts import DecoderModel
    model = DecoderModel(config_from_dict(LOV_A).model_spec())
    names = model.weight_specs()
    for n in ("embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.q", "l0.mix.k.norm", "l0.mix.sink",
              "l0.mix.o", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down", "l1.mlp.router", "l1.mlp.correction", "l1.mlp.e9.gate",
              "l1.mlp.e9.down", "l1.mlp.shared.gate", "l1.mlp.shared.up", "l1.mlp.shared.down"):
        assert n in names, n
    for n in ("head", "final.norm.b", "l0.norm1.b", "l0.mix.q.b", "l0.mix.g", "l1.mlp.e10.gate", "l1.mlp.shared.sg",
              "l2.mlp.shared.gate"):
        assert n not in names, n
    assert names["l0.mix.q.norm"].shape == (64,) and names["l0.mix.k.norm"].shape == (32,)
    assert names["l1.mlp.router"].shape == (12, 64) and names["l1.mlp.correction"].shape == (12,)
    # every pass of a repeated layer keeps keys of its own
    assert model.cache_needs() == [KVNeed(2, 16, 20, value_dim=32), KVNeed(1, 32, 37, value_dim=16), KVNeed(6, 16, None, value_dim=16),
                                   KVNeed(1, 32, 37, value_dim=16), KVNeed(6, 16, None, value_dim=16)]
    assert model.graph_safe
    b = DecoderModel(config_from_dict(LOV_B).model_spec()).weight_specs()
    assert "l1.norm2" not in b and "l1.norm2b" not in b and "l1.norm1b" in b


def test_parts_refuse_what_they_do_not_have():
    from tiny_llm_b200.parts import RoutedExperts, SoftCap
    with pytest.raises(ValueError, match="chosen"):
        RoutedExperts(16, 6, 5, 8, groups=3, keep=2)
    with pytest.raises(ValueError, match="chosen"):
        RoutedExperts(16, 6, 2, 8, groups=4)
    with pytest.raises(ValueError, match="chosen"):
        RoutedExperts(16, 2, 4, 8, identity=1)
    RoutedExperts(16, 2, 3, 8, identity=1)
    with pytest.raises(ValueError, match="shared"):
        RoutedExperts(16, 4, 2, 8, glu="silu", shared_size=8)
    with pytest.raises(ValueError, match="shared"):
        RoutedExperts(16, 4, 2, 8, shared_size=8, shared_gate=False)
    with pytest.raises(ValueError, match="cap"):
        SoftCap(cap=0.0)


class _Norm:
    def __init__(self, name, log, takes):
        self.name, self.log, self.takes = name, log, takes

    def forward(self, ctx, x, rows=None):
        self.log.append(self.name)
        return (self.name, x)[1]

    def add_into(self, ctx, branch, resid, copy=None, then=None):
        self.log.append(self.name + ("+" + then.name if then is not None and self.takes else ""))
        return resid if then is not None and self.takes else None


@pytest.mark.parametrize("takes", [False, True])
def test_a_sandwich_block_takes_the_next_norm_along(takes):
    """Whoever reads the stream next has its norm taken in the kernel that wrote the stream, if that kernel can; a stream
    at another address, of another length or ahead of another norm is normed again."""
    from tiny_llm_b200.config.spec import LayerSpec, PartSpec
    from tiny_llm_b200.parts import SandwichBlock
    norm = PartSpec("layer_norm", {"size": 8, "eps": 1e-5, "has_bias": False})
    spec = LayerSpec("l.", norm, PartSpec("sink_attention", dict(hidden_size=8, num_heads=1, num_kv_heads=1, key_dim=8, value_dim=8,
                                                                 scale=1.0, eps=1e-5)), norm2=norm, ffn=PartSpec("swiglu", {"hidden_size": 8, "intermediate_size": 8}),
                     block="sandwich_norm", more=(("norm1_out", "norm", norm, "a"), ("norm2_out", "norm", norm, "b")))
    log, block = [], SandwichBlock(spec)
    for role in ("norm1", "norm1_out", "norm2", "norm2_out"):
        setattr(block, role, _Norm(role, log, takes))
    block.first_norm = block.norm1
    part = SimpleNamespace(forward=lambda *a: log.append("branch"))
    block.mixer = block.ffn = part
    buf = torch.zeros(3, 8)
    ctx = SimpleNamespace(workspace=SimpleNamespace(get_zeroed=lambda name, shape: torch.zeros(shape)), next_norm=block.norm1, norm_ahead=None)
    block.forward(ctx, buf, None)
    first = ["norm1", "branch", "norm1_out+norm2", "branch", "norm2_out+norm1"] if takes else \
        ["norm1", "branch", "norm1_out", "norm2", "branch", "norm2_out"]
    assert log == first
    log.clear()
    block.forward(ctx, buf, None)
    assert log == (first[1:] if takes else first)
    ctx.next_norm = None                     # the last layer: nothing reads on
    log.clear()
    block.forward(ctx, buf, None)
    assert log == (["branch", "norm1_out+norm2", "branch", "norm2_out"] if takes else first) and ctx.norm_ahead is None
    for other in ((0, block.norm1, buf), (buf.data_ptr(), block.norm2, buf), (buf.data_ptr(), block.norm1, torch.zeros(2, 8))):
        ctx.norm_ahead = other
        log.clear()
        block.forward(ctx, buf, None)
        assert log[0] == "norm1"


def test_plain_pieces_against_closed_forms():
    x = torch.tensor([[1.0, -1.0, 3.0, -3.0]], dtype=torch.float64)
    assert torch.allclose(pl.layer_norm(x + 5.0, torch.ones(4), 0.0), x / math.sqrt(5.0))
    assert torch.allclose(pl.rms_norm(x, torch.full((4,), 2.0), 4.0), 2.0 * x / 3.0)
    z = torch.linspace(-4, 4, 41, dtype=torch.float64)
    assert torch.allclose(pl.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    v = torch.zeros(1, 1, 6, dtype=torch.float64)
    v[0, 0, 0] = v[0, 0, 5] = 1.0
    r = pl.rotate_halves(v, torch.tensor([3]), 4, 10.0)[0, 0]      # value 0 turns with value 2, value 5 passes
    assert torch.allclose(r, torch.tensor([math.cos(3.0), 0, math.sin(3.0), 0, 0, 1.0], dtype=torch.float64))
    # one visible key against a sink of the same score shares the weight in halves; the key before the window counts nothing
    q = torch.ones(1, 1, 1, dtype=torch.float64)
    k, val = torch.tensor([[[50.0]], [[2.0]]], dtype=torch.float64), torch.tensor([[[7.0]], [[1.0]]], dtype=torch.float64)
    o = pl.window_sink_attention(q, k, val, torch.tensor([1]), torch.tensor([0, 1]), 0.5, torch.tensor([1.0]), 1)
    assert torch.allclose(o, torch.full_like(o, 0.5))
    assert float(pl.window_sink_attention(q, k, val, torch.tensor([1]), torch.tensor([0, 1]), 0.5, torch.tensor([1.0]), 2)) > 6.9


def test_plain_router_by_hand():
    s = torch.tensor([0.3, 0.1, 0.25, 0.05, 0.2, 0.1], dtype=torch.float64)
    z = s.log()[None]
    none = torch.zeros(6, dtype=torch.float64)
    ids, w = pl.route(z, none, 2)
    assert ids.tolist() == [[0, 2]] and torch.allclose(w, torch.tensor([[0.3, 0.25]], dtype=torch.float64) / 0.55)
    ids, w = pl.route(z, none, 3, 3, 2)          # groups {0, 1}, {2, 3}, {4, 5}: worth 0.3, 0.25, 0.2
    assert ids.tolist() == [[0, 2, 1]]
    corr = torch.tensor([-0.9, -0.9, -0.5, -0.6, -0.8, -0.1], dtype=torch.float64)   # all choice scores negative but one
    ids, w = pl.route(z, corr, 2, 3, 1)          # the last group is worth 0.0; its members are chosen, nobody else
    assert ids.tolist() == [[5, 4]] and torch.allclose(w, torch.tensor([[1 / 3, 2 / 3]], dtype=torch.float64))
    ids, w = pl.route(z, corr, 4, 3, 2)
    assert ids.tolist() == [[5, 2, 3, 4]]


def test_separate_corrections_fix_the_choice():
    w = separate_corrections({"l.correction": torch.zeros(7), "x": torch.ones(2)}, 3)
    c = w["l.correction"]
    assert torch.equal(w["x"], torch.ones(2)) and float((c.sort().values[1:] - c.sort().values[:-1]).min()) == 1.5
    g = torch.Generator().manual_seed(1)
    ids, _ = pl.route(torch.randn(50, 7, generator=g) * 3, c, 3)
    assert (ids == ids[0]).all()
