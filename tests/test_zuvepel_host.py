"""Host side of the Zuvepel path (no GPU): configuration reader and registry, execution order of repeated layers, checkpoint
tensor names, shapes and ranks, and a few properties of the plain implementation the GPU tests lean on."""
import json
import math

import pytest
import torch

import zuvepel_helpers as zh
from oracle import zuvepel_ref as ref

ALL = [zh.config_a(), zh.config_b(), zh.config_c(), zh.config_d()]


def _model(cfg):
    from nanovllm.models.zuvepel import ZuvepelConfig, ZuvepelForCausalLM
    return ZuvepelForCausalLM(ZuvepelConfig(cfg), device="cpu", max_position=64)


def test_registry_reads_the_configuration(tmp_path):
    from nanovllm.models.registry import model_class, read_config
    from nanovllm.models.zuvepel import ZuvepelConfig, ZuvepelForCausalLM
    (tmp_path / "config.json").write_text(json.dumps(zh.config_a()))
    c = read_config(str(tmp_path))
    assert isinstance(c, ZuvepelConfig) and model_class(c) is ZuvepelForCausalLM
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embed_scale, c.residual_mult) == (97, 64, 2e-5, 3.5, 0.45)
    assert c.num_hidden_layers == 5 and [c.passes_of(i) for i in range(5)] == [1, 3, 3, 3, 1]
    b = ZuvepelConfig(zh.config_b())
    assert b.embed_scale == 1.0 and b.residual_mult == 1.0
    assert ZuvepelConfig(zh.config_c()).loop is None


@pytest.mark.parametrize("cfg", ALL)
def test_execution_order_of_repeated_layers(cfg):
    from nanovllm.models.zuvepel import ZuvepelConfig
    runs = ZuvepelConfig(cfg).runs
    assert [(i, add) for i, _, add in runs] == ref.layer_runs(cfg)
    assert len({(i, k) for i, k, _ in runs}) == len(runs)              # each pass has a cache and state of its own
    assert not runs[0][2]                                              # the first pass adds nothing, wherever the loop starts


def test_bad_configurations_are_refused():
    from nanovllm.models.zuvepel import ZuvepelConfig
    for key, bad in (("type", "lstm"), ("mlp", {"kind": "moe"})):
        cfg = zh.config_a()
        cfg["layers"][1][key] = bad
        with pytest.raises(ValueError):
            ZuvepelConfig(cfg)
    cfg = zh.config_a()
    cfg["layers"][1]["mixer"]["rot"]["dims"] = 18
    with pytest.raises(ValueError):
        _model(cfg)
    cfg = zh.config_a()
    cfg["layers"][2]["mixer"]["kv_heads"] = 3
    with pytest.raises(ValueError):
        _model(cfg)


@pytest.mark.parametrize("cfg", ALL)
@pytest.mark.parametrize("ranks", [{}, {"a1": 8, "g1": 24}, {"a1": 1, "g1": 3}])
def test_checkpoint_tensors_and_ranks_from_their_shapes(cfg, ranks, tmp_path):
    from nanovllm.utils.loader import load_model
    m = _model(cfg)
    W = zh.random_weights(cfg, 1, ranks)
    zh.write_checkpoint(str(tmp_path), cfg, W)
    assert load_model(m, str(tmp_path)) == len(W)
    assert {k: tuple(v) for k, v in m.weight_shapes().items()} == zh.shapes(cfg, ranks)
    with pytest.raises(KeyError):
        m.load_hf_tensor("l0.mix.nothing", torch.zeros(1))
    with pytest.raises(KeyError):
        m.load_hf_tensor("l99.norm1", torch.zeros(1))
    assert m.state_slot_bytes() == sum(b.branches.mixer.state_slot_bytes() * b.passes for b in m.blocks)
    assert m.has_recurrent_state == any(l["type"] != "attention" for l in cfg["layers"]) and m.supports_prefix_cache != m.has_recurrent_state


def test_merged_projections_hold_every_part():
    """The input projection's parts, its zero padding and the merged output projection, on the CPU: every low-rank map and branch
    comes out as its own matrices give."""
    cfg = zh.config_a()
    m = _model(cfg)
    W = zh.random_weights(cfg, 2)
    m.declare_shapes({k: tuple(v.shape) for k, v in W.items()})
    for k, v in W.items():
        m.load_hf_tensor(k, v)
    h = torch.randn(3, cfg["width"], dtype=torch.float64)
    f64 = lambda t: t.double()
    for i, p in ((0, "l0."), (2, "l2."), (3, "l3.")):
        mix = m.blocks[i].branches.mixer
        proj = h @ f64(mix.w_in).T
        for leaf in [l for l, _ in mix.parts()] + [l for l, _ in mix.low_rank()]:
            assert torch.allclose(mix._cols(proj, leaf), h @ f64(W[p + "mix." + leaf]).T), (i, leaf)
        for leaf, _ in mix.low_rank():
            a, second = mix.at[leaf][0], mix.second[leaf[:-1] + "2"]
            want = (h @ f64(W[p + "mix." + leaf]).T) @ f64(W[p + "mix." + leaf[:-1] + "2"]).T
            assert torch.allclose(proj[:, a:a + second.shape[1]] @ f64(second).T, want), (i, leaf)
    att = m.blocks[1].branches.mixer
    q = cfg["layers"][1]["mixer"]["heads"] * cfg["layers"][1]["mixer"]["dim"]
    assert torch.equal(att.w_in[:q], W["l1.mix.q"]) and torch.equal(att.w_in[att.g_off:att.g_off + att.heads], W["l1.mix.g"])
    assert att.in_cols % 8 == 0 and not att.w_in[att.g_off + att.heads:].any() and not att.b_in[att.g_off:].any() and not att.sinks.any()
    assert torch.equal(m.blocks[1].branches.w_out, torch.cat([W["l1.mix.o"], W["l1.mlp.down"]], 1))
    assert torch.equal(m.blocks[2].branches.w_out, W["l2.mix.o"]) and m.blocks[2].branches.ff is None
    assert torch.allclose(m.blocks[2].branches.mixer.rate, -torch.exp(W["l2.mix.A_log"].float()))
    assert torch.allclose(m.blocks[3].branches.mixer.rate, torch.full((2,), -1.0 / 16.0))


def test_decay_forms_agree():
    """exp(rate softplus(sign (z + b))) is both decays: exp(-exp(A) softplus(z + b)) and sigmoid(z + b)^(1 / tau)."""
    z = torch.linspace(-12, 12, 101, dtype=torch.float64)
    sp = torch.nn.functional.softplus
    assert torch.allclose(torch.exp(-(1 / 7.0) * sp(-z)), torch.sigmoid(z) ** (1 / 7.0))
    assert torch.allclose(torch.exp(-math.exp(0.3) * sp(z)), torch.exp(-torch.exp(torch.tensor(0.3, dtype=torch.float64)) * sp(z)))


def test_plain_implementation_is_causal_and_chunks_are_exact():
    cfg = zh.config_a()
    W = zh.random_weights(cfg, 5)
    toks = zh.tokens(40, cfg["vocab"], 1)
    full = ref.forward(cfg, W, toks)
    assert torch.allclose(ref.forward(cfg, W, toks[:23]), full[:23], atol=1e-9)
    see = ref.same_chunk(12, 4)
    assert see[9].tolist() == [False] * 8 + [True, True, False, False] and see[8].tolist() == [False] * 8 + [True] + [False] * 3
    assert see[7].tolist() == [False] * 4 + [True] * 4 + [False] * 4
    p = ref.sink_softmax(torch.tensor([[0.0, 50.0]], dtype=torch.float64), torch.tensor([[True, False]]))
    assert torch.allclose(p, torch.tensor([[0.5, 0.0]], dtype=torch.float64))      # one visible key of score 0 beside the sink
    p = ref.sink_softmax(torch.tensor([[-3.0, -4.0]], dtype=torch.float64), torch.tensor([[True, True]]))
    e = [math.exp(-3.0), math.exp(-4.0)]
    assert torch.allclose(p, torch.tensor([[e[0] / (1 + sum(e)), e[1] / (1 + sum(e))]], dtype=torch.float64))
