"""Host side of the Pekunex path (no GPU): configuration reader and registry, borrowed weights, checkpoint tensor names and shapes, merged
projections, rotation tables, and a few properties of the plain implementation the GPU tests lean on."""
import json
import math

import pytest
import torch

import pekunex_helpers as ph
from oracle import pekunex_ref as ref

ALL = [ph.config_a(), ph.config_b(), ph.config_c(), ph.config_d()]


def _model(cfg):
    from nanovllm.models.pekunex import PekunexConfig, PekunexForCausalLM
    return PekunexForCausalLM(PekunexConfig(cfg), device="cpu", max_position=64)


def test_registry_reads_the_configuration(tmp_path):
    from nanovllm.models.pekunex import PekunexConfig, PekunexForCausalLM
    from nanovllm.models.registry import model_class, read_config
    (tmp_path / "config.json").write_text(json.dumps(ph.config_a()))
    c = read_config(str(tmp_path))
    assert isinstance(c, PekunexConfig) and model_class(c) is PekunexForCausalLM
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embed_scale, c.logit_scale) == (97, 64, 2e-5, 2.5, 1.5)
    assert c.runs == [(0, 0), (1, 0), (2, 0), (0, 1), (1, 1), (5, 0), (2, 1)] and c.copies == {0: 2, 1: 2, 2: 2, 5: 1}
    b = PekunexConfig(ph.config_b())
    assert b.embed_scale == 1.0 and b.logit_scale == 1.0


def test_borrowers_of_borrowers_end_at_the_owner():
    from nanovllm.models.pekunex import PekunexConfig
    cfg = ph.config_a()
    cfg["layers"].append(dict(cfg["layers"][3], weights_of=3))
    c = PekunexConfig(cfg)
    assert c.runs[-1] == (0, 2) and c.copies[0] == 3
    assert len({r for r in c.runs}) == len(c.runs)                     # every run has a cache or state of its own


def test_bad_configurations_are_refused():
    from nanovllm.models.pekunex import PekunexConfig
    for key, bad in (("type", "lstm"), ("mlp", {"kind": "moe"}), ("weights_of", 9), ("weights_of", 1), ("weights_of", 0)):
        cfg = ph.config_a()
        cfg["layers"][1][key] = bad
        with pytest.raises(ValueError):
            PekunexConfig(cfg)
    for layer, path, bad in ((2, ("rot", "dims"), 21), (2, ("kv_heads",), 3), (0, ("groups",), 4), (0, ("norm_groups",), 7), (0, ("state",), 257),
                             (1, ("right", "dim"), 300)):
        cfg = json.loads(json.dumps(ph.config_a()))
        at = cfg["layers"][layer]["mixer"]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = bad
        with pytest.raises(ValueError):
            _model(cfg)


@pytest.mark.parametrize("cfg", ALL)
def test_checkpoint_tensors(cfg, tmp_path):
    from nanovllm.utils.loader import load_model
    m = _model(cfg)
    W = ph.random_weights(cfg, 1)
    ph.write_checkpoint(str(tmp_path), cfg, W)
    assert load_model(m, str(tmp_path)) == len(W)
    assert {k: tuple(v) for k, v in m.weight_shapes().items()} == ph.shapes(cfg)
    for bad in ("l0.mix.nothing", "l99.norm1", "l0.mlp.nothing", "bias", "l0.norm3"):
        with pytest.raises(KeyError):
            m.load_hf_tensor(bad, torch.zeros(1))
    assert m.state_slot_bytes() == sum(b.mixer.state_slot_bytes() * m.cfg.copies[i] for i, b in m.blocks.items())
    assert m.has_recurrent_state == any(l["type"] != "attention" for l in cfg["layers"]) and m.supports_prefix_cache != m.has_recurrent_state


def test_a_borrowing_layer_holds_no_tensors():
    m = _model(ph.config_a())
    assert sorted(m.blocks) == [0, 1, 2, 5]
    with pytest.raises(KeyError):
        m.load_hf_tensor("l3.norm1", torch.zeros(64))


@pytest.mark.parametrize("cfg", [ph.config_a(), ph.config_b(), ph.config_c()])
def test_merged_projections_hold_every_part(cfg):
    m = _model(cfg)
    W = ph.random_weights(cfg, 2)
    for k, v in W.items():
        m.load_hf_tensor(k, v)
    h = torch.randn(3, cfg["width"], dtype=torch.float64)
    f64 = lambda name: W[name].double()
    for i, b in m.blocks.items():
        mix, p, kind = b.mixer, f"l{i}.mix.", cfg["layers"][i]["type"]
        proj = h @ mix.w_in.double().T
        assert mix.w_in.shape[0] % 8 == 0
        if mix.__class__.__name__ == "CappedGatedAttention":
            proj = proj + mix.b_in.double()
            at = 0
            for leaf in ("q", "k", "v", "g"):
                want = h @ f64(p + leaf).T + (f64(p + leaf + ".b") if leaf != "g" else 0.0)
                assert torch.allclose(proj[:, at:at + want.shape[1]], want), (i, leaf)
                at += want.shape[1]
            assert at == mix.in_cols and not mix.w_in[at:].any()
        elif kind == "parallel":
            (li, start, stop), lo = mix.split_in, mix.split_out
            assert start % 8 == 0 and mix.b_in is None
            assert torch.allclose(proj[:, :li], torch.cat([h @ f64(p + "left." + x).T for x in "qkv"], 1))
            assert torch.allclose(proj[:, start:stop], torch.cat([h @ f64(p + "right." + x).T for x in "qkvg"], 1))
            assert torch.equal(mix.w_o, torch.cat([W[p + "left.o"], W[p + "right.o"]], 1)) and lo == W[p + "left.o"].shape[1]
            assert torch.equal(mix.right.w_if, torch.cat([W[p + "right.i"], W[p + "right.f"]], 0))
            assert torch.equal(mix.right.b_if, torch.cat([W[p + "right.i.b"], W[p + "right.f.b"]]).float())
            assert torch.equal(mix.left.sinks, W[p + "left.sink"].float())
        else:
            assert torch.allclose(proj[:, :mix.in_cols], h @ f64(p + "in").T)
            assert torch.allclose(mix.rate, -torch.exp(W[p + "A_log"].float())) and torch.equal(mix.D, W[p + "D"].float())
        if b.ff is not None:
            assert torch.equal(b.ff.w_gate_up, torch.cat([W[f"l{i}.mlp.gate"], W[f"l{i}.mlp.up"]]))


@pytest.mark.parametrize("dims,base", [(12, 900.0), (32, 10000.0), (64, 250.0), (2, 50.0)])
def test_rotation_tables(dims, base):
    """Both frequency scalings against the plain formulas, at positions up to the thousands; the configurations reach all three kinds of pairs."""
    from nanovllm.layers.rotary_embedding import build_scaled_cos_sin
    for sc, plain in ((ph.RAMP, ref.ramp_frequencies), (ph.BANDS, ref.banded_frequencies), (None, ref.banded_frequencies)):
        got = build_scaled_cos_sin(dims, 3000, base, sc)
        freq, mag = plain(dims, base, sc) if plain is ref.ramp_frequencies else (plain(dims, base, sc), 1.0)
        pos = torch.tensor([0, 1, 7, 500, 2999])
        ang = pos[:, None].double() * torch.tensor(freq, dtype=torch.float64)
        want = torch.cat([ang.cos(), ang.sin()], 1) * mag
        assert (got[pos].double() - want).abs().max().item() < 1e-6
    f0 = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if dims == 64:
        for plain, factor in ((lambda *a: ref.ramp_frequencies(*a)[0], 5.0), (ref.banded_frequencies, 3.0)):
            sc = ph.RAMP if factor == 5.0 else ph.BANDS
            ratio = [a / b for a, b in zip(plain(dims, base, sc), f0)]
            assert max(ratio) == 1.0 and abs(min(ratio) - 1.0 / factor) < 1e-12 and any(1.001 / factor < r < 0.999 for r in ratio)


def test_plain_implementation_is_causal_and_its_pieces_are_exact():
    cfg = ph.config_a()
    W = ph.random_weights(cfg, 5)
    toks = ph.tokens(40, cfg["vocab"], 1)
    full = ref.forward(cfg, W, toks)
    assert torch.allclose(ref.forward(cfg, W, toks[:23]), full[:23], atol=1e-9)
    p = ref.causal_softmax(torch.zeros(3, 3, dtype=torch.float64), 0.0)
    assert torch.allclose(p[2], torch.tensor([0.25, 0.25, 0.25], dtype=torch.float64)) and p[0].tolist() == [0.5, 0.0, 0.0]
    # the memory cell's maximum starts at zero: with both gates far below it, the read-out is divided by exp(-m), not by |n . q|
    q, k, v = torch.ones(1, 1), torch.ones(1, 1), torch.full((1, 1), 2.0)
    o = ref.memory_cell(q.double(), k.double(), v.double(), torch.tensor([-3.0]), torch.tensor([-1.0]))
    assert abs(o.item() - 2.0 * math.exp(-2.0) / (math.exp(1.0) + 1e-6)) < 1e-9
    # a state-space step with a huge rate forgets everything but the token itself
    x = torch.randn(4, 3, dtype=torch.float64)
    y = ref.state_space(x, torch.ones(4, 2, dtype=torch.float64), torch.ones(4, 2, dtype=torch.float64), torch.ones(4), 6.0)
    assert torch.allclose(y, 2.0 * x, atol=1e-9)
