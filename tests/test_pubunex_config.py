"""Pubunex without a GPU: the configuration reader and its errors, the lowering to part specs
and a run order, tensor names and the loader, what the cache is asked for, and the plain
implementation's mechanisms on cases worked out by hand."""
import copy
import json
import math

import pytest
import torch

from agave_b200.config import ConfigError, load_config, resolve_architecture
from agave_b200.config.base import (AttentionSpec, ClampedGateSpec, HeadDeltaSpec,
                                    LatentAttentionSpec, LayerCall, NormSpec, ParallelBlockSpec,
                                    RoutedFeedForwardSpec, WavelengthScalingSpec, looped_schedule)
from agave_b200.config.pubunex import PubunexConfig
from agave_b200.models.decoder import DecoderModel, decoder_param_specs
from agave_b200.weights import WeightsError, load_weights
from plain import pubunex_plain as P
from pubunex_util import CONFIGS, folder_for, make_tensors

F64 = torch.float64


# ------------------------------------------------------------------- reading
def test_registry_finds_the_architecture():
    assert resolve_architecture({"architecture": "Pubunex"}).name == "Pubunex"
    assert resolve_architecture({"model_type": "pubunex"}).name == "Pubunex"


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_reading_and_writing_round_trip(name):
    cfg = PubunexConfig.from_dict(CONFIGS[name])
    assert PubunexConfig.from_dict(cfg.to_dict()) == cfg
    assert len(cfg.layers) == len(CONFIGS[name]["layers"])


def test_what_may_be_absent_reads_as_none():
    cfg = PubunexConfig.from_dict(CONFIGS["P3"])
    assert cfg.loop is None and cfg.layers[1].mixer.rot is None
    assert cfg.layers[3].mixer.rot.scaling is None and cfg.layers[3].mlp is None
    assert cfg.layers[0].mlp.shared is None
    raw = copy.deepcopy(CONFIGS["P3"])
    del raw["layers"][2]["mlp"], raw["layers"][1]["mixer"]["kv_heads"]
    cfg = PubunexConfig.from_dict(raw)
    assert cfg.layers[2].mlp is None and cfg.layers[1].mixer.kv_heads == 2


@pytest.mark.parametrize("path, value, match", [
    (("vocab",), None, "vocab"),
    (("width",), 0, "positive"),
    (("norm", "eps"), None, "norm.eps"),
    (("layers", 0, "type"), "conv", "not a mixer"),
    (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "scale"), None, "mixer.scale"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), 12, "rot.dims"),
    (("layers", 0, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 0, "mixer", "rot", "scaling", "fast"), None, "scaling.fast"),
    (("layers", 0, "mixer", "rot", "scaling", "original"), 0, "scaling.original"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "conv"), 2.5, "integer"),
    (("layers", 1, "mixer", "dim"), None, "mixer.dim"),
    (("layers", 2, "mixer", "kv_rank"), 0, "kv_rank"),
    (("layers", 2, "mixer", "rot"), None, "mixer.rot"),
    (("layers", 2, "mixer", "rot", "dims"), 2, "rot_dim"),
    (("layers", 0, "mlp", "kind"), "dense", "not a feed-forward"),
    (("layers", 0, "mlp", "router", "top"), 6, "router.top"),
    (("layers", 0, "mlp", "router", "experts"), None, "router.experts"),
    (("layers", 0, "mlp", "expert", "limit"), None, "expert.limit"),
    (("layers", 0, "mlp", "expert", "ff"), 0, "expert.ff"),
    (("layers", 0, "mlp", "shared", "limit"), -1.0, "shared.limit"),
    (("loop", "stop"), 1, "loop"),
    (("loop", "stop"), 6, "loop"),
    (("loop", "times"), 0, "loop"),
    (("loop", "start"), None, "loop.start"),
])
def test_errors_name_the_key(path, value, match):
    raw = copy.deepcopy(CONFIGS["P1"])
    d = raw
    for k in path[:-1]:
        d = d[k]
    if value is None:
        del d[path[-1]]
    else:
        d[path[-1]] = value
    with pytest.raises(ConfigError, match=match):
        PubunexConfig.from_dict(raw)


# ------------------------------------------------------------------ lowering
def test_lowering_to_parts():
    spec = PubunexConfig.from_dict(CONFIGS["P1"]).to_model_spec()
    assert len(spec.blocks) == 5 and not spec.tie_embeddings and spec.embed_scale == 1.0
    norm = NormSpec(eps=1e-5, zero_centered=True)
    assert spec.final_norm == norm
    for b in spec.blocks:
        assert isinstance(b, ParallelBlockSpec) and not b.gated and b.norm == norm
    b0, b1, b2, b3, b4 = spec.blocks
    a = b0.mixer
    assert isinstance(a, AttentionSpec)
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.scale, a.window, a.chunk) == \
        (4, 2, 10, 14, 0.4, None, None)
    assert a.qkv_bias and a.out_bias and not a.sink and a.qk_norm is None
    assert (a.position.theta, a.position.rotary_dim, a.position.interleaved) == (1000.0, 6, False)
    assert a.position.scaling == WavelengthScalingSpec(factor=8.0, original=64.0, fast=4.0, slow=0.5)
    assert b1.mixer == HeadDeltaSpec(n_heads=4, n_qk_heads=2, head_dim=10, value_dim=14,
                                     conv_taps=3, eps=1e-5, unit_eps=1e-6, gate_activation="silu")
    m = b2.mixer
    assert isinstance(m, LatentAttentionSpec)
    assert (m.n_heads, m.head_dim, m.rot_dim, m.value_dim, m.kv_rank, m.q_rank, m.scale, m.eps,
            m.gate, m.sink) == (3, 10, 4, 6, 20, 0, 0.35, 1e-5, None, True)
    assert m.position.interleaved and m.position.theta == 10000.0 and m.position.scaling is None
    assert b2.feed_forward is None and b4.feed_forward.shared_size == 0
    f = b0.feed_forward
    assert isinstance(f, RoutedFeedForwardSpec)
    assert (f.n_experts, f.top, f.intermediate_size, f.weighting, f.correction, f.weigh_input,
            f.shared_size, f.shared_gate, f.n_groups, f.route_scale) == \
        (5, 2, 24, "sigmoid", False, True, 20, False, 1, 1.0)
    assert f.activation == ClampedGateSpec(limit=0.8, alpha=1.702)
    assert f.shared_activation == ClampedGateSpec(limit=2.5, alpha=1.702)
    # a rotation of the whole head is written as such
    p3 = PubunexConfig.from_dict(CONFIGS["P3"]).to_model_spec()
    assert p3.blocks[3].mixer.position.rotary_dim == 0 and p3.blocks[1].mixer.position is None


def _order(name):
    return [(c.block, c.add_embedding) for c in
            PubunexConfig.from_dict(CONFIGS[name]).to_model_spec().schedule]


def test_run_order():
    assert _order("P1") == [(0, False), (1, False), (2, False), (3, False), (1, True), (2, False),
                            (3, False), (1, True), (2, False), (3, False), (4, False)]
    assert _order("P3") == [(i, False) for i in range(5)]
    assert _order("P5") == [(0, False), (1, False), (1, True), (1, True), (1, True)]
    spec = PubunexConfig.from_dict(CONFIGS["P1"]).to_model_spec()
    # every pass has cache entries of its own
    assert [c.cache for c in spec.schedule] == list(range(11)) and spec.n_cache_entries() == 11
    for name, cfg in CONFIGS.items():
        assert _order(name) == P.run_order(cfg)
    once = copy.deepcopy(CONFIGS["P1"])
    once["loop"]["times"] = 1
    assert [c.block for c in PubunexConfig.from_dict(once).to_model_spec().schedule] == list(range(5))


def test_looped_schedule_without_the_embedding():
    assert looped_schedule(3, 1, 3, 2, add_embedding=False) == tuple(
        LayerCall(block=b, cache=c) for c, b in enumerate((0, 1, 2, 1, 2)))


def test_what_the_cache_is_asked_for():
    """Keys and values, a state alone, a latent row; a pass more asks for as much again."""
    from agave_b200.parts.base import KVRequest, StateRequest
    import agave_b200.models       # registers the parts
    m = DecoderModel(PubunexConfig.from_dict(CONFIGS["P1"]).to_model_spec(), torch.float32,
                     torch.device("cpu"))
    r = m.cache_requests()
    state = StateRequest(4 * 10 * 14 + 2 * (2 * 2 * 10 + 4 * 14))
    row = KVRequest(1, 24, None, value_dim=20, values_in_keys=True)
    assert r[0] == KVRequest(2, 10, None, 14)
    for k in (1, 4, 7):
        assert r[k] == state and r[k + 1] == row
    assert r[10] == KVRequest(1, 22, None, value_dim=14, values_in_keys=True)
    one_tap = DecoderModel(PubunexConfig.from_dict(CONFIGS["P3"]).to_model_spec(), torch.float32,
                           torch.device("cpu")).cache_requests()
    assert one_tap[0] == StateRequest(256)


def test_tensor_names_and_loader():
    folder = folder_for("P1")
    entry, cfg = load_config(folder)
    assert entry.name == "Pubunex"
    specs = decoder_param_specs(cfg.to_model_spec())
    names = entry.weight_names(cfg)
    assert {names.checkpoint_name(n, "") for n in specs} == \
        set(make_tensors(CONFIGS["P1"], 0, torch.float32))
    assert names.checkpoint_name("blocks.0.mixer.o_proj.bias", "") == "l0.mix.o.b"
    assert names.checkpoint_name("blocks.1.mixer.beta_proj.weight", "") == "l1.mix.b"
    assert names.checkpoint_name("blocks.1.mixer.decay_proj.weight", "") == "l1.mix.a"
    assert names.checkpoint_name("blocks.1.mixer.gate_proj.weight", "") == "l1.mix.g"
    assert names.checkpoint_name("blocks.2.mixer.sink", "") == "l2.mix.sink"
    assert names.checkpoint_name("blocks.3.ffn.experts.2.up_proj.weight", "") == "l3.mlp.e2.up"
    assert names.checkpoint_name("blocks.0.ffn.shared.down_proj.weight", "") == "l0.mlp.shared.down"
    assert names.checkpoint_name("lm_head.weight", "") == "head"
    with pytest.raises(KeyError):
        names.checkpoint_name("blocks.0.mixer.sink", "")          # (an attention layer has none)
    tensors = load_weights(folder, specs, names.checkpoint_name, names.prefixes, strict=True)
    assert tensors["blocks.1.mixer.gate_proj.weight"].shape == (56, 72)
    assert not any(n.startswith("blocks.2.ffn") for n in tensors)


def test_loader_reports_what_is_wrong(tmp_path):
    from safetensors.torch import save_file
    t = make_tensors(CONFIGS["P1"], 0, torch.float32)
    del t["l2.mix.sink"]
    t["l1.mix.A_log"] = t["l1.mix.A_log"][:2].contiguous()
    t["l2.mlp.router"] = torch.ones(2, 72)             # (that layer has no feed-forward)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(CONFIGS["P1"], f)
    save_file(t, str(tmp_path / "model.safetensors"))
    entry, cfg = load_config(str(tmp_path))
    names = entry.weight_names(cfg)
    with pytest.raises(WeightsError) as e:
        load_weights(str(tmp_path), decoder_param_specs(cfg.to_model_spec()),
                     names.checkpoint_name, names.prefixes)
    assert e.value.missing == ["l2.mix.sink"]
    assert e.value.unexpected == ["l2.mlp.router"]
    assert [w[0] for w in e.value.wrong_shape] == ["l1.mix.A_log"]


def test_parts_refuse_what_they_cannot_do():
    from agave_b200.parts.delta import HeadDeltaMixer
    from agave_b200.parts.linear import gate_activation
    from agave_b200.parts.moe import RoutedFeedForward
    cpu = torch.device("cpu")
    with pytest.raises(ValueError, match="multiple"):
        HeadDeltaMixer(HeadDeltaSpec(n_heads=4, n_qk_heads=3, head_dim=8, value_dim=8), 16,
                       torch.float32, cpu)
    with pytest.raises(ValueError, match="gate"):
        HeadDeltaMixer(HeadDeltaSpec(n_heads=2, n_qk_heads=2, head_dim=8, value_dim=8,
                                     gate_activation="relu"), 16, torch.float32, cpu)
    with pytest.raises(ValueError, match="identity"):
        RoutedFeedForward(RoutedFeedForwardSpec(n_experts=2, top=1, intermediate_size=8,
                                                correction=False, n_identity=1, weigh_input=True),
                          16, torch.float32, cpu)
    with pytest.raises(ValueError, match="limit"):
        gate_activation(ClampedGateSpec(limit=0.0))
    assert gate_activation("silu") == "silu"
    assert gate_activation(ClampedGateSpec(limit=2.0, alpha=1.0)) == ("clamped", 1.0, 2.0)


# -------------------------------------------------- mechanisms of the plain model, by hand
def test_convolution_by_hand():
    x = torch.tensor([[1.0], [2.0], [-3.0]], dtype=F64)
    w = torch.tensor([[0.5, -1.0, 2.0]], dtype=F64)                   # oldest .. current
    assert P.causal_conv(x, w)[:, 0].tolist() == pytest.approx(
        [2.0, 2.0 * 2 - 1.0, 2.0 * -3 - 1.0 * 2 + 0.5 * 1])


def test_both_rotations_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64).repeat(2, 1, 1)
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    c, s = math.cos, math.sin
    y = P.rotate(x, torch.tensor([0, 3]), {"dims": 4, "base": 100.0}, False)
    assert y[0, 0].tolist() == pytest.approx([1, 2, 3, 4, 5])
    assert y[1, 0].tolist() == pytest.approx(
        [1 * c(a0) - 3 * s(a0), 2 * c(a1) - 4 * s(a1), 3 * c(a0) + 1 * s(a0),
         4 * c(a1) + 2 * s(a1), 5.0])
    y = P.rotate(x, torch.tensor([0, 3]), {"dims": 4, "base": 100.0}, True)
    assert y[1, 0].tolist() == pytest.approx(
        [1 * c(a0) - 2 * s(a0), 2 * c(a0) + 1 * s(a0), 3 * c(a1) - 4 * s(a1),
         4 * c(a1) + 3 * s(a1), 5.0])


def test_scaled_frequencies_by_hand_and_of_the_rotation_part():
    from agave_b200.config.base import RotarySpec
    from agave_b200.parts.rope import RotaryEmbedding
    sc = {"factor": 8.0, "original": 500, "fast": 10.0, "slow": 1.0}
    f, mult = P.frequencies({"dims": 16, "base": 1000.0, "scaling": sc})
    plain = [1000.0 ** (-2.0 * i / 16) for i in range(8)]
    per = 16 / (2 * math.log(1000.0))
    lo = math.floor(per * math.log(500 / (2 * math.pi * 10)))           # 2
    hi = math.ceil(per * math.log(500 / (2 * math.pi)))                 # 6
    assert (lo, hi) == (2, 6)
    for i in range(8):
        ramp = min(1.0, max(0.0, (i - 2) / 4))
        assert f[i] == pytest.approx(plain[i] * ((1 - ramp) + ramp / 8.0))
    assert mult == pytest.approx(1 + 0.1 * math.log(8.0))
    rope = RotaryEmbedding(RotarySpec(theta=1000.0, rotary_dim=16, scaling=WavelengthScalingSpec(
        factor=8.0, original=500, fast=10.0, slow=1.0)), 20)
    got, m2 = rope.frequencies()
    assert got == pytest.approx(f, rel=1e-14) and m2 == pytest.approx(mult)
    x = torch.tensor([[[1.0, 0.0]]], dtype=F64)
    y = P.rotate(x, torch.tensor([0]), {"dims": 2, "base": 9.0, "scaling": sc}, False)
    assert y[0, 0].tolist() == pytest.approx([mult, 0.0])               # (a length is multiplied too)


def test_a_sink_takes_its_share_by_hand():
    q = torch.tensor([[[2.0]], [[1.0]]], dtype=F64)
    k = torch.tensor([[[1.0]], [[3.0]]], dtype=F64)
    v = torch.tensor([[[5.0]], [[-1.0]]], dtype=F64)
    y = P.attend(q, k, v, 0.5, torch.tensor([0.7]))
    s, e = math.exp(0.7), math.exp
    s = math.exp(float(torch.tensor(0.7)))
    assert y[0].item() == pytest.approx(e(1.0) * 5 / (e(1.0) + s))
    assert y[1].item() == pytest.approx((e(0.5) * 5 - e(1.5)) / (e(0.5) + e(1.5) + s))
    assert P.attend(q, k, v, 0.5)[0].item() == pytest.approx(5.0)


def test_delta_recurrence_by_hand():
    """One head, d 2, one value: decay, write against the decayed state, read-out that sees it."""
    q = torch.tensor([[[1.0, 0.5]], [[2.0, 1.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 0.0]], [[0.6, 0.8]]], dtype=F64)
    v = torch.tensor([[[3.0]], [[4.0]]], dtype=F64)
    beta = torch.tensor([[0.5], [0.25]], dtype=F64)
    g = torch.tensor([[0.9], [0.5]], dtype=F64)
    o = P.delta_recurrence(q, k, v, beta, g)
    s0 = [1.5, 0.0]
    assert o[0, 0, 0].item() == pytest.approx(1.5)
    d = [0.75, 0.0]
    u = 0.25 * (4.0 - 0.6 * 0.75)
    s1 = [d[0] + 0.6 * u, d[1] + 0.8 * u]
    assert o[1, 0, 0].item() == pytest.approx(2 * s1[0] + s1[1]) and s0[0] == 1.5
    dec = P.head_decay(torch.tensor([[0.3]], dtype=F64), torch.tensor([0.2], dtype=F64),
                       torch.tensor([-1.0], dtype=F64))
    assert dec.item() == pytest.approx(math.exp(-math.exp(-1.0) * math.log1p(math.exp(0.5))))
    x = torch.tensor([3.0, 4.0], dtype=F64)
    assert torch.allclose(P.unit(x), x / math.sqrt(25 + 1e-6))


def test_a_bounded_expert_by_hand():
    one = torch.ones(1, 1, dtype=F64)
    w = {"gate": 2 * one, "up": -3 * one, "down": 5 * one}
    sg = lambda z: 1 / (1 + math.exp(-1.702 * z))
    # inside the bounds; the gate above its bound and the up projection below its own; a gate far
    # below zero is not bounded
    assert P.clamped_expert(0.1 * one, w, "", 1.0).item() == pytest.approx(
        5 * 0.2 * sg(0.2) * (1 - 0.3))
    assert P.clamped_expert(2 * one, w, "", 1.0).item() == pytest.approx(5 * 1.0 * sg(1.0) * 0.0)
    assert P.clamped_expert(-2 * one, w, "", 1.0).item() == pytest.approx(5 * -4.0 * sg(-4.0) * 2.0)


def test_weights_multiply_the_experts_input():
    """Two experts, top 1: the chosen one sees s * h, not h; the shared one sees h."""
    h = torch.tensor([[0.5, -1.0]], dtype=F64)
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F64)}
    for n, k in (("e0", 1.0), ("e1", 7.0), ("shared", 0.5)):
        w[n + ".gate"] = torch.tensor([[k, 1.0]], dtype=F64)
        w[n + ".up"] = torch.tensor([[1.0, k]], dtype=F64)
        w[n + ".down"] = torch.tensor([[1.0], [2.0]], dtype=F64)
    f = {"expert": {"ff": 1, "limit": 0.9}, "router": {"experts": 2, "top": 1}}
    s = 1 / (1 + math.exp(-0.5))
    want = P.clamped_expert(s * h, w, "e0.", 0.9)
    assert torch.allclose(P.experts(h, f, w, ""), want)
    assert (want - s * P.clamped_expert(h, w, "e0.", 0.9)).abs().max() > 0.01
    f["shared"] = {"ff": 1, "limit": 0.2}
    assert torch.allclose(P.experts(h, f, w, ""), want + P.clamped_expert(h, w, "shared.", 0.2))


def test_small_functions_by_hand():
    z = torch.tensor([-30.0, -0.5, 0.0, 0.7, 40.0], dtype=F64)
    assert P.softplus(z).tolist() == pytest.approx([math.log1p(math.exp(v)) for v in z.tolist()])
    assert P.silu(z).tolist() == pytest.approx([v / (1 + math.exp(-v)) for v in z.tolist()])
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    assert torch.allclose(P.rms(x, 0.5), x / math.sqrt(12.5 + 0.5))


def test_a_looped_layer_by_hand():
    """One attention layer of one head and width 1, run three times: both branches read one norm,
    and the embedding joins before the second and the third pass."""
    cfg = {"layers": [{"type": "attention", "mlp": None,
                       "mixer": {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0}}],
           "loop": {"start": 0, "stop": 1, "times": 3}, "norm": {"eps": 1.0}, "vocab": 2, "width": 1}
    one = torch.ones(1, 1, dtype=F64)
    w = {"embed": torch.tensor([[2.0], [3.0]], dtype=F64), "head": one,
         "final.norm": torch.tensor([0.5], dtype=F64), "l0.norm1": torch.tensor([1.0], dtype=F64)}
    for n, b in (("q", 0.1), ("k", 0.2), ("v", 0.4), ("o", -0.3)):
        w[f"l0.mix.{n}"] = one
        w[f"l0.mix.{n}.b"] = torch.tensor([b], dtype=F64)
    out = []
    y = P.forward(cfg, w, [1], out)
    x = 3.0
    for t in range(3):
        x = x + (3.0 if t else 0.0)
        x = x + 2.0 * x / math.sqrt(x * x + 1) + 0.4 - 0.3
        assert out[t].item() == pytest.approx(x)
    assert y.item() == pytest.approx(x / math.sqrt(x * x + 1) * 1.5)
