"""Savovik without a GPU: the configuration reader and its errors, the lowering to part specs
and a run order, tensor names and the loader, what the cache is asked for, and the plain
implementation's mechanisms on cases worked out by hand."""
import copy
import json
import math

import pytest
import torch

from agave_b200.config import ConfigError, load_config, resolve_architecture
from agave_b200.config.base import (AttentionSpec, BandScalingSpec, DenseFeedForwardSpec, NormSpec,
                                    ParallelBlockSpec, SelectiveScanSpec, SideBySideSpec,
                                    StateSpaceSpec)
from agave_b200.config.savovik import SavovikConfig
from agave_b200.models.decoder import DecoderModel, decoder_param_specs
from agave_b200.weights import WeightsError, load_weights
from plain import savovik_plain as P
from savovik_util import CONFIGS, folder_for, make_tensors

F64 = torch.float64


# ------------------------------------------------------------------- reading
def test_registry_finds_the_architecture():
    assert resolve_architecture({"architecture": "Savovik"}).name == "Savovik"
    assert resolve_architecture({"model_type": "savovik"}).name == "Savovik"


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_reading_and_writing_round_trip(name):
    cfg = SavovikConfig.from_dict(CONFIGS[name])
    assert SavovikConfig.from_dict(cfg.to_dict()) == cfg
    assert len(cfg.layers) == len(CONFIGS[name]["layers"])


def test_what_may_be_absent_reads_as_none():
    cfg = SavovikConfig.from_dict(CONFIGS["S3"])
    m = cfg.layers[0].mixer.left
    assert (m.mask, m.rot, m.softcap) == (1, None, None)
    assert cfg.layers[6].mixer.left.mask is None
    assert cfg.layers[5].mixer.rot.scaling is None
    assert cfg.layers[1].ff is None
    raw = copy.deepcopy(CONFIGS["S3"])
    del raw["layers"][2]["mlp"], raw["layers"][2]["mixer"]["kv_heads"]
    cfg = SavovikConfig.from_dict(raw)
    assert cfg.layers[2].ff is None and cfg.layers[2].mixer.kv_heads == 2


@pytest.mark.parametrize("path, value, match", [
    (("vocab",), None, "vocab"),
    (("width",), 0, "positive"),
    (("norm", "eps"), None, "norm.eps"),
    (("layers", 0, "type"), "conv", "not a mixer"),
    (("layers", 0, "mixer", "left", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "left", "scale"), None, "left.scale"),
    (("layers", 0, "mixer", "left", "mask", "size"), 0, "left.mask.size"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7, "rot.dims"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "high"), 0.5, "rot.scaling"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "low"), None, "rot.scaling.low"),
    (("layers", 0, "mixer", "right", "dt_rank"), None, "right.dt_rank"),
    (("layers", 0, "mixer", "right", "state"), 0, "right.state"),
    (("layers", 0, "mixer", "right_scale"), None, "right_scale"),
    (("layers", 1, "mixer", "groups"), 4, "groups"),
    (("layers", 1, "mixer", "norm_groups"), 7, "norm_groups"),
    (("layers", 1, "mixer", "conv"), 2.5, "integer"),
    (("layers", 2, "mixer", "softcap"), -1.0, "softcap"),
    (("layers", 2, "mixer", "rot", "scaling", "factor"), None, "factor"),
    (("layers", 0, "mlp", "kind"), "moe", "not a feed-forward"),
    (("layers", 0, "mlp", "ff"), None, "mlp.ff"),
    (("layers", 3, "weights_of"), 3, "another layer"),
    (("layers", 3, "weights_of"), 30, "another layer"),
    (("layers", 3, "weights_of"), 1, "must equal"),
])
def test_errors_name_the_key(path, value, match):
    raw = copy.deepcopy(CONFIGS["S1"])
    d = raw
    for k in path[:-1]:
        d = d[k]
    if value is None:
        del d[path[-1]]
    else:
        d[path[-1]] = value
    with pytest.raises(ConfigError, match=match):
        SavovikConfig.from_dict(raw)


# ------------------------------------------------------------------ lowering
def test_lowering_to_parts_and_run_order():
    cfg = SavovikConfig.from_dict(CONFIGS["S1"])
    spec = cfg.to_model_spec()
    assert cfg.owners() == (0, 1, 2, 4) and len(spec.blocks) == 4 and not spec.tie_embeddings
    assert [(c.block, c.cache, c.writes_cache) for c in spec.schedule] == \
        [(0, 0, True), (1, 1, True), (2, 2, True), (0, 3, True), (3, 4, True), (1, 5, True),
         (2, 6, True)]
    norm = NormSpec(eps=1e-5, zero_centered=True)
    assert spec.final_norm == norm and spec.embed_scale == 1.0
    for b in spec.blocks:
        assert isinstance(b, ParallelBlockSpec) and b.gated and b.norm == norm
    b0, b1, b2, b3 = spec.blocks
    assert isinstance(b0.mixer, SideBySideSpec)
    assert (b0.mixer.left_scale, b0.mixer.right_scale) == (1.3, 0.7)
    left = b0.mixer.left
    assert isinstance(left, AttentionSpec)
    assert (left.n_heads, left.n_kv_heads, left.head_dim, left.value_dim, left.scale) == \
        (4, 2, 10, 14, 0.4)
    assert (left.chunk, left.window, left.softcap, left.qkv_bias, left.value_norm_eps) == \
        (7, None, None, True, None)
    assert left.qk_norm == NormSpec(eps=1e-5, zero_centered=False) and not left.qk_norm_whole
    assert (left.position.theta, left.position.rotary_dim, left.position.interleaved,
            left.position.factor) == (1e4, 6, True, 1.0)
    assert left.position.scaling == BandScalingSpec(factor=8.0, original=16.0, low=1.0, high=4.0)
    assert b0.mixer.right == SelectiveScanSpec(inner=36, state=5, dt_rank=3, conv_taps=2)
    assert b0.feed_forward == DenseFeedForwardSpec(intermediate_size=40, activation="gelu_erf")
    assert b1.mixer == StateSpaceSpec(n_heads=6, value_dim=10, state=12, n_groups=3, norm_groups=2,
                                      conv_taps=3, eps=1e-5)
    assert b1.feed_forward is None
    a = b2.mixer
    assert (a.window, a.chunk, a.softcap, a.qkv_bias, a.value_norm_eps, a.qk_norm) == \
        (9, None, 5.0, False, 1e-5, None)
    assert (a.position.factor, a.position.scaling, a.position.interleaved) == (2.5, None, False)
    assert b3.mixer.n_groups == 1 and b3.mixer.norm_groups == 4
    # a rotation of the whole head is written as such
    s2 = SavovikConfig.from_dict(CONFIGS["S2"]).to_model_spec()
    assert s2.blocks[0].mixer.position.rotary_dim == 0 and s2.blocks[0].mixer.value_dim == 0


def test_weights_of_may_lead_through_another_layer():
    raw = copy.deepcopy(CONFIGS["S1"])
    raw["layers"].append(dict(copy.deepcopy(raw["layers"][3]), weights_of=3))
    cfg = SavovikConfig.from_dict(raw)
    assert cfg.owner(7) == 0 and cfg.to_model_spec().schedule[7].block == 0


def test_what_the_cache_is_asked_for():
    """A call has an entry of its own even where it runs another layer's weights: keys and
    values beside the scan's state, a state alone, keys and values alone."""
    from agave_b200.parts.base import KVRequest, StateRequest
    import agave_b200.models       # registers the parts
    spec = SavovikConfig.from_dict(CONFIGS["S1"]).to_model_spec()
    m = DecoderModel(spec, torch.float32, torch.device("cpu"))
    r = m.cache_requests()
    first = (KVRequest(2, 10, 7, 14), StateRequest(36 * 5 + 1 * 36))
    second = StateRequest(6 * 12 * 10 + 2 * (60 + 2 * 36))
    third = KVRequest(1, 12, 9, 6)
    assert r[:3] == [first, second, third] and [r[3], r[5], r[6]] == [first, second, third]
    assert r[4] == StateRequest(4 * 20 * 6 + 3 * (24 + 40))
    s3 = DecoderModel(SavovikConfig.from_dict(CONFIGS["S3"]).to_model_spec(), torch.float32,
                      torch.device("cpu")).cache_requests()
    assert s3[0] == (KVRequest(1, 16, 1, 0), StateRequest(8)) and s3[1] == StateRequest(16)
    assert s3[6][0].window is None


def test_two_mixers_that_cannot_share_a_cache_entry():
    from agave_b200.parts.parallel import SideBySideMixer
    a = AttentionSpec(n_heads=1, n_kv_heads=1, head_dim=8)
    s = SelectiveScanSpec(inner=8, state=2, dt_rank=1, conv_taps=2)
    for l, r, what in ((a, a, "keys and values"), (s, s, "state")):
        with pytest.raises(ValueError, match=what):
            SideBySideMixer(SideBySideSpec(left=l, right=r), 16, torch.float32, torch.device("cpu"))


def test_tensor_names_and_loader():
    folder = folder_for("S1")
    entry, cfg = load_config(folder)
    assert entry.name == "Savovik"
    specs = decoder_param_specs(cfg.to_model_spec())
    names = entry.weight_names(cfg)
    assert {names.checkpoint_name(n, "") for n in specs} == \
        set(make_tensors(CONFIGS["S1"], 0, torch.float32))
    assert names.checkpoint_name("blocks.0.mixer.left.q_proj.bias", "") == "l0.mix.left.q.b"
    assert names.checkpoint_name("blocks.0.mixer.right.dt_proj.bias", "") == "l0.mix.right.dt.b"
    assert names.checkpoint_name("blocks.0.mixer.right.conv.weight", "") == "l0.mix.right.conv"
    assert names.checkpoint_name("blocks.3.mixer.dt_bias", "") == "l4.mix.dt_bias"
    assert names.checkpoint_name("blocks.1.mixer.out_norm.weight", "") == "l1.mix.norm"
    assert names.checkpoint_name("blocks.2.ffn_gate.bias", "") == "l2.rg2.b"
    assert names.checkpoint_name("lm_head.weight", "") == "head"
    with pytest.raises(KeyError):
        names.checkpoint_name("blocks.0.mixer.sink", "")
    tensors = load_weights(folder, specs, names.checkpoint_name, names.prefixes, strict=True)
    assert tensors["blocks.0.mixer.right.a_log"].shape == (36, 5)
    assert tensors["blocks.1.mixer.in_proj.weight"].shape == (60 + 60 + 72 + 6, 72)
    assert not any(n.startswith("blocks.1.ffn") for n in tensors)


def test_loader_reports_what_is_wrong(tmp_path):
    from safetensors.torch import save_file
    t = make_tensors(CONFIGS["S1"], 0, torch.float32)
    del t["l0.mix.right.D"]
    t["l1.mix.A_log"] = t["l1.mix.A_log"][:2].contiguous()
    t["l3.norm1"] = torch.ones(72)             # (that layer has no tensors of its own)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(CONFIGS["S1"], f)
    save_file(t, str(tmp_path / "model.safetensors"))
    entry, cfg = load_config(str(tmp_path))
    names = entry.weight_names(cfg)
    with pytest.raises(WeightsError) as e:
        load_weights(str(tmp_path), decoder_param_specs(cfg.to_model_spec()),
                     names.checkpoint_name, names.prefixes)
    assert e.value.missing == ["l0.mix.right.D"]
    assert e.value.unexpected == ["l3.norm1"]
    assert [w[0] for w in e.value.wrong_shape] == ["l1.mix.A_log"]


# -------------------------------------------------- mechanisms of the plain model, by hand
def test_masks_by_hand():
    see = P.mask(7, P.in_chunk, {"mask": {"size": 3}})
    assert see[2].tolist() == [True, True, True, False, False, False, False]
    assert see[3].tolist() == [False, False, False, True, False, False, False]
    assert see[5].tolist() == [False, False, False, True, True, True, False]
    see = P.mask(7, P.in_window, {"mask": {"size": 3}})
    assert see[5].tolist() == [False, False, False, True, True, True, False]
    assert see[3].tolist() == [False, True, True, True, False, False, False]
    for fn in (P.in_chunk, P.in_window):
        m = P.mask(9, fn, {"mask": {"size": 4}})
        assert all(bool(m[i, j]) == fn(i, j, 4) for i in range(9) for j in range(9))
        assert P.mask(3, fn, {}).tolist() == [[True, False, False], [True, True, False], [True] * 3]


def test_convolution_by_hand():
    x = torch.tensor([[1.0], [2.0], [-3.0]], dtype=F64)
    w = torch.tensor([[0.5, -1.0, 2.0]], dtype=F64)                   # oldest .. current
    y = P.causal_conv(x, w, torch.tensor([0.25], dtype=F64))
    assert y[:, 0].tolist() == pytest.approx(
        [0.25 + 2.0, 0.25 + 2.0 * 2 - 1.0, 0.25 + 2.0 * -3 - 1.0 * 2 + 0.5 * 1])


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


def test_scaled_frequencies_of_the_rotation_part():
    from agave_b200.config.base import RotarySpec
    from agave_b200.parts.rope import RotaryEmbedding
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 16}
    band = BandScalingSpec(factor=8.0, original=16, low=1.0, high=4.0)
    rope = RotaryEmbedding(RotarySpec(theta=100.0, rotary_dim=8, scaling=band), 12)
    f = P.frequencies({"dims": 8, "base": 100.0, "scaling": sc})
    assert rope.frequencies()[0] == pytest.approx(f, rel=1e-14)
    plain = [100.0 ** (-2.0 * i / 8) for i in range(4)]
    s = (16 / (2 * math.pi) - 1.0) / 3.0
    assert f[0] == pytest.approx((1 - s) * plain[0] / 8 + s * plain[0])
    assert f[1:] == pytest.approx([x / 8 for x in plain[1:]])
    assert P.frequencies({"dims": 2, "base": 9.0, "scaling": {**sc, "original": 64}})[0] == 1.0
    lin = P.frequencies({"dims": 8, "base": 100.0, "scaling": {"factor": 2.5}})
    assert lin == pytest.approx([x / 2.5 for x in plain])
    rope = RotaryEmbedding(RotarySpec(theta=100.0, rotary_dim=8, factor=2.5), 12)
    assert rope.frequencies()[0] == pytest.approx(lin)


def test_capped_scores_and_normed_values_by_hand():
    """One head, identity projections: two tokens, the second's weights by hand."""
    eye = torch.eye(2, dtype=F64)
    h = torch.tensor([[3.0, 0.0], [4.0, 1.0]], dtype=F64)
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.5, "softcap": 4.0}
    y = P.window_attention(h, m, {n: eye for n in ("q", "k", "v", "o")}, "", 0.5)
    s = [4.0 * math.tanh(0.5 * z / 4.0) for z in (12.0, 17.0)]
    e = [math.exp(x) for x in s]
    v0 = [3.0 / math.sqrt(9 / 2 + 0.5), 0.0]
    r1 = math.sqrt(17 / 2 + 0.5)
    v1 = [4.0 / r1, 1.0 / r1]
    assert y[1].tolist() == pytest.approx([(e[0] * a + e[1] * b) / sum(e) for a, b in zip(v0, v1)])


def test_biased_and_normed_heads_by_hand():
    """Chunked attention of one token: the value with its bias; of two: the normed, biased keys."""
    eye = torch.eye(2, dtype=F64)
    w = {"q": eye, "k": eye, "v": eye, "o": eye, "q.b": torch.tensor([1.0, 0.0], dtype=F64),
         "k.b": torch.tensor([0.0, 2.0], dtype=F64), "v.b": torch.tensor([5.0, 6.0], dtype=F64),
         "q.norm": torch.tensor([2.0, 1.0], dtype=F64), "k.norm": torch.tensor([1.0, 0.5], dtype=F64)}
    h = torch.tensor([[1.0, 2.0], [3.0, -1.0]], dtype=F64)
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0}
    y = P.chunked_attention(h, m, w, "", 0.0)
    assert y[0].tolist() == pytest.approx([6.0, 8.0])
    q = [4.0 / math.sqrt(17 / 2) * 2, -1.0 / math.sqrt(17 / 2)]
    k = [[1.0 / math.sqrt(17 / 2), 4.0 / math.sqrt(17 / 2) / 2],
         [3.0 / math.sqrt(10 / 2), 1.0 / math.sqrt(10 / 2) / 2]]
    e = [math.exp(q[0] * a + q[1] * b) for a, b in k]
    assert y[1].tolist() == pytest.approx([(e[0] * 6 + e[1] * 8) / sum(e), (e[0] * 8 + e[1] * 5) / sum(e)])
    # chunks of one: every token sees itself alone
    y = P.chunked_attention(h, {**m, "mask": {"size": 1}}, w, "", 0.0)
    assert y[1].tolist() == pytest.approx([8.0, 5.0])


def test_selective_scan_by_hand():
    x = torch.tensor([[2.0], [3.0]], dtype=F64)
    dt = torch.tensor([[0.5], [0.25]], dtype=F64)
    A = torch.tensor([[-1.0, -2.0]], dtype=F64)
    B = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)
    C = torch.tensor([[1.0, 1.0], [0.5, 2.0]], dtype=F64)
    y = P.selective_scan(x, dt, A, B, C, torch.tensor([10.0], dtype=F64))
    s0 = [1.0, 2.0]                                                # dt x B
    s1 = [math.exp(-0.25) * 1.0 + 0.75 * 3, math.exp(-0.5) * 2.0 + 0.75 * 4]
    assert y[:, 0].tolist() == pytest.approx([3.0 + 20.0, 0.5 * s1[0] + 2 * s1[1] + 30.0])
    assert sum(s0) == 3.0


def test_head_scan_by_hand():
    """Two heads of one group: N = 2, one value channel each."""
    x = torch.tensor([[[2.0], [1.0]], [[3.0], [-1.0]]], dtype=F64)
    dt = torch.tensor([[0.5, 1.0], [0.25, 2.0]], dtype=F64)
    a = torch.tensor([1.0, 0.5], dtype=F64)
    B = torch.tensor([[[1.0, 2.0]], [[3.0, 4.0]]], dtype=F64)
    C = torch.tensor([[[1.0, 1.0]], [[0.5, 2.0]]], dtype=F64)
    y = P.ssd(x, dt, a, B, C, torch.tensor([10.0, 0.0], dtype=F64))
    d = math.exp(-0.25)
    assert y[1, 0, 0].item() == pytest.approx(
        0.5 * (d * 1.0 + 0.75 * 3) + 2 * (d * 2.0 + 0.75 * 4) + 30.0)
    d = math.exp(-0.5 * 2.0)
    assert y[1, 1, 0].item() == pytest.approx(0.5 * (d * 1.0 - 2 * 3) + 2 * (d * 2.0 - 2 * 4))


def test_small_functions_by_hand():
    z = torch.tensor([-30.0, -0.5, 0.0, 0.7, 40.0], dtype=F64)
    assert P.softplus(z).tolist() == pytest.approx([math.log1p(math.exp(v)) for v in z.tolist()])
    assert P.silu(z).tolist() == pytest.approx([v / (1 + math.exp(-v)) for v in z.tolist()])
    assert P.gelu_erf(z).tolist() == pytest.approx(
        [v / 2 * (1 + math.erf(v / math.sqrt(2))) for v in z.tolist()])
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    assert torch.allclose(P.rms(x, 0.5), x / math.sqrt(12.5 + 0.5))


def test_a_layer_by_hand():
    """A model of one layer whose mixer and feed-forward are linear enough to write down: both
    branches read the same norm and join through their own gates."""
    cfg = {"layers": [{"type": "attention", "mlp": {"ff": 1, "kind": "dense"},
                       "mixer": {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0}}],
           "norm": {"eps": 1.0}, "vocab": 2, "width": 1}
    one = torch.ones(1, 1, dtype=F64)
    w = {"embed": torch.tensor([[2.0], [3.0]], dtype=F64), "head": one,
         "final.norm": torch.tensor([0.5], dtype=F64), "l0.norm1": torch.tensor([1.0], dtype=F64),
         "l0.rg1": one, "l0.rg1.b": torch.tensor([0.3], dtype=F64), "l0.rg2": -one,
         "l0.rg2.b": torch.tensor([0.1], dtype=F64), "l0.mlp.up": one, "l0.mlp.down": 4 * one}
    w.update({f"l0.mix.{n}": one for n in "qkvo"})
    out = []
    y = P.forward(cfg, w, [1], out)
    h = 3.0 / math.sqrt(9 + 1) * 2.0
    sg = lambda v: 1 / (1 + math.exp(-v))
    x = 3.0 + sg(h + 0.3) * (h / math.sqrt(h * h + 1)) + \
        sg(-h + 0.1) * 4 * (h / 2 * (1 + math.erf(h / math.sqrt(2))))
    assert out[0].item() == pytest.approx(x)
    assert y.item() == pytest.approx(x / math.sqrt(x * x + 1) * 1.5)
