"""Nogavik without a GPU: its configuration checks, its plan (parts, constants, the
caches its layers share, tensor names and shapes), the random-weights writer,
and the plain model's own mechanisms against hand-made cases."""
import copy
import math

import pytest
import torch

from kipp_b200.config import config_from_dict, load_preset
from kipp_b200.config.base import ConfigError
from kipp_b200.config.registry import get_architecture
from nogavik_util import CONFIGS, INIT, random_tokens, write_folder
from tiny import read_weights

import plain_nogavik as P

F64 = torch.float64


def spec_of(cfg):
    c = config_from_dict(cfg)
    return get_architecture(c.architecture).build(c)


def t64(*rows):
    return torch.tensor(rows, dtype=F64)


def test_the_model_class_is_chosen_by_the_architecture_key():
    c = config_from_dict(CONFIGS["A"])
    assert c.architecture == "Nogavik" and c.to_dict()["layers"][0]["type"] == "latent_attention"
    assert config_from_dict(c.to_dict()).to_dict() == c.to_dict()
    assert c.vocab_size == 300 and c.hidden_size == 64 and c.token_side == {"dim": 12}


def test_layers_that_read_another_latent_share_its_cache():
    order = spec_of(CONFIGS["A"]).plan["order"]
    assert [o["cache"] for o in order] == [0, 1, 0, 3, 0]
    assert [o["writes_cache"] for o in order] == [True, True, False, True, False]
    order = spec_of(CONFIGS["B"]).plan["order"]
    assert [o["cache"] for o in order] == [0, 1, 2, 1, 4, 2]
    assert [o["writes_cache"] for o in order] == [True, True, True, False, True, False]


def test_parts_and_their_constants():
    plan = spec_of(CONFIGS["A"]).plan
    assert [e["part"]["kind"] for e in plan["embedding"]] == ["token_embedding", "token_side_table"]
    assert plan["embedding"][1]["part"]["cols"] == 12 * 5 and plan["embedding"][1]["part"]["weight_name"] == "side.embed"
    blocks = [l["part"] for l in plan["layers"]]
    assert all(b["kind"] == "parallel_block" and b["norm"]["weight_offset"] == 1.0 and b["norm"]["eps"] == 1e-5 for b in blocks)
    assert blocks[0]["ffn_norm"]["weight_name"] == "norm2" and blocks[0]["ffn_norm"]["weight_offset"] == 1.0
    assert blocks[2]["ffn"] is None and blocks[2]["ffn_norm"] is None
    assert [b["side"]["offset"] for b in blocks] == [0, 12, 24, 36, 48] and blocks[1]["side"]["table_cols"] == 60
    lat = blocks[0]["mixer"]
    assert lat["kind"] == "latent_attention" and lat["element_gate"] and lat["interleaved"] and not lat["shared_kv"]
    assert (lat["num_heads"], lat["head_dim"], lat["rot_dim"], lat["value_dim"], lat["kv_rank"], lat["q_rank"], lat["scale"]) == \
        (4, 16, 8, 24, 32, 40, 0.25)
    assert lat["position"] == {"kind": "rotary", "head_dim": 8, "rotary_dim": 8, "theta": 10000.0, "exact_exponent": True}
    assert blocks[2]["mixer"]["shared_kv"] and blocks[4]["mixer"]["shared_kv"]
    par = blocks[1]["mixer"]
    assert par["kind"] == "parallel" and par["out_scale"] == 0.5 and par["out_norm"]["eps"] == 1e-5
    assert par["out_norm"].get("offset", 0.0) == 0.0                           # plain weights
    att, gd = (b["part"] for b in par["branches"])
    assert [b["norm"] for b in par["branches"]] == ["left.out", "right.out"]
    assert att["kind"] == "attention" and att["bias"] and att["qk_norm_eps"] == 1e-5 and att["position"]["kind"] == "no_position"
    assert (att["num_heads"], att["num_kv_heads"], att["head_dim"], att["value_dim"], att["scale"]) == (4, 2, 16, 24, 0.3)
    assert gd["kind"] == "gated_delta" and gd["gate"] == "sigmoid"
    assert (gd["num_heads"], gd["num_kv_heads"], gd["head_dim"], gd["value_dim"], gd["conv"]) == (4, 2, 16, 8, 3)
    ssm = blocks[3]["mixer"]
    assert ssm["kind"] == "state_space" and (ssm["num_heads"], ssm["groups"], ssm["value_dim"], ssm["state_dim"], ssm["conv"],
                                             ssm["norm_groups"]) == (4, 2, 16, 24, 3, 2)
    assert blocks[0]["ffn"] == {"kind": "dense_mlp", "hidden_size": 64, "intermediate_size": 96, "activation": "relu_squared"}
    assert plan["final_norm"]["part"]["weight_offset"] == 1.0 and plan["head"]["part"]["tied_to"] == "embed"
    # what the configuration leaves out: no token side, no rotation, sizes that follow from others
    cfg = copy.deepcopy(CONFIGS["E"])
    for side in ("left", "right"):
        for key in ("kv_heads", "vdim"):
            cfg["layers"][1]["mixer"][side].pop(key)
    cfg["layers"][0]["mixer"].pop("vdim")
    plan = spec_of(cfg).plan
    assert len(plan["embedding"]) == 1 and plan["layers"][0]["part"]["side"] is None
    assert plan["layers"][0]["part"]["mixer"]["position"]["kind"] == "no_position"
    att, gd = (b["part"] for b in plan["layers"][1]["part"]["mixer"]["branches"])
    assert att["num_kv_heads"] == 2 and att["value_dim"] == 8 and gd["num_kv_heads"] == 2 and gd["value_dim"] == 8


def test_tensor_names_and_shapes():
    specs = {s.name: tuple(s.shape) for s in spec_of(CONFIGS["A"]).tensor_specs()}
    assert specs["embed"] == (300, 64) and specs["side.embed"] == (300, 60) and specs["final.norm"] == (64,)
    assert specs["l0.norm1"] == specs["l0.norm2"] == (64,) and "l2.norm2" not in specs and "l2.mlp.up" not in specs
    assert specs["l0.mix.dq"] == (40, 64) and specs["l0.mix.dq.norm"] == (40,) and specs["l0.mix.uq"] == (4 * 24, 40)
    assert specs["l0.mix.dkv"] == (40, 64) and specs["l0.mix.dkv.norm"] == (32,)
    assert specs["l0.mix.uk"] == (64, 32) and specs["l0.mix.uv"] == (96, 32) and specs["l0.mix.g"] == (96, 64)
    assert specs["l0.mix.o"] == (64, 96)
    assert "l2.mix.dkv" not in specs and "l2.mix.dkv.norm" not in specs and specs["l2.mix.uk"] == (48, 32)
    assert specs["l1.mix.left.q"] == (64, 64) and specs["l1.mix.left.q.b"] == (64,) and specs["l1.mix.left.k.b"] == (32,)
    assert specs["l1.mix.left.v"] == (48, 64) and specs["l1.mix.left.v.b"] == (48,) and specs["l1.mix.left.o"] == (64, 96)
    assert specs["l1.mix.left.q.norm"] == specs["l1.mix.left.k.norm"] == (16,)
    assert specs["l1.mix.right.q"] == specs["l1.mix.right.k"] == (32, 64) and specs["l1.mix.right.v"] == (32, 64)
    assert specs["l1.mix.right.q.conv"] == (32, 3) and specs["l1.mix.right.v.conv"] == (32, 3)
    assert specs["l1.mix.right.b"] == (4, 64) and specs["l1.mix.right.A_log"] == (4,) and specs["l1.mix.right.dt_bias"] == (64,)
    assert specs["l1.mix.right.a1"] == (12, 64) and specs["l1.mix.right.a2"] == (64, 12)
    assert specs["l1.mix.right.g1"] == (20, 64) and specs["l1.mix.right.g2"] == (32, 20)
    assert specs["l1.mix.right.norm"] == (8,) and specs["l1.mix.right.o"] == (64, 32)
    assert specs["l1.mix.left.out"] == specs["l1.mix.right.out"] == (64,)
    assert specs["l3.side.gate"] == (12, 64) and specs["l3.side.proj"] == (64, 12) and specs["l3.side.norm"] == (64,)
    # the widths of the bottlenecks may be left to the tensors
    cfg = copy.deepcopy(CONFIGS["A"])
    for key in ("decay_rank", "gate_rank"):
        cfg["layers"][1]["mixer"]["right"].pop(key)
    specs = {s.name: tuple(s.shape) for s in spec_of(cfg).tensor_specs()}
    assert specs["l1.mix.right.a1"] == (-1, 64) and specs["l1.mix.right.g2"] == (32, -1)


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["token_side"].update(dim=0), "token_side.dim"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "left.scale"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "right.conv"),
    (lambda c: c["layers"][3]["mixer"].update(groups=3), "multiple of groups"),
    (lambda c: c["layers"][3]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "latent attention layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "latent of its own"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=16), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=3.0), "rotation"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not supported"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "mlp.ff"),
])
def test_what_the_configuration_refuses(change, message):
    cfg = copy.deepcopy(CONFIGS["A"])
    change(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert message in str(e.value)


def test_random_weights_cover_every_declared_tensor(tmp_path):
    for name in ("D", "E"):
        folder = write_folder(str(tmp_path / name), CONFIGS[name], INIT[name])
        w = read_weights(folder)
        specs = {s.name: tuple(s.shape) for s in spec_of(CONFIGS[name]).tensor_specs() if not (s.optional and s.alias_of)}
        assert {k: tuple(v.shape) for k, v in w.items()} == specs
        with torch.no_grad():
            logits = P.forward(CONFIGS[name], w, random_tokens(CONFIGS[name]["vocab"], 12, seed=1))
        assert logits.shape == (12, CONFIGS[name]["vocab"]) and bool(torch.isfinite(logits).all())
    preset, _ = load_preset("nogavik-tiny")
    assert config_from_dict(dict(preset)).architecture == "Nogavik"


def test_the_parts_can_be_described_from_python_for_another_design():
    """A model put together in Python from the descriptions of the same parts gives the tensors and the parts
    the library's own builder makes."""
    from kipp_b200.models.spec import LayerRun, ModelSpec
    from kipp_b200.parts import (AttentionMixer, DenseFeedForward, GatedDeltaMixer, LatentAttentionMixer, NoPositionEncoding, OutputHead,
                                 ParallelBlock, ParallelMixer, RMSNorm, RotaryEncoding, StateSpaceMixer, TokenEmbedding, TokenSide,
                                 TokenSideTable)
    cfg = CONFIGS["A"]
    eps, width, vocab, d = cfg["norm"]["eps"], cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    layers, order = [], []
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        if layer["type"] == "mamba2":
            mixer = StateSpaceMixer(width, m["heads"], m["vdim"], m["state"], m["conv"], eps, groups=m["groups"], norm_groups=m["norm_groups"])
        elif layer["type"] == "latent_attention":
            mixer = LatentAttentionMixer(width, m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"],
                                         RotaryEncoding(m["rot_dim"], m["rot"]["base"], m["rot_dim"]), eps, value_dim=m["vdim"],
                                         scale=m["scale"], element_gate=True, interleaved=True, shared_kv="kv_from" in m)
        else:
            l, r = m["left"], m["right"]
            names = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "q_bias": "q.b", "k_bias": "k.b",
                     "v_bias": "v.b"}
            mixer = ParallelMixer(
                [("left.", AttentionMixer(width, l["heads"], l["kv_heads"], l["dim"], NoPositionEncoding(), eps, 0, l["scale"],
                                          value_dim=l["vdim"], bias=True, names=names)),
                 ("right.", GatedDeltaMixer(width, r["heads"], r["dim"], r["conv"], eps, num_kv_heads=r["kv_heads"], value_dim=r["vdim"],
                                            decay_rank=r["decay_rank"], gate_rank=r["gate_rank"]))],
                out_norms=["left.out", "right.out"], size=width, eps=eps, out_scale=0.5)
        ff = DenseFeedForward(width, layer["mlp"]["ff"], "relu_squared") if layer["mlp"] else None
        block = ParallelBlock(RMSNorm(width, eps, "norm1", 1.0), mixer, ff, ("", "mix.", "mlp.", "", "side."),
                              ffn_norm=RMSNorm(width, eps, "norm2", 1.0) if ff else None,
                              side=TokenSide(vocab, width, d, "side.embed", 5 * d, i * d, eps))
        layers.append((f"l{i}.", block))
        order.append(LayerRun(i, m.get("kv_from", i), "kv_from" not in m))
    spec = ModelSpec(config=None, hidden_size=width, vocab_size=vocab,
                     embedding=[("", TokenEmbedding(vocab, width, weight_name="embed")), ("", TokenSideTable(vocab, 5 * d, "side.embed"))],
                     layers=layers, order=order, final_norm=("", RMSNorm(width, eps, "final.norm", 1.0)),
                     head=("", OutputHead(vocab, width, tied_to="embed", weight_name="head")))
    theirs = spec_of(cfg)
    assert {s.name: tuple(s.shape) for s in spec.tensor_specs()} == {s.name: tuple(s.shape) for s in theirs.tensor_specs()}
    plan, _ = spec.to_plan()
    assert plan["order"] == [{k: o[k] for k in ("layer", "cache", "writes_cache")} for o in theirs.plan["order"]]
    for a, b in zip(plan["layers"], theirs.plan["layers"]):
        assert a["part"]["kind"] == b["part"]["kind"] and a["part"]["mixer"]["kind"] == b["part"]["mixer"]["kind"]
        for key in ("element_gate", "interleaved", "shared_kv", "out_scale"):
            assert a["part"]["mixer"].get(key) == b["part"]["mixer"].get(key)


# ------------------------------------------------------------------ the plain model against hand-made cases
def test_plain_norm_with_a_weight_around_zero():
    got = P.norm_one_plus(t64([3.0, 4.0]), torch.tensor([0.0, 1.0], dtype=F64), 0.5)
    r = math.sqrt(12.5 + 0.5)
    assert torch.allclose(got, t64([3.0 / r, 8.0 / r]))


def test_plain_causal_convolution_and_its_start():
    got = P.causal_conv(t64([1.0], [2.0], [4.0]), t64([100.0, 10.0, 1.0]))       # the last column meets the current token
    assert got.flatten().tolist() == [1.0, 12.0, 124.0]


def test_plain_rotation_turns_neighbours():
    x = torch.zeros(1, 1, 5, dtype=F64)
    x[0, 0] = torch.tensor([1.0, 0.0, 0.0, 1.0, 7.0], dtype=F64)
    got = P.rotate_neighbours(x, torch.tensor([3]), {"base": 100.0, "dims": 4})[0, 0]
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    assert torch.allclose(got, torch.tensor([math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 7.0], dtype=F64))


def test_plain_gated_delta_rule_by_hand():
    """One head, one key channel, one value: the decay acts before the removal, and the read-out sees the write."""
    one = lambda *v: torch.tensor(v, dtype=F64).view(-1, 1, 1)                     # noqa: E731
    q, k, v, g = one(2.0, 3.0), one(0.5, 1.0), one(1.0, -1.0), one(0.9, 0.5)
    beta = torch.tensor([[0.25], [0.8]], dtype=F64)
    s1 = 0.5 * 0.25 * 1.0
    s2 = 0.5 * s1
    s2 = s2 + 1.0 * 0.8 * (-1.0 - s2)
    assert torch.allclose(P.gated_delta_rule(q, k, v, beta, g).flatten(), torch.tensor([2.0 * s1, 3.0 * s2], dtype=F64))


def test_plain_delta_vectors_are_units_and_shared_by_groups():
    m = CONFIGS["A"]["layers"][1]["mixer"]["right"]
    g = torch.Generator().manual_seed(3)
    rand = lambda *s: torch.randn(*s, generator=g, dtype=F64)                       # noqa: E731
    w = {"q": rand(32, 64), "k": rand(32, 64), "v": rand(32, 64), "q.conv": rand(32, 3), "k.conv": rand(32, 3), "v.conv": rand(32, 3),
         "b": rand(4, 64), "a1": rand(12, 64), "a2": rand(64, 12), "dt_bias": rand(64), "A_log": rand(4)}
    q, k, v, beta, decay = P.delta_vectors(m, w, "", rand(5, 64))
    assert torch.allclose(k.norm(dim=-1), torch.ones(5, 4, dtype=F64), atol=1e-4)
    assert torch.allclose(q.norm(dim=-1), torch.full((5, 4), 16 ** -0.5, dtype=F64), atol=1e-4)
    assert torch.equal(k[:, 0], k[:, 1]) and torch.equal(q[:, 2], q[:, 3]) and not torch.equal(k[:, 1], k[:, 2])
    assert v.shape == (5, 4, 8) and bool(((decay > 0) & (decay <= 1)).all()) and bool(((beta > 0) & (beta < 1)).all())


def test_plain_parallel_mixer_is_half_the_sum_of_normed_outputs():
    real_a, real_d = P.attention, P.gated_delta
    P.attention, P.gated_delta = (lambda *a: t64([3.0, 4.0])), (lambda *a: t64([0.0, -2.0]))
    try:
        w = {"left.out": torch.tensor([1.0, 2.0], dtype=F64), "right.out": torch.tensor([5.0, 3.0], dtype=F64)}
        got = P.parallel({"left": {}, "right": {}}, w, "", t64([0.0, 0.0]), 0.5)
    finally:
        P.attention, P.gated_delta = real_a, real_d
    left, right = math.sqrt(13.0), math.sqrt(2.5)
    assert torch.allclose(got, t64([0.5 * 3.0 / left, 0.5 * (8.0 / left - 6.0 / right)]))


def test_plain_latent_attention_of_one_head_by_hand():
    """Two tokens, one dimension each: the second one's softmax over both keys, then the gate per element."""
    m = {"heads": 1, "dim": 1, "rot_dim": 0, "vdim": 1, "kv_rank": 1, "q_rank": 1, "scale": 2.0}
    w = {"dq": t64([1.0, 0.0]), "dq.norm": torch.ones(1, dtype=F64), "uq": t64([1.0]), "uk": t64([0.5]), "uv": t64([3.0]),
         "g": t64([0.0, 1.0]), "o": t64([1.0], [0.0])}
    h = t64([1.0, 0.3], [-1.0, 0.7])
    keys = (t64([0.4], [-0.8]), torch.zeros(2, 0, dtype=F64))
    got = P.latent_attention(m, w, "", h, 1e-12, keys)[:, 0]
    s = torch.tensor([-1.0 * 0.2 * 2.0, -1.0 * -0.4 * 2.0], dtype=F64)
    a = torch.softmax(s, 0)
    want = torch.stack([torch.sigmoid(t64(0.3))[0] * 1.2, torch.sigmoid(t64(0.7))[0] * (a[0] * 1.2 + a[1] * -2.4)])
    assert torch.allclose(got, want, atol=1e-10)


def test_plain_token_side_by_hand():
    w = {"gate": t64([1.0, 1.0]), "proj": t64([2.0], [-1.0]), "norm": torch.tensor([1.0, 0.5], dtype=F64)}
    got = P.token_side(w, "", t64([0.25, 0.75]), t64([3.0]), 0.1)
    g = 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715)) * 3.0
    r = math.sqrt((4 * g * g + g * g) / 2 + 0.1)
    assert torch.allclose(got, t64([2 * g / r, -0.5 * g / r]))


def test_plain_layer_reads_one_stream_twice():
    """Both sublayers read the stream before either adds to it; the token side reads it after both."""
    cfg = {"norm": {"eps": 1e-5}, "token_side": {"dim": 1}, "layers": [{"type": "mamba2", "mixer": {}, "mlp": {"kind": "dense", "ff": 1}}]}
    seen = {}
    real = P.mixer, P.feed_forward, P.token_side

    def fake_mixer(cfg_, w_, i, h, lent):
        seen["mixer"] = h
        return t64([10.0, 0.0])

    def fake_ff(w_, p, h):
        seen["ff"] = h
        return t64([0.0, 100.0])

    def fake_side(w_, p, x, e, eps):
        seen["side"], seen["e"] = x, e
        return t64([1000.0, 1000.0])
    P.mixer, P.feed_forward, P.token_side = fake_mixer, fake_ff, fake_side
    try:
        w = {"l0.norm1": torch.zeros(2, dtype=F64), "l0.norm2": torch.ones(2, dtype=F64), "side.embed": t64([4.0], [5.0])}
        out = P.layer_forward(cfg, w, 0, t64([1.0, 2.0]), torch.tensor([1]), {})
    finally:
        P.mixer, P.feed_forward, P.token_side = real
    assert torch.allclose(seen["ff"], 2 * seen["mixer"]) and torch.equal(seen["side"], t64([11.0, 102.0]))
    assert seen["e"].tolist() == [[5.0]] and torch.equal(out, t64([1011.0, 1102.0]))
