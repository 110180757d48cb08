"""Panolorn without a GPU: its configuration checks, its plan (parts, constants,
tensor names and shapes), what its cache keeps, the random-weights writer, and the
plain model's own mechanisms against hand-made cases."""
import copy
import math

import pytest
import torch

from kipp_b200.config import config_from_dict
from kipp_b200.config.base import ConfigError
from kipp_b200.config.registry import get_architecture
from tiny import read_weights
from panolorn_util import CONFIGS, INIT, random_tokens, write_folder

import plain_panolorn as P

F64 = torch.float64


def spec_of(cfg):
    c = config_from_dict(cfg)
    return get_architecture(c.architecture).build(c)


def test_the_model_class_is_chosen_by_the_architecture_key():
    c = config_from_dict(CONFIGS["A"])
    assert c.architecture == "Panolorn" and c.to_dict()["layers"][1]["mixer"]["mask"] == {"size": 21}
    assert config_from_dict(c.to_dict()).to_dict() == c.to_dict()
    assert c.vocab_size == 300 and c.hidden_size == 64


def test_parts_and_their_constants():
    plan = spec_of(CONFIGS["A"]).plan
    assert plan["embedding"][0]["part"]["scale"] == 3.0
    blocks = [l["part"] for l in plan["layers"]]
    assert all(b["kind"] == "sandwich_norm_block" for b in blocks)
    assert [blocks[0][k]["weight_name"] for k in ("input_norm", "mixer_out_norm", "post_norm", "ffn_out_norm")] == \
        ["norm1", "norm1b", "norm2", "norm2b"]
    att = blocks[1]["mixer"]
    assert att["kind"] == "attention" and att["sink"] == "unit" and att["element_gate"] and att["unit_norm"]
    assert (att["softcap"], att["chunk"], att["scale"], att["qk_norm_eps"]) == (10.0, 21, 0.4, 1e-5)
    assert att["position"]["kind"] == "no_position" and att["forget_blocks"]
    assert att["distance_slopes"] == [2.0 ** (-8.0 * (h + 1) / 6) for h in range(6)]
    ffn = blocks[0]["ffn"]
    assert ffn["kind"] == "gated_mlp" and ffn["activation"] == "gelu_tanh" and ffn["up_add"] == 0.0
    ex = blocks[1]["ffn"]
    assert ex["kind"] == "expert_mixture" and ex["routing"] == "sigmoid_scores" and ex["weight_on_input"] and ex["gated"]
    assert (ex["experts"], ex["top"], ex["renormalize"], ex["up_add"]) == (5, 2, False, 0.0)
    assert ex["shared"]["kind"] == "gated_mlp" and ex["shared"]["activation"] == "swish"
    assert blocks[2]["ffn"] is None and blocks[2]["ffn_out_norm"] is None
    head = plan["head"]["part"]
    assert head["tied_to"] == "embed"
    assert [o["layer"] for o in plan["order"]] == [o["cache"] for o in plan["order"]] == [0, 1, 2, 3]
    # what the configuration leaves out
    plan = spec_of(CONFIGS["B"]).plan
    b0 = plan["layers"][0]["part"]
    assert plan["embedding"][0]["part"]["scale"] == 1.0
    m = b0["mixer"]
    assert (m["num_kv_heads"], m["value_dim"], m["softcap"], m["chunk"], m["forget_blocks"]) == (3, 16, 0.0, 0, False)
    assert b0["ffn"].get("shared") is None and plan["layers"][2]["part"]["ffn"]["shared"] is not None


def test_tensor_names_and_shapes():
    specs = {s.name: tuple(s.shape) for s in spec_of(CONFIGS["A"]).tensor_specs() if not (s.optional and s.alias_of)}
    assert specs["embed"] == (300, 64) and specs["final.norm"] == (64,)
    assert specs["l0.mix.q"] == (64, 64) and specs["l0.mix.k"] == (32, 64) and specs["l0.mix.v"] == (48, 64)
    assert specs["l0.mix.g"] == (96, 64) and specs["l0.mix.o"] == (64, 96)
    assert specs["l0.norm1"] == specs["l0.norm1b"] == specs["l0.norm2"] == specs["l0.norm2b"] == (64,)
    assert specs["l0.mlp.gate"] == (96, 64) and specs["l0.mlp.down"] == (64, 96)
    assert specs["l1.mlp.router"] == (5, 64) and specs["l1.mlp.e4.gate"] == (40, 64) and specs["l1.mlp.e4.down"] == (64, 40)
    assert specs["l1.mlp.shared.up"] == (48, 64) and "l1.mlp.e5.up" not in specs and "l3.mlp.shared.up" not in specs
    assert "l2.norm1b" in specs and "l2.norm2" not in specs and "l2.norm2b" not in specs
    assert not any(n.endswith((".sink", "q.norm", "k.norm", ".b")) or "head" in n for n in specs)


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c["embedding"].update(scale="x"), "embedding.scale"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][1]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "mixer.scale"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1), "mixer.softcap"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "router.top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="other"), "mlp.kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "mlp.ff"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "mlp.expert"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "mlp.shared.ff"),
])
def test_what_the_configuration_refuses(change, message):
    cfg = copy.deepcopy(CONFIGS["A"])
    change(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert message in str(e.value)


def test_random_weights_cover_every_declared_tensor(tmp_path):
    folder = write_folder(str(tmp_path / "m"), CONFIGS["D"], INIT["D"])
    w = read_weights(folder)
    specs = {s.name: tuple(s.shape) for s in spec_of(CONFIGS["D"]).tensor_specs() if not (s.optional and s.alias_of)}
    assert {k: tuple(v.shape) for k, v in w.items()} == specs
    with torch.no_grad():
        logits = P.forward(CONFIGS["D"], w, random_tokens(101, 12, seed=1))
    assert logits.shape == (12, 101) and bool(torch.isfinite(logits).all())


def test_the_parts_can_be_described_from_python_for_another_design():
    """A model put together in Python from the descriptions of the same parts (the layers without experts) gives
    the tensors and the parts the library's own builder makes."""
    from kipp_b200.models.spec import LayerRun, ModelSpec
    from kipp_b200.parts import (AttentionMixer, GatedFeedForward, NoPositionEncoding, OutputHead, RMSNorm, SandwichNormBlock,
                                 TokenEmbedding)
    cfg = copy.deepcopy(CONFIGS["A"])
    cfg["layers"] = [cfg["layers"][0], cfg["layers"][2]]
    eps, width = cfg["norm"]["eps"], cfg["width"]
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        mixer = AttentionMixer(width, m["heads"], m["kv_heads"], m["dim"], NoPositionEncoding(), eps, 0, m["scale"],
                               value_dim=m["vdim"], sink="unit", softcap=m["softcap"], unit_norm=True, element_gate=True,
                               distance_slopes=[2.0 ** (-8.0 * (h + 1) / m["heads"]) for h in range(m["heads"])],
                               chunk=m["mask"]["size"], forget_blocks=True, names={"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g"})
        assert mixer.cache_spec().window == m["mask"]["size"]
        n = lambda name: RMSNorm(width, eps, name)                                  # noqa: E731
        ffn = (n("norm2"), GatedFeedForward(width, layer["mlp"]["ff"], activation="gelu_tanh", up_add=0.0), n("norm2b")) \
            if layer["mlp"] else ()
        layers.append((f"l{i}.", SandwichNormBlock(n("norm1"), mixer, n("norm1b"), *ffn)))
    spec = ModelSpec(config=None, hidden_size=width, vocab_size=cfg["vocab"],
                     embedding=TokenEmbedding(cfg["vocab"], width, weight_name="embed", scale=cfg["embedding"]["scale"]),
                     layers=layers, order=[LayerRun(i, i) for i in range(2)], final_norm=("", RMSNorm(width, eps, "final.norm")),
                     head=("", OutputHead(cfg["vocab"], width, tied_to="embed", weight_name="head")))
    theirs = spec_of(cfg)
    assert {s.name: tuple(s.shape) for s in spec.tensor_specs()} == {s.name: tuple(s.shape) for s in theirs.tensor_specs()}
    plan, _ = spec.to_plan()
    assert plan["embedding"][0]["part"]["scale"] == theirs.plan["embedding"][0]["part"]["scale"] == 3.0
    for a, b in zip(plan["layers"], theirs.plan["layers"]):
        assert a["part"]["kind"] == b["part"]["kind"] and a["part"]["names"] == b["part"]["names"]
        for key in ("distance_slopes", "unit_norm", "element_gate", "chunk", "forget_blocks", "softcap", "scale", "sink"):
            assert a["part"]["mixer"][key] == b["part"]["mixer"][key]


def _plan_with(change):
    plan = copy.deepcopy(spec_of(CONFIGS["A"]).plan)
    change(plan["layers"][0]["part"]["mixer"])
    return plan


@pytest.mark.parametrize("change,message", [
    (lambda m: m.update(distance_slopes=[0.5]), "one number per head"),
    (lambda m: m.update(head_gate=True), "exclude each other"),
    (lambda m: m.update(qk_norm_eps=None), "unit_norm needs"),
    (lambda m: m.update(chunk=0), "forget_blocks needs"),
    (lambda m: m.update(head_mix=True), "head_mix"),
])
def test_what_the_attention_part_refuses(change, message):
    import json
    from kipp_b200 import native as N
    with pytest.raises(Exception) as e:
        N.text_result(N.lib().kipp_plan_tensor_specs, json.dumps(_plan_with(change)).encode())
    assert message in str(e.value)


# ------------------------------------------------------------------ the plain model against hand-made cases
def test_plain_blocks_are_counted_from_the_start_of_the_sequence():
    seen = P.same_block(7, 3)
    assert [seen[i].nonzero().flatten().tolist() for i in range(7)] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    assert bool(P.same_block(4, 0).equal(torch.tril(torch.ones(4, 4, dtype=torch.bool))))


def test_plain_softmax_with_one_in_the_denominator():
    s = torch.tensor([[math.log(2.0), math.log(3.0)]], dtype=F64)
    both, first = torch.tensor([[True, True]]), torch.tensor([[True, False]])
    assert torch.allclose(P.softmax_plus_one(s, both), torch.tensor([[2 / 6, 3 / 6]], dtype=F64))
    assert torch.allclose(P.softmax_plus_one(s, first), torch.tensor([[2 / 3, 0.0]], dtype=F64))
    assert torch.allclose(P.softmax_plus_one(s - 900, both), torch.zeros(1, 2, dtype=F64))


def test_plain_attention_of_two_tokens_by_hand():
    """One head over a width of one: unit norm makes every q and k plus or minus one."""
    m = {"heads": 1, "dim": 1, "scale": 2.0, "softcap": 1.5}
    w = {k: torch.tensor([[v]], dtype=F64) for k, v in dict(q=3.0, k=-0.2, v=10.0, g=0.5, o=1.0).items()}
    h = torch.tensor([[1.0], [-2.0]], dtype=F64)
    got = P.attention(m, w, "", h, 1e-12)
    cap = lambda s: 1.5 * math.tanh(s / 1.5)                                          # noqa: E731
    gate = lambda z: 1 / (1 + math.exp(-z))                                            # noqa: E731
    e00 = math.exp(cap(-2.0))                                      # q_0 = 1, k_0 = -1
    e10, e11 = math.exp(cap(2.0) - 2.0 ** -8), math.exp(cap(-2.0))   # q_1 = -1, k_1 = 1; distance 1 costs the slope
    want = [e00 / (1 + e00) * 10.0 * gate(0.5), (e10 * 10.0 - e11 * 20.0) / (1 + e10 + e11) * gate(-1.0)]
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=F64), atol=1e-9)


def test_plain_slopes():
    assert [P.slope(h, 8) for h in (0, 7)] == [0.5, 2.0 ** -8] and P.slope(0, 1) == 2.0 ** -8
    assert P.slope(2, 6) == 2.0 ** -4


def test_plain_routing_keeps_the_scores_and_weighs_the_input():
    f = {"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 1}}
    one = torch.ones(1, 1, dtype=F64)
    w = {"router": torch.tensor([[1.0], [-1.0], [2.0]], dtype=F64)}
    for e in range(3):
        w.update({f"e{e}.gate": one, f"e{e}.up": (e + 1) * one, f"e{e}.down": one})
    h = torch.tensor([[0.7]], dtype=F64)
    chosen, weights = P.route(f, w, "", h)
    s = [1 / (1 + math.exp(-z)) for z in (0.7, -0.7, 1.4)]
    assert chosen.tolist() == [[2, 0]] and torch.allclose(weights, torch.tensor([[s[2], s[0]]], dtype=F64))
    expert = lambda e, x: x / (1 + math.exp(-x)) * (e + 1) * x                         # noqa: E731
    assert abs(float(P.mixture(f, w, "", h)) - expert(2, s[2] * 0.7) - expert(0, s[0] * 0.7)) < 1e-12


def test_plain_gelu_in_its_tanh_form():
    z = torch.tensor([-3.0, -0.5, 0.0, 2.0], dtype=F64)
    assert torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_plain_layer_norms_on_either_side():
    """A sublayer that doubles its input: x + wb n(2 w n(x))."""
    cfg = {"norm": {"eps": 1e-9}, "layers": [{"mixer": {}, "mlp": None}]}
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    w = {"l0.norm1": torch.tensor([1.0, 2.0], dtype=F64), "l0.norm1b": torch.tensor([10.0, 20.0], dtype=F64)}
    real, P.attention = P.attention, lambda m, w_, p, h, eps: 2 * h
    try:
        got = P.layer_forward(cfg, w, 0, x)
    finally:
        P.attention = real
    v = torch.tensor([3.0, 8.0], dtype=F64)
    v = v / torch.sqrt((v * v).mean())
    assert torch.allclose(got, x + v * w["l0.norm1b"], atol=1e-6)
