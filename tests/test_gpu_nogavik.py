"""Nogavik on the GPU against the plain float64 model (plain_nogavik.py): each
mechanism alone; whole prompts; token-by-token decoding from the first token;
portions down to two tokens; batches of unequal requests; pages and slots used
again; keys far away and at the edges of pages, also through a latent that another
layer cached; the first tokens; states that remember the first token through long
decoding; long decoding through graphs; drawn configurations; greedy generation
through the scheduler; the command line and the trace program."""
import json
import os
import random
import subprocess
import sys

import pytest
import torch

import plain_nogavik as P
from nogavik_util import (CONFIGS, dense, latent_layer, left, mamba_layer, model_folder, parallel_layer, random_tokens, right,
                          set_tensors, write_folder)
from tiny import nmse, read_weights

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# float32: the engine against the float64 plain model.  bfloat16: against the plain model (activations are not
# rounded there, so the bound is that of 16-bit activations through a few layers).
BOUND = {"float32": 1e-9, "bfloat16": 2e-3}
DTYPES = ["float32", "bfloat16"]


def f64(w):
    return {k: (v.double() if v.is_floating_point() else v) for k, v in w.items()}


def weights_for(name):
    return read_weights(model_folder(name))


_plain = {}


def plain_logits(name, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        with torch.no_grad():
            _plain[key] = P.forward(CONFIGS[name], weights_for(name), list(tokens))
    return _plain[key]


def engine_for(name, dtype, **kw):
    from kipp_b200.engine import Engine
    opts = dict(dtype=dtype, page_size=16, cache_tokens=1024, max_requests=4, max_batch_tokens=1024)
    opts.update(kw)
    return Engine.from_folder(model_folder(name), **opts)


def close(got, want, dtype, what="", factor=1.0):
    e = nmse(got.cpu(), want)
    assert e <= BOUND[dtype] * factor, f"{what}: NMSE {e:.3e} > {BOUND[dtype] * factor:.1e}"


def _inputs(name, T, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(T, CONFIGS[name]["width"], generator=g, dtype=torch.float64)


def layers_of(kind):
    return [(n, i) for n in sorted(CONFIGS) for i, l in enumerate(CONFIGS[n]["layers"]) if l["type"] == kind]


def _in_portions(eng, layer, part, h_dev, sizes, rid="a"):
    """The part's output over consecutive portions of one request."""
    from kipp_b200.engine import StepEntry
    out, at = torch.zeros(h_dev.shape[0], h_dev.shape[1], device="cuda"), 0
    for n in sizes:
        eng.run_part([StepEntry(rid, [0] * n, [])], layer, part, input=h_dev[at:at + n].contiguous(), residual=out[at:at + n])
        at += n
    assert at == h_dev.shape[0]
    return out


# ------------------------------------------------------------------ each mechanism alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [x for x in layers_of("latent_attention")
                                        if CONFIGS[x[0]]["layers"][x[1]]["mixer"].get("kv_from") is None])
def test_latent_attention_alone(name, layer, dtype):
    """Two norms, the rotation by neighbours, the gate per element: in three portions, the later
    ones read the latents the earlier ones left."""
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = _inputs(name, 150, 100 + layer).to("cuda", eng.dtype).contiguous()
    w, m, p, eps = f64(weights_for(name)), cfg["layers"][layer]["mixer"], f"l{layer}.mix.", cfg["norm"]["eps"]
    h = h_dev.double().cpu()
    want = P.latent_attention(m, w, p, h, eps, P.latent_keys(m, w, p, h, eps))
    close(_in_portions(eng, layer, "mixer", h_dev, (70, 1, 79)), want, dtype, f"{name} layer {layer}")
    counters = eng.info()["counters"]
    # in bfloat16, where rows go by 16 bytes, prompts make the heads' keys and values first; a token does not
    wide = dtype == "bfloat16" and name != "D"
    assert counters["latent_expansions"] == counters["mix_tc_launches"] == (2 if wide else 0)
    if dtype == "bfloat16" and name == "C":
        assert counters["shared_key_launches"] == 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", layers_of("parallel"))
def test_attention_without_positions_alone(name, layer, dtype):
    """Biases before the norms of q and k, no rotation, values of a size of their own (up to 256)."""
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = _inputs(name, 330, 150 + layer).to("cuda", eng.dtype).contiguous()
    want = P.attention(cfg["layers"][layer]["mixer"]["left"], f64(weights_for(name)), f"l{layer}.mix.left.", h_dev.double().cpu(),
                       cfg["norm"]["eps"])
    before = eng.info()["counters"]
    close(_in_portions(eng, layer, "mixer/0", h_dev, (200, 1, 30, 99)), want, dtype, f"{name} layer {layer}")
    after = eng.info()["counters"]
    if dtype == "bfloat16" and name == "C":             # prompts on the tcgen05 kernel, few tokens on the groups' one
        assert after["mix_tc_launches"] - before["mix_tc_launches"] == 2
        assert after["group_launches"] - before["group_launches"] == 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", layers_of("parallel"))
def test_gated_delta_rule_alone(name, layer, dtype):
    """The state and the convolutions' last inputs cross every cut: portions shorter than the
    convolutions' reach, of one token, and long ones."""
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = _inputs(name, 130, 200 + layer).to("cuda", eng.dtype).contiguous()
    want = P.gated_delta(cfg["layers"][layer]["mixer"]["right"], f64(weights_for(name)), f"l{layer}.mix.right.", h_dev.double().cpu(),
                         cfg["norm"]["eps"])
    close(_in_portions(eng, layer, "mixer/1", h_dev, (1, 2, 1, 1, 3, 17, 2, 39, 64)), want, dtype, f"{name} layer {layer}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", layers_of("mamba2"))
def test_state_space_alone(name, layer, dtype):
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = _inputs(name, 66, 250 + layer).to("cuda", eng.dtype).contiguous()
    want = P.mamba2(cfg["layers"][layer]["mixer"], f64(weights_for(name)), f"l{layer}.mix.", h_dev.double().cpu(), cfg["norm"]["eps"])
    close(_in_portions(eng, layer, "mixer", h_dev, (1, 2, 1, 1, 3, 17, 2, 39)), want, dtype, f"{name} layer {layer}")


def test_decays_and_write_rates_far_from_the_middle(tmp_path):
    """Decays from almost nothing kept to almost all, write rates near 0 and 1, softplus at both of its
    ends: the state follows the equations over 80 tokens."""
    from kipp_b200.engine import Engine
    cfg = {"architecture": "Nogavik", "vocab": 50, "width": 32, "norm": {"eps": 1e-5},
           "layers": [parallel_layer(left(1, 1, 8, 8, 0.5), right(2, 1, 12, 16, 4, 6, 4), None)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=4, sigma=0.5, norm_jitter=0.1))
    bias = torch.linspace(-30.0, 30.0, 24)
    set_tensors(folder, {"l0.mix.right.A_log": torch.tensor([-6.0, 1.0]), "l0.mix.right.dt_bias": bias,
                         "l0.mix.right.b": read_weights(folder)["l0.mix.right.b"] * 4.0})
    w = f64(read_weights(folder))
    h = 2.0 * torch.randn(80, 32, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    *_, beta, g = P.delta_vectors(cfg["layers"][0]["mixer"]["right"], w, "l0.mix.right.", h.float().double())
    assert float(beta.min()) < 0.01 and float(beta.max()) > 0.99 and float(g.min()) < 1e-6 and float(g.max()) > 1 - 1e-6
    want = P.gated_delta(cfg["layers"][0]["mixer"]["right"], w, "l0.mix.right.", h.float().double(), 1e-5)
    eng = Engine.from_folder(folder, dtype="float32", page_size=16, cache_tokens=128, max_requests=1, max_batch_tokens=128, cuda_graphs=False)
    close(_in_portions(eng, 0, "mixer/1", h.float().cuda().contiguous(), (40, 1, 39)), want, "float32", "far from the middle")


def test_states_and_convolutions_start_from_zeros_in_a_slot_used_again():
    """A second request in the slot the first one gave back: no input and no state of the first."""
    name = "A"
    cfg, w = CONFIGS[name], f64(weights_for(name))
    for layer, part, fn in ((3, "mixer", lambda h: P.mamba2(cfg["layers"][3]["mixer"], w, "l3.mix.", h, 1e-5)),
                            (1, "mixer/1", lambda h: P.gated_delta(cfg["layers"][1]["mixer"]["right"], w, "l1.mix.right.", h, 1e-5))):
        eng = engine_for(name, "float32", cuda_graphs=False, max_requests=1)
        for k, rid in enumerate(("first", "second")):
            h_dev = _inputs(name, 9, 700 + k).to("cuda", eng.dtype).contiguous()
            close(_in_portions(eng, layer, part, h_dev, (2, 7), rid), fn(h_dev.double().cpu()), "float32", f"layer {layer} {rid}")
            eng.finish(rid)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("B", 4), ("C", 1), ("D", 1)])
def test_feed_forward_and_its_norm_alone(name, layer, dtype):
    from kipp_b200.engine import StepEntry
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    w = f64(weights_for(name))
    T = 97
    x = _inputs(name, T, 300 + layer).float()
    h_dev = torch.zeros(T, cfg["width"], device="cuda", dtype=eng.dtype)
    eng.run_part([StepEntry("n", [0] * T, [])], layer, "post_norm", residual=x.cuda(), output=h_dev)
    eng.finish("n")
    close(h_dev.float(), P.norm_one_plus(x.double(), w[f"l{layer}.norm2"], cfg["norm"]["eps"]), dtype, "norm", factor=0.1)
    out = torch.zeros(T, cfg["width"], device="cuda")
    eng.run_part([StepEntry("f", [0] * T, [])], layer, "feed_forward", input=h_dev, residual=out)
    close(out, P.feed_forward(w, f"l{layer}.mlp.", h_dev.double().cpu()), dtype, f"{name} layer {layer}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer,T", [(n, i, T) for n, i in (("A", 1), ("A", 3), ("B", 0), ("C", 3), ("D", 0), ("D", 2), ("E", 1))
                                          for T in ((1, 3, 21, 64, 1100) if n in "AD" else (1, 17, 40))])
def test_a_layer_alone(name, layer, T, dtype):
    """Norms, mixer, feed-forward and the token's own embedding of that layer, in steps small and large: the
    stream in and out."""
    from kipp_b200.engine import StepEntry
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False, cache_tokens=2048, max_batch_tokens=2048)
    toks = random_tokens(cfg["vocab"], T, seed=8)
    x_dev = _inputs(name, T, 900 + layer).float().cuda().contiguous()
    with torch.no_grad():
        want = P.layer_forward(cfg, f64(weights_for(name)), layer, x_dev.double().cpu(), torch.tensor(toks), {})
    eng.run_part([StepEntry("b", toks, [])], layer, "block", residual=x_dev)
    close(x_dev, want, dtype, f"{name} layer {layer}")
    # few tokens: the token side is one kernel, where the width goes by 32
    few = dtype == "bfloat16" and T <= 64 and name in ("A", "B", "C")
    assert eng.info()["counters"]["token_side_launches"] == (1 if few else 0)


def test_the_token_side_shows(tmp_path):
    """Another layer's columns of the table, or another token's row, is another result: the
    stream after every layer against the plain model's, with token sides that outweigh it."""
    from kipp_b200.engine import StepEntry
    cfg, w = CONFIGS["A"], weights_for("A")
    toks = random_tokens(cfg["vocab"], 25, seed=3)
    layers = []
    with torch.no_grad():
        P.forward(cfg, w, toks, layers)
        d, moved = cfg["token_side"]["dim"], dict(w)
        moved["side.embed"] = torch.roll(w["side.embed"], d, dims=1)
        assert nmse(P.forward(cfg, moved, toks), P.forward(cfg, w, toks)) > 1e-2
    eng = engine_for("A", "float32", cuda_graphs=False)
    x = torch.zeros(25, cfg["width"], device="cuda")
    eng.run_part([StepEntry("e", toks, [])], 0, "embedding", residual=x)
    eng.finish("e")
    for i in (0, 1):                                     # (a layer that reads another's latent needs the whole step)
        eng.run_part([StepEntry(f"s{i}", toks, [])], i, "block", residual=x)
        eng.finish(f"s{i}")
        assert nmse(x.cpu(), layers[i]) <= 1e-9, f"layer {i}"


# ------------------------------------------------------------------ whole models
LENGTH = {"A": 90, "B": 131, "C": 330, "D": 70, "E": 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_way_of_cutting_it(name, dtype):
    """Whole; token by token from the very first token; portions down to two
    tokens: every position against the plain model, and (32-bit) the ways of
    cutting against one another."""
    from kipp_b200.engine import StepEntry
    toks = random_tokens(CONFIGS[name]["vocab"], LENGTH[name], seed=1)
    want = plain_logits(name, toks)
    eng = engine_for(name, dtype)
    n = len(toks)
    whole = eng.step([StepEntry("w", toks, list(range(n)))], check=True).clone()
    eng.finish("w")
    close(whole, want, dtype, "whole")
    rows = [eng.step([StepEntry("t", [t], [0])]).clone() for t in toks]
    eng.synchronize()
    eng.finish("t")
    single = torch.cat(rows)
    close(single, want, dtype, "token by token")
    cut, at, i = [], 0, 0
    sizes = [2, 7, 2, 19, 3, 33, 2, 16, 17, 5, 64]
    while at < n:
        k = min(sizes[i % len(sizes)], n - at)
        cut.append(eng.step([StepEntry("c", toks[at:at + k], list(range(k)))]).clone())
        at, i = at + k, i + 1
    eng.synchronize()
    eng.finish("c")
    cut = torch.cat(cut)
    close(cut, want, dtype, "portions")
    if dtype == "float32":
        assert nmse(single.cpu(), whole.cpu()) <= 1e-10 and nmse(cut.cpu(), whole.cpu()) <= 1e-10


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(name, dtype):
    """Six requests through two slots and a cache that holds two of them: portions
    of one beside decoded tokens of another; every request's logits are those of
    the request alone (states, kept inputs and pages of a slot's last owner are gone)."""
    from kipp_b200.engine import StepEntry
    vocab = CONFIGS[name]["vocab"]
    lengths = [37, 64, 5, 90, 18, 71]
    seqs = {f"r{i}": random_tokens(vocab, n, seed=20 + i) for i, n in enumerate(lengths)}
    eng = engine_for(name, dtype, cache_tokens=256, max_requests=2, max_batch_tokens=256)
    waiting, live, got = list(seqs), {}, {r: [] for r in seqs}
    tick = 0
    while waiting or live:
        while waiting and len(live) < 2:
            live[waiting.pop(0)] = 0
        entries = []
        for j, (rid, at) in enumerate(live.items()):
            toks = seqs[rid]
            head = max(len(toks) - 9, 1)
            k = 1 if at >= head else min([13, 2, 30, 5][(tick + j) % 4], head - at)
            entries.append(StepEntry(rid, toks[at:at + k], list(range(k))))
        logits = eng.step(entries, check=True)
        row = 0
        for e in entries:
            k = len(e.tokens)
            got[e.request].append(logits[row:row + k].clone())
            row += k
            live[e.request] += k
            if live[e.request] == len(seqs[e.request]):
                eng.finish(e.request)
                del live[e.request]
        eng.cache.check()
        tick += 1
    alone = engine_for(name, dtype)
    for rid, toks in seqs.items():
        close(torch.cat(got[rid]), plain_logits(name, toks), dtype, rid)
        one = alone.step([StepEntry(rid, toks, list(range(len(toks))))], check=True).clone()
        alone.finish(rid)
        assert nmse(torch.cat(got[rid]).cpu(), one.cpu()) <= (1e-10 if dtype == "float32" else BOUND[dtype]), rid


def test_a_request_left_out_of_a_step_goes_on_later():
    """Requests take turns: the one that pauses finds its states, its kept inputs and its
    pages as it left them, whatever the others did meanwhile."""
    from kipp_b200.engine import StepEntry
    name = "A"
    a, b = random_tokens(300, 50, seed=31), random_tokens(300, 44, seed=32)
    eng = engine_for(name, "float32")
    got_a, got_b = [], []
    got_a.append(eng.step([StepEntry("a", a[:7], list(range(7)))]).clone())
    got_b.append(eng.step([StepEntry("b", b[:30], list(range(30)))]).clone())
    lg = eng.step([StepEntry("a", a[7:20], list(range(13))), StepEntry("b", b[30:31], [0])]).clone()
    got_a.append(lg[:13])
    got_b.append(lg[13:])
    got_b.append(eng.step([StepEntry("b", b[31:], list(range(13)))]).clone())
    got_a.append(eng.step([StepEntry("a", a[20:], list(range(30)))], check=True).clone())
    close(torch.cat(got_a), plain_logits(name, a), "float32", "a")
    close(torch.cat(got_b), plain_logits(name, b), "float32", "b")


# ------------------------------------------------------------------ edges, made to show
def _run_both_ways(cfg, folder, dtype, toks, edges, first=11):
    """Every position as a prompt and decoded one by one; those of `edges` are judged one by one."""
    from kipp_b200.engine import Engine, StepEntry
    w = read_weights(folder)
    with torch.no_grad():
        want = P.forward(cfg, w, toks)
    n = len(toks)
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=2 * n + 64, max_requests=2, max_batch_tokens=max(n, 64))
    whole = eng.step([StepEntry("w", toks, list(range(n)))], check=True).clone()
    close(whole, want, dtype, "prompt")
    head = eng.step([StepEntry("d", toks[:first], list(range(first)))]).clone()
    rows = torch.cat([head] + [eng.step([StepEntry("d", [t], [0])]).clone() for t in toks[first:]])
    eng.synchronize()
    close(rows, want, dtype, "decoded")
    row_bound = BOUND[dtype] * (10 if dtype == "bfloat16" else 1)
    for pos in set(edges) & set(range(n)):
        for what, got in (("prompt", whole), ("decoded", rows)):
            e = nmse(got[pos:pos + 1].cpu(), want[pos:pos + 1])
            assert e <= row_bound, f"{what} position {pos}: NMSE {e:.3e}"
    return w, want


EDGES = [0, 1, 15, 16, 17, 31, 32, 63, 64, 127, 128, 511, 512, 590, 599]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds_in_the_attention_without_positions(dtype, tmp_path):
    """600 different tokens.  The query projection is the key projection behind a shift of the
    width's coordinates, and the embeddings of ten tokens of the first page are the shifted
    embeddings of the last ten: each of the last queries meets ONE key hundreds of positions back
    with a score far above all others.  Rows at page borders are judged one by one."""
    cfg = {"architecture": "Nogavik", "vocab": 640, "width": 48, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
           "layers": [parallel_layer(left(4, 2, 16, 24, 1.0), right(2, 1, 8, 8, 2, 8, 8), None)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=77, sigma=0.3, norm_jitter=0.1))
    toks = torch.randperm(640, generator=torch.Generator().manual_seed(9))[:600].tolist()
    w0 = read_weights(folder)
    k, embed = w0["l0.mix.left.k"], w0["embed"].clone()       # k: [2 kv heads x 16, width]; head h reads kv head h // 2
    embed[toks[3:13]] = torch.roll(embed[toks[590:600]], 1, dims=1)
    q = torch.roll(k, -1, dims=1).view(2, 1, 16, 48).expand(2, 2, 16, 48).reshape(64, 48).clone()
    kb = w0["l0.mix.left.k.b"].view(2, 1, 16).expand(2, 2, 16).reshape(64).clone()
    set_tensors(folder, {"l0.mix.left.q": q, "l0.mix.left.q.b": kb, "embed": embed, "l0.norm1": torch.zeros(48)})
    w, want = _run_both_ways(cfg, folder, dtype, toks, EDGES)
    if dtype == "float32":                                # without the first page's keys the last rows are other rows
        with torch.no_grad():
            assert nmse(P.forward(cfg, w, toks[16:])[-5:], want[-5:]) > 1e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("through_another_layer", [False, True])
def test_a_far_latent_among_hundreds(dtype, through_another_layer, tmp_path):
    """The same through the latent: W_dq is W_dkv behind the shift and W_uq makes every head's plain query the
    key of that latent.  Through another layer: the latent is the one layer 0 cached (its own output is nothing), the
    queries are layer 1's."""
    R = 16
    lent = latent_layer(3, 16, 4, 24, R, R, 0.25, None, base=50.0)
    layers = [lent] + ([latent_layer(2, 16, 4, 24, R, R, 4.0, None, base=50.0, kv_from=0)] if through_another_layer else [])
    if not through_another_layer:
        layers[0]["mixer"]["scale"] = 4.0
    cfg = {"architecture": "Nogavik", "vocab": 640, "width": 48, "norm": {"eps": 1e-5}, "layers": layers}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=78, sigma=0.3, norm_jitter=0.1))
    toks = torch.randperm(640, generator=torch.Generator().manual_seed(9))[:600].tolist()
    w0 = read_weights(folder)
    i = len(layers) - 1                                    # the layer whose queries ask
    H = layers[i]["mixer"]["heads"]
    embed = w0["embed"].clone()
    embed[toks[3:13]] = torch.roll(embed[toks[590:600]], 1, dims=1)
    uq = torch.zeros(H, 20, R)
    uq[:, :16] = torch.eye(16)
    changed = {"embed": embed, f"l{i}.mix.dq": torch.roll(w0["l0.mix.dkv"][:R], -1, dims=1), f"l{i}.mix.uq": uq.view(H * 20, R),
               f"l{i}.mix.uk": torch.eye(16).repeat(H, 1), f"l{i}.norm1": torch.zeros(48), "l0.norm1": torch.zeros(48),
               f"l{i}.mix.dq.norm": torch.ones(R), "l0.mix.dkv.norm": torch.ones(R)}
    if through_another_layer:
        changed["l0.mix.o"] = torch.zeros_like(w0["l0.mix.o"])
    set_tensors(folder, changed)
    w, want = _run_both_ways(cfg, folder, dtype, toks, EDGES)
    if dtype == "float32":
        with torch.no_grad():
            assert nmse(P.forward(cfg, w, toks[16:])[-5:], want[-5:]) > 1e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(dtype):
    """Positions 0, 1, 2: one key; convolutions that reach back beyond position 0; a state of nothing."""
    from kipp_b200.engine import StepEntry
    for name in ("A", "D"):
        toks = random_tokens(CONFIGS[name]["vocab"], 3, seed=70)
        eng = engine_for(name, dtype)
        for cuts in ([3], [1, 1, 1], [1, 2], [2, 1]):
            rows, at = [], 0
            for k in cuts:
                rows.append(eng.step([StepEntry("f", toks[at:at + k], list(range(k)))], check=True).clone())
                at += k
            eng.finish("f")
            close(torch.cat(rows), plain_logits(name, toks), dtype, f"{name} {cuts}", factor=5 if dtype == "bfloat16" else 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["mamba2", "gated_delta"])
def test_a_state_that_keeps_the_first_token_through_long_decoding(kind, dtype, tmp_path):
    """Decays next to one: what the first token wrote is still in the state 300 tokens on, so a
    state lost, reset or carried to the wrong slot shows at the end."""
    from kipp_b200.engine import Engine, StepEntry
    layer = mamba_layer(2, 1, 16, 8, 3, 2, None) if kind == "mamba2" else \
        parallel_layer(left(1, 1, 8, 8, 0.5), right(2, 1, 32, 16, 3, 8, 8), None)
    cfg = {"architecture": "Nogavik", "vocab": 60, "width": 32, "norm": {"eps": 1e-5}, "layers": [layer]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=6, sigma=0.4, norm_jitter=0.1))
    if kind == "mamba2":
        set_tensors(folder, {"l0.mix.A_log": torch.tensor([-9.0, -7.0]), "l0.mix.dt_bias": torch.tensor([-1.0, 0.5])})
    else:                                                  # small write rates too, so that later writes do not take it out again
        w0 = read_weights(folder)
        set_tensors(folder, {"l0.mix.right.A_log": torch.tensor([-9.0, -9.0]), "l0.mix.right.b": w0["l0.mix.right.b"] * 3.0,
                             "l0.mix.left.o": torch.zeros_like(w0["l0.mix.left.o"])})
    w = read_weights(folder)
    toks = random_tokens(60, 300, seed=13)
    other = [(toks[0] + 1) % 60] + toks[1:]
    with torch.no_grad():
        want, moved = P.forward(cfg, w, toks), P.forward(cfg, w, other)
    at = 300 if kind == "mamba2" else 40                    # the delta rule takes old writes out as new keys meet them
    assert nmse(moved[at - 1:at], want[at - 1:at]) > 1e-6   # the first token still counts there
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=1024, max_requests=2, max_batch_tokens=64)
    # two requests decode side by side; the second one's state must not leak into the first
    rows = [eng.step([StepEntry("x", [t], [0]), StepEntry("y", [other[i]], [0])]).clone() for i, t in enumerate(toks)]
    eng.synchronize()
    got = torch.stack(rows)                                 # [T, 2, vocab]
    close(got[:, 0], want, dtype, "first request")
    close(got[:, 1], moved, dtype, "second request")
    for pos in (at - 1, 299):
        e = nmse(got[pos:pos + 1, 0].cpu(), want[pos:pos + 1])
        assert e <= BOUND[dtype] * (10 if dtype == "bfloat16" else 1), f"position {pos}: {e:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_of_a_batch_through_graphs(dtype):
    """Three requests of unequal prompts decode 150 tokens each in one batch (decode steps are
    graph replays); every row against the plain model."""
    from kipp_b200.engine import StepEntry
    name = "A"
    vocab = CONFIGS[name]["vocab"]
    seqs = [random_tokens(vocab, n, seed=40 + n) for n in (155, 171, 190)]
    heads = [5, 21, 40]
    eng = engine_for(name, dtype)
    got = [[] for _ in seqs]
    for i, (s, h) in enumerate(zip(seqs, heads)):
        got[i].append(eng.step([StepEntry(i, s[:h], list(range(h)))]).clone())
    for k in range(150):
        lg = eng.step([StepEntry(i, [s[h + k]], [0]) for i, (s, h) in enumerate(zip(seqs, heads))]).clone()
        for i in range(3):
            got[i].append(lg[i:i + 1])
    eng.synchronize()
    assert eng.graph_replays > 100
    for i, (s, h) in enumerate(zip(seqs, heads)):
        close(torch.cat(got[i]), plain_logits(name, s[:h + 150]), dtype, f"request {i}")


# ------------------------------------------------------------------ sizes nobody chose
def _drawn_config(seed):
    r = random.Random(seed)
    cfg = {"architecture": "Nogavik", "vocab": r.choice([64, 99, 130]), "width": r.choice([32, 40, 48, 60, 72]),
           "norm": {"eps": r.choice([1e-5, 1e-6])}}
    if r.random() < 0.85:
        cfg["token_side"] = {"dim": r.choice([4, 8, 11, 24])}

    def mlp():
        return r.choice([None, dense(r.choice([8, 20, 48])), dense(32)])

    layers, lenders = [], []
    for i in range(r.randint(2, 5)):
        kind = r.choice(["mamba2", "latent", "latent", "parallel", "parallel"])
        if kind == "mamba2":
            groups = r.choice([1, 2])
            heads = groups * r.choice([1, 2])
            vdim = r.choice([4, 6, 16, 32])
            parts = r.choice([p for p in (1, 2, heads, heads * 2) if (heads * vdim) % p == 0])
            layers.append(mamba_layer(heads, groups, vdim, r.choice([3, 8, 16, 24]), r.choice([1, 2, 3, 4]), parts, mlp()))
        elif kind == "latent":
            from_ = r.choice(lenders) if lenders and r.random() < 0.6 else None
            if from_ is None:
                rot, rank, base = r.choice([2, 4, 8, 16]), r.choice([5, 8, 24, 32]), r.choice([100.0, 1e4, 5e5])
                lenders.append(i)
            else:
                m = layers[from_]["mixer"]
                rot, rank, base = m["rot_dim"], m["kv_rank"], m["rot"]["base"]
            dim = r.choice([4, 6, 8, 16, 32])
            layers.append(latent_layer(r.choice([1, 2, 3, 5]), dim, rot, r.choice([dim, 4, 12, 24]), rank, r.choice([6, 16, 24]),
                                       r.choice([0.5, 1.0, 2.0]) * (dim + rot) ** -0.5, mlp(), base, from_))
        else:
            kv, gkv = r.choice([1, 2]), r.choice([1, 2])
            dim, gdim = r.choice([4, 6, 8, 16, 32]), r.choice([4, 7, 8, 16, 40])
            layers.append(parallel_layer(left(kv * r.choice([1, 2, 3]), kv, dim, r.choice([dim, 4, 12, 2 * dim]), dim ** -0.5),
                                         right(gkv * r.choice([1, 2]), gkv, gdim, r.choice([gdim, 4, 12, 24]), r.choice([1, 2, 3, 4, 6]),
                                               r.choice([3, 8, 12]), r.choice([4, 7, 16])), mlp()))
    cfg["layers"] = layers
    return cfg


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations(seed, tmp_path):
    """Configurations nobody chose: 32-bit against the plain model (whole, in portions, and two
    requests in one batch through one cache), bfloat16 whole against the plain model."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = _drawn_config(3000 + seed)
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=seed, sigma=0.15, norm_jitter=0.15))
    a, b = random_tokens(cfg["vocab"], 75, seed=seed), random_tokens(cfg["vocab"], 40, seed=100 + seed)
    w = read_weights(folder)
    with torch.no_grad():
        want_a, want_b = P.forward(cfg, w, a), P.forward(cfg, w, b)
    for dtype in DTYPES:
        eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=192, max_requests=2, max_batch_tokens=128)
        whole = eng.step([StepEntry("w", a, list(range(len(a))))], check=True).clone()
        eng.finish("w")
        close(whole, want_a, dtype, f"{cfg} whole")
        if dtype == "bfloat16":
            continue
        got_a, got_b, at_a, at_b, i = [], [], 0, 0, 0
        sizes_a, sizes_b = [2, 21, 1, 9, 30, 5, 7], [3, 1, 1, 17, 2, 16]
        while at_a < len(a) or at_b < len(b):
            entries = []
            if at_a < len(a):
                k = min(sizes_a[i % len(sizes_a)], len(a) - at_a)
                entries.append(StepEntry("a", a[at_a:at_a + k], list(range(k))))
            if at_b < len(b):
                k = min(sizes_b[i % len(sizes_b)], len(b) - at_b)
                entries.append(StepEntry("b", b[at_b:at_b + k], list(range(k))))
            lg, row = eng.step(entries, check=True), 0
            for e in entries:
                k = len(e.tokens)
                (got_a if e.request == "a" else got_b).append(lg[row:row + k].clone())
                row += k
                if e.request == "a":
                    at_a += k
                else:
                    at_b += k
            i += 1
        close(torch.cat(got_a), want_a, dtype, "a in portions beside b")
        close(torch.cat(got_b), want_b, dtype, "b in portions beside a")
        assert nmse(torch.cat(got_a).cpu(), whole.cpu()) <= 1e-10


# ------------------------------------------------------------------ the framework's entry points
def _greedy(name, prompt, n):
    w, seq = weights_for(name), list(prompt)
    with torch.no_grad():
        for _ in range(n):
            seq.append(int(P.forward(CONFIGS[name], w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(name):
    from kipp_b200.engine.llm import LLM
    vocab = CONFIGS[name]["vocab"]
    prompts = [random_tokens(vocab, n, seed=60 + n) for n in (3, 41, 17, 1, 26)]
    llm = LLM(model_folder(name), dtype="float32", kv_tokens=512, max_requests=3, max_batch_tokens=64, chunk=16)
    out = llm.generate(prompts, decode=12)
    for prompt, result in zip(prompts, out):
        assert result.tokens == _greedy(name, prompt, 12)


def test_the_command_line_generates_greedily_and_samples():
    name = "D"
    vocab = CONFIGS[name]["vocab"]
    a, b = random_tokens(vocab, 9, seed=5), random_tokens(vocab, 27, seed=6)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kipp"), "--model", model_folder(name),
                           "--prompt-ids", ",".join(map(str, a)), "--prompt-ids", ",".join(map(str, b)),
                           "--decode", "5", "--dtype", "float32", "--chunk", "16", "--top", "0"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = [[int(t) for t in line.split("\t")[1].split()] for line in proc.stdout.strip().splitlines()]
    assert got == [_greedy(name, a, 5), _greedy(name, b, 5)]
    assert "prefill_tokens=36" in proc.stderr and "decode_tokens=10" in proc.stderr
    sampled = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kipp"), "--random", "nogavik-tiny",
                              "--prompt-ids", "1,2,3,4,5", "--decode", "8", "--temperature", "0.8", "--top-k", "20",
                              "--seed", "3", "--top", "0"], capture_output=True, text=True, timeout=600)
    assert sampled.returncode == 0, sampled.stderr[-2000:]
    tokens = [int(t) for t in sampled.stdout.strip().splitlines()[0].split("\t")[1].split()]
    assert len(tokens) == 8 and all(0 <= t < 320 for t in tokens)


def test_the_trace_program_runs_the_model_step_by_step(tmp_path):
    import numpy as np
    name = "A"
    vocab = CONFIGS[name]["vocab"]
    toks = random_tokens(vocab, 50, seed=77)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:49], "want": []},
                                     {"id": "y", "tokens": toks[:2], "want": [1]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[49:], "want": [0]},
                                     {"id": "z", "tokens": toks[:3], "want": [2]}], "end": ["x", "z"]}]
    out = str(tmp_path / "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", model_folder(name),
                           "--dtype", "float32", "--out", out, "--max-tokens", "128"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = plain_logits(name, toks)
    read = lambda i: torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, vocab))   # noqa: E731
    close(read(0), want[[0, 29]], "float32", "step 0")
    close(read(1), want[[1]], "float32", "step 1")
    close(read(2), want[[49, 2]], "float32", "step 2")
