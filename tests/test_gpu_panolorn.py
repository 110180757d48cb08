"""Panolorn on the GPU against the plain float64 model (plain_panolorn.py): each
mechanism alone; whole prompts; token-by-token decoding from the first token;
portions down to two tokens; batches of unequal requests; pages and slots used
again, also pages of blocks the sequence has left; keys far away, at the edges of
pages and just inside and just outside a block; the sink, the cap and the distance
term; the first tokens; long decoding through graphs; drawn configurations; greedy
generation through the scheduler; the command line and the trace program."""
import copy
import json
import os
import random
import subprocess
import sys

import pytest
import torch

import plain_panolorn as P
from panolorn_util import CONFIGS, attention_layer, dense, model_folder, moe, random_tokens, set_tensors, write_folder
from tiny import nmse, read_weights

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# float32: the engine against the float64 plain model.  bfloat16: against the plain model on the
# same (bfloat16) weights; activations are not rounded there, so the bound is that of 16-bit
# activations through a few layers.
BOUND = {"float32": 1e-9, "bfloat16": 2e-3}


def weights_for(name):
    return read_weights(model_folder(name))


def f64(w):
    return {k: (v.double() if v.is_floating_point() else v) for k, v in w.items()}


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


def close(got, want, dtype, what="", factor=1.0, whole_model=False):
    """whole_model: in bfloat16 a router's close call may go the other way than in the plain model,
    and what that token then leaves in the caches reaches later rows; so the rows of a whole model are
    judged one by one there: half of them within the bound, three quarters within ten times the bound."""
    if whole_model and dtype == "bfloat16":
        g, w = got.cpu().double(), want.cpu().double()
        w = w - w.mean(1, keepdim=True)
        g = g - g.mean(1, keepdim=True)
        rows = (((g - w) ** 2).sum(1) / (w ** 2).sum(1)).sort().values
        n = len(rows)
        median, upper = float(rows[(n - 1) // 2]), float(rows[(3 * (n - 1)) // 4])
        assert median <= BOUND[dtype] * factor and upper <= 10 * BOUND[dtype] * factor, \
            f"{what}: row NMSE median {median:.3e}, third quartile {upper:.3e}"
        return
    e = nmse(got.cpu(), want.cpu())
    assert e <= BOUND[dtype] * factor, f"{what}: NMSE {e:.3e} > {BOUND[dtype] * factor:.1e}"


def _inputs(name, T, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(T, CONFIGS[name]["width"], generator=g, dtype=torch.float64)


LAYERS = [(n, i) for n in sorted(CONFIGS) for i in range(len(CONFIGS[n]["layers"]))]


# ------------------------------------------------------------------ each mechanism alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,layer", LAYERS)
def test_attention_alone(name, layer, dtype):
    """Unit norms, cap, distance term, blocks, sink and gate: in three portions, the later ones
    read the cache the earlier ones left."""
    from kipp_b200.engine import StepEntry
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    T = 150
    h_dev = _inputs(name, T, 100 + layer).to("cuda", eng.dtype).contiguous()
    want = P.attention(cfg["layers"][layer]["mixer"], f64(weights_for(name)), f"l{layer}.mix.", h_dev.double().cpu(), cfg["norm"]["eps"])
    out = torch.zeros(T, cfg["width"], device="cuda")
    at = 0
    for n in (70, 1, 79):
        eng.run_part([StepEntry("a", [0] * n, [])], layer, "mixer", input=h_dev[at:at + n].contiguous(), residual=out[at:at + n])
        at += n
    close(out, want, dtype, f"{name} layer {layer}")


TENSOR_CORE_SIZES = [  # heads, kv heads, key size, value size, cap, block, page
    (4, 2, 128, 128, 20.0, 300, 16), (3, 1, 64, 64, None, 77, 8), (2, 2, 96, 96, 30.0, 130, 16), (4, 1, 40, 104, 5.0, 64, 32),
    (2, 1, 128, 24, 9.0, None, 64), (5, 5, 16, 128, None, None, 16), (2, 1, 72, 64, 15.0, 500, 128), (6, 3, 64, 128, 12.0, 40, 16)]


@pytest.mark.parametrize("heads,kv,dim,vdim,cap,block,page", TENSOR_CORE_SIZES)
def test_prompts_on_the_tensor_cores(heads, kv, dim, vdim, cap, block, page, tmp_path):
    """Portions of more than 64 tokens on the tcgen05 kernel: head sizes that do not fill its tiles, key and
    value tiles of unequal width, every page size, several entries in one step (one of them a single
    token), portions that start anywhere, rows of a tile that see different blocks."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = {"architecture": "Panolorn", "vocab": 30, "width": 64, "norm": {"eps": 1e-5},
           "layers": [attention_layer(heads, kv, dim, vdim, None, 6.0 / dim, cap, block)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=heads + dim, sigma=0.2, norm_jitter=0.1))
    w = f64(read_weights(folder))
    eng = Engine.from_folder(folder, dtype="bfloat16", page_size=page, cache_tokens=2048, max_requests=3, max_batch_tokens=1024,
                             cuda_graphs=False)
    lengths = {"a": 450, "b": 333, "c": 90}
    h = {r: torch.randn(n, 64, generator=torch.Generator().manual_seed(n), dtype=torch.float64).bfloat16() for r, n in lengths.items()}
    want = {r: P.attention(cfg["layers"][0]["mixer"], w, "l0.mix.", h[r].double(), 1e-5) for r in lengths}
    got = {r: torch.zeros(n, 64) for r, n in lengths.items()}
    at, launches = dict.fromkeys(lengths, 0), 0
    for step in ({"a": 200, "b": 129}, {"a": 1, "b": 128, "c": 70}, {"b": 76}, {"a": 249, "c": 20}):
        rows = torch.cat([h[r][at[r]:at[r] + k] for r, k in step.items()]).cuda().contiguous()
        out = torch.zeros(len(rows), 64, device="cuda")
        eng.run_part([StepEntry(r, [0] * k, []) for r, k in step.items()], 0, "mixer", input=rows, residual=out)
        row, out = 0, out.cpu()
        for r, k in step.items():
            got[r][at[r]:at[r] + k] = out[row:row + k]
            row, at[r] = row + k, at[r] + k
        launches += 1
    for r in lengths:
        close(got[r], want[r], "bfloat16", r, factor=0.1)
        worst = (((got[r].double() - want[r]) ** 2).sum(1) / (want[r] ** 2).sum(1)).max()
        assert float(worst) < 2e-3, f"{r}: worst row {float(worst):.2e}"
    assert eng.info()["counters"]["mix_tc_launches"] == launches


@pytest.mark.parametrize("heads,kv,dim,vdim,cap,block,page", [
    (4, 2, 128, 128, 20.0, 300, 16), (3, 1, 64, 64, None, 77, 8), (2, 2, 96, 40, 30.0, 130, 16), (20, 1, 48, 104, 5.0, None, 4),
    (36, 2, 16, 200, 9.0, 50, 64), (5, 5, 32, 8, None, None, 16)])
def test_few_tokens_on_the_tensor_cores(heads, kv, dim, vdim, cap, block, page, tmp_path):
    """Steps of at most 64 tokens (decoded tokens, short portions, both) and a step of 70 single tokens on the
    kernel whose rows are the heads of a group: groups of one head to more than a tile's sixteen, value
    heads up to 200, contexts of several runs of key tiles."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = {"architecture": "Panolorn", "vocab": 30, "width": 64, "norm": {"eps": 1e-5},
           "layers": [attention_layer(heads, kv, dim, vdim, None, 6.0 / dim, cap, block)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=heads + dim, sigma=0.2, norm_jitter=0.1))
    w = f64(read_weights(folder))
    eng = Engine.from_folder(folder, dtype="bfloat16", page_size=page, cache_tokens=8192, max_requests=72, max_batch_tokens=128,
                             cuda_graphs=False)
    h = {r: torch.randn(n, 64, generator=torch.Generator().manual_seed(n), dtype=torch.float64).bfloat16()
         for r, n in (("a", 400), ("b", 170))}
    want = {r: P.attention(cfg["layers"][0]["mixer"], w, "l0.mix.", x.double(), 1e-5) for r, x in h.items()}
    got, at, tick = {r: torch.zeros(len(x), 64) for r, x in h.items()}, dict.fromkeys(h, 0), 0
    while at["a"] < 400:
        step = {"a": min([31, 1, 40, 2, 1][tick % 5], 400 - at["a"]), "b": min([1, 24, 1, 1, 17][tick % 5], 170 - at["b"])}
        step = {r: k for r, k in step.items() if k}
        rows = torch.cat([h[r][at[r]:at[r] + k] for r, k in step.items()]).cuda().contiguous()
        out = torch.zeros(len(rows), 64, device="cuda")
        eng.run_part([StepEntry(r, [0] * k, []) for r, k in step.items()], 0, "mixer", input=rows, residual=out)
        row, out = 0, out.cpu()
        for r, k in step.items():
            got[r][at[r]:at[r] + k] = out[row:row + k]
            row, at[r] = row + k, at[r] + k
        tick += 1
    assert at["b"] == 170
    for r in h:
        close(got[r], want[r], "bfloat16", r, factor=0.1)
        worst = (((got[r].double() - want[r]) ** 2).sum(1) / (want[r] ** 2).sum(1)).max()
        assert float(worst) < 2e-3, f"{r}: worst row {float(worst):.2e}"
        eng.finish(r)
    assert eng.info()["counters"]["group_launches"] == tick
    x = torch.randn(70, 3, 64, generator=torch.Generator().manual_seed(1), dtype=torch.float64).bfloat16()
    for k in range(3):
        out = torch.zeros(70, 64, device="cuda")
        eng.run_part([StepEntry(i, [0], []) for i in range(70)], 0, "mixer", input=x[:, k].cuda().contiguous(), residual=out)
    wanted = torch.stack([P.attention(cfg["layers"][0]["mixer"], w, "l0.mix.", x[i].double(), 1e-5)[2] for i in range(70)])
    close(out, wanted, "bfloat16", "70 single tokens", factor=0.1)
    assert eng.info()["counters"]["group_launches"] == tick + 3


def test_small_queries_and_keys_meet_the_eps_of_their_norm(tmp_path):
    """Projections so small that eps is most of the mean square: the norm is x / sqrt(mean(x^2) + eps)."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = {"architecture": "Panolorn", "vocab": 30, "width": 32, "norm": {"eps": 0.5},
           "layers": [attention_layer(2, 1, 16, 16, None, 2.0)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=2, sigma=0.1, norm_jitter=0.1))
    h = torch.randn(40, 32, generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    w = f64(read_weights(folder))
    want = P.attention(cfg["layers"][0]["mixer"], w, "l0.mix.", h, 0.5)
    assert nmse(P.attention(cfg["layers"][0]["mixer"], w, "l0.mix.", h, 1e-6), want) > 1e-4
    eng = Engine.from_folder(folder, dtype="float32", page_size=16, cache_tokens=64, max_requests=1, max_batch_tokens=64)
    out = torch.zeros(40, 32, device="cuda")
    eng.run_part([StepEntry("a", [0] * 40, [])], 0, "mixer", input=h.float().cuda().contiguous(), residual=out)
    close(out, want, "float32", "eps")


FEED_FORWARDS = [(n, i, T) for n, i in LAYERS if CONFIGS[n]["layers"][i]["mlp"] for T in ((97, 640) if n == "C" else (97,))]


def _sure(mlp, w, p, h, margin):
    """Rows whose choice of experts does not hang on less than `margin`."""
    if mlp["kind"] != "moe" or mlp["router"]["top"] == mlp["router"]["experts"]:
        return torch.ones(h.shape[0], dtype=torch.bool)
    z = torch.sigmoid(h @ w[p + "router"].T).sort(-1, descending=True).values
    top = mlp["router"]["top"]
    return (z[:, top - 1] - z[:, top]) > margin


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,layer,T", FEED_FORWARDS)
def test_feed_forward_alone(name, layer, T, dtype):
    """Dense with gelu; experts chosen by sigmoid scores that weigh the input; the shared expert."""
    from kipp_b200.engine import StepEntry
    cfg = CONFIGS[name]
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = (1.5 * _inputs(name, T, 300 + layer)).to("cuda", eng.dtype).contiguous()
    h_ref = h_dev.double().cpu()
    w = f64(weights_for(name))
    mlp, p = cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    want = P.feed_forward(mlp, w, p, h_ref)
    sure = _sure(mlp, w, p, h_ref, 1e-5)
    assert int(sure.sum()) > T // 2
    out = torch.zeros(T, cfg["width"], device="cuda")
    eng.run_part([StepEntry("f", [0] * T, [])], layer, "feed_forward", input=h_dev, residual=out)
    close(out[sure.cuda()], want[sure], dtype, f"{name} layer {layer}")
    # in bfloat16, sizes that are multiples of 8 run the gated activation inside the products (dense and
    # shared: one each; the experts: their grouped product); 32-bit and odd sizes use the kernel of its own
    fused = eng.info()["counters"]["glu_epilogues"]
    if dtype == "bfloat16" and name in ("A", "B", "C"):
        assert fused == (2 if mlp.get("shared") else 1)
    elif dtype == "float32":
        assert fused == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_weight_on_the_output_is_another_function(dtype):
    """The score multiplies the expert's input: the same score on its output, or divided by the sum of
    the chosen scores, is far from what the engine gives."""
    from kipp_b200.engine import StepEntry
    name, layer = "A", 3
    cfg = CONFIGS[name]
    f, p = cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    eng = engine_for(name, dtype, cuda_graphs=False)
    h_dev = (3.0 * _inputs(name, 40, 17)).to("cuda", eng.dtype).contiguous()
    h, w = h_dev.double().cpu(), f64(weights_for(name))
    sure = _sure(f, w, p, h, 1e-5)
    out = torch.zeros(40, cfg["width"], device="cuda")
    eng.run_part([StepEntry("f", [0] * 40, [])], layer, "feed_forward", input=h_dev, residual=out)
    want = P.feed_forward(f, w, p, h)
    close(out[sure.cuda()], want[sure], dtype)
    chosen, weights = P.route(f, w, p, h)
    on_output = torch.stack([sum(a * P.gated(P.silu, w, f"{p}e{e}.", h[t:t + 1])[0] for e, a in zip(chosen[t].tolist(), weights[t]))
                             for t in range(40)])
    assert nmse(on_output, want) > 0.01
    shares = weights / weights.sum(-1, keepdim=True)
    shared_out = torch.stack([sum(P.gated(P.silu, w, f"{p}e{e}.", a * h[t:t + 1])[0] for e, a in zip(chosen[t].tolist(), shares[t]))
                              for t in range(40)])
    assert nmse(shared_out, want) > 0.01


def test_scores_that_round_to_one_are_still_ordered(tmp_path):
    """Router logits far above zero, where the sigmoid rounds to one in 32 bits: the largest logit wins."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = {"architecture": "Panolorn", "vocab": 30, "width": 32, "norm": {"eps": 1e-5},
           "layers": [attention_layer(2, 1, 16, 16, moe(4, 1, 16), 0.5)]}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=2, sigma=0.3, norm_jitter=0.1))
    router = torch.zeros(4, 32)
    router[:, 0] = torch.tensor([30.0, 32.0, 40.0, 36.0])
    set_tensors(folder, {"l0.mlp.router": router})
    h = torch.randn(20, 32, generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    h[:, 0] = 1.0
    w = f64(read_weights(folder))
    want = P.gated(P.silu, w, "l0.mlp.e2.", h)
    eng = Engine.from_folder(folder, dtype="float32", page_size=16, cache_tokens=64, max_requests=1, max_batch_tokens=64)
    out = torch.zeros(20, 32, device="cuda")
    eng.run_part([StepEntry("f", [0] * 20, [])], 0, "feed_forward", input=h.float().cuda().contiguous(), residual=out)
    close(out, want, "float32", "saturated scores")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 2), ("B", 1), ("C", 1), ("D", 1)])
def test_a_layer_alone(name, layer, dtype):
    """The norms before and after each sublayer and the sums between them."""
    from kipp_b200.engine import StepEntry
    cfg = CONFIGS[name]
    W, T = cfg["width"], 21
    eng = engine_for(name, dtype, cuda_graphs=False)
    x = 2.0 * torch.randn(T, W, generator=torch.Generator().manual_seed(900 + layer), dtype=torch.float64)
    x_dev = x.float().cuda().contiguous()
    with torch.no_grad():
        want = P.layer_forward(cfg, f64(weights_for(name)), layer, x_dev.double().cpu())
    eng.run_part([StepEntry("b", [0] * T, [])], layer, "block", residual=x_dev)
    close(x_dev, want, dtype, f"{name} layer {layer}", factor=3 if dtype == "bfloat16" else 1)


@pytest.mark.parametrize("size", [3, 64, 100, 1000, 4096, 9000, 20001])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("clear", [0, 1])
def test_the_kernel_between_two_sublayers(size, dtype, clear):
    """x += mult wy n(y), h = wh n(x), y cleared or left; rows longer than what a thread keeps."""
    import ctypes
    from kipp_b200.csrc.build import load_library
    f = load_library("elementwise").kipp_norm_add_norm
    f.argtypes = [ctypes.c_void_p, ctypes.c_void_p, ctypes.c_int, ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_float,
                  ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_void_p, ctypes.c_int, ctypes.c_int, ctypes.c_int, ctypes.c_void_p]
    g = torch.Generator().manual_seed(size)
    rows = 5
    x, y = torch.randn(rows, size, generator=g).cuda(), 3 * torch.randn(rows, size, generator=g).cuda()
    wy = (1 + 0.3 * torch.randn(size, generator=g)).bfloat16().cuda()
    wh = (1 + 0.3 * torch.randn(size, generator=g)).cuda()
    h = torch.empty(rows, size, dtype=dtype, device="cuda")
    x0, y0 = x.double(), y.double()
    rc = f(x.data_ptr(), y.data_ptr(), clear, wy.data_ptr(), 1, 1e-5, 0.7, wh.data_ptr(), 0, 1e-3, h.data_ptr(),
           0 if dtype == torch.float32 else 1, rows, size, torch.cuda.current_stream().cuda_stream)
    torch.cuda.synchronize()
    assert rc == 0
    want = x0 + 0.7 * P.norm(y0, wy.double(), 1e-5)
    assert nmse(x.cpu(), want.cpu()) < 1e-12
    assert nmse(h.double().cpu(), P.norm(want, wh.double(), 1e-3).cpu()) < (1e-12 if dtype == torch.float32 else 1e-5)
    assert bool((y == 0).all()) if clear else bool((y.double() == y0).all())


# ------------------------------------------------------------------ whole models
LENGTH = {"A": 130, "B": 131, "C": 330, "D": 70}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    close(whole, want, dtype, "whole", whole_model=True)
    rows = [eng.step([StepEntry("t", [t], [0])]).clone() for t in toks]
    eng.synchronize()
    eng.finish("t")
    single = torch.cat(rows)
    close(single, want, dtype, "token by token", whole_model=True)
    cut, at, i = [], 0, 0
    sizes = [2, 7, 2, 19, 3, 33, 2, 16, 17, 5, 64]
    while at < n:
        k = min(sizes[i % len(sizes)], n - at)
        cut.append(eng.step([StepEntry("c", toks[at:at + k], list(range(k)))]).clone())
        at, i = at + k, i + 1
    eng.synchronize()
    eng.finish("c")
    cut = torch.cat(cut)
    close(cut, want, dtype, "portions", whole_model=True)
    if dtype == "float32":
        assert nmse(single.cpu(), whole.cpu()) <= 1e-10 and nmse(cut.cpu(), whole.cpu()) <= 1e-10


def test_the_stream_after_every_layer():
    from kipp_b200.engine import StepEntry
    name = "A"
    cfg = CONFIGS[name]
    toks = random_tokens(cfg["vocab"], 45, seed=3)
    streams = []
    with torch.no_grad():
        P.forward(cfg, weights_for(name), toks, streams)
    eng = engine_for(name, "float32", cuda_graphs=False)
    x = torch.zeros(len(toks), cfg["width"], device="cuda")
    eng.run_part([StepEntry("e", toks, [])], 0, "embedding", residual=x)
    eng.finish("e")
    close(x, P.embed(cfg, f64(weights_for(name)), toks), "float32", "embedding")
    for r in range(len(cfg["layers"])):
        eng.run_part([StepEntry(f"s{r}", [0] * len(toks), [])], r, "block", residual=x)
        eng.finish(f"s{r}")
        assert nmse(x.cpu(), streams[r]) <= 1e-9, f"layer {r}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(name, dtype):
    """Six requests through two slots and a cache that holds two of them: portions
    of one beside decoded tokens of another; every request's logits are those of
    the request alone."""
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
    # 32-bit: against the plain model.  bfloat16: against the same engine running the request
    # alone in one step (what the batch, the slots and the pages must not do is change a
    # request's own result).
    alone = engine_for(name, dtype) if dtype == "bfloat16" else None
    for rid, toks in seqs.items():
        if alone is None:
            close(torch.cat(got[rid]), plain_logits(name, toks), dtype, rid)
        else:
            want = alone.step([StepEntry(rid, toks, list(range(len(toks))))], check=True).clone()
            alone.finish(rid)
            close(torch.cat(got[rid]), want, dtype, rid, whole_model=True)
    info = eng.info()
    assert info["free_slots"] == 2 and all(g["free_pages"] == g["pages"] for g in info["cache_groups"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_of_blocks_left_behind_serve_again(dtype, tmp_path):
    """Two requests of 300 tokens through a pool that could not hold either of them: a block's pages go
    back once the sequence has left it, and are used again by the same and by the other request."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = {"architecture": "Panolorn", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0},
           "layers": [attention_layer(4, 2, 16, 16, dense(40), 0.5, 9.0, 40)] * 2}
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=31, sigma=0.2, norm_jitter=0.1))
    seqs = [random_tokens(90, 300, seed=s) for s in (1, 2)]
    with torch.no_grad():
        want = [P.forward(cfg, read_weights(folder), s) for s in seqs]
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=192, max_requests=2, max_batch_tokens=64)
    got, at, sizes = [[], []], [0, 0], [11, 1, 2, 17, 1, 5, 23]
    tick = 0
    while min(at) < 300:
        entries = []
        for r in (0, 1):
            k = min(sizes[(tick + 3 * r) % len(sizes)], 300 - at[r])
            if k:
                entries.append(StepEntry(r, seqs[r][at[r]:at[r] + k], list(range(k))))
        lg, row = eng.step(entries, check=True), 0
        for e in entries:
            k = len(e.tokens)
            got[e.request].append(lg[row:row + k].clone())
            row += k
            at[e.request] += k
        eng.cache.check()
        tick += 1
    group = eng.info()["cache_groups"][0]
    assert group["window"] == 40 and group["pages"] <= 14 and len(eng.info()["cache_groups"]) == 1
    for r in (0, 1):
        close(torch.cat(got[r]), want[r], dtype, f"request {r}")


def test_a_request_left_out_of_a_step_goes_on_later():
    from kipp_b200.engine import StepEntry
    name = "A"
    a, b = random_tokens(300, 50, seed=31), random_tokens(300, 44, seed=32)
    eng = engine_for(name, "float32")
    got_a, got_b = [], []
    got_a.append(eng.step([StepEntry("a", a[:7], list(range(7)))]).clone())
    got_b.append(eng.step([StepEntry("b", b[:30], list(range(30)))]).clone())
    lg = eng.step([StepEntry("a", a[7:20], list(range(13))), StepEntry("b", b[30:31], [0])]).clone()
    got_a.append(lg[:13]); got_b.append(lg[13:])
    got_b.append(eng.step([StepEntry("b", b[31:], list(range(13)))]).clone())
    got_a.append(eng.step([StepEntry("a", a[20:], list(range(30)))], check=True).clone())
    close(torch.cat(got_a), plain_logits(name, a), "float32", "a")
    close(torch.cat(got_b), plain_logits(name, b), "float32", "b")


# ------------------------------------------------------------------ edges, made to show
def _run_both_ways(cfg, folder, dtype, toks, edges, first=11):
    """The prompt whole, then the same positions decoded one by one after a portion that ends inside the
    first page; every row at an edge judged alone."""
    from kipp_b200.engine import Engine, StepEntry
    w = read_weights(folder)
    with torch.no_grad():
        want = P.forward(cfg, w, toks)
    n = len(toks)
    eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=2 * n + 64, max_requests=2,
                             max_batch_tokens=max(n, 64))
    whole = eng.step([StepEntry("w", toks, list(range(n)))], check=True).clone()
    close(whole, want, dtype, "prompt")
    head = eng.step([StepEntry("d", toks[:first], list(range(first)))]).clone()
    rows = torch.cat([head] + [eng.step([StepEntry("d", [t], [0])]).clone() for t in toks[first:]])
    eng.synchronize()
    close(rows, want, dtype, "decoded")
    bound = BOUND[dtype] * (10 if dtype == "bfloat16" else 1)
    for pos in set(edges) & set(range(n)):
        for what, got in (("prompt", whole), ("decoded", rows)):
            e = nmse(got[pos:pos + 1].cpu(), want[pos:pos + 1])
            assert e <= bound, f"{what} position {pos}: NMSE {e:.3e}"
    return w, want


def _shifted_model(folder, cfg, seed, pairs, toks):
    """A one-layer model in which the query projection is the key projection behind a shift of the width's
    coordinates; for every (query position, key position) of `pairs` the key's token is given the shifted
    embedding of the query's, so that this one score is as large as a score can be."""
    m = cfg["layers"][0]["mixer"]
    W, G = cfg["width"], m["kv_heads"]
    write_folder(folder, cfg, dict(seed=seed, sigma=0.3, norm_jitter=0.1))
    w = read_weights(folder)
    k, embed = w["l0.mix.k"], w["embed"].clone()
    for query, key in pairs:
        embed[toks[key]] = torch.roll(embed[toks[query]], 1)
    q = torch.roll(k, -1, dims=1).view(G, 1, m["dim"], W).expand(G, m["heads"] // G, m["dim"], W).reshape(-1, W).clone()
    set_tensors(folder, {"l0.mix.q": q, "embed": embed, "l0.norm1": torch.ones(W)})


def _one_layer(scale=1.0, softcap=None, block=None, vocab=97, heads=4, vdim=8):
    return {"architecture": "Panolorn", "vocab": vocab, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
            "layers": [attention_layer(heads, 2, 16, vdim, None, scale, softcap, block)]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("vdim", [8, 16])
def test_a_far_key_among_hundreds_and_the_edges_of_pages(vdim, dtype, tmp_path):
    """600 different tokens; each of the last ten meets ONE key of the first page, hundreds of positions
    back, with a score above all others (the last heads' distance terms are small).  vdim 16 runs the
    prompt on the tensor cores, 8 on the CUDA cores."""
    cfg = _one_layer(scale=1.0, vocab=640, vdim=vdim)
    toks = torch.randperm(640, generator=torch.Generator().manual_seed(9))[:600].tolist()
    folder = str(tmp_path / "m")
    _shifted_model(folder, cfg, 77, [(590 + i, 3 + i) for i in range(10)], toks)
    w, want = _run_both_ways(cfg, folder, dtype, toks, edges=[15, 16, 17, 31, 32, 63, 64, 511, 512, 590, 599])
    if dtype == "float32":                                 # the far keys matter
        with torch.no_grad():
            cut = P.forward(cfg, w, toks[16:])
        assert nmse(cut[-5:], want[-5:]) > 1e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("block,vdim", [(37, 8), (48, 16), (64, 16), (33, 16)])
def test_keys_just_inside_and_just_outside_a_block(block, vdim, dtype, tmp_path):
    """In every block the last query is drawn to the block's first key (just inside), and the first query
    to the last key of the block before (just outside).  A block one position longer or shorter, or
    blocks counted from elsewhere, give other rows there."""
    cfg = _one_layer(scale=1.0, block=block, vocab=400, vdim=vdim)
    n = 5 * block + 3
    toks = torch.randperm(400, generator=torch.Generator().manual_seed(block))[:n].tolist()
    starts = range(block, n, block)
    pairs = [(s + block - 1, s) for s in range(0, n - block, block)] + [(s, s - 1) for s in starts if s % (2 * block) == 0]
    folder = str(tmp_path / "m")
    _shifted_model(folder, cfg, 5, pairs, toks)
    edges = [p for s in starts for p in (s - 1, s, s + 1)] + [s + block - 1 for s in starts]
    w, want = _run_both_ways(cfg, folder, dtype, toks, edges)
    if dtype != "float32":
        return
    inside, outside = 2 * block - 1, 2 * block              # drawn to position block, and to 2 block - 1
    for other, pos in ((block - 1, inside), (block + 1, outside)):
        moved = copy.deepcopy(cfg)
        moved["layers"][0]["mixer"]["mask"]["size"] = other
        with torch.no_grad():
            assert nmse(P.forward(moved, w, toks)[pos:pos + 1], want[pos:pos + 1]) > 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_the_cap_and_the_distance_term_show(dtype, tmp_path, monkeypatch):
    """Leaving any of them out, or taking the distance term off before the cap, is far from the engine."""
    cfg = _one_layer(scale=0.4, softcap=1.5, vocab=97, heads=6, vdim=16)
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=21, sigma=0.3, norm_jitter=0.1))
    toks = random_tokens(97, 90, seed=4)
    w, want = _run_both_ways(cfg, folder, dtype, toks, edges=[0, 1, 15, 16, 31, 32, 89])
    if dtype != "float32":
        return

    def other(**changed):
        with monkeypatch.context() as m, torch.no_grad():
            for name, f in changed.items():
                m.setattr(P, name, f)
            return P.forward(cfg, w, toks)
    assert nmse(other(softmax_plus_one=lambda s, seen: torch.softmax(s.masked_fill(~seen, -1e30), -1)), want) > 1e-3
    assert nmse(other(capped=lambda s, cap: s), want) > 1e-3
    assert nmse(other(slope=lambda h, H: 0.0), want) > 1e-3
    assert nmse(other(slope=lambda h, H: 2.0 ** (-8.0 * h / H)), want) > 1e-3
    # slope * j instead of -slope * (i - j): the same without a sink only
    T = len(toks)
    assert nmse(other(distances=lambda n: -torch.arange(n, dtype=torch.float64)[None, :].expand(n, n)), want) > 1e-3
    assert T == 90


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(dtype):
    """Positions 0, 1, 2: one key and the sink."""
    from kipp_b200.engine import StepEntry
    for name in ("A", "D"):
        toks = random_tokens(CONFIGS[name]["vocab"], 3, seed=70)
        want = plain_logits(name, toks)
        eng = engine_for(name, dtype)
        for cuts in ([3], [1, 1, 1], [1, 2], [2, 1]):
            rows, at = [], 0
            for k in cuts:
                rows.append(eng.step([StepEntry("f", toks[at:at + k], list(range(k)))], check=True).clone())
                at += k
            eng.finish("f")
            close(torch.cat(rows), want, dtype, f"{name} {cuts}", factor=5 if dtype == "bfloat16" else 1, whole_model=True)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_of_a_batch_through_graphs(dtype):
    """Three requests of unequal prompts decode 150 tokens each in one batch (decode steps are
    graph replays), across several blocks of every layer; every row against the plain model."""
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
        close(torch.cat(got[i]), plain_logits(name, s[:h + 150]), dtype, f"request {i}", whole_model=True)


# ------------------------------------------------------------------ sizes nobody chose
def _drawn_config(seed):
    r = random.Random(seed)
    cfg = {"architecture": "Panolorn", "vocab": r.choice([64, 99, 130]), "width": r.choice([32, 40, 48, 64, 72]),
           "norm": {"eps": r.choice([1e-5, 1e-6])}}
    if r.random() < 0.8:
        cfg["embedding"] = {"scale": r.choice([0.5, 4.0, 13.7])}

    def mlp():
        kind = r.choice(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return dense(r.choice([8, 20, 48]))
        experts = r.choice([1, 2, 4, 7])
        return moe(experts, r.randint(1, min(3, experts)), r.choice([8, 12, 32]), r.choice([None, 8, 24]))

    cfg["layers"] = []
    for _ in range(r.randint(2, 4)):
        kv = r.choice([1, 2, 3])
        dim = r.choice([4, 6, 8, 16, 32])
        cfg["layers"].append(attention_layer(kv * r.choice([1, 2, 3]), kv, dim, r.choice([dim, 4, 12, 16, 48]), mlp(),
                                             r.choice([1.0, 3.0, 6.0]) / dim, r.choice([None, 2.0, 30.0]),
                                             r.choice([None, 1, 8, 13, 32, 50])))
    return cfg


@pytest.mark.parametrize("seed", range(10))
def test_drawn_configurations(seed, tmp_path):
    """Ten configurations nobody chose: 32-bit against the plain model (whole, in portions, and two
    requests in one batch through one cache), bfloat16 whole against the plain model row by row."""
    from kipp_b200.engine import Engine, StepEntry
    cfg = _drawn_config(3000 + seed)
    folder = write_folder(str(tmp_path / "m"), cfg, dict(seed=seed, sigma=0.15, norm_jitter=0.15))
    a, b = random_tokens(cfg["vocab"], 75, seed=seed), random_tokens(cfg["vocab"], 40, seed=100 + seed)
    w = read_weights(folder)
    with torch.no_grad():
        want_a, want_b = P.forward(cfg, w, a), P.forward(cfg, w, b)
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(folder, dtype=dtype, page_size=16, cache_tokens=192, max_requests=2, max_batch_tokens=128)
        whole = eng.step([StepEntry("w", a, list(range(len(a))))], check=True).clone()
        eng.finish("w")
        close(whole, want_a, dtype, f"{cfg} whole", whole_model=True)
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
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_scheduler(name):
    from kipp_b200.engine.llm import LLM
    vocab = CONFIGS[name]["vocab"]
    prompts = [random_tokens(vocab, n, seed=60 + n) for n in (3, 41, 17, 1, 26)]
    llm = LLM(model_folder(name), dtype="float32", kv_tokens=512, max_requests=3, max_batch_tokens=64, chunk=16)
    out = llm.generate(prompts, decode=12)
    w = weights_for(name)
    for prompt, result in zip(prompts, out):
        seq = list(prompt)
        with torch.no_grad():
            for _ in range(12):
                seq.append(int(P.forward(CONFIGS[name], w, seq)[-1].argmax()))
        assert result.tokens == seq[len(prompt):]


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
    w = weights_for(name)
    for prompt, tokens in zip((a, b), got):
        seq = list(prompt)
        with torch.no_grad():
            for _ in range(5):
                seq.append(int(P.forward(CONFIGS[name], w, seq)[-1].argmax()))
        assert tokens == seq[len(prompt):]
    assert "prefill_tokens=36" in proc.stderr and "decode_tokens=10" in proc.stderr
    sampled = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kipp"), "--random", "panolorn-tiny",
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
