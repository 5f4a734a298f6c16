"""The Zigolix decoder through the engine against the plain implementation (tests/plain_zigolix.py).

Small configurations of their own sizes and random weights, made here.  On a GPU the engine runs its CUDA kernels in
float32 and bfloat16; without one the same tests run the host-side logic (configuration, loader, cache manager, step
function) over the kernels' plain references.  Covered: each mechanism alone; a prompt whole, against its last tokens
decoded one by one, against portions down to two tokens and one; unequal requests in one batch against each alone, with
pages and slots that are given back and used again; the window's edges, page borders and far keys with one score made to
stand out, in both kinds of attention, in portions and in decoding; the sink; the cap; the looped span and the map that
reads the embedding anew; long decoding from captured steps; a configuration of ones and sizes that are multiples of
nothing; greedy generation through the front end; configuration errors; random-weights mode; each new kernel against its
plain reference.
"""

from __future__ import annotations

import json
import math

import pytest
import torch

import plain_zigolix as P
from helpers import random_tokens

CUDA = torch.cuda.is_available()
DEVICES = [pytest.param("cuda", marks=pytest.mark.gpu), "cpu"]
DTYPES = ["float32", "bfloat16"]


def moe(experts=5, top=2, ff=24, limit=1.4, shared=(40, 0.9)):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def attention(heads=6, kv=2, dim=24, window=19, rot=10, base=3000.0, scaling=(3.0, 64, 8.0, 2.0), scale=0.3, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": m}


def differential(heads=6, kv=3, dim=12, vdim=20, window=13, softcap=5.0, diff=0.3, scale=0.4, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention_2", "mlp": mlp, "mixer": m}


def config(layers, width=48, vocab=97, eps=1e-5, loop=None, logit_scale=None):
    out = {"architecture": "Zigolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    if logit_scale is not None:
        out["logit_scale"] = logit_scale
    return out


CONFIGS = {
    "attention_only": config([attention()]),
    # no window, no scaling of the frequencies, every head its own keys, the whole head rotated
    "attention_plain": config([attention(heads=3, kv=3, dim=16, window=None, rot=16, scaling=None)], logit_scale=0.25),
    "no_rotation": config([attention(heads=2, kv=1, dim=8, rot=None, window=4)]),
    "differential_only": config([differential()]),
    # values wider than both keys together, and no cap; values narrower
    "differential_wide": config([differential(heads=4, kv=2, dim=8, vdim=40, softcap=None, window=None)]),
    "differential_narrow": config([differential(heads=2, kv=2, dim=16, vdim=10, diff=0.7)]),
    "dense_only": config([differential(heads=2, kv=1, dim=4, vdim=8, mlp=dense(56))]),
    "experts_only": config([attention(heads=2, kv=1, dim=8, rot=4, mlp=moe())]),
    "experts_alone": config([attention(heads=2, kv=1, dim=8, rot=4, mlp=moe(experts=4, top=4, shared=None))]),
    # the looped span first, and everything in it
    "loop_all": config([attention(heads=2, kv=1, dim=8, rot=4, window=7), differential(heads=2, kv=2, dim=8, vdim=12, mlp=dense(24))], width=32, vocab=61,
                       loop=(0, 2, 3)),
    # everything at once, no two sizes alike: a loop in the middle, another layer behind it
    "mixed": config([differential(heads=4, kv=2, dim=8, vdim=24, window=9, mlp=dense(40)), attention(mlp=moe()),
                     differential(heads=6, kv=3, dim=12, vdim=20, window=21, softcap=3.0, mlp=moe(experts=7, top=3, ff=16, limit=0.8, shared=(24, 2.0))),
                     attention(heads=4, kv=4, dim=16, window=33, rot=4, base=500.0, scaling=None, mlp=None), differential(heads=3, kv=1, dim=16, vdim=16, mlp=dense(32))],
                    width=56, vocab=131, loop=(1, 4, 2), logit_scale=1.7),
    # one of everything
    "ones": config([attention(heads=1, kv=1, dim=2, window=1, rot=2, scaling=(1.0, 16, 4.0, 1.0), scale=1.0, mlp=moe(experts=1, top=1, ff=8, limit=1.0, shared=(8, 1.0))),
                    differential(heads=1, kv=1, dim=1, vdim=1, window=1, softcap=1.0, diff=0.5, scale=1.0, mlp=dense(8))], width=16, vocab=29, loop=(0, 1, 1),
                   logit_scale=1.0),
    # sizes that are multiples of nothing
    "odd": config([attention(heads=5, kv=5, dim=18, window=10, rot=6, mlp=moe(experts=3, top=2, ff=10, shared=(22, 1.1))),
                   differential(heads=9, kv=3, dim=7, vdim=11, window=17, mlp=dense(27))], width=36, vocab=83, loop=(1, 2, 2)),
    # more rows on one key head than the tile of the decode kernel has
    "many_heads": config([differential(heads=9, kv=1, dim=8, vdim=16, window=30), attention(heads=18, kv=1, dim=16, rot=8, window=25)], width=64, vocab=71),
    # sizes of a real model's layers: on a GPU the tcgen05 attention over heads of 128 and 64, tiles of experts' rows
    "wide": config([differential(heads=4, kv=2, dim=64, vdim=128, window=150, softcap=20.0, scale=0.1, mlp=dense(512)),
                    attention(heads=4, kv=2, dim=128, window=200, rot=64, scale=0.09, mlp=moe(experts=6, top=3, ff=128, shared=(256, 1.0))),
                    differential(heads=4, kv=4, dim=32, vdim=64, window=70, softcap=8.0, scale=0.15, mlp=moe(experts=4, top=2, ff=64)),
                    attention(heads=4, kv=1, dim=64, window=None, rot=32, scale=0.12, mlp=None)], width=256, vocab=512, loop=(1, 3, 2)),
}


def make_weights(cfg, seed):
    """Random tensors for every declared name, large enough that each part moves the logits."""
    from litinfer_b200.config import config_from_dict
    from litinfer_b200.models.decoder import declared_params

    g = torch.Generator().manual_seed(seed)
    out = {}
    for p in declared_params(config_from_dict(cfg).to_model_spec()):
        n, shape = p.name, tuple(p.shape)
        r = torch.randn(shape, generator=g)
        last = n.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or n == "final.norm":
            out[n] = 1.0 + 0.2 * r
        elif last == "b":
            out[n] = 0.3 * r
        elif last == "sink":
            out[n] = 1.0 + r
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            out[n] = r * (0.8 / math.sqrt(shape[0]))
        elif n == "loop.step":
            out[n] = 0.7 * r
        elif last == "router":
            out[n] = r * (3.0 / math.sqrt(shape[-1]))
        elif n == "embed":
            out[n] = r
        else:
            out[n] = r * (1.5 / math.sqrt(shape[-1]))
    return out


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from litinfer_b200.weights.safetensors_io import write_file

    out = {}
    for k, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp("zigolix_" + name)
        w = make_weights(cfg, 711 + k)
        (d / "config.json").write_text(json.dumps(cfg))
        write_file(d / "model.safetensors", w)
        out[name] = (d, cfg, w)
    return out


def use_device(device, request):
    if device == "cpu":
        request.getfixturevalue("cpu_kernels")
    return torch.device("cuda:0" if device == "cuda" else "cpu")


def oracle(cfg, w, tokens, dtype, keep=None):
    if dtype == "bfloat16":
        # what the bfloat16 engine holds: matrices rounded to bfloat16, everything else in float32
        w = {k: (v.to(torch.bfloat16).float() if v.dim() == 2 and k != "loop.step" else v) for k, v in w.items()}
    return P.forward(cfg, {k: v.double() for k, v in w.items()}, tokens, keep).float()


def assert_close(got, ref, dtype, what):
    assert got.shape == ref.shape, what
    assert torch.isfinite(got).all(), what
    d = got - ref
    d = d - d.mean(dim=-1, keepdim=True)
    err = d.pow(2).mean(dim=-1).sqrt() / ref.std(dim=-1).clamp_min(1e-3)
    worst = int(err.argmax())
    if dtype == "float32":
        assert err.max() <= 2e-4, f"{what}: relative error {float(err.max()):.3e} at row {worst}"
        return
    # bfloat16: activations are rounded to 8 bits at a dozen places a layer.  A row may be unlucky, and a token whose
    # choice scores lie within that rounding of each other may go to another expert than in the plain model; most rows may
    # not (a wrong key moves every row behind it by tens of percent)
    assert err.median() <= 0.05, f"{what}: median relative error {float(err.median()):.3e}"
    assert (err > 0.2).float().mean() <= 0.15, f"{what}: {int((err > 0.2).sum())} of {err.numel()} rows are off, the worst ({worst}) by {float(err.max()):.3e}"


class Run:
    """Feeds requests to a Replayer step by step and keeps every position's logits."""

    def __init__(self, folder, dtype, device, max_tokens, max_live=4, graphs=None):
        from litinfer_b200.engine.replay import Replayer
        from litinfer_b200.models import DecoderModel

        self.model = DecoderModel.from_dir(folder, dtype, device)
        self.rp = Replayer(self.model, max_tokens, max_live=max_live, use_graphs=device.type == "cuda" if graphs is None else graphs)
        self.fed = {}
        self.got = {}
        self.n = 0

    def step(self, entries, end=()):
        """entries: (request, all its tokens, how many of them now)."""
        es = []
        for rid, tokens, count in entries:
            lo = self.fed.get(rid, 0)
            es.append({"id": rid, "tokens": tokens[lo:lo + count], "want": list(range(count))})
            self.fed[rid] = lo + count
        logits = self.rp.step({"step": self.n, "entries": es, "end": list(end)}).float().cpu()
        self.n += 1
        row = 0
        for (rid, tokens, count), e in zip(entries, es):
            self.got.setdefault(rid, []).append(logits[row:row + count])
            row += count
        for rid in end:
            self.fed.pop(rid)

    def portions(self, rid, tokens, sizes):
        """The whole request in portions of these sizes (again and again), and its end."""
        at, i = 0, 0
        while at < len(tokens):
            c = min(sizes[i % len(sizes)], len(tokens) - at)
            self.step([(rid, tokens, c)], end=[rid] if at + c == len(tokens) else [])
            at += c
            i += 1

    def logits(self, rid):
        return torch.cat(self.got[rid])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["attention_only", "attention_plain", "no_rotation", "differential_only", "differential_wide", "differential_narrow",
                                  "dense_only", "experts_only", "experts_alone", "loop_all", "ones", "many_heads"])
def test_each_mechanism_alone(name, dtype, device, folders, request):
    dev = use_device(device, request)
    folder, cfg, w = folders[name]
    toks = random_tokens(45, cfg["vocab"], 5)
    ref = oracle(cfg, w, toks, dtype)
    run = Run(folder, dtype, dev, 128)
    run.step([("a", toks, 45)], end=["a"])
    assert_close(run.logits("a"), ref, dtype, f"{name} whole")
    run.step([("b", toks, 30)])
    for _ in range(15):
        run.step([("b", toks, 1)])
    assert_close(run.logits("b"), ref, dtype, f"{name} decoded")
    # portions of two tokens from the start
    for i in range(10):
        run.step([("c", toks, 2)])
    assert_close(run.logits("c"), ref[:20], dtype, f"{name} in twos")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "loop_all"])
def test_the_residual_stream_after_every_layer_run(name, device, folders, request):
    """Float32, layer by layer: the stream after each layer run (every pass of the loop counts) against the plain model's."""
    dev = use_device(device, request)
    folder, cfg, w = folders[name]
    toks = random_tokens(37, cfg["vocab"], 8)
    keep = []
    oracle(cfg, w, toks, "float32", keep)
    run = Run(folder, "float32", dev, 64, graphs=False)
    seen = []

    def observer(i, x, carry):
        # (a block hands its last output on to whatever adds it to the stream next)
        seen.append((x + carry.delta if carry is not None and carry.delta is not None else x).detach().float().cpu().clone())

    run.model.observer = observer
    run.step([("a", toks, 37)])
    assert len(seen) == len(keep) == len(P.order(cfg))
    for i, (a, b) in enumerate(zip(seen, keep)):
        assert (a - b.float()).abs().max() <= 1e-4 * max(1.0, float(b.abs().max())), f"after layer run {i}"


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_whole_decoded_and_in_portions(name, dtype, device, folders, request):
    dev = use_device(device, request)
    folder, cfg, w = folders[name]
    n = 330 if device == "cuda" else (110 if name == "mixed" else 50)
    toks = random_tokens(n, cfg["vocab"], 11)
    ref = oracle(cfg, w, toks, dtype)
    run = Run(folder, dtype, dev, 384)
    run.step([("whole", toks, n)], end=["whole"])
    assert_close(run.logits("whole"), ref, dtype, f"{name} whole")
    # most of it at once, then token by token across page borders (16)
    run.step([("tail", toks, n - 40)])
    for i in range(40):
        run.step([("tail", toks, 1)], end=["tail"] if i == 39 else [])
    assert_close(run.logits("tail"), ref, dtype, f"{name} decoded")
    # portions of changing size, down to two tokens and one; the first token alone
    run.portions("cut", toks, [1, 2, 7, 16, 2, 33, 5, 2, 130, 3, 1, 66, 11, 2, 29])
    assert_close(run.logits("cut"), ref, dtype, f"{name} portions")
    # token by token from the very first one
    for i in range(40):
        run.step([("one", toks, 1)], end=["one"] if i == 39 else [])
    assert_close(run.logits("one"), ref[:40], dtype, f"{name} token by token from the start")
    if dtype == "float32":
        assert (run.logits("whole") - run.logits("cut")).abs().max() < 2e-4
        assert (run.logits("whole") - run.logits("tail")).abs().max() < 2e-4
    run.rp.manager.check()
    assert run.rp.manager.num_free_slots() == 4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(dtype, device, folders, request):
    dev = use_device(device, request)
    folder, cfg, w = folders["mixed"]
    lens = [150, 37, 1, 64, 23, 2, 55, 140] if device == "cuda" else [40, 17, 1, 33, 2, 21]
    reqs = {f"r{j}": random_tokens(n, cfg["vocab"], 40 + j) for j, n in enumerate(lens)}
    # a pool for the most tokens that are live at a time, each request rounded up to 64: pages and slots come back
    run = Run(folder, dtype, dev, 64 * 7, max_live=3)
    queue, live, step_no = list(reqs), [], 0
    portions = [5, 2, 16, 9, 3, 21, 2, 130]
    while queue or live:
        while queue and len(live) < 3:
            live.append(queue.pop(0))
        entries, ending = [], []
        for k, rid in enumerate(live):
            toks, fed = reqs[rid], run.fed.get(rid, 0)
            if (step_no + k) % 5 == 4 and fed > 0:
                continue                                    # left out of this step, goes on later
            c = min(portions[(step_no + k) % len(portions)], len(toks) - fed) if fed < 0.6 * len(toks) else 1
            entries.append((rid, toks, c))
            if fed + c == len(toks):
                ending.append(rid)
        if entries:
            run.step(entries, end=ending)
        live = [r for r in live if r not in ending]
        step_no += 1
    if dtype == "float32":
        for rid, toks in reqs.items():
            assert_close(run.logits(rid), oracle(cfg, w, toks, dtype), dtype, f"{rid} of {len(toks)} tokens in mixed batches")
    else:
        alone = Run(folder, dtype, dev, 64 * 7, max_live=3)
        for rid, toks in reqs.items():
            alone.step([(rid, toks, len(toks))], end=[rid])
            assert_close(run.logits(rid), alone.logits(rid), dtype, f"{rid} of {len(toks)} tokens: in mixed batches against alone")
        assert_close(torch.cat([run.logits(r) for r in reqs]), torch.cat([oracle(cfg, w, t, dtype) for t in reqs.values()]), dtype, "all requests")
    m = run.rp.manager
    m.check()
    assert m.num_free_slots() == 3 and all(m.num_free_pages(g) == m.num_pages for g in range(len(m.groups)))


# ---------------------------------------------------------------------------------------------
# one key that stands out: the window's edges, page borders, far keys, at the model's level
# ---------------------------------------------------------------------------------------------

def _marked_weights(cfg, seed, mark):
    """Weights changed by hand so that one token's key draws every later query of the one layer: residual channel 0 carries a
    constant that the first query elements read, channel 1 is zero but for the token ``mark``, whose key reads it."""
    w = make_weights(cfg, seed)
    m, diff = cfg["layers"][0]["mixer"], cfg["layers"][0]["type"] == "attention_2"
    d = m["dim"]
    w["embed"][:, 0] = 3.0
    w["embed"][:, 1] = 0.0
    w["embed"][mark, 1] = 6.0
    w["l0.norm1"][:2] = 1.0
    q_step = 2 * d if diff else d                              # rows of a head: both maps', of which the first sees the mark
    last = d - 1                                               # an element that is not rotated
    for name in ("q", "k", "v", "g"):
        if f"l0.mix.{name}" in w:
            w[f"l0.mix.{name}"][:, :2] = 0.0                   # nothing else reads the two channels
    for name, col, heads in (("q", 0, m["heads"]), ("k", 1, m["kv_heads"])):
        for h in range(heads):
            w[f"l0.mix.{name}"][h * q_step + last] = 0.0
            w[f"l0.mix.{name}"][h * q_step + last, col] = 12.0
            if diff:
                w[f"l0.mix.{name}.b"][h * q_step + last] = 0.0
    if diff:
        w["l0.mix.v"][:, 1] = 3.0                              # and its value is unmistakable (in the other layer it is the key)
    else:
        w["l0.mix.sink"][:] = -2.0
    return w


MARKED = {
    "attention": config([attention(heads=4, kv=2, dim=16, window=37, rot=6, scale=2.0)]),
    "differential": config([differential(heads=4, kv=2, dim=8, vdim=12, window=37, softcap=40.0, scale=1.0)]),
    "attention_64": config([attention(heads=2, kv=1, dim=64, window=70, rot=32, scale=2.0)], width=64),
    "differential_64": config([differential(heads=2, kv=1, dim=32, vdim=64, window=70, softcap=40.0, scale=1.0)], width=64),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MARKED))
def test_a_key_that_stands_out_is_seen_to_the_edge_of_the_window_and_no_further(name, dtype, device, tmp_path, request):
    """Random weights would bury one key among dozens, so the marked token's score stands out by tens of units for every
    query that sees it: the logits of exactly the queries 0 .. window - 1 behind it move, in the plain model and in the
    engine alike, in prompts, in portions cut around the mark and around the window's end, and in tokens decoded one by one
    while the window's edge passes over the mark."""
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg = MARKED[name]
    window = cfg["layers"][0]["mixer"]["mask"]["size"]
    mark = cfg["vocab"] - 1
    w = _marked_weights(cfg, 900, mark)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    if device == "cpu" and "64" in name:
        pytest.skip("sizes for the tensor-core kernels")
    n = 230 if device == "cuda" else 90
    base = [t if t != mark else 0 for t in random_tokens(n, cfg["vocab"], 77)]
    plain = oracle(cfg, w, base, dtype)
    run = Run(tmp_path, dtype, dev, 512)
    run.step([("plain", base, n)], end=["plain"])
    for k, at in enumerate((0, 15, 16, 20, n - window - 6)):
        toks = list(base)
        toks[at] = mark
        ref = oracle(cfg, w, toks, dtype)
        moved = (ref - plain).abs().max(dim=-1).values / plain.std()
        inside = torch.zeros(n, dtype=torch.bool)
        inside[at:at + window] = True
        assert float(moved[~inside].max()) < 1e-6 and float(moved[inside].min()) > 0.2, f"mark at {at}: the plain model does not see it as made"
        first = max(at + 1, at + window - 8)
        run.step([(f"d{k}", toks, first)])
        for i in range(first, n):
            # the tokens before and behind the window's edge one by one, what is left in one step
            c = 1 if i < min(n, at + window + 8) else n - i
            run.step([(f"d{k}", toks, c)], end=[f"d{k}"] if i + c == n else [])
            if c > 1:
                break
        cuts = sorted({c for c in (at, at + 1, at + window - 1, at + window, at + window + 1, n) if 0 < c <= n})
        lo = 0
        for c in cuts:
            run.step([(f"c{k}", toks, c - lo)], end=[f"c{k}"] if c == n else [])
            lo = c
        run.step([(f"w{k}", toks, n)], end=[f"w{k}"])
        for rid, what in ((f"d{k}", "decoded over the edge"), (f"c{k}", "portions cut around it"), (f"w{k}", "whole")):
            assert_close(run.logits(rid), ref, dtype, f"{name}: mark at {at}, {what}")
            shift = (run.logits(rid) - run.logits("plain")).abs().max(dim=-1).values / plain.std()
            assert float(shift[inside].min()) > 0.1, f"{name}: mark at {at}, {what}: a query inside the window does not see it"
            assert float(shift[~inside].max()) < (1e-3 if dtype == "float32" else 0.1), f"{name}: mark at {at}, {what}: a query outside the window sees it"
    run.rp.manager.check()


@pytest.mark.parametrize("device", DEVICES)
def test_a_far_key_among_hundreds_without_a_window(device, tmp_path, request):
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg = json.loads(json.dumps(MARKED["differential"]))
    del cfg["layers"][0]["mixer"]["mask"]
    mark = cfg["vocab"] - 1
    w = _marked_weights(cfg, 901, mark)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    n = 700 if device == "cuda" else 90
    base = [t if t != mark else 0 for t in random_tokens(n, cfg["vocab"], 78)]
    plain = oracle(cfg, w, base, "float32")
    run = Run(tmp_path, "float32", dev, 1408)
    for at in (0, 31, n // 2):
        toks = list(base)
        toks[at] = mark
        ref = oracle(cfg, w, toks, "float32")
        assert float((ref - plain)[-1].abs().max()) > 0.2
        run.step([(f"a{at}", toks, n - 12)])
        for i in range(12):
            run.step([(f"a{at}", toks, 1)], end=[f"a{at}"] if i == 11 else [])
        assert_close(run.logits(f"a{at}"), ref, "float32", f"mark at {at}")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_takes_its_share(dtype, device, tmp_path, request):
    """The sink moves the logits of short and long contexts in the engine as in the plain model: per head one that takes nearly
    everything, one that counts like a few keys, one that is nothing."""
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg = config([attention(heads=3, kv=1, dim=16, window=12, rot=4)])
    w = make_weights(cfg, 33)
    w["l0.mix.sink"] = torch.tensor([6.0, 1.5, -20.0])
    toks = random_tokens(40, cfg["vocab"], 3)
    ref = oracle(cfg, w, toks, dtype)
    without = oracle(cfg, dict(w, **{"l0.mix.sink": torch.full((3,), -60.0)}), toks, dtype)
    assert float((ref - without).abs().max()) > 0.5
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    run = Run(tmp_path, dtype, dev, 64)
    run.step([("a", toks, 1)])
    run.step([("a", toks, 25)])
    for _ in range(14):
        run.step([("a", toks, 1)])
    assert_close(run.logits("a"), ref, dtype, "with sinks")


@pytest.mark.parametrize("device", DEVICES)
def test_every_pass_of_the_loop_reads_the_embedding_anew(device, folders, request):
    """Without the embedding's half of the map the plain model gives other logits (the map's second half is set to zero), and so
    does one whose passes share their vectors; the engine follows each."""
    from litinfer_b200.models import DecoderModel
    from litinfer_b200.engine.replay import Replayer

    dev = use_device(device, request)
    folder, cfg, w = folders["loop_all"]
    toks = random_tokens(24, cfg["vocab"], 9)
    ref = oracle(cfg, w, toks, "float32")
    half = dict(w, **{"loop.in": torch.cat([w["loop.in"][:, :32], torch.zeros(32, 32)], dim=1)})
    steps = dict(w, **{"loop.step": w["loop.step"][:1].repeat(3, 1)})
    for changed, name in ((half, "loop.in"), (steps, "loop.step")):
        other = oracle(cfg, changed, toks, "float32")
        assert float((other - ref).abs().max()) > 0.3
        model = DecoderModel.from_dir(folder, "float32", dev)
        (model.stream_maps if name == "loop.in" else model.stream_tables)[name].copy_(changed[name])
        rp = Replayer(model, 64, use_graphs=False)
        got = rp.step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": list(range(24))}], "end": ["a"]}).float().cpu()
        assert_close(got, other, "float32", name)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_captured_steps(dtype, folders):
    """300 tokens one by one (steps replayed from a captured graph, pages moving on and given back behind the windows)
    against the prompt whole."""
    folder, cfg, w = folders["mixed"]
    toks = random_tokens(330, cfg["vocab"], 3)
    ref = oracle(cfg, w, toks, dtype)
    run = Run(folder, dtype, torch.device("cuda:0"), 384)
    run.step([("a", toks, 30)])
    for _ in range(300):
        run.step([("a", toks, 1)])
    assert run.rp.runner.graph_replays >= 290
    assert_close(run.logits("a"), ref, dtype, "long decoding")


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_through_the_front_end(device, folders, request):
    dev = use_device(device, request)
    from litinfer_b200.api import CausalLM
    from litinfer_b200.models import DecoderModel

    folder, cfg, w = folders["mixed"]
    w64 = {k: v.double() for k, v in w.items()}
    lm = CausalLM(folder, dtype="float32") if device == "cuda" else CausalLM(folder, device="cpu", model=DecoderModel.from_dir(folder, "float32", dev),
                                                                            use_graphs=False)
    for n, new in ((1, 6), (13, 20), (50, 12)):
        prompt = random_tokens(n, cfg["vocab"], 60 + n)
        toks, margins = list(prompt), []
        for _ in range(new):
            top = torch.topk(P.forward(cfg, w64, toks)[-1], 2)
            margins.append(float(top.values[0] - top.values[1]))
            toks.append(int(top.indices[0]))
        assert min(margins) > 1e-4, "the plain model's own choice is a near-tie; pick another seed"
        out = lm.generate(prompt, max_new_tokens=new)
        assert list(out)[-new:] == toks[n:], f"prompt of {n} tokens"


def test_configuration_is_read_and_refused():
    from litinfer_b200.config import ConfigError, config_from_dict

    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    parsed = config_from_dict(cfg)
    spec = parsed.to_model_spec()
    assert config_from_dict(parsed.to_dict()) == parsed
    assert spec.architecture == "Zigolix" and not spec.tie_word_embeddings
    # the looped span: the same blocks again, every pass behind the map of the stream and with a vector of its own
    assert [e.block for e in spec.schedule] == [0, 1, 2, 3, 1, 2, 3, 4]
    assert [(e.join, e.add) for e in spec.schedule if e.add or e.join] == [("loop.in", ("loop.step", 0)), ("loop.in", ("loop.step", 1))]
    assert [b.parts["mixer"].kind for b in spec.blocks] == ["differential_attention", "attention", "differential_attention", "attention", "differential_attention"]
    a = spec.blocks[1].parts["mixer"]
    assert a["keys_are_values"] and a["sink"] == "sink" and a["window"] == 19 and a["position"]["pairing"] == "interleaved"
    assert a["position"]["scaling"]["kind"] == "yarn" and "scaling" not in spec.blocks[3].parts["mixer"]["position"].params
    ff = spec.blocks[2].parts["feed_forward"]
    assert (ff["experts"], ff["top"], ff["limit"], ff["shared"]["limit"], ff["shared"]["intermediate_size"]) == (7, 3, 0.8, 2.0, 24)
    assert spec.final_norm["gain"] == 1.7

    def broken(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises(ConfigError):
            config_from_dict(c)

    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="glu"))
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][1]["mixer"].update(vdim=12))                   # the values are the keys
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26))
    broken(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"))
    broken(lambda c: c["layers"][0]["mixer"].pop("diff"))
    broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"))
    broken(lambda c: c["loop"].update(stop=6))
    broken(lambda c: c["loop"].update(times=0))
    broken(lambda c: c["norm"].update(eps=0.0))


def test_random_weights_and_a_written_folder(tmp_path, cpu_kernels):
    """Random-weights mode knows the design's tensors; a folder written from it is read back through the registry."""
    from litinfer_b200.config import load_config
    from litinfer_b200.engine.replay import Replayer
    from litinfer_b200.models import DecoderModel
    from litinfer_b200.weights import write_model_folder

    cfg = CONFIGS["mixed"]
    write_model_folder(tmp_path, cfg, seed=5, store_dtype="float32")
    assert load_config(tmp_path).to_model_spec().stream_maps == ("loop.in",)
    model = DecoderModel.from_dir(tmp_path, "float32", torch.device("cpu"))
    rp = Replayer(model, 64, max_live=2, use_graphs=False)
    logits = rp.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3, 4, 5], "want": [4]}], "end": ["a"]})
    assert logits.shape == (1, cfg["vocab"]) and torch.isfinite(logits).all() and float(logits.std()) > 0


# ---------------------------------------------------------------------------------------------
# the new kernels, each against its plain reference
# ---------------------------------------------------------------------------------------------

def _dt(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def _close(a, b, dtype, what, tol=None):
    tol = tol or (2e-5 if dtype == "float32" else 2e-2)
    scale = max(1.0, float(b.float().abs().max()))
    assert torch.isfinite(a.float()).all(), what
    assert float((a.float() - b.float()).abs().max()) <= tol * scale, f"{what}: {float((a.float() - b.float()).abs().max()):.3e} (scale {scale:.2f})"


@pytest.mark.gpu
@pytest.mark.parametrize("implementation,q_lens,ctxs,dh", [
    ("general", [1, 45], [90, 45], 40), ("decode", [1] * 5, [700, 3, 257, 64, 1], 48), ("decode", [1] * 90, [300 + 7 * i for i in range(90)], 64),
    ("decode", [1] * 12, [2000 + 31 * i for i in range(12)], 128), ("decode", [1] * 3, [500, 40, 1000], 256), ("prefill", [130, 7, 1], [333, 7, 50], 96),
    ("prefill", [33, 64], [700, 64], 16), ("prefill_tcgen05", [130, 64, 200], [700, 64, 333], 64), ("prefill_tcgen05", [300, 5], [300, 900], 128),
    ("prefill_tcgen05", [64], [2500], 128)])
@pytest.mark.parametrize("window,softcap", [(None, 0.0), (100, 0.0), (100, 9.0), (None, 0.7), (3, 30.0)])
def test_attention_of_two_maps_a_row(implementation, q_lens, ctxs, dh, window, softcap):
    """Every attention kernel with query rows that stand for two heads each and with capped scores (within and far beyond the
    range where the cap bends), against the plain reference: portions, single tokens, page borders, shared-out tiles."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), torch.bfloat16
    torch.manual_seed(dh + len(q_lens))
    H, G, page = 4, 2, 16
    T, S = sum(q_lens), len(q_lens)
    pages = [-(-c // page) for c in ctxs]
    order = torch.randperm(sum(pages) + 3)
    table = torch.zeros(S, max(pages), dtype=torch.int32)
    at = 0
    for s, p in enumerate(pages):
        table[s, :p] = order[at:at + p].to(torch.int32)
        at += p
    kc = torch.randn(sum(pages) + 3, G, page, dh).to(dev, dt)
    vc = torch.randn(sum(pages) + 3, G, dh, page).to(dev, dt)
    qkv = (1.5 * torch.randn(T, (H + 2 * G) * dh)).to(dev, dt)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    args = dict(k_cache=kc, v_cache=vc, block_table=table.to(dev), q_start=i32(starts), ctx_lens=i32(ctxs),
                seq_of_token=i32([s for s, n in enumerate(q_lens) for _ in range(n)]), positions=i32([c - n + i for n, c in zip(q_lens, ctxs) for i in range(n)]),
                num_heads=2 * H, num_kv_heads=G, head_dim=dh, scale=0.5, window=window, max_q_len=max(q_lens), max_ctx_len=max(ctxs), softcap=softcap,
                sinks=torch.linspace(-1.0, 3.0, 2 * H, device=dev), maps=2)
    out, ref = (torch.empty(T, 2 * H * dh, dtype=dt, device=dev) for _ in range(2))
    more = {}
    if implementation == "prefill_tcgen05":
        from litinfer_b200.engine.batch import attention_units

        units = attention_units(q_lens, ctxs, work_budget=148 // (2 * H))
        more = dict(units=torch.from_numpy(units).to(dev), unit_slots=(int(units[0]), int(units[1])))
    K.paged_attention(qkv, out, **args, implementation=implementation, **more)
    R.paged_attention_dense(qkv, ref, **args)
    _close(out, ref, "bfloat16", f"{implementation}, head of {dh}, window {window}, cap {softcap}")
    # and without the two maps, the cap alone
    one, want = (torch.empty(T, H * dh, dtype=dt, device=dev) for _ in range(2))
    args.update(num_heads=H, maps=1, sinks=None)
    if more:
        units = attention_units(q_lens, ctxs, work_budget=148 // H)
        more = dict(units=torch.from_numpy(units).to(dev), unit_slots=(int(units[0]), int(units[1])))
    K.paged_attention(qkv, one, **args, implementation=implementation, **more)
    R.paged_attention_dense(qkv, want, **args)
    _close(one, want, "bfloat16", f"{implementation}, head of {dh}, window {window}, cap {softcap}, one map")


@pytest.mark.gpu
def test_attention_of_two_maps_in_float32():
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev = torch.device("cuda:0")
    torch.manual_seed(2)
    H, G, dh, page, T, ctx = 6, 3, 26, 16, 9, 60
    kc, vc = torch.randn(5, G, page, dh, device=dev), torch.randn(5, G, dh, page, device=dev)
    qkv = torch.randn(T, (H + 2 * G) * dh, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    args = dict(k_cache=kc, v_cache=vc, block_table=i32([[3, 1, 4, 0]]), q_start=i32([0, T]), ctx_lens=i32([ctx]), seq_of_token=i32([0] * T),
                positions=i32(list(range(ctx - T, ctx))), num_heads=2 * H, num_kv_heads=G, head_dim=dh, scale=0.6, window=21, max_q_len=T, max_ctx_len=ctx,
                softcap=2.5, maps=2)
    out, ref = (torch.empty(T, 2 * H * dh, device=dev) for _ in range(2))
    K.paged_attention(qkv, out, **args)
    R.paged_attention(qkv, ref, **args)
    _close(out, ref, "float32", "two maps")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dh,rot,interleaved,values,weights,norm", [
    (6, 2, 24, 10, True, True, False, True), (4, 1, 128, 64, True, True, False, True), (3, 3, 18, 6, True, True, False, True), (2, 1, 160, 160, True, False, True, True),
    (4, 2, 32, 32, False, False, False, False), (5, 1, 40, 12, False, True, True, True), (2, 2, 8, 0, False, True, False, True), (1, 1, 7, 2, True, True, False, True)])
def test_rotation_norm_values_and_cache_write_kernel(nh, nkv, dh, rot, interleaved, values, weights, norm, dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(dh)
    page = 16
    den = torch.pow(torch.tensor(300.0), 2.0 * torch.arange(rot // 2) / max(rot, 1)).to(dev) if rot else None
    qn, kn = ((1 + 0.2 * torch.randn(dh)).to(dev), (1 + 0.2 * torch.randn(dh)).to(dev)) if weights else (None, None)
    for T in (5, 90):
        slots = torch.randperm(10 * page)[:T].to(torch.int32).to(dev)
        pos = torch.randint(0, 2000, (T,), dtype=torch.int32, device=dev)
        proj = (1.3 * torch.randn(T, (nh + (1 if values else 2) * nkv) * dh + (0 if dh % 4 else 4))).to(dev, dt)
        for to_cache in (True, False):
            res = []
            for F in (K, R):
                out = torch.zeros(T, (nh + 2 * nkv) * dh, dtype=dt, device=dev)
                kc = torch.zeros(11, nkv, page, dh, dtype=dt, device=dev)
                vc = torch.zeros(11, nkv, dh, page, dtype=dt, device=dev)
                F.rope_norm_kv(proj, out, pos, den, rot, 1.17, interleaved, qn, kn, norm, 1e-5, dh, slots, kc, vc, nh, nkv, dh, True, to_cache=to_cache,
                               keys_are_values=values)
                if not to_cache:
                    F.rope_kv_write(out, pos, None, 0, slots, kc, vc, nh, nkv, dh)
                res.append((out, kc, vc))
            for a, b, what in zip(res[0], res[1], ("rows", "keys", "values")):
                _close(a, b, dtype, f"{what}, {T} tokens", 2e-3 if dtype == "float32" else 2e-2)         # (angles of thousands of radians in float32)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv,dl", [(3, 20, 32), (4, 128, 128), (2, 11, 16), (5, 300, 304), (1, 1, 16)])
def test_difference_of_two_maps_kernel(H, dv, dl, dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(dv)
    T = 33
    att = torch.randn(T, 2 * H * dl).to(dev, dt)
    for gate, col in ((torch.randn(T, H * dv + 4).to(dev, dt), 4), (torch.randn(T, H * dv + 3).to(dev, dt), 3), (None, 0)):
        out, ref = (torch.empty(T, H * dv, dtype=dt, device=dev) for _ in range(2))
        K.map_difference(att, dl, gate, col, 0.63, 1e-5, 0.55, out, H, dv)
        R.map_difference(att, dl, gate, col, 0.63, 1e-5, 0.55, ref, H, dv)
        _close(out, ref, dtype, f"difference, gate at {col}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_beside_the_embedding_and_sums_with_a_further_row_kernels(dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(6)
    for T, H in ((7, 48), (3, 50), (5, 33), (300, 1536)):
        x, x0, delta = torch.randn(T, H, device=dev), torch.randn(T, H, device=dev), torch.randn(T, H, device=dev).to(dt)
        for d in (None, delta):
            out, ref = (torch.empty(T, 2 * H, dtype=dt, device=dev) for _ in range(2))
            K.join_rows(x, d, x0, out)
            R.join_rows(x, d, x0, ref)
            assert torch.equal(out, ref)
        # the chosen experts' rows and the shared expert's, inside the pass over the stream and by themselves
        top = 3
        rows = torch.randn(T * top + 5, H, device=dev).to(dt)
        places = torch.randperm(T * top + 5)[:T * top].to(torch.int32).to(dev)
        wts = torch.rand(T, top, device=dev)
        w = (1 + 0.2 * torch.randn(H, device=dev)).contiguous()
        rx, out, ref = x.clone(), torch.empty(T, H, dtype=dt, device=dev), torch.empty(T, H, dtype=dt, device=dev)
        K.norm_add_norm(x, K.RowSum(rows, places, top, wts, extra=delta), None, (w, False, 1e-5), out)
        R.norm_add_norm(rx, K.RowSum(rows, places, top, wts, extra=delta), None, (w, False, 1e-5), ref)
        _close(x, rx, "float32", "stream", 1e-5)
        _close(out, ref, dtype, "next norm")
        y, want = torch.empty(T, H, dtype=dt, device=dev), torch.empty(T, H, dtype=dt, device=dev)
        K.moe_combine(rows, places, wts, top, y, extra=delta)
        R.moe_combine(rows, places, wts, top, want, extra=delta)
        _close(y, want, dtype, "combined")
        both, ref2 = (torch.empty(T, 2 * H, dtype=dt, device=dev) for _ in range(2))
        K.join_rows(x, K.RowSum(rows, places, top, wts, extra=delta), x0, both)
        R.join_rows(x, K.RowSum(rows, places, top, wts, extra=delta), x0, ref2)
        _close(both, ref2, dtype, "joined with a sum of rows")
        rx = x.clone()
        K.residual_add(x, K.RowSum(rows, places, top, None, extra=None))
        R.residual_add(rx, K.RowSum(rows, places, top, None, extra=None))
        _close(x, rx, "float32", "a sum of rows added to the stream", 1e-5)


@pytest.mark.gpu
def test_gelu_unit_as_a_kernel_and_as_an_epilogue_of_every_product():
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev = torch.device("cuda:0")
    torch.manual_seed(8)
    for dtype in DTYPES:
        both = (4.0 * torch.randn(9, 2 * 56)).to(dev, _dt(dtype))
        both[0, :4] = torch.tensor([-40.0, 40.0, 0.0, -1e-3], device=dev).to(both.dtype)
        out, ref = (torch.empty(9, 56, dtype=both.dtype, device=dev) for _ in range(2))
        K.geglu(both, out)
        R.geglu(both, ref)
        _close(out, ref, dtype, "gelu unit")
    for which, M, N, Kd in (("gemv", 5, 96, 64), ("gemv", 40, 160, 72), ("gemv_tcgen05", 3, 1024, 512), ("gemv_tcgen05", 33, 256, 4096), ("tcgen05", 130, 512, 256),
                            ("tcgen05", 600, 1056, 128), ("tcgen05", 2048, 8192, 256)):
        a = torch.randn(M, Kd).to(dev, torch.bfloat16)
        w = (2.0 * torch.randn(N, Kd) / math.sqrt(Kd)).to(dev, torch.bfloat16)
        out, ref = (torch.empty(M, N // 2, dtype=torch.bfloat16, device=dev) for _ in range(2))
        K.linear_with(which, a, w, None, out, epilogue="geglu")
        R.linear(a, w, None, ref, epilogue="geglu")
        _close(out, ref, "bfloat16", f"{which} {M} x {N} x {Kd}")
    # rows in groups: the weight-streaming tiles and the tcgen05 tiles
    E, W, F = 4, 64, 48
    w = (torch.randn(E, 2 * F, W) / 8).to(dev, torch.bfloat16)
    for per in (3, 128):
        offsets = torch.arange(0, E * per + 1, per, dtype=torch.int32, device=dev)
        tiles = torch.arange(E, dtype=torch.int32, device=dev) if per == 128 else None
        a = torch.randn(E * per, W).to(dev, torch.bfloat16)
        out, ref = (torch.empty(E * per, F, dtype=torch.bfloat16, device=dev) for _ in range(2))
        K.grouped_linear(a, w, out, offsets, tile_group=tiles, epilogue="geglu")
        R.grouped_linear(a, w, ref, offsets, tile_group=tiles, epilogue="geglu")
        _close(out, ref, "bfloat16", f"groups of {per} rows")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_front_of_a_mixture_in_one_launch_and_rows_read_in_place(dtype):
    """Router, choice and sort of a small step against the kernels they stand for; the first product of the experts with the
    tokens' rows read where they are against the gathered rows."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(12)
    for T, E, top, H, scoring, groups, keep in ((1, 8, 2, 64, "softmax_grouped", 1, 1), (9, 5, 3, 48, "softmax_grouped", 5, 4), (10, 12, 4, 96, "sigmoid", 1, 1),
                                                (30, 3, 1, 1536, "softmax_chosen", 1, 1), (16, 8, 3, 256, "softmax_grouped", 4, 2), (1, 100, 6, 128, "softmax_grouped", 1, 1)):
        h = torch.randn(T, H).to(dev, dt)
        w = (2.0 * torch.randn(E, H) / math.sqrt(H)).to(dev, dt)
        bias = (0.3 * torch.randn(E)).to(dev) if scoring == "softmax_chosen" else None
        corr = (0.05 * torch.randn(E)).to(dev) if groups > 1 else None
        assert K.moe_small_step_accepts(h, E, top)
        res = []
        for F in (K, R):
            wt = torch.empty(T, top, device=dev)
            off, at, place = (torch.empty(n, dtype=torch.int32, device=dev) for n in (E + 1, T * top, T * top))
            F.moe_small_step(h, w, bias, top, scoring, corr, groups, keep, 1.3, wt, off, at, place)
            res.append((wt, off, at, place))
        assert torch.equal(res[0][1], res[1][1]) and torch.equal(res[0][2], res[1][2]) and torch.equal(res[0][3], res[1][3]), f"{T} tokens, {E} experts"
        assert (res[0][0] - res[1][0]).abs().max() < 1e-4
        if dtype == "bfloat16":
            _, off, at, _ = res[0]
            gu = (torch.randn(E, 96, H) / math.sqrt(H)).to(dev, dt)
            params = torch.tensor([1.2, 1.702], device=dev)
            rows = torch.empty(T * top, H, dtype=dt, device=dev)
            K.moe_gather(h, at, None, top, rows)
            out, want = (torch.empty(T * top, 48, dtype=dt, device=dev) for _ in range(2))
            K.grouped_linear(h, gu, out, off, epilogue="glu_clamped", epilogue_params=params, row_source=(at, top))
            K.grouped_linear(rows, gu, want, off, epilogue="glu_clamped", epilogue_params=params)
            assert torch.equal(out, want)
    assert not K.moe_small_step_accepts(torch.empty(300, 64, dtype=dt, device=dev), 8, 2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [3, 20, 70])
def test_projection_with_a_gate_behind_it_kernel(T, dtype):
    """q|k|v and a further map of the same input in one call: one kernel for few tokens, separate products otherwise."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(T)
    nh, nkv, dh, more, W, page = 3, 2, 32, 3, 64, 16
    w = (torch.randn((nh + 2 * nkv + more) * dh, W) / 8).to(dev, dt)
    b = (0.2 * torch.randn((nh + 2 * nkv + more) * dh)).to(dev)
    a = torch.randn(T, W).to(dev, dt)
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    slots = (torch.arange(T, dtype=torch.int32) + 16).to(dev)
    ssq = (torch.rand(T, 4, device=dev) + 0.5).contiguous()
    for scale in (None, (ssq, W, 1e-5)):
        if scale is not None and (dtype == "float32" or T > 64):
            continue
        res = []
        for F in (K, R):
            qkv, gate = torch.zeros(T, (nh + 2 * nkv) * dh, dtype=dt, device=dev), torch.zeros(T, more * dh, dtype=dt, device=dev)
            kc, vc = torch.zeros(8, nkv, page, dh, dtype=dt, device=dev), torch.zeros(8, nkv, dh, page, dtype=dt, device=dev)
            F.linear_rope_kv(a, w, b, qkv, pos, None, 0, slots, kc, vc, nh, nkv, dh, row_scale=scale, extra=gate)
            res.append((qkv[:, :nh * dh], gate, kc, vc))
        for x, y, what in zip(res[0], res[1], ("queries", "gate", "keys", "values")):
            _close(x, y, dtype, f"{what}, {T} tokens")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dh,page", [(24, 16), (128, 32), (20, 16), (9, 16)])
def test_keys_and_values_of_a_long_step_into_pages_kernel(dh, page, dtype):
    """Runs of consecutive slots (whole pieces of pages), a ragged end, and slots in any order."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(dh)
    nh, nkv = 2, 3
    for T, order in ((96, "run"), (101, "run"), (75, "any"), (80, "late")):
        qkv = torch.randn(T, (nh + 2 * nkv) * dh).to(dev, dt)
        slots = torch.randperm(12 * page)[:T] if order == "any" else torch.arange(T) + (page if order == "run" else 5)
        slots = slots.to(torch.int32).to(dev)
        res = []
        for F in (K, R):
            kc, vc = torch.zeros(13, nkv, page, dh, dtype=dt, device=dev), torch.zeros(13, nkv, dh, page, dtype=dt, device=dev)
            F.rope_kv_write(qkv.clone(), torch.zeros(T, dtype=torch.int32, device=dev), None, 0, slots, kc, vc, nh, nkv, dh)
            res.append((kc, vc))
        assert torch.equal(res[0][0], res[1][0]) and torch.equal(res[0][1], res[1][1]), f"{T} tokens, {order}"


@pytest.mark.gpu
@pytest.mark.parametrize("epilogue", [None, "swiglu", "glu_clamped", "geglu"])
def test_products_of_experts_on_pairs_of_ctas(epilogue):
    """Runs padded to 256 rows in the persistent kernel: uneven runs, an expert that nobody chose, tiles of no group among and
    behind the others, columns that are no whole tile, more tiles than pairs of multiprocessors and fewer; against the
    reference and, bit for bit, against a second run."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), torch.bfloat16
    params = torch.tensor([1.1, 1.702], device=dev) if epilogue == "glu_clamped" else None
    for T, E, top, W, F, extra in ((700, 3, 2, 64, 80, 1), (2048, 5, 2, 128, 2000, 0), (1500, 4, 1, 264, 304, 0), (512, 2, 1, 1024, 64, 2)):
        torch.manual_seed(T)
        ids = torch.randint(0, E + extra, (T, top), dtype=torch.int32, device=dev)
        if E == 5:
            ids[ids == 1] = 4
        n_rows = K.sorted_rows(T * top, E + extra, 256)
        offsets, pair_at, place_of = (torch.empty(n, dtype=torch.int32, device=dev) for n in (E + extra + 1, n_rows, T * top))
        tiles = torch.empty(n_rows // 256, dtype=torch.int32, device=dev)
        K.moe_sort(ids, E + extra, offsets, pair_at, place_of, 256, tiles, matrices=E)
        a = torch.randn(n_rows, W, device=dev).to(dt)
        w = (2.0 * torch.randn(E, F, W, device=dev) / math.sqrt(W)).to(dt)
        cols = F if epilogue is None else F // 2
        outs = [torch.full((n_rows, cols), 3.0, dtype=dt, device=dev) for _ in range(3)]
        for out, fn in zip(outs, (K, R, K)):
            fn.grouped_linear(a, w, out, offsets[:E + 1], tile_group=tiles, tile_rows=256, epilogue=epilogue, epilogue_params=params)
        lo = int(offsets[E])
        live = pair_at[:lo] >= 0
        _close(outs[0][:lo][live], outs[1][:lo][live], "bfloat16", f"{T} tokens, {E} experts")
        assert torch.equal(outs[0], outs[2])
        assert (outs[0][lo:] == 3.0).all(), "rows of no expert were written"
