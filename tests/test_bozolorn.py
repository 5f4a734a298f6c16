"""The Bozolorn decoder through the engine against the plain implementation (tests/plain_bozolorn.py).

Small configurations of their own sizes and random weights, made here.  On a GPU the engine runs its CUDA kernels in
float32 and bfloat16; without one the same tests run the host-side logic (configuration, loader, cache manager, step
function) over the kernels' plain references.  Covered: each mechanism alone; a prompt whole, against its last tokens
decoded one by one, against portions down to two tokens and one; unequal requests in one batch against each alone, with
pages and slots that are given back and used again; a key made to stand out that its own chunk sees to the chunk's last
position and the next chunk does not, at page borders, in portions and in decoding, in a layer with keys of its own and in
one that reads another's; far keys among hundreds; the one in the denominator; the delta rule's state and convolution; the
routing's groups; the token's row; long decoding from captured steps; a configuration of ones and sizes that are multiples
of nothing; greedy generation through the front end and the scheduler; configuration errors; random-weights mode; each new
kernel or form against its plain reference.
"""

from __future__ import annotations

import json
import math

import pytest
import torch

import plain_bozolorn as P
from helpers import random_tokens

CUDA = torch.cuda.is_available()
DEVICES = [pytest.param("cuda", marks=pytest.mark.gpu), "cpu"]
DTYPES = ["float32", "bfloat16"]


def moe(experts=6, top=2, groups=(3, 2), ff=24, limit=1.3):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}


def attention(heads=6, kv=2, dim=12, vdim=20, size=21, scale=0.3, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def left(heads=4, kv=2, dim=16, vdim=12, rot=10, base=3000.0, scaling=(3.0, 64, 8.0, 2.0), scale=0.4):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def right(heads=4, kv=2, dim=12, vdim=20, conv=4):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(a=None, b=None, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a or left(), "right": b or right()}}


def config(layers, width=48, vocab=97, eps=1e-5, scale=2.5, side=12):
    out = {"architecture": "Bozolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if side:
        out["token_side"] = {"dim": side}
    return out


CONFIGS = {
    "attention_only": config([attention()]),
    # every head its own keys, values narrower than keys, the token's row left out
    "attention_narrow": config([attention(heads=3, kv=3, dim=24, vdim=8, size=7, scale=0.5)], side=0),
    "attention_equal": config([attention(heads=2, kv=1, dim=16, vdim=16, size=40)], scale=1.0),
    # the reader's chunks are longer than the owner's, and the other way round
    "shared_longer": config([attention(size=10), attention(size=33, kv_from=0)]),
    "shared_shorter": config([attention(size=33), attention(size=10, kv_from=0, mlp=moe())]),
    "parallel_only": config([parallel()]),
    "parallel_plain": config([parallel(left(heads=3, kv=3, dim=8, vdim=24, rot=8, scaling=None), right(heads=3, kv=3, dim=8, vdim=8, conv=2))], side=0),
    # a rule whose key heads serve three value heads each, another number of taps
    "parallel_groups": config([parallel(left(heads=4, kv=1, dim=20, vdim=20, rot=4), right(heads=6, kv=2, dim=24, vdim=12, conv=3))]),
    "experts_only": config([attention(heads=2, kv=1, dim=8, vdim=8, mlp=moe())]),
    "experts_one_group": config([attention(heads=2, kv=1, dim=8, vdim=8, mlp=moe(experts=5, top=3, groups=None))]),
    "experts_groups_of_one": config([attention(heads=2, kv=1, dim=8, vdim=8, mlp=moe(experts=4, top=2, groups=(4, 3)))]),
    # everything at once, no two sizes alike
    "mixed": config([parallel(mlp=moe()), attention(heads=4, kv=2, dim=16, vdim=24, size=29, mlp=moe(experts=8, top=3, groups=(2, 1), ff=16, limit=0.8)),
                     parallel(left(heads=6, kv=3, dim=24, vdim=8, rot=24, base=500.0, scaling=None), right(heads=2, kv=1, dim=40, vdim=16, conv=3), mlp=None),
                     attention(heads=4, kv=2, dim=16, vdim=24, size=37, kv_from=1, mlp=moe(experts=9, top=4, groups=(3, 2), ff=40, limit=2.0)),
                     attention(heads=6, kv=6, dim=8, vdim=8, size=16, mlp=None)], width=56, vocab=131, side=20),
    # one of everything
    "ones": config([parallel(left(heads=1, kv=1, dim=2, vdim=1, rot=2, scaling=(1.0, 16, 4.0, 1.0), scale=1.0), right(heads=1, kv=1, dim=1, vdim=1, conv=1),
                             mlp=moe(experts=1, top=1, groups=(1, 1), ff=8, limit=1.0)), attention(heads=1, kv=1, dim=1, vdim=1, size=1, scale=1.0, mlp=None)],
                   width=16, vocab=29, scale=1.0, side=1),
    # sizes that are multiples of nothing
    "odd": config([parallel(left(heads=5, kv=5, dim=18, vdim=11, rot=6), right(heads=3, kv=3, dim=7, vdim=11, conv=5), mlp=moe(experts=3, top=2, groups=(3, 3), ff=10)),
                   attention(heads=9, kv=3, dim=7, vdim=13, size=17, mlp=moe(experts=10, top=3, groups=(5, 2), ff=27))], width=36, vocab=83, side=7),
    # more rows on one key head than the tile of the decode kernel has; more experts and groups than a warp has lanes
    "many": config([attention(heads=18, kv=1, dim=16, vdim=16, size=25, mlp=moe(experts=80, top=5, groups=(40, 9), ff=8)),
                    parallel(left(heads=18, kv=1, dim=16, vdim=16, rot=8), right(heads=8, kv=1, dim=16, vdim=8))], width=64, vocab=71),
    # sizes of a real model's layers: on a GPU the tcgen05 attention over heads of 128 and 64, tiles of experts' rows
    "wide": config([parallel(left(heads=4, kv=2, dim=128, vdim=96, rot=64, scale=0.09), right(heads=4, kv=2, dim=128, vdim=128), mlp=moe(experts=8, top=2, groups=(4, 2), ff=128)),
                    attention(heads=4, kv=2, dim=64, vdim=64, size=150, scale=0.12, mlp=moe(experts=4, top=2, groups=(2, 1), ff=64)),
                    attention(heads=4, kv=2, dim=64, vdim=64, size=90, kv_from=1, scale=0.12),
                    parallel(left(heads=4, kv=1, dim=64, vdim=64, rot=32, scale=0.12), right(heads=2, kv=2, dim=64, vdim=128))], width=256, vocab=512, side=64),
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
        if last in ("norm1", "norm2", "norm1b", "norm2b", "norm", "out"):
            out[n] = 1.0 + 0.2 * r
        elif n.endswith((".q.b", ".k.b", ".v.b")):
            out[n] = 0.3 * r
        elif last == "conv":
            out[n] = r * 0.7
        elif last in ("dt_bias", "A_log"):
            out[n] = 0.7 * r - 0.5
        elif last == "correction":
            out[n] = 0.2 * r
        elif last == "router":
            out[n] = r * (3.0 / math.sqrt(shape[-1]))
        elif n in ("embed", "side.embed"):
            out[n] = r
        else:
            out[n] = r * (1.5 / math.sqrt(shape[-1]))
    return out


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from litinfer_b200.weights.safetensors_io import write_file

    out = {}
    for k, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp("bozolorn_" + name)
        w = make_weights(cfg, 811 + k)
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
        # what the bfloat16 engine holds: matrices rounded to bfloat16, vectors (the convolutions' taps among them) in float32
        w = {k: (v.to(torch.bfloat16).float() if v.dim() == 2 and not k.endswith(".conv") else v) for k, v in w.items()}
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
    assert err.median() <= 0.06, f"{what}: median relative error {float(err.median()):.3e}"
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
        for rid, tokens, count in entries:
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
@pytest.mark.parametrize("name", ["attention_only", "attention_narrow", "attention_equal", "shared_longer", "shared_shorter", "parallel_only", "parallel_plain",
                                  "parallel_groups", "experts_only", "experts_one_group", "experts_groups_of_one", "ones", "many"])
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
@pytest.mark.parametrize("name", ["mixed", "shared_longer"])
def test_the_residual_stream_after_every_layer(name, device, folders, request):
    """Float32, layer by layer: the stream after each layer against the plain model's."""
    dev = use_device(device, request)
    folder, cfg, w = folders[name]
    toks = random_tokens(37, cfg["vocab"], 8)
    keep, seen = [], []
    oracle(cfg, w, toks, "float32", keep)
    run = Run(folder, "float32", dev, 64, graphs=False)
    run.model.observer = lambda i, x, carry: seen.append(x.detach().float().cpu().clone())
    run.step([("a", toks, 37)])
    assert len(seen) == len(keep) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, keep)):
        assert (a - b.float()).abs().max() <= 1e-4 * max(1.0, float(b.abs().max())), f"after layer {i}"


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_whole_decoded_and_in_portions(name, dtype, device, folders, request):
    dev = use_device(device, request)
    folder, cfg, w = folders[name]
    n = 330 if device == "cuda" else (90 if name == "mixed" else 50)
    toks = random_tokens(n, cfg["vocab"], 11)
    ref = oracle(cfg, w, toks, dtype)
    run = Run(folder, dtype, dev, 384)
    run.step([("whole", toks, n)], end=["whole"])
    assert_close(run.logits("whole"), ref, dtype, f"{name} whole")
    # most of it at once, then token by token across page borders (16) and chunks
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
        got, one = (torch.cat([r.logits(i) for i in reqs]) for r in (run, alone))
        assert_close(got, one, dtype, "all requests in mixed batches against alone")
        assert_close(got, torch.cat([oracle(cfg, w, t, dtype) for t in reqs.values()]), dtype, "all requests")
    m = run.rp.manager
    m.check()
    assert m.num_free_slots() == 3 and all(m.num_free_pages(g) == m.num_pages for g in range(len(m.groups)))


# ---------------------------------------------------------------------------------------------
# one key that stands out: a chunk's edges, page borders, far keys, at the model's level
# ---------------------------------------------------------------------------------------------

def _marked_weights(cfg, seed, mark, layer, mix, slope=True):
    """Weights changed by hand so that one token's key draws every later query of one layer: residual channel 0 carries a
    constant that the first query element reads, channel 1 is zero but for the token ``mark``, whose key reads it and whose value is
    unmistakable."""
    w = make_weights(cfg, seed)
    m = cfg["layers"][layer]["mixer"]
    m = m.get("left", m)
    owner = m.get("kv_from", layer)
    q, kv = f"l{layer}.{mix}", f"l{owner}.{mix}"
    w["embed"][:, 0] = 3.0
    w["embed"][:, 1] = 0.0
    w["embed"][mark, 1] = 6.0
    for i in range(len(cfg["layers"])):
        w[f"l{i}.norm1"][:2] = 1.0
        w[f"l{i}.norm1b"][:2] = 0.0                            # the two channels stay as they are from layer to layer
        w[f"l{i}.side.norm"][:2] = 0.0
        for name, t in w.items():
            if name.startswith(f"l{i}.mix.") and t.dim() == 2 and t.shape[1] == cfg["width"]:
                t[:, :2] = 0.0                                 # nothing else reads the two channels
    d, last = m["dim"], m["dim"] - 1                           # an element that is not rotated
    for name, p, col, heads in (("q", q, 0, m["heads"]), ("k", kv, 1, m["kv_heads"])):
        for h in range(heads):
            w[f"{p}{name}"][h * d + last] = 0.0
            w[f"{p}{name}"][h * d + last, col] = 12.0
            if f"{p}{name}.b" in w:
                w[f"{p}{name}.b"][h * d + last] = 0.0
    w[f"{kv}v"][:, 1] = 3.0
    return w


MARKED = {
    # (configuration, the layer that is watched, below its mixer)
    "attention": (config([attention(heads=4, kv=2, dim=16, vdim=12, size=37, scale=4.0)]), 0),
    # the layer with the keys has long chunks; the watched one reads them in short ones, and the other way round
    "reader": (config([attention(heads=4, kv=2, dim=16, vdim=12, size=16, scale=0.02), attention(heads=4, kv=2, dim=16, vdim=12, size=37, scale=4.0, kv_from=0)]), 1),
    "attention_64": (config([attention(heads=2, kv=1, dim=64, vdim=64, size=70, scale=4.0)], width=64), 0),
    "attention_128": (config([attention(heads=2, kv=1, dim=128, vdim=96, size=150, scale=4.0)], width=64), 0),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MARKED))
def test_a_key_that_stands_out_is_seen_to_the_end_of_its_chunk_and_no_further(name, dtype, device, tmp_path, request):
    """Random weights would bury one key among dozens, so the marked token's score stands out by tens of units for every query
    that sees it: the logits of exactly the queries from the mark to the last of its chunk move, in the plain model and in the
    engine alike, in prompts, in portions cut around the mark and around the chunk's end, and in tokens decoded one by one across
    the chunk's end.  (The layers that are not watched move the mark's own logits only.)"""
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg, layer = MARKED[name]
    if device == "cpu" and ("64" in name or "128" in name):
        pytest.skip("sizes for the tensor-core kernels")
    size = cfg["layers"][layer]["mixer"]["mask"]["size"]
    mark = cfg["vocab"] - 1
    w = _marked_weights(cfg, 900, mark, layer, "mix.")
    if layer:
        w["l0.mix.v"][:, 1] = 0.0                              # layer 0 passes nothing of the mark on: only its keys carry it
        for h in range(cfg["layers"][0]["mixer"]["kv_heads"]):
            w["l0.mix.v"][h * 12, 1] = 3.0
        w["l0.norm1b"][:] = 0.0
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    n = 330 if device == "cuda" else 100
    base = [t if t != mark else 0 for t in random_tokens(n, cfg["vocab"], 77)]
    plain = oracle(cfg, w, base, dtype)
    run = Run(tmp_path, dtype, dev, 512)
    run.step([("plain", base, n)], end=["plain"])
    for k, at in enumerate((0, 15, 16, size - 1, size, size + 5, 2 * size - 3)):
        toks = list(base)
        toks[at] = mark
        ref = oracle(cfg, w, toks, dtype)
        moved = (ref - plain).abs().max(dim=-1).values / plain.std()
        inside = torch.zeros(n, dtype=torch.bool)
        edge = (at // size + 1) * size                         # the first position of the next chunk
        inside[at:edge] = True
        assert float(moved[~inside].max()) < 1e-6 and float(moved[inside].min()) > 0.2, f"mark at {at}: the plain model does not see it as made"
        first = max(at + 1, edge - 8)
        run.step([(f"d{k}", toks, first)])
        for i in range(first, n):
            # the tokens before and behind the chunk's edge one by one, what is left in one step
            c = 1 if i < min(n, edge + 8) else n - i
            run.step([(f"d{k}", toks, c)], end=[f"d{k}"] if i + c == n else [])
            if c > 1:
                break
        cuts = sorted({c for c in (at, at + 1, edge - 1, edge, edge + 1, n) if 0 < c <= n})
        lo = 0
        for c in cuts:
            run.step([(f"c{k}", toks, c - lo)], end=[f"c{k}"] if c == n else [])
            lo = c
        run.step([(f"w{k}", toks, n)], end=[f"w{k}"])
        for rid, what in ((f"d{k}", "decoded over the edge"), (f"c{k}", "portions cut around it"), (f"w{k}", "whole")):
            assert_close(run.logits(rid), ref, dtype, f"{name}: mark at {at}, {what}")
            shift = (run.logits(rid) - run.logits("plain")).abs().max(dim=-1).values / plain.std()
            assert float(shift[inside].min()) > 0.1, f"{name}: mark at {at}, {what}: a query of its chunk does not see it"
            assert float(shift[~inside].max()) < (1e-3 if dtype == "float32" else 0.1), f"{name}: mark at {at}, {what}: a query of another chunk sees it"
    run.rp.manager.check()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
def test_a_far_key_among_hundreds_in_the_rotated_half(dtype, dim, device, tmp_path, request):
    """The rotated attention of a parallel layer, in which a marked key stands out for every later query, however far."""
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg = config([parallel(left(heads=2, kv=1, dim=dim, vdim=12, rot=6, scale=9.0), right(heads=2, kv=1, dim=4, vdim=4, conv=2))], width=48)
    mark = cfg["vocab"] - 1
    w = _marked_weights(cfg, 901, mark, 0, "mix.left.")
    w["l0.mix.right.out"][:] = 0.0                             # the other half says nothing
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    n = 700 if device == "cuda" else 80
    base = [t if t != mark else 0 for t in random_tokens(n, cfg["vocab"], 78)]
    plain = oracle(cfg, w, base, dtype)
    run = Run(tmp_path, dtype, dev, 1408)
    for at in (0, 31, n // 2):
        toks = list(base)
        toks[at] = mark
        ref = oracle(cfg, w, toks, dtype)
        assert float((ref - plain)[-1].abs().max()) > 0.2
        assert float((ref - plain)[:at].abs().max() if at else 0.0) < 1e-6
        run.step([(f"a{at}", toks, n - 12)])
        for i in range(12):
            run.step([(f"a{at}", toks, 1)], end=[f"a{at}"] if i == 11 else [])
        assert_close(run.logits(f"a{at}"), ref, dtype, f"mark at {at}")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_the_one_in_the_denominator_takes_its_share(dtype, device, tmp_path, request):
    """With small scores the first tokens' outputs shrink by what the one takes (half at the first token); the norm over the
    head's map hides a common factor, so the values of one head are made large against the others'."""
    from litinfer_b200.weights.safetensors_io import write_file

    dev = use_device(device, request)
    cfg = config([parallel(left(heads=2, kv=2, dim=16, vdim=16, rot=4, scale=0.05), right(heads=1, kv=1, dim=4, vdim=4))])
    w = make_weights(cfg, 33)
    w["l0.mix.left.k.norm"][:] = 40.0                          # head 0 and head 1: scores far from zero on either side
    toks = random_tokens(30, cfg["vocab"], 3)
    ref = oracle(cfg, w, toks, dtype)
    weights = P.weights_of_scores

    def without(s, seen, one_more=False):
        return weights(s, seen, False)

    P.weights_of_scores = without
    try:
        other = oracle(cfg, w, toks, dtype)
    finally:
        P.weights_of_scores = weights
    assert float((ref - other).abs().max() / ref.std()) > 0.2
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_file(tmp_path / "model.safetensors", w)
    run = Run(tmp_path, dtype, dev, 64)
    run.step([("a", toks, 1)])
    run.step([("a", toks, 20)])
    for _ in range(9):
        run.step([("a", toks, 1)])
    assert_close(run.logits("a"), ref, dtype, "with the one in the denominator")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("change", ["state", "conv"])
def test_a_lost_state_shows(change, device, folders, request):
    """Zeros in place of the rule's state or of the convolution's rows between two portions move the logits behind the cut far
    beyond the tolerance, so the portions of the other tests would show either; a slot used again starts from zeros."""
    dev = use_device(device, request)
    folder, cfg, w = folders["parallel_only"]
    toks = random_tokens(40, cfg["vocab"], 21)
    ref = oracle(cfg, w, toks, "float32")
    run = Run(folder, "float32", dev, 64, max_live=1, graphs=False)
    run.step([("a", toks, 20)])
    entry = run.rp.manager.entries[0].parts[1]
    r = cfg["layers"][0]["mixer"]["right"]
    cut = r["heads"] * r["dim"] * r["vdim"]
    slot = run.rp.live["a"].slot
    part = entry.state[slot, :cut] if change == "state" else entry.state[slot, cut:]
    assert float(part.abs().max()) > 0
    part.zero_()
    run.step([("a", toks, 20)], end=["a"])
    assert (run.logits("a")[20:] - ref[20:]).abs().max() > 1e-2 * ref.std()
    run.step([("b", toks, 40)], end=["b"])                     # the same slot, cleared at admission
    assert_close(run.logits("b"), ref, "float32", "slot used again")


@pytest.mark.parametrize("device", DEVICES)
def test_the_token_row_and_the_correction_count(device, folders, request):
    """Another table of token rows and another correction give other logits in the plain model; the engine follows each."""
    from litinfer_b200.engine.replay import Replayer
    from litinfer_b200.models import DecoderModel

    dev = use_device(device, request)
    folder, cfg, w = folders["mixed"]
    toks = random_tokens(24, cfg["vocab"], 9)
    ref = oracle(cfg, w, toks, "float32")
    table = dict(w, **{"side.embed": torch.roll(w["side.embed"], cfg["token_side"]["dim"], dims=1)})     # every layer another's columns
    corr = dict(w, **{"l1.mlp.correction": torch.linspace(2.0, -2.0, 8)})
    for changed, name in ((table, "table"), (corr, "correction")):
        other = oracle(cfg, changed, toks, "float32")
        assert float((other - ref).abs().max()) > 0.3
        model = DecoderModel.from_dir(folder, "float32", dev)
        target = model.token_tables["side.embed"] if name == "table" else model.blocks[1].feed_forward.correction
        target.copy_(changed["side.embed" if name == "table" else "l1.mlp.correction"])
        rp = Replayer(model, 64, use_graphs=False)
        got = rp.step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": list(range(24))}], "end": ["a"]}).float().cpu()
        assert_close(got, other, "float32", name)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_captured_steps(dtype, folders):
    """300 tokens one by one (steps replayed from a captured graph, chunks ending and their pages given back) against the
    prompt whole."""
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


def test_pages_of_chunks_that_are_over_go_back(cpu_kernels):
    """A group keeps the pages of the newest token's chunk, of every size that a layer reads it with, and no others; a page that a
    chunk's end cuts stays as long as one of its keys can be read."""
    from litinfer_b200.cache.manager import CacheManager
    from litinfer_b200.parts.base import PagedKV

    for chunks in ((40,), (24, 40), (16,), (1,), (100,)):
        m = CacheManager([PagedKV(1, 16, chunks=chunks)], [None], 16, 16, 2, torch.float32, "cpu")
        rc = m.admit(7)
        for n in range(1, 200):
            m.extend(rc, n)
            m.commit(rc, n)
            # the next query stands at position n or later: the first key it can still read
            first = min(n // c * c for c in chunks)
            held = [p >= 0 for p in m.table(rc, 0)]
            assert held == [(b + 1) * 16 > first for b in range(len(held))], f"chunks of {chunks}, {n} tokens"
            m.check()
        m.release(rc)
        assert m.num_free_pages(0) == 16


def test_what_a_reading_layer_needs_is_kept(folders):
    from litinfer_b200.config import config_from_dict
    from litinfer_b200.models.decoder import DecoderModel
    from litinfer_b200.parts.base import PagedKV

    for name, sizes in (("shared_longer", (10, 33)), ("shared_shorter", (10, 33))):
        model = DecoderModel(config_from_dict(CONFIGS[name]).to_model_spec(), "float32", "meta")
        own, reads = model.cache_requirements()
        assert reads is None and own == PagedKV(2, 32, chunks=sizes)
    assert PagedKV(2, 32, chunks=(8,)).covering(PagedKV(2, 32)) == PagedKV(2, 32)
    assert PagedKV(2, 32, window=5).covering(PagedKV(2, 32, window=9, keep_first=2)) == PagedKV(2, 32, window=9, keep_first=2)
    with pytest.raises(ValueError, match="is read as"):
        PagedKV(2, 32).covering(PagedKV(1, 32))


def test_configuration_is_read_and_refused():
    from litinfer_b200.config import ConfigError, config_from_dict

    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    parsed = config_from_dict(cfg)
    spec = parsed.to_model_spec()
    assert config_from_dict(parsed.to_dict()) == parsed
    assert spec.architecture == "Bozolorn" and not spec.tie_word_embeddings and spec.embedding_scale == 2.5
    assert spec.token_tables == {"side.embed": 5 * 20} and [b.parts["token_input"]["column"] for b in spec.blocks] == [0, 20, 40, 60, 80]
    assert [b.parts["mixer"].kind for b in spec.blocks] == ["parallel", "attention", "parallel", "attention", "attention"]
    assert [e.cache_from for e in spec.schedule] == [None, None, None, 1, None]
    a = spec.blocks[1].parts["mixer"]
    assert a["chunk"] == 29 and a["element_gate"] == "g" and a["distance_slopes"] == tuple(2.0 ** (-2.0 * h) for h in (1, 2, 3, 4)) and a["position"] is None
    p = spec.blocks[0].parts["mixer"]
    assert p["left"]["sink_score"] == 0.0 and p["left"]["qkv_bias"] and p["left"]["position"]["scaling"]["kind"] == "yarn"
    assert p["right"]["decay"] == "head" and p["right"]["gate"] == "silu" and (p["left_scale"], p["right_scale"]) == (0.5, 0.5)
    ff = spec.blocks[3].parts["feed_forward"]
    assert (ff["experts"], ff["top"], ff["groups"], ff["keep_groups"], ff["limit"], ff["scoring"]) == (9, 4, 3, 2, 2.0, "sigmoid_grouped")

    def broken(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises(ConfigError):
            config_from_dict(c)

    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mixer"].pop("right"))
    broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"))
    broken(lambda c: c["layers"][0]["mixer"]["right"].pop("conv"))
    broken(lambda c: c["layers"][1]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][1]["mixer"]["mask"].pop("size"))
    broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=5))            # one group of four is kept
    broken(lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3))
    broken(lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"))
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=0))                 # no attention layer
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=4))                 # behind it
    broken(lambda c: c["layers"][3]["mixer"].update(vdim=16))
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=3))                 # no keys of its own
    broken(lambda c: c["token_side"].update(dim=0))
    broken(lambda c: c["norm"].update(eps=0.0))


def test_random_weights_and_a_written_folder(tmp_path, cpu_kernels):
    """Random-weights mode knows the design's tensors; a folder written from it is read back through the registry."""
    from litinfer_b200.config import load_config
    from litinfer_b200.engine.replay import Replayer
    from litinfer_b200.models import DecoderModel
    from litinfer_b200.weights import write_model_folder

    cfg = CONFIGS["mixed"]
    write_model_folder(tmp_path, cfg, seed=5, store_dtype="float32")
    assert load_config(tmp_path).to_model_spec().token_tables == {"side.embed": 100}
    model = DecoderModel.from_dir(tmp_path, "float32", torch.device("cpu"))
    rp = Replayer(model, 64, max_live=2, use_graphs=False)
    logits = rp.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3, 4, 5], "want": [4]}], "end": ["a"]})
    assert logits.shape == (1, cfg["vocab"]) and torch.isfinite(logits).all() and float(logits.std()) > 0


# ---------------------------------------------------------------------------------------------
# the new kernels and forms, each against its plain reference
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
@pytest.mark.parametrize("chunk,slopes,gated,narrow", [(100, True, "elements", False), (100, True, "elements", True), (None, True, None, False), (37, False, "heads", False),
                                                       (1, True, "elements", True), (128, True, "heads", True)])
def test_attention_in_chunks_with_slopes_and_gates(implementation, q_lens, ctxs, dh, chunk, slopes, gated, narrow):
    """Every attention kernel with chunks (smaller and larger than its tiles), a penalty linear in the distance, a gate per head or
    per output element, and queries in q|k|v rows or alone beside the gate."""
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
    rows = (1.5 * torch.randn(T, 2 * H * dh if narrow else (H + 2 * G) * dh)).to(dev, dt)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    gate, more = None, {}
    if gated == "elements":
        gate, more = (rows, {"gate_col": H * dh}) if narrow else (torch.randn(T, H * dh).to(dev, dt), {})
        more["gate_elements"] = True
    elif gated == "heads":
        gate, more = torch.randn(T, H + 8).to(dev, dt), {"gate_col": 8}
    args = dict(k_cache=kc, v_cache=vc, block_table=table.to(dev), q_start=i32(starts), ctx_lens=i32(ctxs),
                seq_of_token=i32([s for s, n in enumerate(q_lens) for _ in range(n)]), positions=i32([c - n + i for n, c in zip(q_lens, ctxs) for i in range(n)]),
                num_heads=H, num_kv_heads=G, head_dim=dh, scale=1.0 / math.sqrt(dh), window=None, max_q_len=max(q_lens), max_ctx_len=max(ctxs), chunk=chunk or 0,
                slopes=torch.tensor([0.4, 0.1, 0.02, 0.003], device=dev) if slopes else None, gate=gate, **more)
    out, ref = (torch.empty(T, H * dh, dtype=dt, device=dev) for _ in range(2))
    lists = {}
    if implementation == "prefill_tcgen05":
        from litinfer_b200.engine.batch import attention_units

        units = attention_units(q_lens, ctxs, work_budget=148 // H)
        lists = dict(units=torch.from_numpy(units).to(dev), unit_slots=(int(units[0]), int(units[1])))
    K.paged_attention(rows, out, **args, implementation=implementation, **lists)
    R.paged_attention_dense(rows, ref, **args)
    _close(out, ref, "bfloat16", f"{implementation}, head of {dh}, chunk {chunk}")


@pytest.mark.gpu
def test_attention_in_chunks_in_float32():
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev = torch.device("cuda:0")
    torch.manual_seed(2)
    H, G, dh, page, T, ctx = 6, 3, 26, 16, 33, 60
    kc, vc = torch.randn(5, G, page, dh, device=dev), torch.randn(5, G, dh, page, device=dev)
    rows = torch.randn(T, 2 * H * dh, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    args = dict(k_cache=kc, v_cache=vc, block_table=i32([[3, 1, 4, 0]]), q_start=i32([0, T]), ctx_lens=i32([ctx]), seq_of_token=i32([0] * T),
                positions=i32(list(range(ctx - T, ctx))), num_heads=H, num_kv_heads=G, head_dim=dh, scale=0.3, window=None, max_q_len=T, max_ctx_len=ctx,
                chunk=14, slopes=torch.rand(H, device=dev), gate=rows, gate_col=H * dh, gate_elements=True)
    out, ref = (torch.empty(T, H * dh, device=dev) for _ in range(2))
    K.paged_attention(rows, out, **args)
    R.paged_attention(rows, ref, **args)
    _close(out, ref, "float32", "chunks of 14")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dh,real,rot,interleaved", [(6, 2, 24, 20, 10, True), (4, 1, 128, 128, 64, True), (3, 3, 18, 18, 6, True), (2, 1, 160, 150, 150, True),
                                                           (4, 2, 32, 32, 32, False), (2, 2, 8, 8, 0, False)])
def test_norm_before_the_rotation_kernel(nh, nkv, dh, real, rot, interleaved, dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(dh)
    page = 16
    den = torch.pow(torch.tensor(300.0), 2.0 * torch.arange(rot // 2) / max(rot, 1)).to(dev) if rot else None
    qn, kn = ((1 + 0.2 * torch.randn(dh)).to(dev) for _ in range(2))
    for T in (5, 90):
        slots = torch.randperm(10 * page)[:T].to(torch.int32).to(dev)
        pos = torch.randint(0, 2000, (T,), dtype=torch.int32, device=dev)
        proj = (1.3 * torch.randn(T, (nh + 2 * nkv) * dh + 40)).to(dev, dt)
        res = []
        for F in (K, R):
            out = torch.zeros(T, (nh + 2 * nkv) * dh, dtype=dt, device=dev)
            kc = torch.zeros(11, nkv, page, dh, dtype=dt, device=dev)
            vc = torch.zeros(11, nkv, dh, page, dtype=dt, device=dev)
            F.rope_norm_kv(proj, out, pos, den, rot, 1.17, interleaved, qn, kn, 2, 1e-5, real, slots, kc, vc, nh, nkv, dh, True)
            res.append((out[:, :nh * dh], kc, vc))
        for a, b, what in zip(res[0], res[1], ("queries", "keys", "values")):
            _close(a, b, dtype, f"{what}, {T} tokens", 2e-3 if dtype == "float32" else 2e-2)         # (angles of thousands of radians in float32)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,d,dv,taps", [(4, 2, 12, 20, 4), (3, 3, 7, 11, 5), (2, 1, 128, 128, 4), (6, 2, 64, 48, 3), (1, 1, 1, 1, 1), (2, 2, 200, 32, 2)])
def test_delta_rule_with_one_decay_a_head(heads, kv, d, dv, taps, dtype):
    """Preparation and walk: portions and single tokens beside each other, then single tokens whose convolution moves its state on."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(d + dv)
    C, DP = 2 * kv * d + heads * dv, K.delta_row_elements(d)
    col, width = 8, C + 2 * heads + 24
    conv_w = (0.6 * torch.randn(C, taps)).to(dev)
    A_log, dt_bias = (0.5 * torch.randn(heads) - 0.5).to(dev), (0.5 * torch.randn(heads)).to(dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    first = 0.3 * torch.randn(5, heads * d * dv + (taps - 1) * C, device=dev)
    for lens in ([37, 1, 80, 2], [1, 1, 1, 1], [150, 0, 1, 64]):
        T = sum(lens)
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        seq, slots = i32([s for s, n in enumerate(lens) for _ in range(n)]), i32([2, 0, 4, 1])
        proj = torch.randn(T, width).to(dev, dt)
        res = []
        for F in (K, R):
            state = first.clone()
            qk, g, v, o = (torch.empty(s, device=dev) for s in ((T, kv, 2 * DP + 4), (T, heads, 4), (T, heads * dv), (T, heads * dv)))
            single = max(lens) == 1
            F.delta_prepare(proj, col, col + C, conv_w, state, heads * d * dv, i32(starts), seq, slots, None, 0, A_log, qk, g, v, heads, kv, d, dv, shift=single,
                            a_col=col + C + heads, dt_bias=dt_bias)
            if not single and taps > 1:
                F.conv_state_shift(proj, col, C, taps, state, heads * d * dv, i32(starts), slots)
            F.delta_scan(qk, g, v, state, i32(starts), slots, o, heads, kv, d, dv)
            res.append((qk[..., :2 * DP + 1], g[..., :2], v, o, state))
        for a, b, what in zip(res[0], res[1], ("q and k", "decay and beta", "values", "outputs", "state")):
            _close(a, b, "float32", f"{what}, portions of {lens}", 1e-4)
    # one token a sequence, from the projections to the gated norm, as one kernel; twice, so that the second reads what the first left
    proj = torch.randn(4, width + heads * dv).to(dev, dt)
    w = 1 + 0.2 * torch.randn(heads * dv, device=dev)
    assert K.delta_step_accepts(heads, kv, d, dv)
    res = []
    for F in (K, R):
        state, y = first.clone(), torch.empty(4, heads * dv, dtype=dt, device=dev)
        for again in range(2):
            F.delta_step(proj if not again else (0.5 * proj), col, col + C, col + C + heads, width, conv_w, state, heads * d * dv, i32([2, 0, 4, 1]), dt_bias, A_log, w,
                         1e-5, y, heads, kv, d, dv)
        res.append((y, state))
    _close(res[0][0], res[1][0], dtype, "outputs of single tokens", 2e-4 if dtype == "float32" else 2e-2)
    _close(res[0][1], res[1][1], "float32", "state after single tokens", 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,d,dv", [(4, 2, 12, 20), (3, 3, 7, 11), (2, 1, 128, 128), (6, 2, 64, 48), (1, 1, 1, 1), (2, 2, 200, 160), (2, 1, 40, 130)])
@pytest.mark.parametrize("forget", [0.3, 60.0, 0.0])
def test_delta_rule_in_chunks(heads, kv, d, dv, forget, dtype):
    """Chunks as matrix products against the walk: portions that end on a chunk's edge, one token before and behind it, single tokens,
    several sequences, states of their own; heads that forget slowly, at once (decays of nothing), and never."""
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(d + dv)
    DP = K.delta_row_elements(d)
    first = 0.5 * torch.randn(6, heads * d * dv + 8, device=dev)
    for lens, slots in (([64, 63, 65, 1, 200], [4, 0, 2, 1, 3]), ([129, 0, 128], [1, 0, 2]), ([300], [5])):
        T = sum(lens)
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        q, k = (torch.nn.functional.normalize(torch.randn(T, kv, d, device=dev) + 0.7, dim=-1) for _ in range(2))
        qk = torch.zeros(T, kv, 2 * DP + 4, device=dev)
        qk[..., :d], qk[..., DP:DP + d], qk[..., 2 * DP] = q, k, (q * k).sum(-1)
        g = torch.zeros(T, heads, 4, device=dev)
        g[..., 2] = -forget * torch.rand(T, heads, device=dev) ** 2
        g[..., 0], g[..., 1] = torch.exp(g[..., 2]), torch.rand(T, heads, device=dev)
        v, gate = torch.randn(T, heads * dv, device=dev), torch.randn(T, heads * dv + 7).to(dev, dt)
        w = 1 + 0.2 * torch.randn(heads * dv, device=dev)
        chunks = K.ScanChunks(starts, slots, dev)
        res = []
        for F in (K, R):
            state, y = first.clone(), torch.empty(T, heads * dv, dtype=dt, device=dev)
            F.delta_chunks(qk, g, v, state, chunks, heads, kv, d, dv, gate, 7, w, 1e-5, y)
            res.append((state, y))
        _close(res[0][0], res[1][0], "float32", f"states, portions of {lens}", 1e-5)
        _close(res[0][1], res[1][1], dtype, f"outputs, portions of {lens}", 2e-4 if dtype == "float32" else 2e-2)
        # and the walk's kernel gives the same states
        state, o = first.clone(), torch.empty(T, heads * dv, device=dev)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        K.delta_scan(qk, g, v, state, i32(starts), i32(slots), o, heads, kv, d, dv)
        _close(res[0][0], state, "float32", "states of the walk", 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_routing_by_sigmoid_scores_in_groups(dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(4)
    for T, E, top, groups, keep in ((70, 6, 2, 3, 2), (5, 16, 4, 2, 1), (33, 80, 5, 40, 9), (9, 256, 8, 8, 3), (3, 4, 2, 4, 3), (300, 5, 3, 1, 1), (2, 1, 1, 1, 1), (64, 192, 6, 64, 20)):
        logits = (2.0 * torch.randn(T, E)).to(dev)
        for corr in ((0.3 * torch.randn(E) - 0.8).to(dev), None):      # (choice scores below zero: the others count as minus infinity, not as nothing)
            res = []
            for F in (K, R):
                ids, wt = torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev)
                F.moe_route_grouped(logits, corr, top, groups, keep, 1.5, ids, wt, scoring="sigmoid_grouped")
                res.append((ids, wt))
            assert torch.equal(res[0][0], res[1][0]), f"{T} tokens, {E} experts in {groups} groups"
            _close(res[0][1], res[1][1], "float32", "weights", 1e-6)
    for T, E, top, H, groups, keep in ((1, 16, 2, 64, 2, 1), (9, 6, 3, 48, 3, 2), (16, 8, 2, 256, 4, 2), (1, 100, 6, 128, 50, 7)):
        h, w = torch.randn(T, H).to(dev, dt), (2.0 * torch.randn(E, H) / math.sqrt(H)).to(dev, dt)
        corr = (0.3 * torch.randn(E)).to(dev)
        assert K.moe_small_step_accepts(h, E, top)
        res = []
        for F in (K, R):
            wt = torch.empty(T, top, device=dev)
            off, at, place = (torch.empty(n, dtype=torch.int32, device=dev) for n in (E + 1, T * top, T * top))
            F.moe_small_step(h, w, None, top, "sigmoid_grouped", corr, groups, keep, 1.0, wt, off, at, place)
            res.append((wt, off, at, place))
        assert all(torch.equal(a, b) for a, b in zip(res[0][1:], res[1][1:])), f"{T} tokens, {E} experts"
        _close(res[0][0], res[1][0], "float32", "weights", 1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_two_outputs_with_norms_into_the_stream_and_an_opened_token_row(dtype):
    import kernel_refs as R
    from litinfer_b200 import kernels as K

    dev, dt = torch.device("cuda:0"), _dt(dtype)
    torch.manual_seed(6)
    for T, H in ((7, 48), (3, 50), (5, 33), (40, 1536), (2, 8192)):
        a, b = torch.randn(T, H).to(dev, dt), (5.0 * torch.randn(T, H)).to(dev, dt)
        ws = [(1 + 0.2 * torch.randn(H, device=dev)).contiguous() for _ in range(4)]
        for norms in ((ws[0], ws[1], 1e-5), None):
            x = torch.randn(T, H, device=dev)
            rx, out, ref = x.clone(), torch.empty(T, H, dtype=dt, device=dev), torch.empty(T, H, dtype=dt, device=dev)
            K.norm_add_norm(x, K.WeightedPair(a, b, 0.5, 0.25, norms), (ws[2], False, 1e-5), (ws[3], False, 1e-5), out)
            R.norm_add_norm(rx, K.WeightedPair(a, b, 0.5, 0.25, norms), (ws[2], False, 1e-5), (ws[3], False, 1e-5), ref)
            _close(x, rx, "float32", "stream", 1e-5)
            _close(out, ref, dtype, "next norm")
            y = K.WeightedPair(a, b, 0.5, 0.25, norms).materialize()
            _close(y, R._pair_sum(K.WeightedPair(a, b, 0.5, 0.25, norms)), dtype, "sum")
    z = 3.0 * torch.randn(9, 20, device=dev)
    z[0, :3] = torch.tensor([-40.0, 40.0, 0.0], device=dev)
    table = torch.randn(50, 60).to(dev, dt)
    ids = torch.randint(0, 50, (12,), dtype=torch.int32, device=dev)
    out, ref = (torch.empty(9, 20, dtype=dt, device=dev) for _ in range(2))
    K.gelu_token_rows(z, table, 40, ids, out)
    R.gelu_token_rows(z, table, 40, ids, ref)
    _close(out, ref, dtype, "opened rows")
    with pytest.raises(K.KernelError, match="columns"):
        K.gelu_token_rows(z, table, 41, ids, out)
    for T, H, n in ((1, 64, 20), (9, 1536, 13), (16, 40, 60), (11, 2056, 24)):
        x, w = torch.randn(T, H).to(dev, dt), (2.0 * torch.randn(n, H) / math.sqrt(H)).to(dev, dt)
        ids = torch.randint(0, 50, (T,), dtype=torch.int32, device=dev)
        out, ref = (torch.empty(T, n, dtype=dt, device=dev) for _ in range(2))
        assert K.token_gate_accepts(x)
        K.token_gate(x, w, table, 60 - n, ids, out)
        R.token_gate(x, w, table, 60 - n, ids, ref)
        _close(out, ref, dtype, f"gate of {T} tokens")
    assert not K.token_gate_accepts(torch.empty(17, 64, dtype=dt, device=dev)) and not K.token_gate_accepts(torch.empty(3, 50, dtype=dt, device=dev))
