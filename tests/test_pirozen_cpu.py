"""The Pirozen design through the engine's host logic on the CPU: the step function, the cache (pages under windows, caches of its
own for every pass of a layer that runs several times) and the batch description run with the plain PyTorch kernels of
tests/ref_ops.py in place of the CUDA kernels and are compared with the plain whole-sequence implementation
(tests/plain_pirozen.py): each mechanism alone, whole prompts, token-by-token decoding, portions down to two tokens, batches of
unequal requests in a pool so small that pages and slots are used again, keys at page borders and just inside and outside the
window with attention made sharp, the first tokens of a request, long decoding, passes that must not share a cache, what the
correction, the groups, the identities and the weight factor do to the choice, the token's side rows, and greedy generation
through the entry point."""
import json
import os
import random

import pytest
import torch

import plain_pirozen as P
import ref_ops
from pirozen_configs import ALL, ONLY, PAGE_SIZE, att, config, moe, write_model, yarn
from zig_ai_b200.config import ConfigError, config_from_dict
from zig_ai_b200.engine import Engine
from zig_ai_b200.engine.runner import load_runner
from zig_ai_b200.models import build_model
from zig_ai_b200.weights.safetensors_io import SafetensorsFile, write_safetensors

ATOL = 3e-4          # float32 on the CPU against float64, logits of size one to ten


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("pirozen")
    out = {}
    for name, (cfg, seed) in list(ALL.items())[:2] + [(k, (c, 5)) for k, c in ONLY.items()]:
        out[name] = write_model(cfg, seed, str(root / name))
    return out


def read_model(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    f = SafetensorsFile(os.path.join(model_dir, "model.safetensors"))
    return cfg, {n: f.read(n) for n in f.names()}


def plain(model_dir, tokens):
    cfg, tensors = read_model(model_dir)
    return P.forward(cfg, tensors, tokens)


def runner(model_dir, page_size=8, max_tokens=512, max_requests=4):
    return load_runner(model_dir, "float32", max_tokens=max_tokens, max_requests=max_requests, page_size=page_size,
                       device="cpu", ops=ref_ops)


def tokens(vocab, n, seed):
    g = random.Random(seed)
    return [g.randrange(vocab) for _ in range(n)]


def close(got, want, what="", atol=ATOL):
    err = (got.double() - want).abs().max()
    assert err < atol, f"{what}: off by {float(err):.3e}"


def run_cut(r, rid, toks, cuts):
    r.add_request(rid)
    got, at = [], 0
    for n in cuts:
        got.append(r.step([(rid, toks[at:at + n], list(range(n)))]))
        at += n
    assert at == len(toks)
    r.end_request(rid)
    return torch.cat(got)


def with_tensors(model_dir, out_dir, change):
    """A copy of a model folder whose stored tensors `change` has altered (it gets them by name, bfloat16 as stored, and
    alters the dict in place)."""
    os.makedirs(out_dir, exist_ok=True)
    f = SafetensorsFile(os.path.join(model_dir, "model.safetensors"))
    tensors = {n: f.read(n).clone() for n in f.names()}
    change(tensors)
    write_safetensors(os.path.join(out_dir, "model.safetensors"), tensors)
    with open(os.path.join(model_dir, "config.json")) as src, open(os.path.join(out_dir, "config.json"), "w") as dst:
        dst.write(src.read())
    return out_dir


def altered(cfg, path, value):
    out = json.loads(json.dumps(cfg))
    at = out
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return out


@pytest.mark.parametrize("name", sorted(ONLY))
def test_each_mechanism_alone(models, name):
    r = runner(models[name])
    toks = tokens(r.model.vocab_size, 45, 1)
    want = plain(models[name], toks)
    close(run_cut(r, "w", toks, [45]), want, "whole")
    close(run_cut(r, "d", toks, [1] * 45), want, "token by token")
    close(run_cut(r, "p", toks, [2, 7, 1, 3, 16, 2, 9, 5]), want, "portions")


@pytest.mark.parametrize("name", ["A", "B"])
def test_whole_decode_and_portions(models, name):
    r = runner(models[name], PAGE_SIZE[name])
    toks = tokens(r.model.vocab_size, 75, 2)
    want = plain(models[name], toks)
    close(run_cut(r, "w", toks, [75]), want, "whole")
    close(run_cut(r, "d", toks, [43] + [1] * 32), want, "decoded tail")
    for seed, sizes in ((3, (2, 3, 5)), (4, (2, 11, 17)), (5, (7, 8, 9, 16))):
        g, cuts, left = random.Random(seed), [], 75
        while left:
            n = min(g.choice(sizes), left)
            cuts.append(n)
            left -= n
        close(run_cut(r, f"p{seed}", toks, cuts), want, f"portions {sizes}")
    assert r.cache.stats()["slots_used"] == 0


@pytest.mark.parametrize("name", ["A", "B"])
def test_first_tokens_and_tiny_requests(models, name):
    r = runner(models[name], PAGE_SIZE[name])
    for n in (1, 2, 3):
        toks = tokens(r.model.vocab_size, n, 10 + n)
        close(run_cut(r, f"t{n}", toks, [n]), plain(models[name], toks), f"{n} tokens")
    toks = tokens(r.model.vocab_size, 9, 20)
    close(run_cut(r, "s", toks, [1, 2, 1, 2, 3]), plain(models[name], toks), "small portions from the start")


@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_together_in_a_small_pool(models, name):
    """Four slots and a pool of a few pages: requests wait for room, and the pages and slots of finished requests go to the
    next ones; a request is sometimes left out of a step; every row equals the request alone."""
    ps = PAGE_SIZE[name]
    lengths = [23, 40, 9, 31, 1, 17, 28, 2, 36]
    r = runner(models[name], ps, max_tokens=6 * 16, max_requests=4)
    V = r.model.vocab_size
    reqs = {f"r{i}": tokens(V, n, 100 + i) for i, n in enumerate(lengths)}
    want = {k: plain(models[name], t) for k, t in reqs.items()}
    g = random.Random(9)
    waiting, live, at, got = list(reqs), [], {}, {k: [] for k in reqs}
    room = r.cache.num_pages * ps
    slots_seen = []
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-len(reqs[x]) // ps) * ps for x in live + [waiting[0]]) <= room:
            k = waiting.pop(0)
            live.append(k)
            at[k] = 0
            r.add_request(k)
            slots_seen.append(r.cache.requests[k].slot)
        entries = []
        for k in live:
            if len(live) > 1 and g.random() < 0.25:
                continue
            left = len(reqs[k]) - at[k]
            n = 1 if left <= len(reqs[k]) // 3 else min(g.choice([2, 3, 5, 8]), left)
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
        if not entries:
            continue
        logits = r.step(entries)
        row = 0
        for k, toks, w in entries:
            got[k].append(logits[row:row + len(w)].clone())
            row += len(w)
        for k in [k for k in live if at[k] == len(reqs[k])]:
            live.remove(k)
            r.end_request(k)
        r.cache.check()
    for k in reqs:
        close(torch.cat(got[k]), want[k], f"request {k} among others")
    assert len(slots_seen) > len(set(slots_seen)) and r.cache.pages_reused > 0     # slots and pages were used again


def test_window_edges(models):
    """A key just inside the window and just outside it shows in the logits: every cut of the request agrees with the whole
    sequence, for queries in portions and decoded one by one, with pages of 4 (the window ends inside pages); pages behind the
    window go back to the pool while the request runs."""
    d = models["sharp_attention"]
    cfg, tensors = read_model(d)
    r = runner(d, page_size=4)
    toks = tokens(cfg["vocab"], 60, 7)
    want = P.forward(cfg, tensors, toks)
    path = ("layers", 0, "mixer")
    for key, value in (("mask", {"size": 14}), ("mask", {"size": 12}), ("scale", 2.2)):
        assert (P.forward(altered(cfg, path + (key,), value), tensors, toks) - want).abs().max() > 1e-2, key
    for key, value in (("factor", 3.3), ("original", 20), ("fast", 1.0), ("slow", 0.9)):
        assert (P.forward(altered(cfg, path + ("rot", "scaling", key), value), tensors, toks) - want).abs().max() > 1e-2, key
    close(run_cut(r, "w", toks, [60]), want, "whole")
    close(run_cut(r, "d", toks, [5] + [1] * 55), want, "decoded across the window's edge")
    close(run_cut(r, "p", toks, [3, 10, 2, 13, 1, 14, 2, 2, 13]), want, "portions that end at the window's edges")
    r.add_request("k")
    r.step([("k", toks[:40], [])])
    r.step([("k", toks[40:41], [])])
    table = r.cache.requests["k"].tables[r.cache.paged_groups()[0]]
    assert -1 in table and table[-1] > 0
    r.end_request("k")


def test_every_pass_has_caches_of_its_own(models):
    """A looped layer's passes hold different keys: the passes' pages differ, and every pass counts in the logits."""
    d = models["loop_at_the_end"]
    cfg, tensors = read_model(d)
    r = runner(d)
    assert [k for k, _ in r.model.cache_needs()] == ["own"] * 9          # two layers, the second four times, each behind a merge
    assert sum(len(n) > 0 for _, n in r.model.cache_needs()) == 5
    toks = tokens(cfg["vocab"], 30, 4)
    want = P.forward(cfg, tensors, toks)
    r.add_request("a")
    r.step([("a", toks[:29], [])])
    rows = r.cache.requests["a"]
    assert rows is not None
    close(r.step([("a", toks[29:], [0])]), want[29:], "decoded behind four passes")
    r.end_request("a")
    for times in (1, 2, 3):
        assert (P.forward(altered(cfg, ("loop", "times"), times), tensors, toks) - want).abs().max() > 1e-2
    no_embedding = dict(tensors)
    no_embedding["loop.in"] = tensors["loop.in"].clone()
    no_embedding["loop.in"][:, cfg["width"]:] = 0
    assert (P.forward(cfg, no_embedding, toks) - want).abs().max() > 1e-2


def test_running_order_of_a_loop():
    for loop, want in ((None, [0, 1, 2, 3]), ((1, 3, 3), [0, 4, 1, 2, 4, 1, 2, 4, 1, 2, 3]), ((0, 4, 1), [4, 0, 1, 2, 3]),
                       ((0, 1, 2), [4, 0, 4, 0, 1, 2, 3]), ((3, 4, 2), [0, 1, 2, 4, 3, 4, 3])):
        model = build_model(config_from_dict(config(50, 24, 1e-5, [att(2, 1, 8, 8, 0.3, 9, 4)] * 4, loop=loop)))
        assert [c.layer for c in model.spec.order] == want


def test_what_the_choice_goes_by(models):
    """The correction moves tokens to other experts without changing a weight's score, the groups take experts away, the factor
    scales: leaving any of it out gives other logits, and the framework's equal the plain ones."""
    cfg, tensors = read_model(models["experts"])
    toks = tokens(cfg["vocab"], 30, 3)
    want = P.forward(cfg, tensors, toks)
    router = ("layers", 0, "mlp", "router")
    for key, value in (("scale", 1.6), ("groups", None), ("groups", {"count": 4, "keep": 3}), ("groups", {"count": 2, "keep": 1}), ("top", 2)):
        assert (P.forward(altered(cfg, router + (key,), value), tensors, toks) - want).abs().max() > 1e-2, (key, value)
    for change in (lambda c: c * 0, lambda c: c - 1.0 * torch.arange(len(c))):
        other = dict(tensors, **{"l0.mlp.correction": change(tensors["l0.mlp.correction"].float())})
        assert (P.forward(cfg, other, toks) - want).abs().max() > 1e-2
    same = dict(tensors, **{"l0.mlp.correction": tensors["l0.mlp.correction"].double() - 5.0})     # all negative: no other choice
    assert (P.forward(cfg, same, toks) - want).abs().max() < 1e-9


def test_corrections_that_send_every_token_to_identities(models, tmp_path):
    """All chosen outputs are identities: no row enters an expert, and the sum is the input times the factor, plus the expert for
    every token; and the other way round, no identity is chosen.  All choice values are negative: a group that is left out must
    count as less than any of them."""
    for sign, tag in ((1.0, "only"), (-1.0, "none")):
        def change(t):
            c = torch.full((8,), -9.0)
            c[6:] += 4.0 * sign
            t["l0.mlp.correction"] = c.to(torch.bfloat16)
        d = with_tensors(models["experts"], str(tmp_path / tag), change)
        with open(os.path.join(d, "config.json")) as f:
            cfg = json.load(f)
        cfg["layers"][0]["mlp"]["router"].update(top=2, groups={"count": 4, "keep": 1} if sign > 0 else {"count": 4, "keep": 2})
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        toks = tokens(cfg["vocab"], 25, 8)
        r = runner(d)
        close(run_cut(r, "w", toks, [25]), plain(d, toks), tag)
        close(run_cut(r, "d", toks, [9] + [1] * 16), plain(d, toks), tag)


def test_side_rows_go_by_token_and_layer(models):
    cfg, tensors = read_model(models["side_rows"])
    toks = tokens(cfg["vocab"], 30, 3)
    want = P.forward(cfg, tensors, toks)
    dim = cfg["token_side"]["dim"]
    swapped = torch.cat([tensors["side.embed"][:, dim:], tensors["side.embed"][:, :dim]], dim=1)
    rolled = tensors["side.embed"].roll(1, 0)
    for t in (swapped, rolled):
        assert (P.forward(cfg, dict(tensors, **{"side.embed": t}), toks) - want).abs().max() > 1e-2
    close(run_cut(runner(models["side_rows"]), "w", toks, [30]), want, "whole")


def test_long_decoding(models):
    r = runner(models["A"], PAGE_SIZE["A"], max_tokens=256)
    toks = tokens(r.model.vocab_size, 160, 17)
    close(run_cut(r, "d", toks, [4] + [1] * 156), plain(models["A"], toks), "156 decoded tokens")


def test_config_errors():
    good = ALL["A"][0]
    mixer, router = ("layers", 0, "mixer"), ("layers", 0, "mlp", "router")
    for path, value in ((("layers", 0, "type"), "conv"), (mixer + ("mask", "size"), 0), (mixer + ("kv_heads",), 3), (mixer + ("rot", "dims"), 5),
                        (mixer + ("rot", "dims"), 14), (mixer + ("rot", "base"), 0.0), (mixer + ("rot", "scaling", "factor"), 0.0),
                        (mixer + ("rot", "scaling", "fast"), None), (mixer + ("scale",), None), (("norm",), None), (("loop", "stop"), 4),
                        (("loop", "start"), 3), (("loop", "times"), 0), (("token_side", "dim"), 0), (router + ("groups", "count"), 3),
                        (router + ("groups", "keep"), 5), (router + ("top",), 9), (router + ("identity",), -1), (router + ("top",), 5),
                        (("layers", 0, "mlp"), {"kind": "dense", "ff": 8})):
        with pytest.raises(ConfigError):
            config_from_dict(altered(good, path, value))


def test_configuration_round_trip():
    cfg = config_from_dict(ALL["B"][0])
    assert cfg.architecture == "Pirozen" and cfg.vocab_size == 257 and cfg.hidden_size == 66 and len(cfg.layers) == 4
    assert cfg.token_side == 12 and cfg.loop == {"start": 0, "stop": 2, "times": 2}
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    bare = config_from_dict(ONLY["attention"])
    assert bare.loop is None and bare.token_side is None and config_from_dict(bare.to_dict()).to_dict() == bare.to_dict()
    names = build_model(cfg).param_decls()
    assert tuple(names["side.embed"].shape) == (257, 48) and tuple(names["loop.in"].shape) == (66, 132)
    assert tuple(names["l1.mlp.router"].shape) == (9, 66) and tuple(names["l0.mlp.correction"].shape) == (8,)
    assert "l0.mlp.e1.gate" in names and "l0.mlp.e2.gate" not in names          # the other six are identities


def random_router(g, most=8):
    """Sizes of a router that fit together: equal groups, of which the kept ones hold enough to choose from."""
    groups = None if g.random() < 0.3 else g.randrange(1, 6)
    total = (groups or 1) * g.randrange(1, 5)
    identity = g.randrange(0, total) if g.random() < 0.8 else 0
    keep = g.randrange(1, groups + 1) if groups else None
    room = total if groups is None else keep * (total // groups)
    return dict(experts=total - identity, identity=identity, top=min(g.randrange(1, room + 1), most),
                groups=None if groups is None else (groups, keep), scale=round(g.uniform(0.4, 3.0), 2))


def random_config(g, heads=4, dims=(4, 20), windows=40, ff=(4, 30), vocab=(40, 200), width=None, sizes=None):
    layers = []
    n = g.randrange(1, 5)
    for i in range(n):
        mlp = None if g.random() < 0.25 else moe(g.randrange(*ff), shared=None if g.random() < 0.4 else g.randrange(*ff), **random_router(g))
        kv, per = g.randrange(1, heads), g.randrange(1, heads)
        dim, vdim = (g.choice(sizes), g.choice(sizes)) if sizes else (g.randrange(*dims), g.randrange(*dims))
        scaling = None if g.random() < 0.25 else yarn(round(g.uniform(1.5, 16.0), 2), g.randrange(16, 300), g.uniform(2.0, 32.0), g.uniform(0.2, 1.5))
        layers.append(att(kv * per, kv, dim, vdim, g.uniform(0.5, 1.5) * dim ** -0.5, g.randrange(1, windows), 2 * g.randrange(0, dim // 2 + 1),
                          g.choice([20.0, 500.0, 10000.0, 1e6]), scaling, mlp))
    loop = None
    if g.random() < 0.7:
        start = g.randrange(n)
        loop = (start, g.randrange(start + 1, n + 1), g.randrange(1, 4))
    return config(g.randrange(*vocab), width(g) if width else g.randrange(12, 70), 10.0 ** -g.randrange(4, 7), layers,
                  None if g.random() < 0.25 else g.randrange(1, 20), loop)


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes, layer orders, loops and constants drawn at random, each whole, in portions and decoded."""
    g = random.Random(50 + seed)
    cfg = random_config(g)
    d = write_model(cfg, seed, str(tmp_path / "m"))
    r = runner(d, page_size=g.choice([4, 8, 16]))
    toks = tokens(cfg["vocab"], 50, seed)
    want = plain(d, toks)
    close(run_cut(r, "w", toks, [50]), want, "whole")
    close(run_cut(r, "p", toks, [2, 5, 13, 2, 9, 16, 3]), want, "portions")
    close(run_cut(r, "d", toks, [30] + [1] * 20), want, "decoded")


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_entry_point(models, name):
    """`Engine.generate` (scheduler, sampler, step function, prompts in portions of six tokens beside decoding requests)
    against the plain implementation's choice at every produced token."""
    cfg, tensors = read_model(models[name])
    g = random.Random(3)
    prompts = [[g.randrange(cfg["vocab"]) for _ in range(n)] for n in (7, 13, 1, 22)]
    eng = Engine(models[name], "float32", max_num_seqs=3, max_batched_tokens=6, max_model_len=64,
                 page_size=PAGE_SIZE[name], device="cpu", ops=ref_ops)
    got = eng.generate(prompts, max_new_tokens=8, temperature=0.0)
    for p, out in zip(prompts, got):
        assert len(out) == 8
        logits = P.forward(cfg, tensors, p + out)
        for i, tok in enumerate(out):
            row = logits[len(p) + i - 1]
            assert float(row.max() - row[tok]) < ATOL, f"token {i} is not the plain implementation's choice"
    assert eng.stats()["slots_used"] == 0
