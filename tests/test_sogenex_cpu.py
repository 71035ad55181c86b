"""The Sogenex design through the engine's host logic on the CPU: the step function, the cache (pages of keys of two maps and
their values under a window, slots of recurrent state and of the convolution's history, an own cache and state for layers that
run on another layer's tensors) and the batch description run with the plain PyTorch kernels of tests/ref_ops.py in place of
the CUDA kernels and are compared with the plain whole-sequence implementation (tests/plain_sogenex.py): each mechanism alone,
whole prompts, token-by-token decoding, portions down to two tokens, batches of unequal requests in a pool so small that
pages and slots are used again, keys at page borders and just inside and outside the window with attention made sharp in
either map, far tokens that the state keeps, the first tokens of a request, long decoding, the router's bias and the gated
unit, and greedy generation through the entry point."""
import json
import os
import random

import pytest
import torch

import plain_sogenex as P
import ref_ops
from sogenex_configs import ALL, ONLY, PAGE_SIZE, config, diff, moe, ssm, write_model
from zig_ai_b200.config import ConfigError, config_from_dict
from zig_ai_b200.engine import Engine
from zig_ai_b200.engine.runner import load_runner
from zig_ai_b200.weights.safetensors_io import SafetensorsFile, write_safetensors

ATOL = 3e-4          # float32 on the CPU against float64, logits of size one to ten


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("sogenex")
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
    """Requests of one to three tokens and small portions from the start: the empty state and history, position zero's
    vector, a first token that attends to itself alone."""
    r = runner(models[name], PAGE_SIZE[name])
    for n in (1, 2, 3):
        toks = tokens(r.model.vocab_size, n, 10 + n)
        close(run_cut(r, f"t{n}", toks, [n]), plain(models[name], toks), f"{n} tokens")
    toks = tokens(r.model.vocab_size, 9, 20)
    close(run_cut(r, "s", toks, [1, 2, 1, 2, 3]), plain(models[name], toks), "small portions from the start")


@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_together_in_a_small_pool(models, name):
    """Four slots and a pool of a few pages: requests wait for room, and the pages and slots of finished requests go to the
    next ones (whose state and history start from zero all the same); a request is sometimes left out of a step; every row
    equals the request alone."""
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


def sharp_map(tensors, pre, heads, dim, which):
    """Make layer `pre`'s attention depend on single keys in one of its maps: that map's rows of the k projection are scaled
    up so that scores differ by many units."""
    k = tensors[pre + "k"].float()
    k = k.reshape(-1, 2, dim, k.shape[1])
    k[:, which] *= 6.0
    tensors[pre + "k"] = k.reshape(tensors[pre + "k"].shape).to(torch.bfloat16)
    # the difference's weights: lambda away from zero and from one, so that both maps count
    for name, value in (("lq1", 0.3), ("lk1", 0.2), ("lq2", 0.1), ("lk2", -0.4)):
        tensors[pre + name] = torch.full_like(tensors[pre + name], value)


@pytest.mark.parametrize("which", [0, 1])
def test_window_edges_in_either_map(models, tmp_path, which):
    """With one map made sharp a key just inside the window and just outside it shows in the logits: every cut of the request
    agrees with the whole sequence, for queries in portions and decoded one by one, with pages of 4 (the window ends inside
    pages); pages behind the window go back to the pool while the request runs."""
    d = with_tensors(models["sharp_maps"], str(tmp_path / "sharp"), lambda t: sharp_map(t, "l0.mix.", 3, 10, which))
    cfg, tensors = read_model(d)
    r = runner(d, page_size=4)
    toks = tokens(cfg["vocab"], 60, 7)
    want = P.forward(cfg, tensors, toks)
    path = ("layers", 0, "mixer")
    for key, value in (("mask", {"size": 14}), ("mask", {"size": 12}), ("diff", 0.35), ("scale", 2.1)):
        assert (P.forward(altered(cfg, path + (key,), value), tensors, toks) - want).abs().max() > 1e-2, key
    close(run_cut(r, "w", toks, [60]), want, "whole")
    close(run_cut(r, "d", toks, [5] + [1] * 55), want, "decoded across the window's edge")
    close(run_cut(r, "p", toks, [3, 10, 2, 13, 1, 14, 2, 2, 13]), want, "portions that end at the window's edges")
    r.add_request("k")
    r.step([("k", toks[:40], [])])
    r.step([("k", toks[40:41], [])])
    table = r.cache.requests["k"].tables[r.cache.paged_groups()[0]]
    assert -1 in table and table[-1] > 0
    r.end_request("k")


def test_maps_share_pages_without_copies(models):
    """A page holds a key head's two maps side by side and its values once: two times the map's size, or the values' if wider."""
    r = runner(models["two_maps"])
    need = [g.need for g in r.cache.groups if g.paged][0]
    assert (need.kv_heads, need.head_dim, need.window) == (2, 16, 13)
    r = runner(models["experts_all"])
    need = [g.need for g in r.cache.groups if g.paged][0]
    assert (need.kv_heads, need.head_dim, need.window) == (1, 16, 9)


def test_the_state_keeps_a_far_token(models, tmp_path):
    """Decays near one and a step size that is large for one token: the state holds that token for the rest of the request, and
    portions, single tokens and the whole sequence agree."""
    def change(t):
        t["l0.mix.A_log"] = torch.full_like(t["l0.mix.A_log"], -7.0)
        t["l0.mix.dt_bias"] = torch.full_like(t["l0.mix.dt_bias"], -3.0)
        t["l0.mix.in"][-4:] = (t["l0.mix.in"][-4:].float() * 6.0).to(torch.bfloat16)       # the heads' step sizes
    d = with_tensors(models["state_space"], str(tmp_path / "far"), change)
    cfg, tensors = read_model(d)
    toks = tokens(cfg["vocab"], 90, 13)
    want = P.forward(cfg, tensors, toks)
    other = list(toks)
    other[3] = (toks[3] + 1) % cfg["vocab"]
    assert (P.forward(cfg, tensors, other)[-1] - want[-1]).abs().max() > 1e-3              # the third token is still seen at the end
    r = runner(d, page_size=8)
    close(run_cut(r, "w", toks, [90]), want, "whole")
    close(run_cut(r, "d", toks, [20] + [1] * 70), want, "long decoding")
    close(run_cut(r, "p", toks, [2, 2, 31, 16, 17, 2, 20]), want, "portions")


def test_router_bias_and_gated_unit_count(models):
    """The bias moves tokens to other experts and changes the weights, the unit's gate is one number per token: leaving either
    out, or weighing by the softmax over all experts, gives other logits."""
    cfg, tensors = read_model(models["experts"])
    toks = tokens(cfg["vocab"], 30, 3)
    want = P.forward(cfg, tensors, toks)
    for name, change in (("router.b", lambda t: t + 2.0 * torch.arange(len(t))), ("shared.sg", lambda t: t + 1.0), ("router", lambda t: t * 2.0)):
        other = dict(tensors)
        other["l0.mlp." + name] = change(tensors["l0.mlp." + name].float())
        assert (P.forward(cfg, other, toks) - want).abs().max() > 1e-2, name
    r = runner(models["experts"])
    close(run_cut(r, "w", toks, [30]), want, "whole")


def test_long_decoding(models):
    r = runner(models["A"], PAGE_SIZE["A"], max_tokens=256)
    toks = tokens(r.model.vocab_size, 160, 17)
    close(run_cut(r, "d", toks, [4] + [1] * 156), plain(models["A"], toks), "156 decoded tokens")


def test_config_errors():
    good = ONLY["tensors_used_again"]
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "groups"), 3), (("layers", 0, "mixer", "norm_groups"), 3),
                        (("layers", 1, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "kv_heads"), 4), (("norm",), None),
                        (("layers", 2, "weights_of"), 2), (("layers", 2, "weights_of"), 1), (("layers", 2, "mixer", "state"), 9),
                        (("logit_softcap",), 0.0), (("layers", 0, "mlp"), {"kind": "dense", "ff": 8}),
                        (("layers", 0, "mlp"), moe(8, 2, 3))):
        with pytest.raises(ConfigError):
            config_from_dict(altered(good, path, value))


def test_configuration_round_trip():
    cfg = config_from_dict(ALL["B"][0])
    assert cfg.architecture == "Sogenex" and cfg.vocab_size == 257 and cfg.hidden_size == 66 and len(cfg.layers) == 5
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    chained = config_from_dict(ONLY["tensors_used_again"])
    assert [la.get("weights_of") for la in chained.layers] == [None, None, 0, 1, 0]


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes, layer orders and constants drawn at random, each whole, in portions and decoded."""
    g = random.Random(50 + seed)
    layers = []
    for i in range(g.randrange(1, 5)):
        mlp = None if g.random() < 0.3 else moe(g.randrange(4, 30), *(lambda e: (e, g.randrange(1, e + 1)))(g.randrange(1, 8)),
                                                shared=None if g.random() < 0.4 else g.randrange(3, 30))
        if layers and g.random() < 0.3:
            of = g.randrange(len(layers))
            layers.append(dict({k: v for k, v in layers[of].items() if k != "weights_of"}, weights_of=of))
        elif g.random() < 0.5:
            groups, per, parts = g.randrange(1, 4), g.randrange(1, 4), g.randrange(1, 4)
            layers.append(ssm(groups * per, parts * g.randrange(1, 9), g.randrange(1, 24), groups, g.randrange(1, 6), parts, mlp))
        else:
            kv, per = g.randrange(1, 4), g.randrange(1, 4)
            layers.append(diff(kv * per, kv, g.randrange(2, 16), g.randrange(2, 30), g.uniform(0.2, 0.8), g.randrange(1, 40),
                               round(g.uniform(-0.2, 0.9), 3), mlp))
    cfg = config(g.randrange(40, 200), g.randrange(12, 70), 10.0 ** -g.randrange(4, 7), layers, g.uniform(0.5, 2.0), g.uniform(5.0, 40.0))
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
