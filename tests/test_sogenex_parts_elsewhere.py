"""The parts and options that came with the Sogenex design are parts like any other: a sixth toy architecture, defined in
this file, puts the state-space mixer (without a convolution bias) into the block with a norm before and after each sublayer
in front of experts whose units are plain SwiGLU, chosen by softmax scores with a bias and with a gated SwiGLU unit beside
them; and, into the block with the norm behind the sublayers, differential attention without a window in front of a dense
feed-forward with the square of relu.  Its embedding is scaled and its position vectors have another base.  Registered, written
with random weights, stepped in portions and single tokens, and compared with plain formulas; nothing under the package
changes."""
import random
from dataclasses import dataclass

import pytest
import torch

import plain_sogenex as P
import ref_ops
from zig_ai_b200.config import ModelConfig, register_architecture, unregister_architecture
from zig_ai_b200.engine.runner import load_runner
from zig_ai_b200.parts import LayerCall, LayerSpec, ModelSpec, PartSpec
from zig_ai_b200.weights import write_random_model
from zig_ai_b200.weights.safetensors_io import SafetensorsFile

T6 = dict(hidden=40, vocab=83, eps=1e-5, mult=0.8, scale=30.0, base=500.0, heads=6, vdim=5, state=9, groups=3, taps=3, parts=2,
          att_heads=4, att_kv=2, dim=6, att_vdim=10, att_scale=0.5, diff=0.25, experts=5, top=2, ff=24, unit_ff=16, dense_ff=56)
SSM = {"in": "s.in", "conv": "s.conv", "dt_bias": "s.dt", "a_log": "s.a", "d": "s.d", "norm": "s.norm", "o": "s.o"}
ATT = {k: "a." + k for k in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")}
EXPERTS = {"router": "x.router", "router_bias": "x.bias", "gate": "x.e{e}.gate", "up": "x.e{e}.up", "down": "x.e{e}.down", "shared_gate": "x.sg"}


@dataclass
class Toy6Config(ModelConfig):
    @classmethod
    def from_dict(cls, d):
        return cls("Toy6ForTests")

    def to_dict(self):
        return {"architectures": ["Toy6ForTests"]}


def toy6_spec(cfg):
    a, W = T6, T6["hidden"]
    norm = lambda name: PartSpec("rmsnorm", dict(size=W, eps=a["eps"], weight=name))
    mixer = PartSpec("mamba2", dict(hidden=W, heads=a["heads"], vdim=a["vdim"], state=a["state"], groups=a["groups"], taps=a["taps"],
                                    norm_parts=a["parts"], eps=a["eps"], conv_bias=False, names=SSM))
    unit = PartSpec("swiglu", dict(hidden=W, ff_dim=a["unit_ff"], names={"gate": "x.u.gate", "up": "x.u.up", "down": "x.u.down"}))
    experts = PartSpec("routed_experts", dict(hidden=W, ff_dim=a["ff"], experts=a["experts"], top=a["top"], renormalize=True, weight_on="output",
                                              score="softmax", router_bias=True, shared=unit, shared_gate=True, names=EXPERTS))
    att = PartSpec("attention", dict(hidden=W, heads=a["att_heads"], kv_heads=a["att_kv"], head_dim=a["dim"], value_dim=a["att_vdim"], qk_norm=False,
                                     eps=a["eps"], position=PartSpec("none", {}), scale=a["att_scale"], differential={"diff": a["diff"]}, names=ATT))
    dense = PartSpec("dense", dict(hidden=W, ff_dim=a["dense_ff"], activation="relu2", names={"up": "f.up", "down": "f.down"}))
    layers = [
        LayerSpec("l0.", PartSpec("sandwich_residual", dict(mixer=mixer, mixer_norm=norm("n0"), mixer_post_norm=norm("n1"), feed_forward=experts,
                                                            ff_norm=norm("n2"), ff_post_norm=norm("n3")))),
        LayerSpec("l1.", PartSpec("postnorm_residual", dict(mixer=att, mixer_norm=norm("n0"), feed_forward=dense, ff_norm=norm("n1"), mult=a["mult"]))),
    ]
    return ModelSpec("Toy6ForTests", W, a["vocab"], 256, PartSpec("embedding", dict(weight="emb", scale=a["scale"], sinusoidal=a["base"])), layers,
                     [LayerCall(0), LayerCall(1)], norm("final"), PartSpec("linear_head", dict(weight="head", tied=False)))


def toy6_plain(W, tokens):
    a, dt = T6, torch.float64
    w = lambda name: W[name].to(dt)
    n = lambda x, name: P.rms(x, a["eps"]) * w(name)
    T, H, V, N, G = len(tokens), a["heads"], a["vdim"], a["state"], a["groups"]
    t, c = torch.arange(T, dtype=dt)[:, None], torch.arange(a["hidden"])
    angle = t * a["base"] ** (-2.0 * (c // 2).to(dt) / a["hidden"])
    h = w("emb")[torch.tensor(tokens)] * a["scale"] + torch.where(c % 2 == 0, torch.sin(angle), torch.cos(angle))
    # the state-space mixer between two norms
    y = n(h, "l0.n0") @ w("l0.s.in").T
    I, ch = H * V, H * V + 2 * G * N
    u = P.convolve(y[:, I:I + ch], w("l0.s.conv"), torch.zeros(ch, dtype=dt))
    d = torch.nn.functional.softplus(y[:, I + ch:] + w("l0.s.dt"))
    o = P.state_space(u[:, :I].reshape(T, H, V), u[:, I:I + G * N].reshape(T, G, N), u[:, I + G * N:].reshape(T, G, N), d, w("l0.s.a"), w("l0.s.d"))
    h = h + n(P.gated_norm(o.reshape(T, I), y[:, :I], a["parts"], w("l0.s.norm"), a["eps"]) @ w("l0.s.o").T, "l0.n1")
    # experts by softmax scores of biased logits, and a gated unit
    r = n(h, "l0.n2")
    glu = lambda x, pre: (P.silu(x @ w(pre + "gate").T) * (x @ w(pre + "up").T)) @ w(pre + "down").T
    s = torch.softmax(r @ w("l0.x.router").T + w("l0.x.bias"), dim=-1)
    f = torch.sigmoid(r @ w("l0.x.sg").T) * glu(r, "l0.x.u.")
    for i in range(T):
        chosen = sorted(range(a["experts"]), key=lambda e: (-float(s[i, e]), e))[:a["top"]]
        for e in chosen:
            f[i] += s[i, e] / sum(s[i, k] for k in chosen) * glu(r[i:i + 1], f"l0.x.e{e}.")[0]
    h = h + n(f, "l0.n3")
    # two maps over all earlier positions, on the stream itself
    m = dict(heads=a["att_heads"], kv_heads=a["att_kv"], dim=a["dim"], vdim=a["att_vdim"], scale=a["att_scale"], mask={"size": 10 ** 6}, diff=a["diff"])
    h = h + a["mult"] * n(P.attention(m, W, "l1.a.", h, a["eps"], dt), "l1.n0")
    h = h + a["mult"] * n(torch.relu(h @ w("l1.f.up").T) ** 2 @ w("l1.f.down").T, "l1.n1")
    return n(h, "final") @ w("head").T


@pytest.fixture
def toy6_registered():
    register_architecture("Toy6ForTests", Toy6Config, toy6_spec)
    yield
    unregister_architecture("Toy6ForTests")


def run_toy6(tmp_path, device):
    d = write_random_model(Toy6Config("Toy6ForTests"), 71, str(tmp_path / "toy6"), matrix_std="fan_in")
    kw = dict(device="cpu", ops=ref_ops) if device == "cpu" else {}
    runner = load_runner(d, "float32", max_tokens=128, max_requests=3, page_size=8, **kw)
    f = SafetensorsFile(str(tmp_path / "toy6" / "model.safetensors"))
    W = {name: f.read(name) for name in f.names()}
    g = random.Random(8)
    reqs = {k: [g.randrange(T6["vocab"]) for _ in range(n)] for k, n in (("x", 33), ("y", 12), ("z", 1))}
    for k, toks in reqs.items():
        want = toy6_plain(W, toks)
        for tag, cuts in (("w", [len(toks)]), ("p", [2, 5, 1, 3] + [1] * (len(toks) - 11) if len(toks) > 11 else [1] * len(toks))):
            runner.add_request(k + tag)
            got, at = [], 0
            for n_ in cuts:
                got.append(runner.step([(k + tag, toks[at:at + n_], list(range(n_)))]).double().cpu())
                at += n_
            runner.end_request(k + tag)
            err = (torch.cat(got) - want).abs().max() / want.abs().max()
            assert err < 5e-5, (k, tag, float(err))


def test_sixth_toy_architecture_on_the_cpu_stand_ins(toy6_registered, tmp_path):
    run_toy6(tmp_path, "cpu")


@pytest.mark.gpu
def test_sixth_toy_architecture_on_the_gpu(toy6_registered, tmp_path):
    run_toy6(tmp_path, "cuda")
