"""The parts and options that came with the Pirozen design are parts like any other: a seventh toy architecture, defined in this
file, puts a state-space mixer beside a dense tanh-GELU feed-forward in the parallel block, with a term from a table's row; puts
attention with a bias on every projection, pairs (2i, 2i + 1) turned and frequencies stretched by wavelength, in front of experts
with sigmoid scores, a correction, groups and identities whose weights scale the inputs, into the block with a norm before and
after each sublayer; and merges the stream with the embedding's output between the two, and once more behind them in front of the
first layer's second run.  Registered, written with random weights, stepped in portions and single tokens, and compared with
plain formulas; nothing under the package changes."""
import math
import random
from dataclasses import dataclass

import pytest
import torch

import plain_pirozen as P
import plain_sogenex as S
import ref_ops
from zig_ai_b200.config import ModelConfig, register_architecture, unregister_architecture
from zig_ai_b200.engine.runner import load_runner
from zig_ai_b200.parts import LayerCall, LayerSpec, ModelSpec, PartSpec
from zig_ai_b200.weights import write_random_model
from zig_ai_b200.weights.safetensors_io import SafetensorsFile

T7 = dict(hidden=40, vocab=83, eps=1e-5, side=6, columns=9, at=3, scale=30.0, heads=4, vdim=6, state=7, groups=2, taps=3, parts=2, ff=36,
          att_heads=4, att_kv=2, dim=10, att_vdim=7, dims=8, base=60.0, att_scale=0.4, window=12, experts=3, identities=3, top=2,
          count=3, keep=2, factor=1.4, expert_ff=20)
WAVES = dict(kind="wavelength", factor=4.0, low=1.0, high=4.0, original=40)
SSM = {"in": "s.in", "conv": "s.conv", "dt_bias": "s.dt", "a_log": "s.a", "d": "s.d", "norm": "s.norm", "o": "s.o"}
ATT = {"q": "a.q", "k": "a.k", "v": "a.v", "o": "a.o", "g": "a.g", "q_bias": "a.qb", "k_bias": "a.kb", "v_bias": "a.vb", "o_bias": "a.ob",
       "q_norm": "a.qn", "k_norm": "a.kn"}
EXPERTS = {"router": "x.router", "correction": "x.c", "gate": "x.e{e}.gate", "up": "x.e{e}.up", "down": "x.e{e}.down"}


@dataclass
class Toy7Config(ModelConfig):
    @classmethod
    def from_dict(cls, d):
        return cls("Toy7ForTests")

    def to_dict(self):
        return {"architectures": ["Toy7ForTests"]}


def toy7_spec(cfg):
    a, W = T7, T7["hidden"]
    norm = lambda name: PartSpec("rmsnorm", dict(size=W, eps=a["eps"], weight=name))
    ssm = PartSpec("mamba2", dict(hidden=W, heads=a["heads"], vdim=a["vdim"], state=a["state"], groups=a["groups"], taps=a["taps"],
                                  norm_parts=a["parts"], eps=a["eps"], conv_bias=False, names=SSM))
    dense = PartSpec("swiglu", dict(hidden=W, ff_dim=a["ff"], activation="gelu_tanh", names={"gate": "f.gate", "up": "f.up", "down": "f.down"}))
    side = PartSpec("side_rows", dict(hidden=W, dim=a["side"], at=a["at"], eps=a["eps"], table="rows", names={"gate": "t.gate", "proj": "t.proj", "norm": "t.norm"}))
    att = PartSpec("attention", dict(
        hidden=W, heads=a["att_heads"], kv_heads=a["att_kv"], head_dim=a["dim"], value_dim=a["att_vdim"], qk_norm=True, eps=a["eps"],
        position=PartSpec("rotary_interleaved", dict(head_dim=a["dim"], theta=a["base"], rotary_dim=a["dims"], scaling=WAVES)), window=a["window"],
        scale=a["att_scale"], bias=True, out_bias=True, gate="head", names=ATT))
    experts = PartSpec("routed_experts", dict(
        hidden=W, ff_dim=a["expert_ff"], experts=a["experts"], top=a["top"], weight_on="input", score="sigmoid", correction=True,
        groups={"count": a["count"], "keep": a["keep"]}, identities=a["identities"], weight_scale=a["factor"], names=EXPERTS))
    layers = [
        LayerSpec("l0.", PartSpec("parallel_residual", dict(mixer=ssm, mixer_norm=norm("n0"), feed_forward=dense, ff_norm=norm("n1"), token_input=side))),
        LayerSpec("l1.", PartSpec("sandwich_residual", dict(mixer=att, mixer_norm=norm("n0"), mixer_post_norm=norm("n1"), feed_forward=experts,
                                                            ff_norm=norm("n2"), ff_post_norm=norm("n3")))),
        LayerSpec("m.", PartSpec("stream_merge", dict(hidden=W, weight="w"))),
    ]
    return ModelSpec("Toy7ForTests", W, a["vocab"], 256, PartSpec("embedding", dict(weight="emb", scale=a["scale"])), layers,
                     [LayerCall(0), LayerCall(2), LayerCall(1), LayerCall(2), LayerCall(0)], norm("final"),
                     PartSpec("linear_head", dict(weight="head", tied=False)), tables={"rows": PartSpec("token_table", dict(weight="rows", columns=a["columns"]))})


def toy7_plain(W, tokens):
    a, dt = T7, torch.float64
    w = lambda name: W[name].to(dt)
    n = lambda x, name: P.rms(x, a["eps"]) * w(name)
    T, ids = len(tokens), torch.tensor(tokens)
    x0 = w("emb")[ids] * a["scale"]

    def first(h):
        H, V, N, G = a["heads"], a["vdim"], a["state"], a["groups"]
        I, ch = H * V, H * V + 2 * G * N
        y = n(h, "l0.n0") @ w("l0.s.in").T
        u = S.convolve(y[:, I:I + ch], w("l0.s.conv"), torch.zeros(ch, dtype=dt))
        d = torch.nn.functional.softplus(y[:, I + ch:] + w("l0.s.dt"))
        o = S.state_space(u[:, :I].reshape(T, H, V), u[:, I:I + G * N].reshape(T, G, N), u[:, I + G * N:].reshape(T, G, N), d, w("l0.s.a"), w("l0.s.d"))
        m = S.gated_norm(o.reshape(T, I), y[:, :I], a["parts"], w("l0.s.norm"), a["eps"]) @ w("l0.s.o").T
        r = n(h, "l0.n1")
        h = h + (m + (P.gelu_tanh(r @ w("l0.f.gate").T) * (r @ w("l0.f.up").T)) @ w("l0.f.down").T)
        g = P.gelu_tanh(h @ w("l0.t.gate").T) * w("rows")[ids][:, a["at"]:a["at"] + a["side"]]
        return h + n(g @ w("l0.t.proj").T, "l0.t.norm")

    def attention(r):
        H, G, D, V, dims = a["att_heads"], a["att_kv"], a["dim"], a["att_vdim"], a["dims"]
        q, k, v = (r @ w(f"l1.a.{c}").T + w(f"l1.a.{c}b") for c in "qkv")
        q, k = n_head(q.reshape(T, H, D), "l1.a.qn"), n_head(k.reshape(T, G, D), "l1.a.kn")
        freqs = []
        for i in range(dims // 2):
            f = a["base"] ** (-2.0 * i / dims)
            wave = 2 * math.pi / f
            s = (WAVES["original"] / wave - WAVES["low"]) / (WAVES["high"] - WAVES["low"])
            freqs.append(f if s > 1 else f / WAVES["factor"] if s < 0 else (1 - s) * f / WAVES["factor"] + s * f)
        t = torch.arange(T, dtype=dt)[:, None]
        for x in (q, k):
            for i, f in enumerate(freqs):
                u, z = x[..., 2 * i].clone(), x[..., 2 * i + 1].clone()
                x[..., 2 * i], x[..., 2 * i + 1] = u * torch.cos(t * f) - z * torch.sin(t * f), z * torch.cos(t * f) + u * torch.sin(t * f)
        k, v = k.permute(1, 0, 2).repeat_interleave(H // G, dim=0), v.reshape(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, dim=0)
        o = P.windowed_softmax(q.permute(1, 0, 2), k, v, a["att_scale"], a["window"]).permute(1, 0, 2) * torch.sigmoid(r @ w("l1.a.g").T)[:, :, None]
        return o.reshape(T, H * V) @ w("l1.a.o").T + w("l1.a.ob")

    def n_head(x, name):
        return P.rms(x, a["eps"]) * w(name)

    def second(h):
        h = h + n(attention(n(h, "l1.n0")), "l1.n1")
        r = n(h, "l1.n2")
        s, f = torch.sigmoid(r @ w("l1.x.router").T), torch.zeros_like(r)
        router = {"top": a["top"], "groups": {"count": a["count"], "keep": a["keep"]}}
        for i in range(T):
            for e in P.choose(s[i].tolist(), w("l1.x.c").tolist(), router):
                x = (s[i, e] * a["factor"] * r[i])[None]
                f[i] += P.unit(W, f"l1.x.e{e}.", x, dt)[0] if e < a["experts"] else x[0]
        return h + n(f, "l1.n3")

    merge = lambda h: torch.cat([h, x0], dim=-1) @ w("m.w").T
    return n(first(merge(second(merge(first(x0))))), "final") @ w("head").T


@pytest.fixture
def toy7_registered():
    register_architecture("Toy7ForTests", Toy7Config, toy7_spec)
    yield
    unregister_architecture("Toy7ForTests")


def run_toy7(tmp_path, device):
    d = write_random_model(Toy7Config("Toy7ForTests"), 71, str(tmp_path / "toy7"), matrix_std="fan_in")
    kw = dict(device="cpu", ops=ref_ops) if device == "cpu" else {}
    runner = load_runner(d, "float32", max_tokens=128, max_requests=3, page_size=8, **kw)
    f = SafetensorsFile(str(tmp_path / "toy7" / "model.safetensors"))
    W = {name: f.read(name) for name in f.names()}
    g = random.Random(8)
    reqs = {k: [g.randrange(T7["vocab"]) for _ in range(n)] for k, n in (("x", 33), ("y", 12), ("z", 1))}
    for k, toks in reqs.items():
        want = toy7_plain(W, toks)
        for tag, cuts in (("w", [len(toks)]), ("p", [2, 5, 1, 3] + [1] * (len(toks) - 11) if len(toks) > 11 else [1] * len(toks))):
            runner.add_request(k + tag)
            got, at = [], 0
            for n_ in cuts:
                got.append(runner.step([(k + tag, toks[at:at + n_], list(range(n_)))]).double().cpu())
                at += n_
            runner.end_request(k + tag)
            err = (torch.cat(got) - want).abs().max() / want.abs().max()
            assert err < 5e-5, (k, tag, float(err))


def test_seventh_toy_architecture_on_the_cpu_stand_ins(toy7_registered, tmp_path):
    run_toy7(tmp_path, "cpu")


@pytest.mark.gpu
def test_seventh_toy_architecture_on_the_gpu(toy7_registered, tmp_path):
    run_toy7(tmp_path, "cuda")
