"""Small configurations of the Sogenex design for the tests.  Between them they differ in every size and option: layer order
and count, each mixer in front of experts and of none, layers that run on an earlier layer's tensors (one and several times,
also on another such layer's), one group of B and C for many heads and as many as there are heads, one norm part and several,
one tap and several, states smaller and larger than a head's values, one key/value head for many query heads and as many as
there are, maps' sizes whose double is smaller and larger than the values' size, windows of one position, smaller and larger
than a page, differences' constants of zero and others, one expert a token, several and all, experts with and without a unit
for every token, logit factors and bounds, widths that are no multiple of four."""


def ssm(heads, vdim, state, groups, conv, norm_groups, mlp=None, of=None):
    m = {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}
    return layer("mamba2", m, mlp, of)


def diff(heads, kv_heads, dim, vdim, scale, size, const, mlp=None, of=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}, "diff": const}
    return layer("attention", m, mlp, of)


def layer(kind, mixer, mlp, of):
    out = {"type": kind, "mixer": mixer, "mlp": mlp}
    if of is not None:
        out["weights_of"] = of
    return out


def moe(ff, experts, top, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": None if shared is None else {"ff": shared}}


def config(vocab, width, eps, layers, scale=1.0, cap=20.0):
    return {"architecture": "Sogenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": cap,
            "layers": layers}


A_SSM = lambda of=None: ssm(4, 6, 10, 2, 3, 3, moe(20, 5, 2, shared=28), of)
S_A = config(131, 48, 1e-5, [
    diff(4, 2, 6, 10, 0.4, 11, 0.3, moe(24, 4, 4)),
    A_SSM(),
    ssm(3, 12, 8, 1, 4, 1),
    A_SSM(of=1),
    diff(3, 1, 10, 8, 0.3, 5, 0.0),
    A_SSM(of=3),
], scale=1.5, cap=12.0)

B_DIFF = lambda of=None: diff(6, 3, 8, 20, 0.35, 40, 0.55, moe(40, 7, 3), of)
S_B = config(257, 66, 1e-6, [
    ssm(6, 10, 20, 3, 2, 5, moe(32, 3, 1, shared=16)),
    B_DIFF(),
    ssm(2, 30, 12, 2, 1, 2, moe(16, 2, 2, shared=40)),
    B_DIFF(of=1),
    diff(2, 2, 12, 24, 0.3, 1, 0.8, moe(12, 9, 4, shared=20)),
], scale=0.7, cap=50.0)

# one layer of each kind, alone: a fault shows in the mechanism that has it
ONLY = {
    "state_space": config(97, 40, 1e-5, [ssm(4, 10, 14, 2, 4, 4)]),
    "state_space_one_group": config(97, 40, 1e-5, [ssm(5, 8, 6, 1, 2, 1)]),
    "state_space_no_history": config(97, 40, 1e-5, [ssm(2, 12, 20, 2, 1, 3)]),
    "two_maps": config(97, 40, 1e-5, [diff(4, 2, 8, 12, 0.4, 13, 0.4)]),
    "two_maps_wide_keys": config(97, 40, 1e-5, [diff(3, 3, 14, 10, 0.3, 20, 0.7)]),
    "experts": config(97, 40, 1e-5, [ssm(2, 8, 6, 1, 2, 1, moe(24, 6, 2, shared=12))]),
    "experts_one_of_many": config(97, 40, 1e-5, [ssm(2, 8, 6, 1, 2, 1, moe(12, 9, 1))]),
    "experts_all": config(97, 40, 1e-5, [diff(2, 1, 8, 16, 0.3, 9, 0.2, moe(16, 3, 3, shared=20))], scale=3.0, cap=4.0),
    "tensors_used_again": config(97, 40, 1e-5, [ssm(2, 10, 8, 1, 4, 2), diff(2, 1, 6, 12, 0.4, 7, 0.3), ssm(2, 10, 8, 1, 4, 2, of=0),
                                               diff(2, 1, 6, 12, 0.4, 7, 0.3, of=1), ssm(2, 10, 8, 1, 4, 2, of=2)]),
    # attention made sharp by its scale: nearly all weight on one key a map, so a key lost or seen too early shows
    "sharp_maps": config(97, 40, 1e-5, [diff(3, 1, 10, 14, 2.0, 13, 0.3)]),
}

# sizes that the tensor-core kernels and the few-rows product kernels take, for the whole-model GPU tests in bfloat16
C_SSM = lambda of=None: ssm(6, 64, 96, 3, 4, 3, moe(128, 8, 2, shared=192), of)
S_C = config(1000, 320, 1e-6, [
    C_SSM(),
    diff(4, 1, 32, 64, 0.18, 100, 0.5, moe(64, 4, 1)),
    ssm(10, 32, 128, 2, 3, 2, None),
    C_SSM(of=0),
    diff(2, 2, 64, 128, 0.125, 300, 0.35, moe(96, 6, 3, shared=64)),
], scale=1.2, cap=30.0)

ALL = {"A": (S_A, 31), "B": (S_B, 37), "C": (S_C, 41)}
PAGE_SIZE = {"A": 8, "B": 16, "C": 64}


def write_model(cfg, seed, model_dir):
    """A model folder with random tensors of sizes at which every mechanism counts: token rows as large as the position vectors,
    convolutions of size one (so that B, C and the states are, too), decays from nearly one to nearly none, difference weights
    away from their constant."""
    import os
    import torch
    from zig_ai_b200.config import config_from_dict
    from zig_ai_b200.weights import write_random_model
    from zig_ai_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
    write_random_model(config_from_dict(cfg), seed, model_dir, matrix_std="fan_in")
    path = os.path.join(model_dir, "model.safetensors")
    f = SafetensorsFile(path)
    tensors = {n: f.read(n).clone() for n in f.names()}
    for name, t in tensors.items():
        factor = 40.0 if name == "embed" else 8.0 if name.endswith(".mix.conv") else 4.0 if name[-4:-1] in (".lq", ".lk") else None
        if factor is not None:
            tensors[name] = (t.float() * factor).to(t.dtype)
        elif name.endswith(".A_log"):
            tensors[name] = torch.linspace(-4.0, 1.0, len(t)).to(t.dtype)
        elif name.endswith(".dt_bias"):
            tensors[name] = (t.float() * 5.0 - 1.0).to(t.dtype)
    write_safetensors(path, tensors)
    return model_dir
