"""Small configurations of the Pirozen design for the tests.  Between them they differ in every size and option: layer counts,
layers with experts and without a feed-forward, windows of one position, smaller and larger than a page, rotations of all, some and
no dimensions, with stretched frequencies and without, keys wider and narrower than values and equal, one key/value head for many
query heads and as many as there are, no groups of experts, one group, groups of one expert, groups that are all kept, no
identities, one, more than there are experts, one choice a token and all of them, weight factors of one and others, experts with
and without one more for every token, side rows or none, loops at the start, in the middle, at the end and over everything, of one
layer and of several, passed once and several times, no loop, widths that are no multiple of four."""


def att(heads, kv_heads, dim, vdim, scale, size, dims, base=10000.0, scaling=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
         "rot": {"base": base, "dims": dims, "scaling": scaling}}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def moe(ff, experts, identity, top, groups=None, scale=1.0, shared=None):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "identity": identity, "top": top, "scale": scale,
                       "groups": None if groups is None else {"count": groups[0], "keep": groups[1]}},
            "shared": None if shared is None else {"ff": shared}}


def config(vocab, width, eps, layers, side=None, loop=None):
    out = {"architecture": "Pirozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side is not None:
        out["token_side"] = {"dim": side}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


P_A = config(131, 48, 1e-5, [
    att(4, 2, 12, 8, 0.3, 11, 8, 500.0, yarn(4.0, 30, 6.0, 0.5), moe(20, 5, 3, 2, (4, 2), 1.7, shared=28)),
    att(6, 2, 8, 14, 0.4, 5, 8, 300.0, None, None),
    att(3, 1, 10, 10, 0.35, 30, 4, 2000.0, yarn(8.0, 64, 4.0, 0.3), moe(12, 3, 1, 3, (2, 2), 0.6)),
], side=5, loop=(1, 3, 3))

P_B = config(257, 66, 1e-6, [
    att(6, 3, 16, 24, 0.3, 40, 10, 10000.0, yarn(2.0, 128, 8.0, 1.0), moe(24, 2, 6, 3, (2, 1), 2.5, shared=16)),
    att(2, 2, 20, 12, 0.25, 7, 20, 100.0, yarn(16.0, 20, 3.0, 0.2), moe(16, 9, 0, 2, (3, 2), 1.0, shared=40)),
    att(8, 1, 8, 8, 0.4, 300, 0, 10000.0, None, moe(12, 4, 2, 1, None, 3.0)),
    att(5, 5, 12, 16, 0.3, 1, 2, 50.0, None, moe(8, 1, 7, 4, (8, 5), 0.8, shared=20)),
], side=12, loop=(0, 2, 2))

# one mechanism at a time: a fault shows in the mechanism that has it
L_ATT = lambda mlp=None: att(4, 2, 12, 8, 0.3, 13, 6, 200.0, yarn(4.0, 32, 4.0, 0.5), mlp)
ONLY = {
    "attention": config(97, 40, 1e-5, [L_ATT()]),
    "attention_wide_values": config(97, 40, 1e-5, [att(3, 3, 8, 18, 0.35, 20, 8, 77.0)]),
    "attention_no_rotation": config(97, 40, 1e-5, [att(4, 1, 10, 10, 0.35, 9, 0)]),
    # attention made sharp by its scale: nearly all weight on one key, so a key lost or seen too early shows
    "sharp_attention": config(97, 40, 1e-5, [att(3, 1, 10, 14, 2.0, 13, 10, 50.0, yarn(3.0, 50, 5.0, 0.4))]),
    "experts": config(97, 40, 1e-5, [L_ATT(moe(24, 6, 2, 3, (4, 2), 1.5, shared=12))]),
    "experts_one_of_many": config(97, 40, 1e-5, [L_ATT(moe(12, 9, 1, 1, (5, 1), 2.0))]),
    "experts_all": config(97, 40, 1e-5, [L_ATT(moe(16, 3, 2, 5, None, 1.0, shared=20))]),
    "experts_no_identity": config(97, 40, 1e-5, [L_ATT(moe(16, 8, 0, 2, (2, 1), 0.5))]),
    "mostly_identities": config(97, 40, 1e-5, [L_ATT(moe(16, 1, 11, 2, (6, 4), 1.2))]),
    "side_rows": config(97, 40, 1e-5, [L_ATT(), L_ATT()], side=7),
    "loop_over_all": config(97, 40, 1e-5, [L_ATT(), L_ATT(moe(12, 3, 1, 2))], loop=(0, 2, 2)),
    "loop_of_one_once": config(97, 40, 1e-5, [L_ATT(), L_ATT(), L_ATT()], loop=(1, 2, 1)),
    "loop_at_the_end": config(97, 40, 1e-5, [L_ATT(), L_ATT()], side=4, loop=(1, 2, 4)),
}

# sizes that the tensor-core kernels and the few-rows product kernels take, for the whole-model GPU tests in bfloat16
P_C = config(1000, 256, 1e-6, [
    att(8, 2, 64, 64, 0.125, 100, 32, 50000.0, yarn(8.0, 512, 16.0, 1.0), moe(128, 6, 2, 2, (4, 2), 2.0, shared=192)),
    att(4, 1, 96, 64, 0.1, 70, 96, 10000.0, yarn(4.0, 256, 32.0, 1.0), moe(64, 12, 4, 4, (2, 1), 1.5, shared=64)),
    att(6, 3, 32, 48, 0.18, 300, 16, 10000.0, None, moe(96, 4, 0, 1, None, 1.0)),
    att(4, 4, 128, 128, 0.09, 33, 64, 1000.0, yarn(2.0, 100, 8.0, 0.5), None),
], side=24, loop=(1, 3, 2))

ALL = {"A": (P_A, 31), "B": (P_B, 37), "C": (P_C, 41)}
PAGE_SIZE = {"A": 8, "B": 16, "C": 64}


def write_model(cfg, seed, model_dir):
    """A model folder with random tensors of sizes at which every mechanism counts: rows of the embedding and of the side table
    of size one, routers whose scores differ, corrections as large as the scores' differences (some negative), biases and gates
    away from zero."""
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
        factor = 50.0 if name in ("embed", "side.embed") else 5.0 if name[-2:] == ".b" else 3.0 if name.endswith(".mix.g") else None
        if name.endswith(".mlp.router"):
            factor = 20.0 * t.shape[1] ** -0.5
        if factor is not None:
            tensors[name] = (t.float() * factor).to(t.dtype)
    write_safetensors(path, tensors)
    return model_dir
