"""Small Merusun configurations for the tests.  Between them every size differs, and sizes that are often equal are not
(key and value size, heads of the mixers, the windows of a layer and of the layers that read its keys and values); every
kind of layer comes with and without a feed-forward, routing with and without groups, with and without a shared expert."""
import copy


def memory(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale, base, mlp=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, window, scale, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def moe(ff, experts, top, count=1, keep=1, scale=1.0, shared=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if count > 1:
        r["groups"] = {"count": count, "keep": keep}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, scale, layers):
    return {"architecture": "Merusun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": layers}


def every_expert(config):
    """The same configuration with every expert chosen: in bfloat16 a row's rounding can swap two experts (or groups) with
    close scores, which is no fault and moves the row by far more than rounding does."""
    c = copy.deepcopy(config)
    for L in c["layers"]:
        if L["mlp"]:
            r = L["mlp"]["router"]
            r["top"] = r["experts"]
            if "groups" in r:
                r["groups"]["keep"] = r["groups"]["count"]
    return c


# attention whose keys and values two later layers read, one behind a longer window and one behind a shorter one; a latent
# narrow enough for the kernels of the latent space; a value of 24 against a key of 20 in the matrix memory
MERUSUN_A = model(211, 64, 1e-5, 5.0, [
    attention(6, 3, 24, 40, 21, 0.25, mlp=moe(24, 10, 3, count=5, keep=2, scale=2.5, shared=40)),
    memory(3, 20, 24, 4.0, mlp=moe(16, 6, 2, scale=0.7)),
    attention(6, 3, 24, 40, 37, 0.3, kv_from=0),
    latent(5, 16, 8, 12, 32, 19, 0.2, 700.0, mlp=moe(8, 4, 1, count=2, keep=1, shared=24)),
    attention(6, 3, 24, 40, 9, 0.4, kv_from=0, mlp=moe(32, 3, 3, scale=1.3)),
])
# a latent wider than the tensor-core kernels take as a key (per-head keys in a prompt), two latent layers that differ, a
# window of one, one memory head with long keys, a feed-forward of one expert
MERUSUN_B = model(320, 96, 1e-6, 0.5, [
    latent(4, 40, 24, 56, 128, 33, 0.13, 1e6, mlp=moe(40, 12, 4, count=3, keep=2, scale=1.7, shared=16)),
    memory(1, 136, 40, 15.0),
    latent(2, 64, 2, 32, 62, 70, 0.12, 50.0, mlp=moe(48, 1, 1, scale=0.5)),
    attention(4, 1, 64, 16, 1, 0.2, mlp=moe(24, 8, 2, count=8, keep=3)),
    memory(4, 16, 64, 0.75, mlp=moe(56, 16, 5, count=2, keep=2, shared=72)),
])
# a width that is no multiple of 8 (no tensor-core product), an odd vocabulary, head sizes that are no multiple of 4, a
# window wider than any test sequence, a memory whose values are one number each; an eps so large that it counts
MERUSUN_C = model(97, 42, 0.2, 2.0, [
    memory(2, 6, 10, 30.0, mlp=moe(10, 5, 2, shared=14)),
    attention(3, 1, 20, 12, 400, 0.3),
    latent(3, 10, 6, 14, 18, 11, 0.3, 99.0, mlp=moe(7, 6, 2, count=3, keep=1, scale=3.0)),
    memory(5, 3, 1, 2.0),
    attention(3, 1, 20, 12, 16, 0.2, kv_from=1, mlp=moe(12, 9, 4, count=3, keep=2, scale=1.1)),
])
CONFIGS = {"A": MERUSUN_A, "B": MERUSUN_B, "C": MERUSUN_C}
