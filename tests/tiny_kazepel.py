"""Small Kazepel configurations for the tests.  They differ from one another in every size, in the order and
kinds of the layers, in which layers have a feed-forward, in the loop, in windows, kept first tokens, rotated
lanes, the rotation's scaling, the router's groups and identity experts, the bottlenecks' ranks, and in the
constants."""
import torch

import plain_kazepel as plain
from tokenizer_b200 import write_random_model
from tokenizer_b200.config import KazepelConfig


def attention(heads, kv_heads, dim, vdim, scale, size=None, keep=None, rot=None, mlp=None):
    """rot = (base, dims, (factor, original, fast, slow) or None)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts, top, ff, limit, groups=None, identity=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if identity is not None:
        router["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}


def config(layers, vocab, width, eps, logit_scale=None, loop=None):
    raw = {"architecture": "Kazepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if logit_scale is not None:
        raw["logit_scale"] = logit_scale
    if loop is not None:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return KazepelConfig.from_dict(raw)


# name -> (configuration, seed, page size, the bottlenecks' ranks by tensor name)
def tiny_a():
    """A window of 20 keys with the first five kept on pages of 8, keys narrower than values; two value heads a
    key head in the delta rule; identity experts in groups; the middle two layers run three times."""
    return config([delta(4, 2, 24, 16, 3, mlp=moe(5, 2, 40, 1.5, groups=(2, 1), identity=1)),
                   attention(6, 3, 16, 32, 0.3, size=20, keep=5, rot=(5000.0, 8, (3.0, 256, 16.0, 1.5)),
                             mlp=moe(6, 3, 24, 0.7, groups=(3, 2), identity=3)),
                   delta(2, 2, 40, 12, 4),
                   attention(4, 1, 48, 48, 0.15, size=33, keep=11, rot=(300.0, 48, None))],
                  vocab=301, width=96, eps=1e-5, logit_scale=0.3, loop=(1, 3, 3)), 3, 8, \
        {"l0.mix.a1": 9, "l0.mix.g1": 20, "l2.mix.a1": 16, "l2.mix.g1": 5}


def tiny_b():
    """Sizes the tensor-core kernels take (cache rows of 64 and 128 lanes, matrices of 128 x 128 and 64 x 64): a window
    of 130 with 20 first tokens kept, more than one page; a window with none kept; the first three layers looped
    twice; every expert counts in one group."""
    return config([attention(4, 2, 64, 64, 0.125, size=130, keep=20, rot=(9000.0, 64, (8.0, 512, 20.0, 2.0)), mlp=moe(4, 2, 64, 3.0)),
                   delta(2, 2, 128, 128, 4, mlp=moe(6, 2, 32, 2.5, groups=(4, 2), identity=2)),
                   delta(3, 1, 64, 64, 2),
                   attention(2, 2, 128, 96, 0.09, size=70, rot=(70000.0, 32, (2.0, 64, 8.0, 0.5)), mlp=moe(3, 2, 128, 1.0, identity=1))],
                  vocab=1000, width=128, eps=1e-6, logit_scale=0.125, loop=(0, 3, 2)), 4, 16, {"l1.mix.a1": 32, "l1.mix.g1": 48}


def tiny_c():
    """Sizes that no vector load fits (a width of 50, a vocabulary of 77, heads of 10 and 6 lanes), a window of one
    key with one first token kept, no rotation, a convolution of one tap, one head, no constant on the logits,
    every expert chosen, a loop of a single pass, pages of 32."""
    return config([attention(3, 3, 10, 20, 0.3, size=1, keep=1, rot=(100.0, 2, (4.0, 32, 4.0, 1.0)), mlp=moe(3, 3, 14, 0.5)),
                   delta(1, 1, 6, 10, 1, mlp=moe(2, 1, 8, 4.0, identity=1)),
                   attention(5, 1, 6, 6, 0.5, mlp=moe(5, 2, 8, 1.0, groups=(5, 3))),
                   delta(3, 3, 10, 7, 5)],
                  vocab=77, width=50, eps=3e-6, loop=(1, 2, 1)), 5, 32, {"l1.mix.a1": 1, "l1.mix.g1": 3, "l3.mix.a1": 7, "l3.mix.g1": 10}


def tiny_d():
    """The loop in the middle of the layers and over all kinds; the kept tokens fill pages exactly; a window wider
    than any prompt; heads of 136 and 260 lanes in the delta rule; more identity experts than experts; no feed-forward
    at the end."""
    return config([delta(2, 1, 136, 8, 4, mlp=moe(2, 2, 24, 2.0, groups=(4, 2), identity=6)),
                   attention(2, 1, 48, 16, 0.14, size=50, keep=16, rot=(1000.0, 16, (16.0, 32, 8.0, 2.0)), mlp=moe(8, 3, 16, 1.2, groups=(2, 1))),
                   delta(2, 2, 260, 20, 2, mlp=moe(4, 2, 16, 0.9, identity=2)),
                   attention(6, 3, 16, 32, 0.25, size=4096, keep=3, rot=(50.0, 16, (1.5, 128, 3.0, 1.0)))],
                  vocab=120, width=64, eps=2e-6, logit_scale=0.7, loop=(1, 4, 2)), 6, 16, {"l0.mix.a1": 8, "l0.mix.g1": 8}


TINY = {"a": tiny_a, "b": tiny_b, "c": tiny_c, "d": tiny_d}
# logits of a size against which a tolerance means something, a stream large enough for the norms to bend, router
# logits that differ from token to token, attention that is sharp enough for a wrong key to show
SHARPEN = {r"^embed$": 40.0, r"^loop\.in$": 4.0, r"^loop\.step$": 20.0, r"\.router$": 10.0, r"\.mix\.(q|k)$": 5.0,
           r"\.mix\.(v|b|a1|g1)$": 5.0, r"\.mix\.(a2|g2)$": 4.0, r"\.mix\.o$": 5.0, r"\.(gate|up|down)$": 4.0,
           r"norm[12]\.b$": 5.0}


def make_folder(tmp_path_factory, name, scale=SHARPEN):
    cfg, seed, page, sizes = TINY[name]()
    folder = str(tmp_path_factory.mktemp(f"kazepel_{name}"))
    write_random_model(folder, cfg, seed, scale=scale, sizes=sizes)
    return folder, cfg, page


def reference_logits(folder, requests):
    """{request: array [len, vocab]} from the plain implementation (float64, kept as float32)."""
    cfg, weights = plain.load_folder(folder)
    return {name: plain.forward(cfg, weights, ids).to(torch.float32).numpy() for name, ids in requests.items()}
