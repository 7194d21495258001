"""Small Kerudra configurations for the tests.  They differ from one another in every size, in the number of streams, in
the order and kinds of the layers, in which layers have a feed-forward, in the loop, in windows, rotated lanes, ranks
and in the constants."""
import torch

import plain_kerudra as plain
from tokenizer_b200 import write_random_model
from tokenizer_b200.config import KerudraConfig


def dense(ff):
    return {"kind": "dense", "ff": ff}


def attention(heads, kv_heads, dim, scale, rot=None, mlp=None):
    """rot = (base, dims)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, size=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def memory(heads, dim, vdim, gate_cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def config(layers, vocab, width, eps, streams, mult=None, embedding=None, logit_scale=None, loop=None):
    raw = {"architecture": "Kerudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if mult is not None:
        raw["residual_mult"] = mult
    if embedding is not None:
        raw["embedding"] = {"scale": embedding}
    if logit_scale is not None:
        raw["logit_scale"] = logit_scale
    if loop is not None:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return KerudraConfig.from_dict(raw)


# name -> (configuration, seed, page size)
def tiny_a():
    """Three streams; a window of 20 keys on pages of 8; half of the attention's lanes rotated; one key head for
    every three query heads; the middle two layers run three times."""
    return config([memory(3, 24, 16, 9.0, mlp=dense(72)),
                   latent(5, 16, 8, 24, 40, 0.22, 5000.0, size=20, mlp=dense(104)),
                   attention(6, 2, 32, 0.19, rot=(8000.0, 16), mlp=dense(56)),
                   latent(2, 40, 12, 8, 20, 0.14, 300.0, size=33)],
                  vocab=301, width=96, eps=2e-5, streams=3, mult=0.6, embedding=9.0, logit_scale=0.3, loop=(1, 3, 3)), 3, 8


def tiny_b():
    """Sizes the tensor-core kernels take (cache rows of 64 and 128 lanes, matrices of 128 x 128 and 64 x 96); a window
    of 130; four streams; the first three layers looped twice."""
    return config([latent(4, 48, 32, 64, 96, 0.11, 20000.0, size=130, mlp=dense(384)),
                   memory(2, 128, 128, 2.0, mlp=dense(192)),
                   attention(4, 2, 64, 0.07, rot=(90000.0, 64), mlp=dense(256)),
                   memory(3, 64, 96, 1.2),
                   attention(2, 1, 128, 0.05, rot=(700.0, 64), mlp=dense(128)),
                   latent(2, 32, 16, 32, 48, 0.15, 2000.0, size=64, mlp=dense(64))],
                  vocab=1000, width=128, eps=1e-2, streams=4, mult=0.5, embedding=6.0, logit_scale=0.125, loop=(0, 3, 2)), 4, 16


def tiny_c():
    """Sizes that no vector load fits (a width of 50, a vocabulary of 77, heads of 10, 6 and 7 lanes), one stream, a window
    of one key, no rotation, one head, no constants, a loop of a single pass, pages of 32."""
    return config([latent(3, 10, 2, 7, 11, 0.3, 100.0, size=1, mlp=dense(37)),
                   memory(1, 6, 10, 3.0, mlp=dense(14)),
                   attention(5, 1, 6, 0.5, mlp=dense(9)),
                   memory(3, 7, 5, 20.0)],
                  vocab=77, width=50, eps=4e-3, streams=1, loop=(1, 2, 1)), 5, 32


def tiny_d():
    """Five streams; the loop in the middle of the layers and over all kinds; a window wider than any prompt and an open
    one; heads of 136 and 256 lanes in the memory; cache rows wider than the tensor-core kernels take; no feed-forward at
    the end."""
    return config([attention(4, 4, 16, 0.25, rot=(50.0, 4), mlp=dense(48)),
                   memory(2, 136, 8, 12.0, mlp=dense(40)),
                   latent(3, 24, 10, 20, 150, 0.2, 1000.0, size=4096, mlp=dense(64)),
                   memory(1, 256, 20, 6.0),
                   latent(2, 8, 4, 12, 24, 0.3, 10.0)],
                  vocab=120, width=64, eps=1e-4, streams=5, mult=0.9, embedding=3.0, logit_scale=0.7, loop=(1, 4, 2)), 6, 16


TINY = {"a": tiny_a, "b": tiny_b, "c": tiny_c, "d": tiny_d}
# logits of a size against which a tolerance means something, attention that is sharp enough for a wrong key to show,
# gates that open and close, streams that stay apart without running away
SHARPEN = {r"^embed$": 30.0, r"\.mix\.q$": 3.5, r"\.mix\.k$": 3.5, r"\.mix\.(dkv|uk)$": 3.5, r"\.mix\.(v|uv|g|i|f)$": 5.0,
           r"\.mix\.(q|k)\.b$": 10.0, r"\.mix\.o$": 5.0, r"\.(up|down)$": 4.0}


def make_folder(tmp_path_factory, name, scale=SHARPEN):
    cfg, seed, page = TINY[name]()
    folder = str(tmp_path_factory.mktemp(f"kerudra_{name}"))
    write_random_model(folder, cfg, seed, scale=scale)
    return folder, cfg, page


def reference_logits(folder, requests):
    """{request: array [len, vocab]} from the plain implementation (float64, kept as float32)."""
    cfg, weights = plain.load_folder(folder)
    return {name: plain.forward(cfg, weights, ids).to(torch.float32).numpy() for name, ids in requests.items()}
