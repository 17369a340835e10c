"""Small random Logesun configurations shared by the tests."""
from oracle import logesun as lo

import torch

from vodavik_util import rel_error, tokens  # noqa: F401  (shared by the test files)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=2.0, shared=None, shared_limit=1.5):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, mlp=None, base=10000.0, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def config(width, vocab, layers, loop=None, eps=1e-5):
    c = {"architecture": "Logesun", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# name -> configuration; together: every order of feed-forwards and none, sizes at and off the padded ones, one and many
# heads, windows of one token and beyond the sequence, one and several experts per token, with and without a shared
# one, loops over some, all and none of the layers, several passes
CONFIGS = {
    "mixed": config(200, 331, [latent(5, 40, 24, 56, 72, 48, 50, dense(300)),
                               latent(3, 24, 16, 40, 56, 72, 33, moe(7, 3, 40, shared=72)),
                               latent(4, 48, 8, 24, 100, 40, 130)], loop=(1, 3, 3)),
    "no_loop": config(128, 256, [latent(4, 64, 64, 64, 128, 128, 128, moe(9, 2, 64, limit=0.7)),
                                 latent(4, 64, 64, 64, 128, 128, 64, dense(256))], eps=1e-4),
    "many_heads": config(320, 100, [latent(20, 32, 32, 32, 96, 200, 90, moe(33, 4, 48, shared=200), base=500.0),
                                    latent(40, 16, 48, 72, 160, 130, 200, dense(130))], loop=(0, 2, 2)),
    "single_head": config(96, 65, [latent(1, 24, 2, 120, 17, 33, 1, dense(48)), latent(1, 72, 6, 9, 33, 17, 4000, moe(2, 2, 5, shared=3))],
                          loop=(1, 2, 1)),
    "wide_latent": config(160, 77, [latent(6, 128, 64, 128, 300, 512, 140, moe(5, 1, 136, shared=40)), latent(34, 30, 20, 30, 64, 400, 70)],
                          loop=(0, 1, 2)),
    "head_blocks": config(136, 90, [latent(70, 20, 12, 16, 48, 250, 60, dense(72)), latent(37, 16, 64, 20, 40, 384, 45, dense(40))]),
}
# sizes the tensor-core attention kernels leave to the plain ones: heads above 128, rotated parts above 64, latents above 512
BIG = config(144, 81, [latent(3, 150, 32, 140, 80, 64, 40, dense(100)), latent(2, 40, 100, 40, 80, 96, 64),
                       latent(2, 40, 16, 200, 80, 600, 50, moe(4, 2, 24))])


def oracle_logits(cfg, w, toks, dtype=torch.float64):
    return lo.Sequence(cfg, w, dtype).step(toks)
