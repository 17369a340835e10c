"""Small random Vodavik configurations shared by the tests."""
import torch

from oracle import vodavik as vo


def attention(heads, kv_heads, dim, vdim, ff=None, scale=None, coef=0.4, every=16, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
         "scale": dim ** -0.5 if scale is None else scale, "q_temp": {"coef": coef, "every": every}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mlstm(heads, dim, vdim, cap=9.0, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5, alpha=1.7, logit_scale=0.5):
    return {"architecture": "Vodavik", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "postln_alpha": alpha, "logit_scale": logit_scale}


# name -> configuration; together: grouped, shared and plain heads, sizes at and off the padded sizes, all
# orders, feed-forwards on both kinds of layer and on neither, constants that are 1
CONFIGS = {
    "mixed": config(200, 331, [mlstm(3, 40, 56), attention(6, 2, 40, 72, ff=300), attention(6, 2, 40, 72, kv_from=1),
                               mlstm(2, 72, 40, ff=136)]),
    "plain_heads": config(128, 256, [attention(4, 4, 64, 64, ff=256, every=1), mlstm(2, 64, 64, cap=1.0)], alpha=1.0,
                          logit_scale=1.0),
    "wide_group": config(320, 100, [attention(10, 2, 128, 128, ff=130, every=7), attention(10, 2, 128, 128, ff=64, kv_from=0),
                                    mlstm(3, 128, 128)], eps=1e-4),
    "single_head": config(96, 65, [attention(1, 1, 24, 136, coef=1.0, every=3), mlstm(1, 33, 17, ff=48)]),
    "unequal": config(136, 500, [attention(8, 1, 100, 30, ff=72), mlstm(2, 20, 130), attention(3, 3, 16, 200)]),
}
BIG_HEADS = config(160, 77, [attention(3, 1, 200, 256, ff=100), mlstm(1, 256, 150), mlstm(2, 130, 256), mlstm(1, 250, 40)])


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def rel_error(got, want):
    """Largest over rows of the rms difference of the centred logits over the rms of all logits."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    c = want - want.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / c.pow(2).mean().sqrt().clamp_min(1e-12))


def oracle_logits(cfg, w, toks, dtype=torch.float64):
    return vo.Sequence(cfg, w, dtype).step(toks)
