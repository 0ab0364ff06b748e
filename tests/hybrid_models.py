"""Small layer-listed configurations and weights of the tests (random, made here)."""
import json
import os

import torch

from megaqwen_b200.spec import read_hybrid_config
from megaqwen_b200.synthetic import random_hybrid_weights


def lightning(heads, dim, vdim, decay=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                           "decay": decay or [1.0 - 0.4 / 2 ** (1.5 * i) for i in range(heads)]}}


def latent(heads, dim, rot, vdim, rank, base=5000.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                  "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5}}


def config(layers, width=96, vocab=331, ff=160, loop=None, eps=1e-5, embed_scale=7.0, mult=0.4):
    """layers: mixers; a pair (mixer, ff) overrides ff, None for no feed-forward."""
    out = []
    for entry in layers:
        mixer, f = entry if isinstance(entry, tuple) else (entry, ff)
        out.append(dict(mixer, mlp=None if f is None else {"kind": "dense", "ff": f}))
    return {"architecture": "Satosun", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps},
            "residual_mult": mult, "layers": out, "loop": loop}


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


# Models that differ in everything config.json gives: sizes off the multiples of 16, 8 and 4, more than 16 heads, one
# head, layers without feed-forward, loops at the start, in the middle, of one pass and none.
MODELS = {
    "mixed": config([latent(5, 40, 12, 24, 56, scale=0.5), lightning(3, 24, 40), latent(5, 40, 12, 24, 56, scale=0.4), lightning(3, 24, 40)],
                    loop=loop(1, 3, 3)),
    "latent first, loop to the end": config([(latent(2, 64, 32, 64, 80), None), (lightning(4, 16, 16), 72)], width=128, loop=loop(0, 2, 2), eps=1e-3),
    "no loop, other layers": config([lightning(7, 48, 8), latent(17, 8, 2, 8, 24, base=90.0), (lightning(1, 80, 112), 40), latent(1, 112, 64, 128, 256)],
                                    width=72, vocab=509, mult=1.0, embed_scale=1.0),
    "one pass": config([latent(3, 128, 16, 72, 32), lightning(2, 136, 24)], width=64, vocab=1000, loop=loop(0, 1, 1), mult=0.2),
    "wide feed-forward": config([(lightning(2, 16, 16), 8160), (latent(1, 16, 4, 16, 24), 12000), (lightning(2, 16, 16), 9000)], width=32, vocab=130),
    "large heads": config([latent(2, 136, 72, 136, 520), lightning(2, 264, 20)], width=80, loop=None),
}


def weights(cfg, seed=0):
    return random_hybrid_weights(read_hybrid_config(cfg), seed=seed)


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(9000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def save_checkpoint(cfg, w, folder):
    from safetensors.torch import save_file
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({k: v.contiguous() for k, v in w["tensors"].items()}, os.path.join(folder, "model.safetensors"))


def errors(got, ref):
    """Per position: rms of the logit difference (its mean taken off) over the rms of the reference's deviation."""
    got, ref = got.double().cpu(), ref.double()
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    s = (ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / s
