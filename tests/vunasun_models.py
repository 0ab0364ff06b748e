"""Small configurations and weights of design "Vunasun" for the tests (random, made here)."""
import math

import torch

import hybrid_models as hm
from megaqwen_b200.spec import read_hybrid_config
from megaqwen_b200.synthetic import random_hybrid_weights


def gla(heads, dim, vdim, tau=8.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def attention(heads, kv_heads, dim, rot, size, base=3000.0, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"base": base, "dims": rot},
                                           "scale": scale or dim ** -0.5, "mask": {"size": size}}}


def config(layers, width=96, vocab=331, ff=176, eps=1e-5):
    """layers: mixers; a pair (mixer, ff) overrides ff, None for no feed-forward."""
    out = []
    for entry in layers:
        mixer, f = entry if isinstance(entry, tuple) else (entry, ff)
        out.append(dict(mixer, mlp=None if f is None else {"kind": "dense", "ff": f}))
    return {"architecture": "Vunasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}


# Models that differ in everything config.json gives: sizes off the multiples of 16, 8 and 4, one head, many heads, one key
# head and as many as heads, parts of a norm that end inside a head, filters of one to many taps, chunks shorter and longer
# than a tile, every mixer with and without a feed-forward.
MODELS = {
    "all three": config([mamba2(6, 24, 20, groups=3, norm_groups=2), attention(6, 2, 40, 24, 50), (gla(3, 24, 40), None)]),
    "attention first": config([(attention(4, 4, 64, 64, 17, base=50.0, scale=0.3), None), (gla(1, 80, 112, tau=1.0), 72),
                               (mamba2(4, 32, 16, groups=4, conv=1, norm_groups=4), None)], width=128, eps=1e-3),
    "one key head": config([gla(7, 8, 8, tau=30.0), attention(17, 1, 16, 2, 129, base=9.0), (mamba2(2, 72, 136, conv=7), 40), attention(2, 1, 128, 96, 64)],
                           width=72, vocab=509),
    "odd parts": config([(mamba2(5, 6, 10, groups=5, conv=3, norm_groups=3), 24), (mamba2(3, 20, 34, conv=2, norm_groups=12), None)], width=40, vocab=130),
    "large heads": config([attention(2, 1, 136, 136, 70), (gla(2, 264, 20), None), (gla(1, 200, 72), None), (mamba2(1, 136, 264), None),
                           attention(2, 2, 264, 10, 100)], width=80),
    "wide feed-forward": config([(gla(2, 16, 16), 8160), (attention(2, 1, 16, 8, 40), 9000)], width=32, vocab=130),
    "wide": config([(gla(2, 32, 16), None), (mamba2(1, 16, 16), 80)], width=2200, vocab=90),       # more than two quads per thread
}
GATE_RANK = 11         # inner width of the decay projections: comes from the tensors, not from config.json


def weights(cfg, seed=0, gate_rank=GATE_RANK):
    return random_hybrid_weights(read_hybrid_config(cfg, gate_rank=gate_rank), seed=seed)


tokens, save_checkpoint, errors = hm.tokens, hm.save_checkpoint, hm.errors


LOUD = 96              # the token whose key every other token's query matches


def loud_model(kind, size=64):
    """One layer whose logits follow one token far back: LOUD has a feature that no other token has, its key answers to the
    feature that all others share, so losing (or double counting) it changes the logits by their own size."""
    mixer = {"attention": attention(2, 1, 32, 8, size, base=1e9, scale=1.0), "gla": gla(2, 24, 48, tau=16.0),
             "mamba2": mamba2(2, 48, 24, conv=2)}[kind]
    cfg = config([(mixer, None)], width=64, vocab=LOUD + 1)
    w = weights(cfg, 5)
    t = {k: v.float() for k, v in w["tensors"].items()}
    e = t["embed"]
    e[:, 0], e[:, 1] = 1.0, 0.0
    e[LOUD, 0], e[LOUD, 1] = 0.0, 8.0
    if kind == "attention":                           # dimension 31 is not rotated; the value is the key as projected
        t["l0.mix.q.b"] *= 0
        t["l0.mix.k.b"] *= 0
        t["l0.mix.q.norm"][:] = 1.0
        t["l0.mix.k.norm"][:] = 0.2
        t["l0.mix.k.norm"][31] = 4.0
        for h in range(2):
            t["l0.mix.q"][h * 32 + 31] = 0
            t["l0.mix.q"][h * 32 + 31, 0] = 2.0
        t["l0.mix.k"][31] = 0
        t["l0.mix.k"][31, 1] = 3.0
    elif kind == "gla":
        t["l0.mix.a2.b"][:] = 12.0                    # hardly any decay
        t["l0.mix.a2"] *= 0.1
        for h in range(2):
            t["l0.mix.q"][h * 24], t["l0.mix.k"][h * 24] = 0, 0
            t["l0.mix.q"][h * 24, 0], t["l0.mix.k"][h * 24, 1] = 8.0, 8.0
    else:
        n, inner = 24, 96
        t["l0.mix.A_log"][:] = -8.0
        t["l0.mix.in"][2 * inner + 2 * n:] = 0        # step sizes all alike
        t["l0.mix.dt_bias"][:] = -2.0
        b, c = 2 * inner, 2 * inner + n
        t["l0.mix.in"][b], t["l0.mix.in"][c] = 0, 0
        t["l0.mix.in"][b, 1], t["l0.mix.in"][c, 0] = 30.0, 30.0
        t["l0.mix.conv"][inner], t["l0.mix.conv"][inner + n] = torch.tensor([0.0, 1.0]), torch.tensor([0.0, 1.0])
        t["l0.mix.conv.b"][inner:] = 0
    w["tensors"] = {k: v.bfloat16() for k, v in t.items()}
    return cfg, w


def recurrence_exact(q, k, v, log_decay, state, scale=1.0):
    """Token by token in 64-bit.  q, k [T, H, d], v [T, H, dv], log_decay [T, H, d] (natural), state [H, d, dv]."""
    S, out = state.double().clone(), []
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t].double())[:, :, None] * S + k[t].double()[:, :, None] * v[t].double()[:, None, :]
        out.append((S * q[t].double()[:, :, None]).sum(1) * scale)
    return torch.stack(out), S


def attention_exact(q, k, v, pos0, size, scale, gate=None):
    """q [n, H, d] at positions pos0 .., k, v [pos0 + n, G, ..], size 0: no chunks; gate [n, H] before its sigmoid."""
    n, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    kk, vv = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)
    s = torch.einsum("thd,khd->htk", q.double(), kk) * scale
    i, j = pos0 + torch.arange(n)[:, None], torch.arange(k.shape[0])[None, :]
    hidden = (j > i) | ((j < i // size * size) if size else torch.zeros_like(j > i))
    out = torch.einsum("htk,khv->thv", torch.softmax(s.masked_fill(hidden[None], -math.inf), -1), vv)
    return out * torch.sigmoid(gate.double())[:, :, None] if gate is not None else out
