"""Plain CPU oracle of the layer-listed decoder (design "Satosun"), one function per mechanism.

TEST INFRASTRUCTURE ONLY (see oracle/__init__.py).  Written from the equations,
token by token where the mechanism is a recurrence, with explicit loops and no
code of the product: slow, and meant to be read.  Everything is evaluated in
one floating dtype (float64 by default), so it is the exact value that the
kernels approximate with either of their weight types.

A model is ``(config, tensors)``: the parsed config.json and a dict name ->
torch tensor.
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------- elementary functions
def rms(x, eps):
    """x divided by its root mean square; eps is added inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(z):
    return z * torch.sigmoid(z)


def rotate_interleaved(x, position, base):
    """x [..., dims]: the pair (2i, 2i + 1) turns by position * base^(-2i / dims)."""
    dims = x.shape[-1]
    out = x.clone()
    for i in range(dims // 2):
        a = position * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def softmax_with_sink(scores, sink):
    """Weights of the keys when the denominator also holds exp(sink); scores [keys]."""
    m = max(float(scores.max()), float(sink))
    e = torch.exp(scores - m)
    return e / (e.sum() + math.exp(float(sink) - m))


# ---------------------------------------------------------------- mixers
def lightning(h, w, mixer, eps, state=None):
    """h [tokens, width].  w: dict of the mixer's tensors by short name.  Returns (out, state);
    state [heads, dim, vdim] is the recurrent state after the last token."""
    H, d, dv = mixer["heads"], mixer["dim"], mixer["vdim"]
    T = h.shape[0]
    q = silu(h @ w["q"].T).reshape(T, H, d)
    k = silu(h @ w["k"].T).reshape(T, H, d)
    v = silu(h @ w["v"].T).reshape(T, H, dv)
    S = torch.zeros(H, d, dv, dtype=h.dtype) if state is None else state.clone()
    decay = torch.tensor(mixer["decay"], dtype=h.dtype).reshape(H, 1, 1)
    o = torch.empty(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    y = norm_plain(o.reshape(T, H * dv), w["norm"], eps) * torch.sigmoid(h @ w["g"].T)
    return y @ w["o"].T, S


def latent_attention(h, w, mixer, eps, cache=None):
    """cache: (c [past, kv_rank], rotated key [past, rot_dim]) of earlier tokens, or None."""
    H, d, r, dv, R = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    base = mixer["rot"]["base"]
    T = h.shape[0]
    past = 0 if cache is None else cache[0].shape[0]
    q = (h @ w["q"].T).reshape(T, H, d + r)
    down = h @ w["dkv"].T
    c_new = norm_plain(down[:, :R], w["dkv.norm"], eps)
    k_new = torch.stack([rotate_interleaved(down[t, R:], past + t, base) for t in range(T)])
    c = c_new if cache is None else torch.cat([cache[0], c_new])
    kr = k_new if cache is None else torch.cat([cache[1], k_new])
    ku = (c @ w["uk"].T).reshape(past + T, H, d)
    v = (c @ w["uv"].T).reshape(past + T, H, dv)
    out = torch.empty(T, H * dv, dtype=h.dtype)
    for t in range(T):
        n = past + t + 1                       # keys 0 .. position
        qr = rotate_interleaved(q[t, :, d:], past + t, base)
        for a in range(H):
            s = (ku[:n, a] @ q[t, a, :d] + kr[:n] @ qr[a]) * mixer["scale"]
            out[t, a * dv:(a + 1) * dv] = softmax_with_sink(s, w["sink"][a]) @ v[:n, a]
    return out @ w["o"].T, (c, kr)


MIXERS = {"lightning": lightning, "latent_attention": latent_attention}


# ---------------------------------------------------------------- feed-forward, layer, model
def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def parallel_layer(x, entry, mix, mlp, norm_w, eps, mult, state):
    """One norm; the mixer and the feed-forward both read it; their sum is added once."""
    h = norm_zero_centred(x, norm_w, eps)
    y, state = MIXERS[entry["type"]](h, mix, entry["mixer"], eps, state)
    if entry["mlp"] is not None:
        y = y + feed_forward(h, mlp)
    return x + mult * y, state


def loop_input(x, x0, w):
    return torch.cat([x, x0], -1) @ w.T


def layer_order(cfg):
    """[(layer index, is it the first layer of a pass)] in running order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        runs += [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, False) for i in range(lp["stop"], n)]


class HybridReference:
    """``forward(tokens)`` continues the sequence and returns logits [tokens, vocab]; ``trace`` then
    holds the residual stream after every layer run of that call."""

    def __init__(self, cfg, tensors, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.runs = layer_order(cfg)
        self.reset()

    def reset(self):
        self.states = [None] * len(self.runs)

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def forward(self, tokens):
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = self.t["embed"][torch.as_tensor(tokens).long()] * cfg["embedding"]["scale"]
        x0 = x
        self.trace = []
        for n, (i, first) in enumerate(self.runs):
            if first:
                x = loop_input(x, x0, self.t["loop.in"])
            p = f"l{i}."
            x, self.states[n] = parallel_layer(x, cfg["layers"][i], self._sub(p + "mix."), self._sub(p + "mlp."), self.t[p + "norm1"],
                                               eps, cfg["residual_mult"], self.states[n])
            self.trace.append(x)
        return norm_zero_centred(x, self.t["final.norm"], eps) @ self.t["head"].T

    def greedy(self, prompt, n):
        """n greedy tokens after the prompt, and the margin between the two best logits at each."""
        out, margins = [], []
        lg = self.forward(prompt)[-1]
        for _ in range(n):
            top = torch.topk(lg, 2).values
            out.append(int(lg.argmax()))
            margins.append(float(top[0] - top[1]))
            lg = self.forward([out[-1]])[-1]
        return out, margins
