"""Plain CPU oracle of the layer-listed design "Vunasun", one function per mechanism.

TEST INFRASTRUCTURE ONLY (see oracle/__init__.py), in the manner of hybrid_reference.py: written
from the equations, token by token, in one floating dtype (float64 by default), with no code of
the product.  A layer is two sublayers one after the other; each reads the residual stream itself,
and only its RESULT is normed, scaled element by element and added.
"""
from __future__ import annotations

import math

import torch

from .hybrid_reference import feed_forward, norm_plain, rms, silu


# ---------------------------------------------------------------- elementary functions
def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_halves(x, position, base, dims):
    """x [..., dim]: element i < dims/2 turns together with element i + dims/2 by position * base^(-2i / dims);
    elements from dims on stay as they are."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = position * base ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * math.cos(a) - v * math.sin(a)
        out[..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def causal_conv(x, w, b, past):
    """x [T, channels], w [channels, taps]: y_t = b + sum_j w[:, j] x_(t - taps + 1 + j).  past [taps - 1, channels] are the
    inputs before x (zeros where a sequence starts).  Returns (y, the last taps - 1 inputs)."""
    T, taps = x.shape[0], w.shape[1]
    ext = torch.cat([past, x])
    y = torch.empty_like(x)
    for t in range(T):
        y[t] = b + (ext[t:t + taps].T * w).sum(1)
    return y, ext[ext.shape[0] - (taps - 1):]


def chunk_mask(position, size):
    """First key that a position of a chunk sees; the last one is itself."""
    return position // size * size


# ---------------------------------------------------------------- mixers
def gla(h, w, mixer, eps, state=None):
    """Gated linear attention: every key channel of the state decays by a rate of its own that the token sets."""
    H, d, dv, tau = mixer["heads"], mixer["dim"], mixer["vdim"], mixer["tau"]
    T = h.shape[0]
    q = (h @ w["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w["k"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, dv)
    z = ((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).reshape(T, H, d)
    alpha = torch.sigmoid(z) ** (1.0 / tau)
    S = torch.zeros(H, d, dv, dtype=h.dtype) if state is None else state.clone()
    o = torch.empty(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    y = norm_plain(o, w["norm"], eps).reshape(T, H * dv) * silu(h @ w["g"].T)
    return y @ w["o"].T, S


def mamba2(h, w, mixer, eps, state=None):
    """state: (S [heads, N, vdim], the last inputs of the convolution)."""
    H, dv, N, G = mixer["heads"], mixer["vdim"], mixer["state"], mixer["groups"]
    inner, T = H * dv, h.shape[0]
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], -1)
    if state is None:
        state = (torch.zeros(H, N, dv, dtype=h.dtype), torch.zeros(mixer["conv"] - 1, xbc.shape[1], dtype=h.dtype))
    S, past = state[0].clone(), state[1]
    xbc, past = causal_conv(xbc, w["conv"], w["conv.b"], past)
    x, B, C = torch.split(silu(xbc), [inner, G * N, G * N], -1)
    x, B, C = x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N)
    dt = softplus(dt + w["dt_bias"])
    y = torch.empty(T, H, dv, dtype=h.dtype)
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            S[a] = torch.exp(-torch.exp(w["A_log"][a]) * dt[t, a]) * S[a] + dt[t, a] * B[t, g][:, None] * x[t, a][None, :]
            y[t, a] = S[a].T @ C[t, g] + w["D"][a] * x[t, a]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.reshape(T, mixer["norm_groups"], -1), eps).reshape(T, inner) * w["norm"]
    return y @ w["o"].T, (S, past)


def attention(h, w, mixer, eps, cache=None):
    """cache: (keys after norm and rotation, values) of earlier tokens, [past, kv_heads, dim] each."""
    H, G, d, rot = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["rot"]
    T = h.shape[0]
    past = 0 if cache is None else cache[0].shape[0]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = k
    q, k = norm_plain(q, w["q.norm"], eps), norm_plain(k, w["k.norm"], eps)
    q = torch.stack([rotate_halves(q[t], past + t, rot["base"], rot["dims"]) for t in range(T)])
    k = torch.stack([rotate_halves(k[t], past + t, rot["base"], rot["dims"]) for t in range(T)])
    if cache is not None:
        k, v = torch.cat([cache[0], k]), torch.cat([cache[1], v])
    gate = torch.sigmoid(h @ w["g"].T)
    out = torch.empty(T, H, d, dtype=h.dtype)
    for t in range(T):
        p = past + t
        lo = chunk_mask(p, mixer["mask"]["size"])
        for a in range(H):
            g = a // (H // G)
            s = (k[lo:p + 1, g] @ q[t, a]) * mixer["scale"]
            out[t, a] = (torch.softmax(s, 0) @ v[lo:p + 1, g]) * gate[t, a]
    return out.reshape(T, H * d) @ w["o"].T, (k, v)


MIXERS = {"gla": gla, "mamba2": mamba2, "attention": attention}


# ---------------------------------------------------------------- layer, model
def add_normed(x, y, norm_w, scale_w, eps):
    return x + norm_plain(y, norm_w, eps) * scale_w


class VunasunReference:
    """``forward(tokens)`` continues the sequence and returns logits [tokens, vocab]; ``trace`` then holds the residual
    stream after every layer of that call."""

    def __init__(self, cfg, tensors, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.states = [None] * len(self.cfg["layers"])

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def forward(self, tokens):
        eps = self.cfg["norm"]["eps"]
        x = self.t["embed"][torch.as_tensor(tokens).long()]
        self.trace = []
        for i, entry in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            y, self.states[i] = MIXERS[entry["type"]](x, self._sub(p + "mix."), entry["mixer"], eps, self.states[i])
            x = add_normed(x, y, self.t[p + "norm1"], self.t[p + "ls1"], eps)
            if entry["mlp"] is not None:
                x = add_normed(x, feed_forward(x, self._sub(p + "mlp.")), self.t[p + "norm2"], self.t[p + "ls2"], eps)
            self.trace.append(x)
        return norm_plain(x, self.t["final.norm"], eps) @ self.t["head"].T

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
