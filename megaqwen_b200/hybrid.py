"""Decoder of layer-listed models: each layer has its own mixer and an optional
gated feed-forward.  Design "Satosun": lightning or latent attention beside the
feed-forward, and a stretch of layers may run several times with the same
weights.  Design "Vunasun": gated linear attention, Mamba-2 or chunked attention,
the feed-forward after it, norms on their results.

The object has the interface of ``MegakernelDecoder`` (engine.py): prompts,
portions of prompts, single steps, device-resident chains replayed from CUDA
graphs.  This file packs checkpoint tensors into the layout that
include/megaqwen_hybrid.h describes and calls that C ABI; all arithmetic of a
token is in the CUDA kernels.
"""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib
from ._lib import MqhBuffers, MqhLayer, MqhModel
from .engine import DecodeEngine, _ptr
from .spec import HybridSpec, MixerSpec
from .state import SequenceState

_DTYPES = {"bfloat16": (_lib.MQH_BF16, torch.bfloat16), "float32": (_lib.MQH_F32, torch.float32)}


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def _segment(rows: torch.Tensor) -> torch.Tensor:
    """Zero rows up to a multiple of MQH_SEGMENT."""
    extra = -rows.shape[0] % _lib.MQH_SEGMENT
    return torch.nn.functional.pad(rows, (0, 0, 0, extra)) if extra else rows


def _pad_rows(w: torch.Tensor, heads: int, d: int) -> torch.Tensor:
    """[heads*d, k] -> [heads*pad16(d), pad16(k)]: every head's rows, and the columns, filled up with zeros."""
    k = w.shape[1]
    w = torch.nn.functional.pad(w.reshape(heads, d, k), (0, pad16(k) - k, 0, pad16(d) - d))
    return w.reshape(heads * pad16(d), pad16(k))


def _pad_cols(w: torch.Tensor, heads: int, d: int) -> torch.Tensor:
    """[n, heads*d] -> [pad16(n), heads*pad16(d)]."""
    n = w.shape[0]
    w = torch.nn.functional.pad(w.reshape(n, heads, d), (0, pad16(d) - d, 0, 0, 0, pad16(n) - n))
    return w.reshape(pad16(n), heads * pad16(d))


def _pad_vec(v: torch.Tensor, heads: int, d: int) -> torch.Tensor:
    return torch.nn.functional.pad(v.reshape(heads, d), (0, pad16(d) - d)).reshape(-1).contiguous()


def decay_powers(decay, count: int) -> torch.Tensor:
    """[heads, count] fp32: decay^0, decay^1, .. of every head, each rounded once."""
    d = torch.tensor(decay, dtype=torch.float64)
    return (d[:, None] ** torch.arange(count, dtype=torch.float64)[None, :]).to(torch.float32)


def rope_table(max_seq_len: int, dims: int, base: float, padded: int | None = None) -> torch.Tensor:
    """[max_seq_len, padded/2, 2] fp32: cos, sin of position * base^(-2i/dims) for pair i, (2i, 2i + 1) or
    (i, i + dims/2); pairs of the padding do not turn."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    a = torch.arange(max_seq_len, dtype=torch.float64)[:, None] * f[None, :]
    a = torch.nn.functional.pad(a, (0, ((padded or dims) - dims) // 2))
    return torch.stack([torch.cos(a), torch.sin(a)], -1).to(torch.float32).contiguous()


class HybridDecoder(DecodeEngine):
    """Batch-1 greedy decoder of a layer-listed model.

    ``weights``: {"spec": HybridSpec, "tensors": name -> tensor}.  ``dtype`` "bfloat16" computes matrix
    products in bf16 with 32-bit accumulation and everything else that the design keeps in 32-bit (residual
    stream, norms, scores, recurrent state, logits) in 32-bit; "float32" computes everything in 32-bit.
    """

    def __init__(self, weights: dict, max_seq_len: int, max_prefill_len: int = 512, dtype: str = "bfloat16", device="cuda"):
        if not torch.cuda.is_available():
            raise RuntimeError("megaqwen_b200 needs a CUDA device (sm_100a); there is no CPU fallback")
        if dtype not in _DTYPES:
            raise ValueError(f"dtype must be one of {sorted(_DTYPES)}, got {dtype!r}")
        self.spec: HybridSpec = weights["spec"]
        self.dtype = dtype
        device = torch.device(device)
        if device.type != "cuda":
            raise RuntimeError("a CUDA device is needed")
        if device.index is None:
            device = torch.device("cuda", torch.cuda.current_device())
        self._init_engine(_lib.hybrid_lib(), device, self.spec.vocab_size, max_seq_len, min(int(max_prefill_len), int(max_seq_len)))
        with torch.cuda.device(device):
            self._pack(weights["tensors"])
            lib = self._lib
            runs = lib.mqh_run_count(C.byref(self._model))
            self.state = SequenceState([(lib.mqh_state_bytes(C.byref(self._model), r), lib.mqh_state_recurrent(C.byref(self._model), r))
                                        for r in range(runs)], device)
            nbytes = lib.mqh_workspace_bytes(C.byref(self._model), self.max_prefill_len_)
            if nbytes == 0:
                raise RuntimeError("this model has sizes that the kernels do not hold "
                                   "(a head's query / key or state size <= 512, latent rank <= 2048, latent vdim <= 512, convolution <= 64 taps)")
            self._workspace = torch.zeros(nbytes, dtype=torch.uint8, device=device)
            self._buf = MqhBuffers(_ptr(self._workspace), nbytes, self.max_prefill_len_, self.state.pointers, _ptr(self._scalars) + 4)
            self._step_launches = lib.mqh_decode_launch_count(C.byref(self._model))

    # ------------------------------------------------------------------ packing
    def _keep(self, t: torch.Tensor) -> int:
        """Hold a packed tensor for the lifetime of the decoder (the C side has only its pointer)."""
        t = t.contiguous()
        self._packed.append(t)
        return _ptr(t)

    def _pack(self, tensors: dict) -> None:
        spec, dev = self.spec, self.device
        code, dt = _DTYPES[self.dtype]
        self._packed = []
        self._ropes = {}

        def mat(name):
            return tensors[name].to(device=dev, dtype=dt)

        def vec(name):
            return tensors[name].to(device=dev, dtype=torch.float32)

        w = spec.hidden_size

        def gain(name, scale=None):          # norms over the width: stored around zero, or plain with a layer scale
            g = 1.0 + vec(name) if not spec.post_norm else vec(name) * (vec(scale) if scale else 1.0)
            return self._keep(_pad_vec(g, 1, w))

        pack = {"lightning": self._pack_lightning, "latent_attention": self._pack_latent, "gla": self._pack_gla, "mamba2": self._pack_mamba2,
                "attention": self._pack_attention}
        form = _lib.MQH_POST_NORM if spec.post_norm else _lib.MQH_PARALLEL
        self._layers = (MqhLayer * spec.num_layers)()
        for i, layer in enumerate(spec.layers):
            p, m, out = f"l{i}.", layer.mixer, self._layers[i]
            out.heads, out.dim, out.vdim, out.ff = m.heads, pad16(m.dim), pad16(m.vdim), pad16(layer.ff)
            out.vdim_n, out.norm_parts = m.vdim, 1
            out.norm = gain(p + "norm1", p + "ls1")
            rows = pack[m.kind](out, m, p + "mix.", mat, vec)
            cols = [_pad_cols(mat(p + "mix.o"), m.heads, m.vdim)]
            if layer.ff:
                gate, up = (_pad_rows(mat(p + "mlp." + n), 1, layer.ff) for n in ("gate", "up"))
                gu, down = torch.stack([gate, up], 1).reshape(2 * gate.shape[0], -1), _pad_cols(mat(p + "mlp.down"), 1, layer.ff)
                if spec.post_norm:
                    out.w_gu, out.w_down, out.norm2 = self._keep(_segment(gu)), self._keep(down), gain(p + "norm2", p + "ls2")
                else:
                    rows.append(gu)
                    cols.append(down)
            w_in = torch.cat([_segment(r) for r in rows])
            if w_in.shape[0] != self._lib.mqh_in_rows(C.byref(out), form):
                raise RuntimeError("packed input projection does not have the rows the library expects")
            out.w_in = self._keep(w_in)
            out.w_out = self._keep(torch.cat(cols, 1))
        wp = pad16(w)
        loop = spec.loop or (0, 0, 0)
        self._model = MqhModel(
            code, form, wp, w, spec.vocab_size, self.max_seq_len_, spec.embed_scale, spec.rms_eps, spec.residual_mult, spec.num_layers, *loop,
            self._layers, self._keep(_pad_cols(mat("loop.in"), 2, w)) if spec.loop else None,
            self._keep(torch.nn.functional.pad(mat("embed"), (0, wp - w))), gain("final.norm"),
            self._keep(torch.nn.functional.pad(mat("head"), (0, wp - w))))

    def _pack_lightning(self, out: MqhLayer, m: MixerSpec, p: str, mat, vec) -> list:
        out.kind, out.mix_norm_n = _lib.MQH_LIGHTNING, m.heads * m.vdim
        out.mix_norm = self._keep(_pad_vec(vec(p + "norm"), m.heads, m.vdim))
        out.decay_pow = self._keep(decay_powers(m.decay, _lib.MQH_CHUNK + 1).to(self.device))
        return [_pad_rows(mat(p + n), m.heads, d) for n, d in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim))]

    def _rope(self, dims: int, base: float, padded: int) -> int:
        key = (dims, base, padded)
        if key not in self._ropes:
            self._ropes[key] = self._keep(rope_table(self.max_seq_len_, dims, base, padded).to(self.device))
        return self._ropes[key]

    def _pack_gla(self, out: MqhLayer, m: MixerSpec, p: str, mat, vec) -> list:
        out.kind, out.rank, out.scale, out.inv_tau = _lib.MQH_GLA, pad16(m.rank), m.dim ** -0.5, 1.0 / m.tau
        out.mix_norm_n, out.norm_parts = m.vdim, m.heads                     # every head by itself, one weight for all
        out.mix_norm = self._keep(_pad_vec(vec(p + "norm").repeat(m.heads), m.heads, m.vdim))
        a2 = _pad_rows(mat(p + "a2"), m.heads, m.dim)
        out.gate_w = self._keep(a2.reshape(m.heads, pad16(m.dim), pad16(m.rank)).transpose(1, 2))
        out.gate_b = self._keep(_pad_vec(vec(p + "a2.b"), m.heads, m.dim))
        return [_pad_rows(mat(p + n), h, d) for n, h, d in
                (("q", m.heads, m.dim), ("k", m.heads, m.dim), ("v", m.heads, m.vdim), ("g", m.heads, m.vdim), ("a1", 1, m.rank))]

    def _pack_mamba2(self, out: MqhLayer, m: MixerSpec, p: str, mat, vec) -> list:
        out.kind, out.kv_heads, out.conv = _lib.MQH_MAMBA2, m.kv_heads, m.conv
        out.mix_norm_n, out.norm_parts = m.heads * m.vdim // m.norm_groups, m.norm_groups
        out.mix_norm = self._keep(_pad_vec(vec(p + "norm"), m.heads, m.vdim))
        out.dt_bias, out.skip = self._keep(vec(p + "dt_bias")), self._keep(vec(p + "D"))
        out.a_neg = self._keep((-torch.exp(vec(p + "A_log").double())).float())
        inner, gn = m.heads * m.vdim, m.kv_heads * m.dim
        parts = ((inner, m.heads, m.vdim), (gn, m.kv_heads, m.dim), (gn, m.kv_heads, m.dim))           # x, B, C
        sizes = [n for n, _, _ in parts]
        conv = [_pad_rows(c, h, d) for c, (_, h, d) in zip(vec(p + "conv").split(sizes), parts)]
        out.conv_w = self._keep(torch.cat(conv)[:, :m.conv].T)
        out.conv_b = self._keep(torch.cat([_pad_vec(c, h, d) for c, (_, h, d) in zip(vec(p + "conv.b").split(sizes), parts)]))
        z, x, b, c, dt = mat(p + "in").split([inner] + sizes + [m.heads])
        return [_pad_rows(z, m.heads, m.vdim)] + [_pad_rows(r, h, d) for r, (_, h, d) in zip((x, b, c), parts)] + [_pad_rows(dt, 1, m.heads)]

    def _pack_attention(self, out: MqhLayer, m: MixerSpec, p: str, mat, vec) -> list:
        out.kind, out.kv_heads, out.rot, out.scale, out.chunk, out.mix_norm_n = _lib.MQH_ATTENTION, m.kv_heads, m.rot, m.scale, m.chunk, m.dim
        out.rope = self._rope(m.rot, m.rot_base, m.rot)
        out.q_bias, out.k_bias = (self._keep(_pad_vec(vec(p + n + ".b"), h, m.dim)) for n, h in (("q", m.heads), ("k", m.kv_heads)))
        out.q_norm, out.k_norm = (self._keep(_pad_vec(vec(p + n + ".norm"), 1, m.dim)) for n in ("q", "k"))
        return [_pad_rows(mat(p + "q"), m.heads, m.dim), _pad_rows(mat(p + "k"), m.kv_heads, m.dim), _pad_rows(mat(p + "g"), 1, m.heads)]

    def _pack_latent(self, out: MqhLayer, m: MixerSpec, p: str, mat, vec) -> list:
        out.kind, out.mix_norm_n, out.rank, out.rot, out.scale = _lib.MQH_LATENT, m.rank, pad16(m.rank), pad16(m.rot), m.scale
        out.mix_norm = self._keep(_pad_vec(vec(p + "dkv.norm"), 1, m.rank))
        out.sink = self._keep(vec(p + "sink"))
        out.rope = self._rope(m.rot, m.rot_base, pad16(m.rot))
        uk, uv = _pad_rows(mat(p + "uk"), m.heads, m.dim), _pad_rows(mat(p + "uv"), m.heads, m.vdim)
        w_ukv = torch.cat([_segment(uk), _segment(uv)])
        if w_ukv.shape[0] != self._lib.mqh_ukv_rows(C.byref(out)):
            raise RuntimeError("packed key / value projection does not have the rows the library expects")
        out.w_ukv = self._keep(w_ukv)
        out.w_uk_t = self._keep(uk.reshape(m.heads, pad16(m.dim), pad16(m.rank)).transpose(1, 2))
        q = mat(p + "q").reshape(m.heads, m.dim + m.rot, -1)
        dkv = mat(p + "dkv")
        return [_pad_rows(q[:, :m.dim].reshape(m.heads * m.dim, -1), m.heads, m.dim),
                _pad_rows(q[:, m.dim:].reshape(m.heads * m.rot, -1), m.heads, m.rot),
                torch.cat([_pad_rows(dkv[:m.rank], 1, m.rank), _pad_rows(dkv[m.rank:], 1, m.rot)])]

    # ------------------------------------------------------------------ launches
    @property
    def step_launches(self) -> int:
        return self._step_launches

    def _launch(self, in_ptr, out_ptr, pos_ptr, logits_ptr, chained) -> None:
        flags = (_lib.MQ_FLAG_CHAINED if chained else 0) | (0 if self.use_pdl else _lib.MQ_FLAG_NO_PDL)
        _lib.check(self._lib.mqh_launch_decode(C.byref(self._model), C.byref(self._buf), in_ptr, out_ptr, pos_ptr, logits_ptr, flags,
                                               self._stream()), "mqh_launch_decode")
        self.launches += self.step_launches

    def _prefill(self, ids: torch.Tensor, want=None):
        """Tokens that continue the sequence at ``position()``.  Returns (next token, logits [len(want), vocab] or None)."""
        n = int(ids.numel())
        with torch.cuda.device(self.device):
            dev_ids = ids.to(self.device, non_blocking=True)
            rows = logits = None
            if want:
                rows = torch.tensor(want, dtype=torch.int32, device=self.device)
                logits = torch.empty((len(want), self._lib.mqh_logits_ld(C.byref(self._model))), dtype=torch.float32, device=self.device)
            count = C.c_int(0)
            rc = self._lib.mqh_launch_prefill(C.byref(self._model), C.byref(self._buf), _ptr(dev_ids), n, self.position_,
                                              _ptr(rows) if want else None, len(want) if want else 0, _ptr(self._scalars),
                                              _ptr(logits) if want else None, C.byref(count), self._stream())
            _lib.check(rc, "mqh_launch_prefill")
            self.launches += count.value
            self.position_ += n
            tok, status = self._scalars[:2].tolist()
        self._check_status(status)
        return tok, (logits[:, :self.vocab_size_] if want else None)

    # ------------------------------------------------------------------ prompts
    def reset(self) -> None:
        self.position_ = 0
        with torch.cuda.device(self.device):
            self.state.reset()

    def prefill_step(self, input_ids) -> int:
        """A whole prompt from position 0; returns the token that follows it."""
        ids = torch.as_tensor(input_ids, dtype=torch.int32).reshape(-1)
        self._check_prefill(ids, 0)
        self.reset()
        return self._prefill(ids)[0]

    def prefill_append(self, input_ids) -> int:
        """A portion of a prompt: the tokens continue the sequence at ``position()``."""
        ids = torch.as_tensor(input_ids, dtype=torch.int32).reshape(-1)
        self._check_prefill(ids, self.position_)
        return self._prefill(ids)[0]

    def prefill_step_logits(self, input_ids, append: bool = False):
        """prefill_step (or prefill_append) that also returns the fp32 logits after the last token."""
        ids = torch.as_tensor(input_ids, dtype=torch.int32).reshape(-1)
        self._check_prefill(ids, self.position_ if append else 0)
        if not append:
            self.reset()
        tok, lg = self._prefill(ids, [int(ids.numel()) - 1])
        return tok, lg[0].clone()

    def step_logits(self, input_ids, want):
        """The next tokens of the sequence in one forward pass; fp32 logits [len(want), vocab] at the places
        ``want`` among them.  One token goes through the decode step, more through prefill (in pieces of at
        most ``max_prefill_len()``)."""
        ids, want = [int(t) for t in input_ids], [int(i) for i in want]
        if any(i < 0 or i >= len(ids) for i in want):
            raise ValueError("a wanted place lies outside the tokens of the step")
        if len(ids) == 1:
            if not want:
                self.decode_step(ids[0])
                return torch.empty((0, self.vocab_size_), dtype=torch.float32, device=self.device)
            lg = self.decode_step_logits(ids[0])[1]
            return lg.unsqueeze(0).expand(len(want), -1)
        got, step = {}, self.max_prefill_len_
        for at in range(0, len(ids), step):
            part = torch.tensor(ids[at:at + step], dtype=torch.int32)
            self._check_prefill(part, self.position_)
            here = sorted({i for i in want if at <= i < at + step})
            lg = self._prefill(part, [i - at for i in here])[1]
            got.update({i: lg[j] for j, i in enumerate(here)})
        return torch.stack([got[i] for i in want]) if want else torch.empty((0, self.vocab_size_), dtype=torch.float32, device=self.device)
