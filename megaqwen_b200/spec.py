"""Model dimensions of the decode/prefill paths.

``ModelSpec`` is the Qwen3 block: its CUDA kernels are specialised at compile time for the Qwen3-0.6B block
geometry (hidden 1024, intermediate 3072, 16 query heads / 8 KV heads of
dimension 128), as the reference is (csrc/megakernel/config.cuh:64-73,
csrc/megakernel/megakernel_kernels.py:13-21).  The number of layers, the
vocabulary size and the cache length are run-time values, so the parity tests
can use a 2-layer / small-vocabulary model with the same kernels.

``HybridSpec`` is a model whose layers are listed one by one in config.json
(designs "Satosun" and "Vunasun"): every size and constant comes from there, and
the sizes that config.json leaves open from the shapes of the tensors.
"""
from __future__ import annotations

from dataclasses import dataclass


@dataclass(frozen=True)
class ModelSpec:
    hidden_size: int = 1024
    intermediate_size: int = 3072
    num_q_heads: int = 16
    num_kv_heads: int = 8
    head_dim: int = 128
    num_layers: int = 28
    vocab_size: int = 151936
    rms_eps: float = 1e-6
    rope_theta: float = 1e6

    @property
    def q_size(self) -> int:
        return self.num_q_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def weight_bytes(self) -> int:
        """Bytes of weights one decoded token must read (bf16).

        Per layer: q,k,v,o,gate,up,down matrices plus four norm vectors; then
        the tied LM head read once, the final norm and one embedding row.
        """
        h, i, q, kv, d = self.hidden_size, self.intermediate_size, self.q_size, self.kv_size, self.head_dim
        per_layer = (q * h + 2 * kv * h + h * q + 2 * i * h + h * i) + (2 * h + 2 * d)
        return 2 * (self.num_layers * per_layer + self.vocab_size * h + h + h)

    def kv_bytes_per_position(self) -> int:
        """Bytes of K plus V one cached position holds over all layers (bf16)."""
        return self.num_layers * 2 * self.kv_size * 2

    def decode_bytes(self, cache_len: int) -> int:
        """Algorithmic HBM bytes of one batch-1 decode step that ends with
        ``cache_len`` cached positions: all weights, a read of every cached
        position and the write of the new one."""
        return self.weight_bytes() + self.kv_bytes_per_position() * (cache_len + 1)

    def prefill_flops(self, seq_len: int) -> float:
        h, i, q, kv, d = self.hidden_size, self.intermediate_size, self.q_size, self.kv_size, self.head_dim
        lin = q * h + 2 * kv * h + h * q + 3 * i * h
        attn = self.num_layers * self.num_q_heads * (2 * 2 * d) * seq_len * (seq_len + 1) / 2
        return 2.0 * seq_len * self.num_layers * lin + attn + 2.0 * self.vocab_size * h


QWEN3_0_6B = ModelSpec()

# Same block geometry, two layers and a 4096-entry vocabulary: runs through the
# CPU oracle in well under a second.
QWEN3_TINY = ModelSpec(num_layers=2, vocab_size=4096)


# ---------------------------------------------------------------- layer-listed models
@dataclass(frozen=True)
class MixerSpec:
    """One layer's token mixer.  All kinds: heads, dim (query / key size; state size of mamba2), vdim.

    ``lightning``: decay.  ``latent_attention``: dim (unrotated), rot (rotated), rank, rot_base, scale.
    ``gla``: tau, rank (inner width of the decay projection).  ``mamba2``: kv_heads (groups of B and C),
    conv (taps), norm_groups.  ``attention``: kv_heads, rot (rotated dimensions), rot_base, scale, chunk
    (positions see their own chunk of that many)."""
    kind: str
    heads: int
    dim: int
    vdim: int
    decay: tuple = ()
    rank: int = 0
    rot: int = 0
    rot_base: float = 0.0
    scale: float = 0.0
    kv_heads: int = 0
    conv: int = 0
    norm_groups: int = 1
    tau: float = 1.0
    chunk: int = 0

    @property
    def conv_channels(self) -> int:
        return self.heads * self.vdim + 2 * self.kv_heads * self.dim

    def tensor_shapes(self, w: int) -> dict:
        """name after 'mix.' -> shape, for a model of width ``w``."""
        hd, hv, kd = self.heads * self.dim, self.heads * self.vdim, self.kv_heads * self.dim
        if self.kind == "lightning":
            out = {"q": (hd, w), "k": (hd, w), "v": (hv, w), "g": (hv, w), "norm": (hv,)}
        elif self.kind == "latent_attention":
            out = {"q": (self.heads * (self.dim + self.rot), w), "dkv": (self.rank + self.rot, w), "dkv.norm": (self.rank,),
                   "uk": (hd, self.rank), "uv": (hv, self.rank), "sink": (self.heads,)}
        elif self.kind == "gla":
            out = {"q": (hd, w), "k": (hd, w), "v": (hv, w), "g": (hv, w), "a1": (self.rank, w), "a2": (hd, self.rank), "a2.b": (hd,),
                   "norm": (self.vdim,)}
        elif self.kind == "mamba2":
            cc = self.conv_channels
            out = {"in": (hv + cc + self.heads, w), "conv": (cc, self.conv), "conv.b": (cc,), "dt_bias": (self.heads,), "A_log": (self.heads,),
                   "D": (self.heads,), "norm": (hv,)}
        else:
            out = {"q": (hd, w), "q.b": (hd,), "k": (kd, w), "k.b": (kd,), "q.norm": (self.dim,), "k.norm": (self.dim,), "g": (self.heads, w)}
        out["o"] = (w, hv)
        return out

    @property
    def state_elems(self) -> int:
        """Elements of the recurrent matrix state, 0 for attention."""
        return self.heads * self.dim * self.vdim if self.kind in ("lightning", "gla", "mamba2") else 0

    def visible(self, position: int) -> int:
        """Keys that a position of an attention layer sees."""
        return position % self.chunk + 1 if self.chunk else position + 1

    def cache_elems(self) -> int:
        """Elements that one cached position holds, 0 for recurrent mixers."""
        return {"latent_attention": self.rank + self.rot, "attention": 2 * self.kv_heads * self.dim}.get(self.kind, 0)

    def score_flops(self, seq_len: int) -> float:
        """FLOPs of everything between the projections of a prompt, by the recurrence's or the attention's definition."""
        if self.state_elems:
            return 4.0 * seq_len * self.state_elems
        full, rest = (seq_len // self.chunk, seq_len % self.chunk) if self.chunk else (0, seq_len)
        pairs = full * self.chunk * (self.chunk + 1) / 2 + rest * (rest + 1) / 2
        own_rot = self.rot if self.kind == "latent_attention" else 0
        return self.heads * 2.0 * (self.dim + own_rot + self.vdim) * pairs


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    ff: int                  # width of the gated feed-forward, 0 for none


@dataclass(frozen=True)
class HybridSpec:
    vocab_size: int
    hidden_size: int
    embed_scale: float
    rms_eps: float
    residual_mult: float
    layers: tuple
    loop: tuple | None = None        # (start, stop, times)
    architecture: str = "Satosun"
    # False: one norm, stored around zero, feeds mixer and feed-forward side by side.  True: the two follow one
    # another, read the residual stream itself, and their results are normed and scaled (layer scale).
    post_norm: bool = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def runs(self) -> list:
        """Layer of every layer run of one forward pass, in order."""
        n = self.num_layers
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a checkpoint."""
        w, out = self.hidden_size, {"embed": (self.vocab_size, self.hidden_size)}
        if self.loop is not None:
            out["loop.in"] = (w, 2 * w)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            out[p + "norm1"] = (w,)
            out.update({p + "mix." + k: v for k, v in layer.mixer.tensor_shapes(w).items()})
            if self.post_norm:
                out[p + "ls1"] = (w,)
            if layer.ff:
                if self.post_norm:
                    out[p + "norm2"] = out[p + "ls2"] = (w,)
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (layer.ff, w)
                out[p + "mlp.down"] = (w, layer.ff)
        out["final.norm"] = (w,)
        out["head"] = (self.vocab_size, w)
        return out

    def decode_bytes(self, context: int, elem: int = 2) -> int:
        """Algorithmic HBM bytes of one decode step at ``context`` cached positions: every weight that the
        step reads (looped layers count each time), the cached rows it sees, recurrent states read and written."""
        shapes = self.tensor_shapes()
        total = elem * (_count(shapes["head"]) + 2 * self.hidden_size)
        if self.loop is not None:
            total += elem * self.loop[2] * _count(shapes["loop.in"])
        for i in self.runs():
            m = self.layers[i].mixer
            total += elem * sum(_count(s) for k, s in shapes.items() if k.startswith(f"l{i}."))
            total += 2 * 4 * m.state_elems
            if m.kind == "mamba2":
                total += elem * m.conv * m.conv_channels
            total += elem * m.cache_elems() * m.visible(context)
        return total

    def prefill_flops(self, seq_len: int) -> float:
        shapes, total = self.tensor_shapes(), 2.0 * _count(self.tensor_shapes()["head"])
        if self.loop is not None:
            total += 2.0 * seq_len * self.loop[2] * _count(shapes["loop.in"])
        for i in self.runs():
            total += 2.0 * seq_len * sum(_count(s) for k, s in shapes.items() if k.startswith(f"l{i}.") and len(s) == 2)
            total += self.layers[i].mixer.score_flops(seq_len)
        return total


def _count(shape) -> int:
    n = 1
    for s in shape:
        n *= s
    return n


def _positive(value, what: str) -> int:
    if not isinstance(value, int) or value <= 0:
        raise ValueError(f"{what} must be a positive integer, got {value!r}")
    return value


def _divides(part: int, whole: int, what: str) -> None:
    if whole % part:
        raise ValueError(f"{what}: {part} does not divide {whole}")


def _read_mixer(entry: dict, where: str, gate_rank: int) -> MixerSpec:
    kind, m = entry["type"], entry["mixer"]
    heads, vdim = (_positive(m[k], f"{where}.{k}") for k in ("heads", "vdim"))
    dim = _positive(m["state" if kind == "mamba2" else "dim"], f"{where}.dim")
    if kind == "lightning":
        decay = tuple(float(d) for d in m["decay"])
        if len(decay) != heads:
            raise ValueError(f"{where}: {len(decay)} decays for {heads} heads")
        return MixerSpec(kind, heads, dim, vdim, decay=decay)
    if kind == "latent_attention":
        rot = _positive(m["rot_dim"], f"{where}.rot_dim")
        if m["rot"]["dims"] != rot or rot % 2:
            raise ValueError(f"{where}: the rotation covers the whole rotated part, an even number of dimensions "
                             f"(rot.dims {m['rot']['dims']}, rot_dim {rot})")
        return MixerSpec(kind, heads, dim, vdim, rank=_positive(m["kv_rank"], f"{where}.kv_rank"), rot=rot,
                         rot_base=float(m["rot"]["base"]), scale=float(m["scale"]))
    if kind == "gla":
        if not m["tau"] > 0:
            raise ValueError(f"{where}.tau must be positive, got {m['tau']!r}")
        return MixerSpec(kind, heads, dim, vdim, tau=float(m["tau"]), rank=_positive(gate_rank, f"{where}: rank of a1"))
    if kind == "mamba2":
        groups, parts = (_positive(m[k], f"{where}.{k}") for k in ("groups", "norm_groups"))
        _divides(groups, heads, f"{where}.groups")
        _divides(parts, heads * vdim, f"{where}.norm_groups")
        return MixerSpec(kind, heads, dim, vdim, kv_heads=groups, conv=_positive(m["conv"], f"{where}.conv"), norm_groups=parts)
    if kind == "attention":
        kv_heads, rot = _positive(m["kv_heads"], f"{where}.kv_heads"), _positive(m["rot"]["dims"], f"{where}.rot.dims")
        _divides(kv_heads, heads, f"{where}.kv_heads")
        if vdim != dim:
            raise ValueError(f"{where}: the values are the keys, so vdim is dim ({vdim}, {dim})")
        if rot % 2 or rot > dim:
            raise ValueError(f"{where}: an even number of at most {dim} dimensions is rotated, not {rot}")
        return MixerSpec(kind, heads, dim, vdim, kv_heads=kv_heads, rot=rot, rot_base=float(m["rot"]["base"]), scale=float(m["scale"]),
                         chunk=_positive(m["mask"]["size"], f"{where}.mask.size"))
    raise ValueError(f"{where}: unknown mixer type {kind!r}")


# mixers of each design
DESIGN_MIXERS = {"Satosun": ("lightning", "latent_attention"), "Vunasun": ("gla", "mamba2", "attention")}


def read_hybrid_config(cfg: dict, shapes: dict | None = None, gate_rank: int = 16) -> HybridSpec:
    """The spec of a config.json of a layer-listed design.  ``shapes``: tensor name -> shape of the checkpoint, for
    the sizes config.json does not give (the rank of a gla layer's decay projection; without a checkpoint ``gate_rank``)."""
    name = cfg.get("architecture", "Satosun")
    if name not in DESIGN_MIXERS:
        raise ValueError(f"unknown layer-listed design {name!r}")
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        if entry["type"] not in DESIGN_MIXERS[name]:
            raise ValueError(f"layers[{i}].mixer: unknown mixer type {entry['type']!r}")
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"layers[{i}]: unknown feed-forward kind {mlp.get('kind')!r}")
        a1 = (shapes or {}).get(f"l{i}.mix.a1")
        mixer = _read_mixer(entry, f"layers[{i}].mixer", int(a1[0]) if a1 else gate_rank)
        layers.append(LayerSpec(mixer, 0 if mlp is None else _positive(mlp["ff"], f"layers[{i}].mlp.ff")))
    vocab, width, eps = _positive(cfg["vocab"], "vocab"), _positive(cfg["width"], "width"), float(cfg["norm"]["eps"])
    if name == "Vunasun":
        return HybridSpec(vocab, width, 1.0, eps, 1.0, tuple(layers), architecture=name, post_norm=True)
    loop = cfg.get("loop")
    if loop is not None:
        loop = (int(loop["start"]), int(loop["stop"]), _positive(loop["times"], "loop.times"))
        if not 0 <= loop[0] < loop[1] <= len(layers):
            raise ValueError(f"loop {loop[0]} .. {loop[1]} does not lie within {len(layers)} layers")
    return HybridSpec(vocab, width, float(cfg["embedding"]["scale"]), eps, float(cfg["residual_mult"]), tuple(layers), loop=loop, architecture=name)
