"""Model dimensions of the decode/prefill paths.

``ModelSpec`` is the Qwen3 block: its CUDA kernels are specialised at compile time for the Qwen3-0.6B block
geometry (hidden 1024, intermediate 3072, 16 query heads / 8 KV heads of
dimension 128), as the reference is (csrc/megakernel/config.cuh:64-73,
csrc/megakernel/megakernel_kernels.py:13-21).  The number of layers, the
vocabulary size and the cache length are run-time values, so the parity tests
can use a 2-layer / small-vocabulary model with the same kernels.

``HybridSpec`` is a model whose layers are listed one by one in config.json
(design "Satosun"): every size and constant comes from there.
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
    """One layer's token mixer.  ``lightning``: heads, dim, vdim, decay.  ``latent_attention``: heads,
    dim (unrotated), rot (rotated), vdim, rank, rot_base, scale."""
    kind: str
    heads: int
    dim: int
    vdim: int
    decay: tuple = ()
    rank: int = 0
    rot: int = 0
    rot_base: float = 0.0
    scale: float = 0.0


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
            m, p = layer.mixer, f"l{i}."
            out[p + "norm1"] = (w,)
            if m.kind == "lightning":
                out[p + "mix.q"] = out[p + "mix.k"] = (m.heads * m.dim, w)
                out[p + "mix.v"] = out[p + "mix.g"] = (m.heads * m.vdim, w)
                out[p + "mix.norm"] = (m.heads * m.vdim,)
            else:
                out[p + "mix.q"] = (m.heads * (m.dim + m.rot), w)
                out[p + "mix.dkv"] = (m.rank + m.rot, w)
                out[p + "mix.dkv.norm"] = (m.rank,)
                out[p + "mix.uk"] = (m.heads * m.dim, m.rank)
                out[p + "mix.uv"] = (m.heads * m.vdim, m.rank)
                out[p + "mix.sink"] = (m.heads,)
            out[p + "mix.o"] = (w, m.heads * m.vdim)
            if layer.ff:
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (layer.ff, w)
                out[p + "mlp.down"] = (w, layer.ff)
        out["final.norm"] = (w,)
        out["head"] = (self.vocab_size, w)
        return out

    def decode_bytes(self, context: int, elem: int = 2) -> int:
        """Algorithmic HBM bytes of one decode step at ``context`` cached positions: every weight that the
        step reads (looped layers count each time), cached latents, recurrent states read and written."""
        shapes = self.tensor_shapes()

        def layer_elems(i):
            return sum(_count(s) for k, s in shapes.items() if k.startswith(f"l{i}."))

        total = elem * (_count(shapes["head"]) + 2 * self.hidden_size)
        if self.loop is not None:
            total += elem * self.loop[2] * _count(shapes["loop.in"])
        for i in self.runs():
            m = self.layers[i].mixer
            total += elem * layer_elems(i)
            if m.kind == "lightning":
                total += 2 * 4 * m.heads * m.dim * m.vdim
            else:
                total += elem * (m.rank + m.rot) * (context + 1)
        return total

    def prefill_flops(self, seq_len: int) -> float:
        shapes, total = self.tensor_shapes(), 2.0 * _count(self.tensor_shapes()["head"])
        if self.loop is not None:
            total += 2.0 * seq_len * self.loop[2] * _count(shapes["loop.in"])
        for i in self.runs():
            m = self.layers[i].mixer
            total += 2.0 * seq_len * sum(_count(s) for k, s in shapes.items() if k.startswith(f"l{i}.") and len(s) == 2)
            if m.kind == "lightning":
                total += 4.0 * seq_len * m.heads * m.dim * m.vdim
            else:
                total += m.heads * 2.0 * (m.dim + m.rot + m.vdim) * seq_len * (seq_len + 1) / 2
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


def _read_mixer(entry: dict, where: str) -> MixerSpec:
    kind, m = entry["type"], entry["mixer"]
    heads, dim, vdim = (_positive(m[k], f"{where}.{k}") for k in ("heads", "dim", "vdim"))
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
    raise ValueError(f"{where}: unknown mixer type {kind!r}")


def read_hybrid_config(cfg: dict) -> HybridSpec:
    """The spec of a config.json of design "Satosun"."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"layers[{i}]: unknown feed-forward kind {mlp.get('kind')!r}")
        layers.append(LayerSpec(_read_mixer(entry, f"layers[{i}].mixer"), 0 if mlp is None else _positive(mlp["ff"], f"layers[{i}].mlp.ff")))
    loop = cfg.get("loop")
    if loop is not None:
        loop = (int(loop["start"]), int(loop["stop"]), _positive(loop["times"], "loop.times"))
        if not 0 <= loop[0] < loop[1] <= len(layers):
            raise ValueError(f"loop {loop[0]} .. {loop[1]} does not lie within {len(layers)} layers")
    return HybridSpec(vocab_size=_positive(cfg["vocab"], "vocab"), hidden_size=_positive(cfg["width"], "width"),
                      embed_scale=float(cfg["embedding"]["scale"]), rms_eps=float(cfg["norm"]["eps"]),
                      residual_mult=float(cfg["residual_mult"]), layers=tuple(layers), loop=loop)
