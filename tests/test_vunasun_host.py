"""Design "Vunasun" without a GPU: configuration, tensor names, packing, C ABI, and the
oracle's own consistency with mistakes planted in it."""
import ctypes
import json
import math

import pytest
import torch

import vunasun_models as vm
from megaqwen_b200 import _lib, registry
from megaqwen_b200.spec import read_hybrid_config
from oracle import vunasun_reference as ref


def copy(cfg):
    return json.loads(json.dumps(cfg))


# ---------------------------------------------------------------- configuration
def test_config_gives_every_size():
    spec = read_hybrid_config(vm.MODELS["all three"], gate_rank=11)
    assert spec.post_norm and spec.architecture == "Vunasun" and spec.loop is None and spec.runs() == [0, 1, 2]
    m, a, g = (layer.mixer for layer in spec.layers)
    assert (m.heads, m.vdim, m.dim, m.kv_heads, m.conv, m.norm_groups) == (6, 24, 20, 3, 4, 2) and m.conv_channels == 144 + 120
    assert (a.heads, a.kv_heads, a.dim, a.rot, a.chunk, a.rot_base) == (6, 2, 40, 24, 50, 3000.0)
    assert (g.heads, g.dim, g.vdim, g.tau, g.rank) == (3, 24, 40, 8.0, 11) and [x.ff for x in spec.layers] == [176, 176, 0]
    s = spec.tensor_shapes()
    assert s["l0.mix.in"] == (144 + 264 + 6, 96) and s["l0.mix.conv"] == (264, 4) and s["l0.mix.norm"] == (144,) and s["l0.ls2"] == (96,)
    assert s["l1.mix.k"] == (80, 96) and s["l1.mix.g"] == (6, 96) and s["l1.mix.q.norm"] == (40,) and "l1.mix.v" not in s
    assert s["l2.mix.a1"] == (11, 96) and s["l2.mix.a2"] == (72, 11) and s["l2.mix.norm"] == (40,) and s["l2.ls1"] == (96,)
    assert not any(k.startswith("l2.mlp") or k in ("l2.norm2", "l2.ls2") for k in s)


def test_the_rank_of_the_decay_projection_comes_from_the_tensors(tmp_path):
    from megaqwen_b200.weights import load_hybrid_weights
    cfg = vm.config([vm.gla(2, 16, 24), vm.gla(3, 8, 8)])
    w = vm.weights(cfg, gate_rank=21)
    vm.save_checkpoint(cfg, w, tmp_path)
    got = load_hybrid_weights(str(tmp_path))
    assert [layer.mixer.rank for layer in got["spec"].layers] == [21, 21]
    assert all(torch.equal(got["tensors"][k], v) for k, v in w["tensors"].items())
    w["tensors"]["l1.mix.a2"] = w["tensors"]["l1.mix.a2"][:, :-1].contiguous()
    vm.save_checkpoint(cfg, w, tmp_path)
    with pytest.raises(RuntimeError, match="l1.mix.a2"):
        load_hybrid_weights(str(tmp_path))


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].__setitem__("type", "lightning"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("groups", 4), "does not divide"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("norm_groups", 7), "does not divide"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("conv", 0), "positive integer"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 4), "does not divide"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("vdim", 48), "values are the keys"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 42), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "positive integer"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("tau", 0), "tau"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "routed"), "unknown feed-forward"),
])
def test_config_errors(change, message):
    cfg = copy(vm.MODELS["all three"])
    change(cfg)
    with pytest.raises(ValueError, match=message):
        read_hybrid_config(cfg)


def test_the_mixers_of_one_design_are_not_those_of_another():
    cfg = copy(vm.MODELS["all three"])
    cfg.update(architecture="Satosun", embedding={"scale": 1.0}, residual_mult=1.0)
    with pytest.raises(ValueError, match="unknown mixer type"):
        read_hybrid_config(cfg)


def test_registry_and_command_line(tmp_path, capsys):
    from megaqwen_b200 import generate
    (tmp_path / "config.json").write_text(json.dumps(vm.MODELS["all three"]))
    entry = registry.find_model(str(tmp_path))
    assert entry.name == "Vunasun" and entry.library == "hybrid" and entry.dtypes == ("bfloat16", "float32")
    assert generate.main(["--list"]) == 0 and "Vunasun: bfloat16, float32" in capsys.readouterr().out


def test_work_counts_follow_the_chunks():
    spec = read_hybrid_config(vm.config([(vm.attention(2, 1, 16, 8, 10), None)], width=32, vocab=50))
    m = spec.layers[0].mixer
    assert [m.visible(p) for p in (0, 9, 10, 25)] == [1, 10, 1, 6]
    assert m.score_flops(25) == 2 * 2.0 * 32 * (2 * 55 + 15)
    assert spec.decode_bytes(25) - spec.decode_bytes(20) == 2 * 32 * 5


# ---------------------------------------------------------------- packing
def test_rope_table_of_halves_has_no_padding():
    from megaqwen_b200.hybrid import rope_table
    t = rope_table(40, 10, 700.0)
    assert t.shape == (40, 5, 2)
    a = 39 * 700.0 ** (-2 * 3 / 10)
    assert abs(float(t[39, 3, 0]) - math.cos(a)) < 1e-6 and abs(float(t[39, 3, 1]) - math.sin(a)) < 1e-6


def _layer(kind, **sizes):
    one = ctypes.c_void_p(256)            # never dereferenced by the host functions below
    layer = _lib.MqhLayer()
    for n, t in layer._fields_:
        if t is ctypes.c_void_p:
            setattr(layer, n, one)
    base = dict(kind=kind, heads=6, dim=32, vdim=48, kv_heads=2, rank=16, rot=8, ff=80, mix_norm_n=6 * 42, norm_parts=1, vdim_n=42, conv=4, chunk=9)
    for k, v in dict(base, **sizes).items():
        setattr(layer, k, v)
    return layer


def _model(*layers, form=_lib.MQH_POST_NORM, loop_times=0):
    one = ctypes.c_void_p(256)
    arr = (_lib.MqhLayer * len(layers))(*layers)
    return _lib.MqhModel(_lib.MQH_BF16, form, 64, 64, 333, 100, 1.0, 1e-6, 1.0, len(layers), 0, 1, loop_times, arr, one, one, one, one)


def test_host_entry_points():
    from megaqwen_b200.csrc.build import build
    build(name="hybrid")
    lib = _lib.hybrid_lib()
    mamba, att, gla = _layer(_lib.MQH_MAMBA2), _layer(_lib.MQH_ATTENTION, vdim=32, ff=0), _layer(_lib.MQH_GLA)
    m = _model(mamba, att, gla)
    p = ctypes.byref(m)
    assert lib.mqh_run_count(p) == 3 and [lib.mqh_state_recurrent(p, r) for r in range(3)] == [1, 0, 1]
    channels = 6 * 48 + 2 * 2 * 32
    assert lib.mqh_state_bytes(p, 0) == 6 * 32 * 48 * 4 + 4 * channels * 2
    assert lib.mqh_state_bytes(p, 1) == 100 * 2 * 2 * 32 * 2 and lib.mqh_state_bytes(p, 2) == 6 * 32 * 48 * 4
    rows = [lib.mqh_in_rows(ctypes.byref(x), m.form) for x in (mamba, att, gla)]
    assert rows == [288 + 288 + 64 + 64 + 32, 192 + 64 + 32, 192 + 192 + 288 + 288 + 32]
    assert lib.mqh_in_rows(ctypes.byref(gla), _lib.MQH_PARALLEL) == rows[2] + 160
    assert lib.mqh_decode_launch_count(p) == (3 + 2) + 3 + (3 + 2) + 1
    assert 0 < lib.mqh_workspace_bytes(p, 16) < lib.mqh_workspace_bytes(p, 32)
    # rejected before anything runs
    for bad in (_layer(_lib.MQH_MAMBA2, kv_heads=4), _layer(_lib.MQH_MAMBA2, conv=65), _layer(_lib.MQH_MAMBA2, norm_parts=2),
                _layer(_lib.MQH_ATTENTION), _layer(_lib.MQH_ATTENTION, vdim=32, rot=34), _layer(_lib.MQH_ATTENTION, vdim=32, rot=7),
                _layer(_lib.MQH_GLA, dim=528), _layer(_lib.MQH_GLA, rank=10), _layer(_lib.MQH_GLA, vdim_n=49), _layer(7)):
        assert lib.mqh_workspace_bytes(ctypes.byref(_model(bad)), 16) == 0
    assert lib.mqh_workspace_bytes(ctypes.byref(_model(gla, loop_times=2)), 16) == 0          # loops are of the parallel form
    assert lib.mqh_workspace_bytes(ctypes.byref(_model(gla, form=2)), 16) == 0


# ---------------------------------------------------------------- the oracle
@pytest.mark.parametrize("name", ["all three", "attention first", "odd parts"])
def test_oracle_does_not_depend_on_the_cut(name):
    cfg = vm.MODELS[name]
    m = ref.VunasunReference(cfg, vm.weights(cfg)["tensors"])
    ids = vm.tokens(cfg, 23)
    whole = m.forward(ids)
    m.reset()
    cut = torch.cat([m.forward(ids[:4]), m.forward(ids[4:5]), m.forward(ids[5:7]), m.forward(ids[7:])])
    assert torch.allclose(whole, cut, atol=1e-10) and len(m.trace) == len(cfg["layers"])


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0], dtype=torch.float64)
    y = ref.rotate_halves(x, 3, 16.0, 4)              # pairs (0, 2) by 3, (1, 3) by 3 / 4; the fifth stays
    assert torch.allclose(y[0], torch.tensor(math.cos(3) - 3 * math.sin(3), dtype=torch.float64)) and y[4] == 5
    assert torch.allclose(y[3], torch.tensor(4 * math.cos(.75) + 2 * math.sin(.75), dtype=torch.float64))
    assert [ref.chunk_mask(p, 5) for p in (0, 4, 5, 11)] == [0, 0, 5, 10]
    out, past = ref.causal_conv(torch.tensor([[1.0], [2.0], [3.0]]), torch.tensor([[10.0, 1.0]]), torch.tensor([0.5]), torch.zeros(1, 1))
    assert out.flatten().tolist() == [1.5, 12.5, 23.5] and past.tolist() == [[3.0]]
    assert abs(float(ref.softplus(torch.tensor(-40.0, dtype=torch.float64))) - math.exp(-40)) < 1e-20


MISTAKES = {
    "chunk from 1": lambda mp: mp.setattr(ref, "chunk_mask", lambda p, size: (p + 1) // size * size),
    "no chunk": lambda mp: mp.setattr(ref, "chunk_mask", lambda p, size: 0),
    "interleaved rotation": lambda mp: mp.setattr(ref, "rotate_halves", lambda x, p, base, dims: _interleaved(x, p, base, dims)),
    "tap order": lambda mp: mp.setattr(ref, "causal_conv", _wrap_conv(lambda w: w.flip(1))),
    "no layer scale": lambda mp: mp.setattr(ref, "add_normed", lambda x, y, n, s, eps: x + ref.norm_plain(y, n, eps)),
    "norm of the sum": lambda mp: mp.setattr(ref, "add_normed", lambda x, y, n, s, eps: ref.norm_plain(x + y, n, eps) * s),
    "sigmoid for softplus": lambda mp: mp.setattr(ref, "softplus", torch.sigmoid),
}


def _interleaved(x, p, base, dims):
    from oracle.hybrid_reference import rotate_interleaved
    return torch.cat([rotate_interleaved(x[..., :dims], p, base), x[..., dims:]], -1)


def _wrap_conv(change):
    real = ref.causal_conv
    return lambda x, w, b, past: real(x, change(w), b, past)


TENSOR_MISTAKES = ["l0.mix.conv.b", "l0.mix.D", "l0.mix.dt_bias", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.g", "l2.mix.a2", "l2.mix.a2.b", "l2.mix.g", "l0.ls2"]


@pytest.mark.parametrize("mistake", list(MISTAKES) + TENSOR_MISTAKES)
def test_a_planted_mistake_shows_in_the_oracle(mistake, monkeypatch):
    """Each mistake moves the logits by far more than the tolerances of the GPU tests allow."""
    cfg = copy(vm.MODELS["all three"])
    cfg["layers"][1]["mixer"]["mask"]["size"] = 9
    w, ids = vm.weights(cfg), vm.tokens(cfg, 30)
    right = ref.VunasunReference(cfg, w["tensors"]).forward(ids)
    tensors = dict(w["tensors"])
    if mistake in MISTAKES:
        MISTAKES[mistake](monkeypatch)
    else:
        assert mistake in tensors
        tensors[mistake] = tensors[mistake] * 0
    assert float(vm.errors(ref.VunasunReference(cfg, tensors).forward(ids), right).max()) > 0.1


@pytest.mark.parametrize("kind", ["attention", "gla", "mamba2"])
def test_loud_models_are_decided_by_the_far_token(kind):
    cfg, w = vm.loud_model(kind, size=200)
    oracle = ref.VunasunReference(cfg, w["tensors"])
    ids = [t % vm.LOUD for t in vm.tokens(cfg, 150, 2)]
    quiet = oracle.forward(ids)
    oracle.reset()
    loud = oracle.forward([vm.LOUD] + ids[1:])
    assert float(vm.errors(quiet[100:], loud[100:]).min()) > 0.3
