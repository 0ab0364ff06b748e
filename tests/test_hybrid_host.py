"""Layer-listed models without a GPU: configuration, packing, registry, trace
runner, C ABI, and the oracle's own consistency."""
import ctypes
import io
import json
import math
import os
import re

import numpy as np
import pytest
import torch

import hybrid_models as hm
from megaqwen_b200 import _lib, registry, trace
from megaqwen_b200.spec import read_hybrid_config
from oracle import hybrid_reference as ref

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---------------------------------------------------------------- configuration
def test_config_gives_every_size_and_the_order_of_runs():
    spec = read_hybrid_config(hm.MODELS["mixed"])
    assert spec.runs() == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [i for i, _ in ref.layer_order(hm.MODELS["mixed"])] == spec.runs()
    assert spec.layers[0].mixer.rank == 56 and spec.layers[1].mixer.kind == "lightning" and spec.layers[1].ff == 160
    assert read_hybrid_config(hm.MODELS["latent first, loop to the end"]).layers[0].ff == 0
    shapes = spec.tensor_shapes()
    assert shapes["loop.in"] == (96, 192) and shapes["l0.mix.q"] == (5 * 52, 96) and shapes["l1.mix.g"] == (120, 96)
    assert "loop.in" not in read_hybrid_config(hm.MODELS["no loop, other layers"]).tensor_shapes()


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].__setitem__("type", "other"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("decay", [0.5]), "decays for"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 4), "rotation covers"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "routed"), "unknown feed-forward"),
    (lambda c: c.__setitem__("loop", hm.loop(1, 5, 2)), "does not lie within"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("dim", 0), "positive integer"),
])
def test_config_errors(change, message):
    cfg = json.loads(json.dumps(hm.config([hm.lightning(3, 16, 16), hm.latent(2, 16, 8, 16, 24)])))
    change(cfg)
    with pytest.raises(ValueError, match=message):
        read_hybrid_config(cfg)


def test_registry_chooses_by_architecture(tmp_path):
    assert registry.find_model("synthetic").name == "Qwen3ForCausalLM"
    for cfg, name in ((hm.MODELS["mixed"], "Satosun"), ({"architectures": ["Qwen3ForCausalLM"]}, "Qwen3ForCausalLM")):
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        assert registry.find_model(str(tmp_path)).name == name
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.find_model(str(tmp_path))


def test_weights_are_read_and_checked(tmp_path):
    from megaqwen_b200.weights import load_hybrid_weights
    cfg = hm.MODELS["mixed"]
    w = hm.weights(cfg)
    hm.save_checkpoint(cfg, w, tmp_path)
    got = load_hybrid_weights(str(tmp_path))
    assert set(got["tensors"]) == set(w["tensors"]) and got["tokenizer"] is None
    assert all(torch.equal(got["tensors"][k], v) for k, v in w["tensors"].items())
    w["tensors"]["l1.mix.k"] = w["tensors"]["l1.mix.k"][:-1]
    hm.save_checkpoint(cfg, w, tmp_path)
    with pytest.raises(RuntimeError, match="l1.mix.k"):
        load_hybrid_weights(str(tmp_path))
    del w["tensors"]["l2.mix.sink"]
    w["tensors"]["l1.mix.k"] = got["tensors"]["l1.mix.k"]
    hm.save_checkpoint(cfg, w, tmp_path)
    with pytest.raises(KeyError, match="l2.mix.sink"):
        load_hybrid_weights(str(tmp_path))


def test_generate_command_line(capsys, tmp_path):
    from megaqwen_b200 import generate
    assert generate.main(["--list"]) == 0
    assert "Satosun: bfloat16, float32" in capsys.readouterr().out
    with pytest.raises(SystemExit):
        generate.main([str(tmp_path)])                       # neither ids nor text
    with pytest.raises(SystemExit):
        generate.main([str(tmp_path), "--ids", "1", "--prompt", "x"])


def test_dtype_is_checked_before_anything_is_built():
    with pytest.raises(ValueError, match="runs in bfloat16"):
        registry.build_decoder(weights={"spec": None}, dtype="float32")


# ---------------------------------------------------------------- packing
def test_padding_keeps_products():
    from megaqwen_b200.hybrid import _pad_cols, _pad_rows, _segment
    g = torch.Generator().manual_seed(1)
    w, x = torch.randn(3 * 20, 40, generator=g), torch.randn(40, generator=g)
    p = _pad_rows(w, 3, 20)
    assert p.shape == (96, 48)
    y = (p @ torch.nn.functional.pad(x, (0, 8))).reshape(3, 32)
    assert torch.allclose(y[:, :20].reshape(-1), w @ x, atol=1e-5) and not y[:, 20:].any()
    back = _pad_cols(w.T.contiguous(), 3, 20)                        # a product over padded heads
    assert back.shape == (48, 96) and torch.allclose((back @ y.reshape(-1))[:40], w.T @ (w @ x), atol=1e-3)
    assert _segment(torch.ones(33, 2)).shape == (64, 2) and _segment(torch.ones(64, 2)).shape == (64, 2)


def test_decay_powers_and_rope_table():
    from megaqwen_b200.hybrid import decay_powers, rope_table
    d = decay_powers([0.0, 0.5, 0.999, 1.0], 129)
    assert d[:, 0].tolist() == [1.0] * 4 and d[0, 1] == 0 and d[1, 10] == 2.0 ** -10 and d[3, 128] == 1
    assert abs(float(d[2, 128]) - 0.999 ** 128) < 1e-7
    t = rope_table(50, 6, 300.0, 16)
    assert t.shape == (50, 8, 2)
    for p, i in ((0, 0), (1, 1), (49, 2)):
        a = p * 300.0 ** (-2 * i / 6)
        assert abs(float(t[p, i, 0]) - math.cos(a)) < 1e-6 and abs(float(t[p, i, 1]) - math.sin(a)) < 1e-6
    assert t[:, 3:, 0].eq(1).all() and t[:, 3:, 1].eq(0).all()


def test_random_weights_are_deterministic():
    a, b = hm.weights(hm.MODELS["mixed"], 3), hm.weights(hm.MODELS["mixed"], 3)
    assert all(torch.equal(a["tensors"][k], b["tensors"][k]) for k in a["tensors"])


# ---------------------------------------------------------------- C ABI
def test_library_exports_what_its_header_declares():
    from megaqwen_b200.csrc.build import build
    lib = ctypes.CDLL(build(name="hybrid"))
    text = open(os.path.join(ROOT, "include", "megaqwen_hybrid.h")).read()
    names = set(re.findall(r"\b(mqh?_\w+)\s*\(", re.sub(r"/\*.*?\*/", "", text, flags=re.S)))
    assert names == set(_lib.HYBRID_SIGNATURES)
    for name in names:
        assert hasattr(lib, name)


def _c_model(max_seq=100):
    one = ctypes.c_void_p(256)            # never dereferenced by the host functions below
    layers = (_lib.MqhLayer * 2)()
    for layer, kind in zip(layers, (_lib.MQH_LATENT, _lib.MQH_LIGHTNING)):
        layer.kind, layer.heads, layer.dim, layer.vdim, layer.rank, layer.rot, layer.ff, layer.mix_norm_n = kind, 3, 32, 48, 64, 16, 80, 126
        layer.norm_parts, layer.vdim_n = 1, 42
        for n in ("norm", "w_in", "w_out", "mix_norm", "decay_pow", "w_ukv", "w_uk_t", "sink", "rope"):
            setattr(layer, n, one)
    return _lib.MqhModel(_lib.MQH_BF16, _lib.MQH_PARALLEL, 64, 64, 333, max_seq, 1.0, 1e-6, 1.0, 2, 0, 1, 3, layers, one, one, one, one)


def test_host_entry_points():
    from megaqwen_b200.csrc.build import build
    build(name="hybrid")
    lib, m = _lib.hybrid_lib(), _c_model()
    p = ctypes.byref(m)
    assert lib.mqh_run_count(p) == 4 and [lib.mqh_run_layer(p, r) for r in range(5)] == [0, 0, 0, 1, -1]
    assert lib.mqh_state_bytes(p, 0) == 100 * 80 * 2 and lib.mqh_state_bytes(p, 3) == 3 * 32 * 48 * 4
    assert not lib.mqh_state_recurrent(p, 0) and lib.mqh_state_recurrent(p, 3)
    assert lib.mqh_in_rows(ctypes.byref(m.layers[0]), m.form) == 96 + 64 + 96 + 160
    assert lib.mqh_in_rows(ctypes.byref(m.layers[1]), m.form) == 2 * 96 + 2 * 160 + 160
    assert lib.mqh_ukv_rows(ctypes.byref(m.layers[0])) == 96 + 160 and lib.mqh_ukv_rows(ctypes.byref(m.layers[1])) == 0
    assert lib.mqh_logits_ld(p) == 512
    assert lib.mqh_decode_launch_count(p) == 3 * (1 + 5) + 3 + 1
    small, large = lib.mqh_workspace_bytes(p, 16), lib.mqh_workspace_bytes(p, 32)
    assert 0 < small < large
    m.width = 60                           # not padded: rejected before anything runs
    assert lib.mqh_workspace_bytes(p, 16) == 0
    assert lib.mqh_launch_decode(p, None, None, None, None, None, 0, None) == -1
    assert lib.mqh_launch_prefill(None, None, None, 1, 0, None, 0, None, None, None, None) == -1


# ---------------------------------------------------------------- state
def test_state_resets_what_recurs():
    from megaqwen_b200.state import SequenceState
    s = SequenceState([(64, 0), (32, 1)], "cpu")
    for b in s.buffers:
        b.fill_(7)
    saved = s.snapshot()
    s.reset()
    assert s.buffers[0].eq(7).all() and not s.buffers[1].any() and s.nbytes() == 96
    s.restore(saved)
    assert s.buffers[1].eq(7).all()


# ---------------------------------------------------------------- trace runner
class FakeDecoder:
    """Logits that spell the history: [number of tokens so far, sum of them]."""

    def __init__(self):
        self.resets = 0
        self.reset()

    def reset(self):
        self.seen, self.resets = [], self.resets + 1

    def step_logits(self, ids, want):
        rows = []
        for i, t in enumerate(ids):
            self.seen.append(t)
            if i in want:
                rows.append([len(self.seen), sum(self.seen)])
        return torch.tensor(rows, dtype=torch.float32)


def test_trace_runner_keeps_and_gives_back_a_request(tmp_path):
    run = trace.TraceRunner(FakeDecoder(), str(tmp_path))
    run.run_step({"step": 0, "entries": [{"id": "a", "tokens": [5, 6], "want": []}], "end": []})
    assert not os.listdir(tmp_path)
    run.run_step({"step": 1, "entries": [{"id": "a", "tokens": [1, 1, 1], "want": [0, 2]}], "end": ["a"]})
    assert np.fromfile(tmp_path / "1.f32", dtype="<f4").tolist() == [3, 12, 5, 14]
    with_next = {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": []}
    run.run_step(with_next)
    assert np.fromfile(tmp_path / "2.f32", dtype="<f4").tolist() == [1, 9]
    with pytest.raises(ValueError, match="before"):
        run.run_step({"step": 3, "entries": [{"id": "c", "tokens": [9], "want": []}], "end": []})
    with pytest.raises(ValueError, match="one entry"):
        run.run_step({"step": 3, "entries": with_next["entries"] * 2, "end": []})


def test_trace_runner_main(tmp_path, monkeypatch, capsys):
    (tmp_path / "config.json").write_text(json.dumps(hm.MODELS["mixed"]))
    made = {}

    def fake(model, max_seq_len, max_prefill_len, dtype):
        made.update(max_seq_len=max_seq_len, dtype=dtype)
        return FakeDecoder(), None
    monkeypatch.setattr(registry, "build_decoder", fake)
    monkeypatch.setattr("megaqwen_b200.csrc.build.build", lambda name: made.update(library=name))
    monkeypatch.setattr("sys.stdin", io.StringIO('{"step": 0, "entries": [{"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]}\n'))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "50"]) == 0
    assert "done 0" in capsys.readouterr().out.split("\n")
    assert made["dtype"] == "float32" and made["library"] == "hybrid" and made["max_seq_len"] >= 50
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["Qwen3ForCausalLM"]}))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "50"]) == 3


def test_step_logits_of_the_base_class_cuts_at_the_wanted_places():
    from megaqwen_b200.engine import DecodeEngine

    class Scripted(DecodeEngine):
        def __init__(self):
            self.vocab_size_, self.device, self.calls, self.n = 2, "cpu", [], 0

        def decode_step_logits(self, t):
            self.calls.append([t])
            self.n += 1
            return 0, torch.tensor([float(self.n), 0.0])

        def prefill_step_logits(self, ids, append=False):
            assert append
            self.calls.append(list(ids))
            self.n += len(ids)
            return 0, torch.tensor([float(self.n), 0.0])
    d = Scripted()
    lg = d.step_logits([1, 2, 3, 4, 5], [0, 3])
    assert lg[:, 0].tolist() == [1.0, 4.0] and d.calls == [[1], [2, 3, 4], [5]]
    assert d.step_logits([6], []).shape == (0, 2) and d.n == 6


# ---------------------------------------------------------------- the oracle
def test_oracle_does_not_depend_on_the_cut():
    cfg = hm.MODELS["mixed"]
    m = ref.HybridReference(cfg, hm.weights(cfg)["tensors"])
    ids = hm.tokens(cfg, 9)
    whole = m.forward(ids)
    m.reset()
    cut = torch.cat([m.forward(ids[:4]), m.forward(ids[4:5]), m.forward(ids[5:])])
    assert torch.allclose(whole, cut, atol=1e-10)
    assert len(m.trace) == len(read_hybrid_config(cfg).runs())


def _logits(cfg, w, ids):
    return ref.HybridReference(cfg, w["tensors"]).forward(ids)


@pytest.mark.parametrize("mistake", ["sink", "decay", "key", "rotation", "gain", "loop state", "gate", "loop input"])
def test_a_planted_mistake_shows_in_the_oracle(mistake, monkeypatch):
    """Each mistake moves the logits by far more than the tolerances of the GPU tests allow."""
    cfg = hm.MODELS["mixed"]
    w, ids = hm.weights(cfg), hm.tokens(cfg, 12)
    right = _logits(cfg, w, ids)
    if mistake == "sink":
        monkeypatch.setattr(ref, "softmax_with_sink", lambda s, sink: torch.softmax(s, 0))
    elif mistake == "decay":
        cfg = json.loads(json.dumps(cfg))
        for e in cfg["layers"]:
            if e["type"] == "lightning":
                e["mixer"]["decay"] = [1.0] * e["mixer"]["heads"]
    elif mistake == "key":
        keep = ref.softmax_with_sink
        monkeypatch.setattr(ref, "softmax_with_sink", lambda s, sink: keep(torch.cat([torch.full((1,), -1e30, dtype=s.dtype), s[1:]]), sink) if len(s) > 1
                            else keep(s, sink))
    elif mistake == "rotation":
        monkeypatch.setattr(ref, "rotate_interleaved", lambda x, p, base: x)
    elif mistake == "gain":
        monkeypatch.setattr(ref, "norm_zero_centred", lambda x, g, eps: ref.rms(x, eps) * (0.9 + g))
    elif mistake == "loop state":
        class Shared(ref.HybridReference):
            def forward(self, t):
                out = []
                for one in t:                 # a pass leaves its state to the next pass of the layer
                    for n, (i, _) in enumerate(self.runs):
                        self.states[n] = self.states[[j for j, (k, _) in enumerate(self.runs) if k == i][-1]]
                    out.append(super().forward([one]))
                return torch.cat(out)
        wrong = Shared(cfg, w["tensors"]).forward(ids)
        assert float(hm.errors(wrong, right).max()) > 0.1
        return
    elif mistake == "gate":
        w["tensors"] = dict(w["tensors"], **{"l1.mix.g": w["tensors"]["l1.mix.g"] * 0})
    elif mistake == "loop input":
        monkeypatch.setattr(ref, "loop_input", lambda x, x0, m: torch.cat([x0, x], -1) @ m.T)
    assert float(hm.errors(_logits(cfg, w, ids), right).max()) > 0.1
