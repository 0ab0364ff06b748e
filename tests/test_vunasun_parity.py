"""Design "Vunasun" on the GPU against the plain oracle: every mechanism through the C ABI,
whole models in both compute types, and the public entry points."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import vunasun_models as vm
from oracle import vunasun_reference as ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

# rms logit error over the rms of the logits, per position; see test_hybrid_parity.py.  In bfloat16 a sublayer's small
# result is normed up together with its rounding: rounding the operands and results of the oracle's products alone moves
# single positions of these models by up to 0.053 (0.006 on average).  Every mistake planted in test_vunasun_host.py
# moves the logits by more than 0.1.
TOL = {"float32": 1e-5, "bfloat16": 0.06}
DTYPES = ("bfloat16", "float32")


@pytest.fixture(scope="module", autouse=True)
def built():
    from megaqwen_b200.csrc.build import build
    build(name="hybrid")


@pytest.fixture(scope="module")
def lib(built):
    from megaqwen_b200 import _lib
    return _lib.hybrid_lib()


_decoders, _logits = {}, {}


def model(cfg, dtype, max_seq=400, max_prefill=300, w=None, key=None):
    """(config, weights, decoder) with the decoder at the start of a sequence; decoders are kept over the module."""
    from megaqwen_b200.hybrid import HybridDecoder
    cfg = vm.MODELS[cfg] if isinstance(cfg, str) else cfg
    key = (key or json.dumps(cfg, sort_keys=True), dtype, max_seq, max_prefill)
    if key not in _decoders:
        w = w or vm.weights(cfg)
        _decoders[key] = (w, HybridDecoder(w, max_seq, max_prefill, dtype=dtype))
    w, dec = _decoders[key]
    dec.reset()
    return cfg, w, dec


def exact(cfg, w, ids, key=None):
    key = (key or json.dumps(cfg, sort_keys=True), tuple(ids))
    if key not in _logits:
        _logits[key] = ref.VunasunReference(cfg, w["tensors"]).forward(ids)
    return _logits[key]


def feed(dec, ids, portions):
    """Logits at every position, the tokens cut into the given portions (the rest one by one)."""
    dec.reset()
    out, at, cuts = [], 0, []
    for n in portions:
        cuts.append(min(n, len(ids) - sum(cuts)))
    for n in [n for n in cuts if n] + [1] * (len(ids) - sum(cuts)):
        out.append(dec.step_logits(ids[at:at + n], list(range(n))).cpu())
        at += n
    assert at == len(ids) and dec.position() == len(ids)
    return torch.cat(out)


def check(got, want, dtype, what=""):
    e = vm.errors(got, want)
    print(f"{what} {dtype}: max {float(e.max()):.2e} mean {float(e.mean()):.2e}")
    assert float(e.max()) <= TOL[dtype] and float(e.mean()) <= TOL[dtype] / 3, (what, dtype, float(e.max()), int(e.argmax()), float(e.mean()))


# ---------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(vm.MODELS))
def test_prompt_portions_and_decoding(name, dtype):
    """A whole prompt, portions of several sizes, and token by token from the first: every position."""
    cfg, w, dec = model(name, dtype)
    ids = vm.tokens(cfg, 150)
    want = exact(cfg, w, ids)
    for portions in ([150], [], [130], [2] * 20, [17, 2, 3, 50, 2, 64], [127, 2, 15]):
        check(feed(dec, ids, portions), want, dtype, f"{name} {portions[:6]}")


ALONE = {
    "gla": [(vm.gla(3, 48, 32), None)],
    "gla, fast decay": [(vm.gla(2, 32, 48, tau=0.25), None)],
    "gla, slow decay": [(vm.gla(2, 32, 48, tau=200.0), None)],
    "mamba2": [(vm.mamba2(4, 32, 48, groups=2, norm_groups=2), None)],
    "mamba2, one tap": [(vm.mamba2(3, 16, 32, conv=1), None)],
    "mamba2, many taps": [(vm.mamba2(2, 16, 16, conv=40), None)],
    "mamba2, a group per head": [(vm.mamba2(4, 24, 32, groups=4, norm_groups=4), None)],
    "attention": [(vm.attention(6, 3, 48, 16, 1000), None)],
    "attention, short chunks": [(vm.attention(4, 2, 32, 32, 3), None)],
    "attention, chunks of one": [(vm.attention(2, 2, 16, 4, 1), None)],
    "attention, one pair turns": [(vm.attention(2, 1, 64, 2, 33, base=2.0), None)],
    "feed-forward": [(vm.attention(1, 1, 16, 16, 1), 208)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALONE))
def test_each_mechanism_alone(name, dtype):
    """One mechanism per model: its normed result carries the logits."""
    cfg, w, dec = model(vm.config(ALONE[name], width=80, vocab=211), dtype)
    ids = vm.tokens(cfg, 140, 11)
    want = exact(cfg, w, ids)
    for portions in ([140], [], [2, 63, 2, 66]):
        check(feed(dec, ids, portions), want, dtype, f"{name} {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_from_nothing_to_everything(dtype):
    """Heads that forget within a token beside heads that keep everything, in one chunk: no factor overflows or vanishes."""
    cfg = vm.config([(vm.gla(3, 32, 32, tau=1.0), None), (vm.mamba2(3, 32, 32), None)], width=64, vocab=150)
    w = vm.weights(cfg, 3)
    t = w["tensors"]
    b = torch.linspace(-80.0, 40.0, 96)
    t["l0.mix.a2.b"] = b[torch.randperm(96, generator=torch.Generator().manual_seed(1))].bfloat16()
    t["l1.mix.A_log"], t["l1.mix.dt_bias"] = torch.tensor([4.0, -6.0, 0.0]).bfloat16(), torch.tensor([2.0, -1.0, -9.0]).bfloat16()
    cfg, w, dec = model(cfg, dtype, w=w, key="decays")
    ids = vm.tokens(cfg, 300, 3)
    want = exact(cfg, w, ids, "decays")
    for portions in ([300], [], [20, 250]):
        check(feed(dec, ids, portions), want, dtype, f"decays {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [64, 100, 128, 129, 300])
def test_long_sequence_over_tile_and_chunk_edges(size, dtype):
    """Positions around the attention's chunks, 64-key pieces, 128-key tiles and the recurrence's chunks of 128."""
    cfg = vm.config([(vm.attention(4, 2, 24, 8, size, scale=0.9), None), vm.gla(2, 40, 24), (vm.mamba2(2, 24, 40, groups=2), None)], width=64, vocab=257)
    cfg, w, dec = model(cfg, dtype)
    ids = vm.tokens(cfg, 390, 1)
    want = exact(cfg, w, ids)
    for portions in ([300, 86], [60], [128, 128, 120], [129, 127, 129], [size, 390 - size - 20], [size - 1, 2, 2]):
        check(feed(dec, ids, portions), want, dtype, f"{size} {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_several_chunks(dtype):
    cfg = vm.config([(vm.attention(8, 1, 64, 32, 640), None), (vm.gla(1, 16, 16), None)], width=48, vocab=64)
    cfg, w, dec = model(cfg, dtype, max_seq=1500, max_prefill=700)
    ids = vm.tokens(cfg, 1400, 4)
    want = exact(cfg, w, ids)
    check(feed(dec, ids, [600]), want, dtype, "decoded from 600")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gla", "mamba2"])
@pytest.mark.parametrize("place", [0, 1, 15, 16, 127, 128, 191])
def test_one_loud_token_far_away(kind, place, dtype):
    """The loud token sits at block and chunk edges and is read hundreds of tokens later."""
    cfg, w = vm.loud_model(kind)
    cfg, w, dec = model(cfg, dtype, 330, 330, w, "loud " + kind)
    ids = [t % vm.LOUD for t in vm.tokens(cfg, 320, 2)]
    ids[place] = vm.LOUD
    want = exact(cfg, w, ids, "loud " + kind)
    check(feed(dec, ids, [320]), want, dtype, f"{kind} prompt {place}")
    check(feed(dec, ids, [max(place, 2), 250 - max(place, 2)]), want, dtype, f"{kind} decoded {place}")
    check(feed(dec, ids, [place + 1, 60]), want, dtype, f"{kind} cut behind {place}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [64, 100, 150])
def test_loud_keys_at_the_edges_of_a_chunk(size, dtype):
    """The first and the last position of a chunk are loud in turn: every position of the chunk sees the one, none of the
    next chunk either, in prompts and in decoding."""
    cfg, w = vm.loud_model("attention", size)
    key = f"loud attention {size}"
    cfg, w, dec = model(cfg, dtype, 330, 330, w, key)
    base = [t % vm.LOUD for t in vm.tokens(cfg, 310, 2)]
    for place in (0, size - 1, size, size + 1, 2 * size - 1, 2 * size):
        ids = list(base)
        ids[place] = vm.LOUD
        want = exact(cfg, w, ids, key)
        quiet = exact(cfg, w, base, key)
        end = min((place // size + 1) * size, 310)
        moved = vm.errors(quiet, want)
        assert float(moved[place:end].min()) > 0.3 and float(moved[:place].sum()) == 0 and float(moved[end:].sum()) == 0
        for portions in ([310], [place + 1, 20], [max(place, 2), 2, 30], [size // 2, size, size // 2]):
            check(feed(dec, ids, portions), want, dtype, f"{size} {place} {portions}")


# ---------------------------------------------------------------- cache and state
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_that_is_used_again(dtype):
    """A sequence after a longer one in the same decoder, after a reset: nothing of it is left, also beyond the end."""
    cfg, w, dec = model("all three", dtype)
    a, b = vm.tokens(cfg, 140, 3), vm.tokens(cfg, 40, 4)
    feed(dec, a, [140])
    first = feed(dec, b, [30])
    check(first, exact(cfg, w, b), dtype)
    for short in ([1], [2], [1, 2]):                 # the filter's first taps, with what the longer sequence left in its ring
        feed(dec, a, [100])
        check(feed(dec, b, short), exact(cfg, w, b), dtype, f"{short}")
    assert torch.equal(first, feed(dec, b, [30]))    # same cut, same bits
    for buf, recurrent in zip(dec.state.buffers, dec.state.recurrent):      # whatever a cache holds beyond the position is never read
        if not recurrent:
            buf.view(torch.bfloat16 if dtype == "bfloat16" else torch.float32).fill_(float("nan"))
    assert torch.equal(feed(dec, b, [30]), first)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_snapshot_continues_two_ways(dtype):
    cfg, w, dec = model("all three", dtype)
    ids = vm.tokens(cfg, 60, 5)
    dec.step_logits(ids[:50], [])
    saved, pos = dec.state.snapshot(), dec.position()
    one = dec.step_logits(ids[50:], list(range(10))).cpu()
    dec.state.restore(saved)
    dec.position_ = pos
    two = dec.step_logits(ids[50:], list(range(10))).cpu()
    assert torch.equal(one, two)
    check(one, exact(cfg, w, ids)[50:], dtype)


def test_prompt_longer_than_one_prefill_call():
    cfg, w, dec = model("all three", "float32", max_seq=170, max_prefill=48)
    ids = vm.tokens(cfg, 150)
    want = exact(cfg, w, ids)
    places = [0, 47, 48, 49, 95, 96, 149]
    check(dec.step_logits(ids, places).cpu(), want[places], "float32")


# ---------------------------------------------------------------- generation
def same_tokens(got, tokens, margins, tie):
    for i, (g, t, m) in enumerate(zip(got, tokens, margins)):
        if g != t:
            assert m <= tie, (i, g, t, m)
            return                                  # the sequences part here
    assert len(got) == len(tokens)


@pytest.mark.parametrize("dtype, tie", [("bfloat16", 0.3), ("float32", 1e-4)])
@pytest.mark.parametrize("name", ["all three", "attention first"])
def test_greedy_generation_through_the_generators(name, dtype, tie, tmp_path):
    from megaqwen_b200.generators import MegakernelGenerator, MegakernelPrefillGenerator
    cfg = vm.MODELS[name]
    w = vm.weights(cfg)
    vm.save_checkpoint(cfg, w, tmp_path)
    prompt = vm.tokens(cfg, 37, 6)
    tokens, margins = ref.VunasunReference(cfg, w["tensors"]).greedy(prompt, 40)
    gen = MegakernelPrefillGenerator(str(tmp_path), max_seq_len=128, max_prefill_len=64, dtype=dtype)
    got = gen.generate_ids(prompt, 40)
    same_tokens(got, tokens, margins, tie)
    assert gen.generate_ids_fast(prompt, 40) == got                  # the device-resident chain
    one = MegakernelGenerator(str(tmp_path), max_seq_len=128, dtype=dtype)
    same_tokens(one.generate_ids(prompt, 40), tokens, margins, tie)   # the prompt token by token
    stop = got[7]
    assert gen.generate_ids(prompt, 40, stop_tokens=[stop]) == got[:got.index(stop)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["all three", "one key head"])
def test_chains_equal_single_steps(name, dtype):
    """Graph replay, eager chain, no programmatic launches, and the greedy loop with its EOS scan."""
    cfg, _, dec = model(name, dtype)
    prompt = vm.tokens(cfg, 20, 7)

    def start():
        dec.reset()
        return dec.prefill_step(prompt)
    t = first = start()
    steps = []
    for _ in range(140):
        t = dec.decode_step(t)
        steps.append(t)
    assert start() == first and dec.decode_steps(first, 140).tolist() == steps
    start()
    assert dec.decode_steps_cuda(first, 140).tolist() == steps
    start()
    assert dec.decode_steps_cuda_graph(first, 33).tolist() == steps[:33] and dec.decode_steps_cuda_graph(steps[32], 33).tolist() == steps[33:66]
    dec.use_pdl = False
    start()
    assert dec.decode_steps_cuda(first, 140).tolist() == steps
    dec.use_pdl = True
    start()
    out, n, reason = dec.decode_greedy_cuda(first, 60, [cfg["vocab"] + 1])
    assert (n, reason) == (60, 0) and out.tolist() == ([first] + steps)[:60]


def test_launch_counts():
    cfg, _, dec = model("all three", "bfloat16")
    before = dec.launches
    dec.decode_step(1)
    assert dec.launches - before == dec.step_launches == 5 + 5 + 3 + 1


def test_bad_tokens_and_the_end():
    cfg, _, dec = model("all three", "bfloat16", max_seq=20, max_prefill=20)
    dec.prefill_step(vm.tokens(cfg, 19))
    dec.decode_step(1)
    with pytest.raises(RuntimeError, match="max_seq_len"):
        dec.decode_step(1)
    dec.reset()
    with pytest.raises(RuntimeError, match="vocabulary"):
        dec.decode_step(cfg["vocab"])
    dec.reset()
    dec.decode_step(1)                              # the status word was cleared


def test_generate_command(tmp_path):
    cfg = vm.MODELS["all three"]
    w = vm.weights(cfg)
    vm.save_checkpoint(cfg, w, tmp_path)
    prompt = vm.tokens(cfg, 21, 10)
    tokens, margins = ref.VunasunReference(cfg, w["tensors"]).greedy(prompt, 12)
    res = subprocess.run([sys.executable, "-m", "megaqwen_b200.generate", str(tmp_path), "--ids", ",".join(map(str, prompt)), "--max-new", "12",
                          "--max-seq-len", "64", "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    same_tokens([int(t) for t in res.stdout.split()], tokens, margins, 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_program(dtype, tmp_path):
    cfg = vm.MODELS["all three"]
    w = vm.weights(cfg)
    vm.save_checkpoint(cfg, w, tmp_path)
    a, b = vm.tokens(cfg, 70, 8), vm.tokens(cfg, 12, 9)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:65], "want": [3, 49, 50, 64]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[65:69], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[69:], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "y", "tokens": b[1:], "want": [10]}], "end": ["y"]}]
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                          "--max-tokens", "70"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(5)]
    wa, wb = exact(cfg, w, a), exact(cfg, w, b)
    for step, rows in ((0, wa[[3, 49, 50, 64]]), (2, wa[[69]]), (3, wb[[0]]), (4, wb[[11]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(rows), -1))
        check(got, rows, dtype, f"step {step}")


# ---------------------------------------------------------------- recurrences alone
LENGTHS = [1, 2, 15, 16, 17, 127, 128, 129, 300]


def run_recurrence(lib, layer, q, k, v, decay_in, state, want, end, tols):
    """Both forms in both types.  tols: (32-bit, bf16 token by token, chunked)."""
    from megaqwen_b200 import _lib
    n, heads, dim, vdim = q.shape[0], layer.heads, layer.dim, layer.vdim
    scratch = torch.zeros(lib.mqh_recurrence_scratch_bytes(n, heads, dim, vdim), dtype=torch.uint8, device="cuda")
    gate = layer.gate_w_host if layer.kind == _lib.MQH_GLA else None
    for (code, dt, chunked), tol in zip(((_lib.MQH_F32, torch.float32, 0), (_lib.MQH_BF16, torch.bfloat16, 0), (_lib.MQH_BF16, torch.bfloat16, 1)), tols):
        a, b, c = (x.to("cuda", dt).contiguous() for x in (q, k, v))
        if gate is not None:
            g = gate.to("cuda", dt).contiguous()
            layer.gate_w = g.data_ptr()
        s, o, d = state.cuda(), torch.full((n, heads, vdim), float("nan"), device="cuda"), decay_in.cuda()
        _lib.check(lib.mqh_launch_recurrence(code, C.byref(layer), a.data_ptr(), b.data_ptr(), c.data_ptr(), d.data_ptr(), d.shape[1], s.data_ptr(),
                                             o.data_ptr(), n, chunked, scratch.data_ptr(), torch.cuda.current_stream().cuda_stream), "recurrence")
        eo = float((o.double().cpu() - want).abs().max() / want.abs().max())
        es = float((s.double().cpu() - end).abs().max() / end.abs().max())
        assert eo < tol and es < tol, (chunked, dt, eo, es)


@pytest.mark.parametrize("n", LENGTHS)
@pytest.mark.parametrize("heads, dim, vdim, rank, inv_tau", [(3, 32, 48, 16, 0.1), (1, 16, 16, 32, 1.0), (2, 144, 80, 16, 0.05), (2, 64, 128, 48, 0.02),
                                                             (1, 208, 64, 16, 4.0)])
def test_gla_kernels(lib, n, heads, dim, vdim, rank, inv_tau):
    """Decays between 1 and far below the smallest float, side by side."""
    from megaqwen_b200 import _lib
    g = torch.Generator().manual_seed(n * 31 + dim)
    q, k = (torch.randn(n, heads, dim, generator=g).bfloat16() for _ in range(2))
    v = torch.randn(n, heads, vdim, generator=g).bfloat16()
    u = torch.randn(n, rank, generator=g)
    a2, bias = (torch.randn(heads, rank, dim, generator=g) * rank ** -0.5).bfloat16(), torch.randn(heads, dim, generator=g) * 3
    bias[:, ::5] = 30.0
    bias[:, 1::7] = -60.0
    state = torch.randn(heads, dim, vdim, generator=g)
    z = torch.einsum("tr,hrd->thd", u.double(), a2.double()) + bias.double()
    want, end = vm.recurrence_exact(q, k, v, torch.nn.functional.logsigmoid(z) * inv_tau, state, 0.3)
    b = bias.cuda()
    layer = _lib.MqhLayer(kind=_lib.MQH_GLA, heads=heads, dim=dim, vdim=vdim, rank=rank, scale=0.3, inv_tau=inv_tau, gate_b=b.data_ptr())
    layer.gate_w_host = a2
    run_recurrence(lib, layer, q, k, v, u, state, want, end, (3e-6, 3e-6, 4e-5))


@pytest.mark.parametrize("n", LENGTHS)
@pytest.mark.parametrize("heads, groups, dim, vdim", [(4, 2, 32, 48), (3, 1, 16, 16), (2, 2, 144, 80), (6, 2, 128, 64), (2, 1, 64, 128)])
def test_mamba2_kernels(lib, n, heads, groups, dim, vdim):
    from megaqwen_b200 import _lib
    g = torch.Generator().manual_seed(n * 17 + dim)
    q, k = (torch.randn(n, groups, dim, generator=g).bfloat16() for _ in range(2))
    v = torch.randn(n, heads, vdim, generator=g).bfloat16()
    raw, bias, skip = torch.randn(n, heads + 3, generator=g), torch.randn(heads, generator=g), torch.randn(heads, generator=g)
    a_neg = -torch.tensor([0.02, 40.0, 1.0, 0.001, 8.0, 0.3][:heads])
    state = torch.randn(heads, dim, vdim, generator=g)
    dt = ref.softplus(raw[:, :heads].double() + bias.double())
    rep = heads // groups
    want, end = vm.recurrence_exact(q.repeat_interleave(rep, 1), dt[:, :, None] * k.double().repeat_interleave(rep, 1), v,
                                    (dt * a_neg.double())[:, :, None].expand(-1, -1, dim), state)
    want = want + skip.double()[None, :, None] * v.double()
    dev = [x.cuda() for x in (bias, a_neg, skip)]
    layer = _lib.MqhLayer(kind=_lib.MQH_MAMBA2, heads=heads, dim=dim, vdim=vdim, kv_heads=groups, dt_bias=dev[0].data_ptr(), a_neg=dev[1].data_ptr(),
                          skip=dev[2].data_ptr())
    run_recurrence(lib, layer, q, k, v, raw, state, want, end, (3e-6, 3e-6, 4e-5))


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 9, 64])
@pytest.mark.parametrize("pos0, cuts", [(0, [200]), (0, [1, 2, 3, 70, 1, 64, 59]), (7, [63, 65])])
def test_convolution_kernel(lib, taps, pos0, cuts):
    """Portions of a sequence against one pass over it; a state with rubbish where no position was."""
    from megaqwen_b200 import _lib
    ch, n = 48, sum(cuts)
    g = torch.Generator().manual_seed(taps)
    x, w, b = torch.randn(n, ch, generator=g).bfloat16(), torch.randn(taps, ch, generator=g), torch.randn(ch, generator=g)
    past = torch.randn(taps - 1, ch, generator=g).bfloat16()                        # inputs of positions pos0 - taps + 1 ..
    past[[i for i in range(taps - 1) if pos0 - taps + 1 + i < 0]] = 0
    y, _ = ref.causal_conv(x.double(), w.T.double(), b.double(), past.double())
    want = y * torch.sigmoid(y)
    for code, dt, tol in ((_lib.MQH_F32, torch.float32, 2e-6), (_lib.MQH_BF16, torch.bfloat16, 8e-3)):
        ring = torch.full((taps, ch), 1e4, dtype=dt)
        for i in range(taps - 1):
            if pos0 - taps + 1 + i >= 0:
                ring[(pos0 - taps + 1 + i) % taps] = past[i].to(dt)
        xd, wd, bd, ring = x.to("cuda", dt), w.cuda(), b.cuda(), ring.cuda()
        out, at = torch.full((n, ch), float("nan"), dtype=dt, device="cuda"), 0
        for m in cuts:
            _lib.check(lib.mqh_launch_conv(code, xd[at:].data_ptr(), wd.data_ptr(), bd.data_ptr(), ring.data_ptr(), out[at:].data_ptr(), m, pos0 + at,
                                           ch, taps, torch.cuda.current_stream().cuda_stream), "conv")
            at += m
        assert float((out.double().cpu() - want).abs().max() / want.abs().max()) < tol
        for t in range(max(0, n - taps + 1), n):                                    # what the next token will need
            assert torch.equal(ring[(pos0 + t) % taps].cpu(), x[t].to(dt))


def test_convolution_rejects_what_it_does_not_hold(lib):
    from megaqwen_b200 import _lib
    x = torch.zeros(1 << 14, device="cuda")
    p = x.data_ptr()
    assert lib.mqh_launch_conv(_lib.MQH_F32, p, p, p, p, p, 2, 0, 16, 65, None) == -3
    assert lib.mqh_launch_conv(_lib.MQH_F32, p, p, p, p, p, 2, 0, 20, 4, None) == -1


# ---------------------------------------------------------------- attention alone
@pytest.mark.parametrize("n, pos0", [(1, 0), (2, 127), (64, 64), (128, 0), (129, 128), (200, 57), (130, 255), (300, 3)])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, chunk", [(4, 2, 64, 64, 0), (3, 1, 32, 112, 50), (2, 2, 112, 48, 128), (4, 1, 128, 128, 129),
                                                               (2, 1, 16, 16, 7)])
def test_grouped_chunked_attention_kernels(lib, n, pos0, heads, kv_heads, dim, vdim, chunk):
    """Both kernels, heads in groups, a gate per head, keys aligned with the queries at the edges of chunks and tiles."""
    from megaqwen_b200 import _lib
    g = torch.Generator().manual_seed(n + dim)
    keys = pos0 + n
    q, k, v = (torch.randn(r, h, d, generator=g) for r, h, d in ((n, heads, dim), (keys, kv_heads, dim), (keys, kv_heads, vdim)))
    for j in {0, 63, 64, 127, 128, 255, keys - 1, chunk, chunk - 1, 2 * chunk, 2 * chunk - 1}:
        if 0 <= j < keys:
            k[j] = 2 * q.mean(0)[:kv_heads].sign()
    q, k, v = (x.bfloat16() for x in (q, k, v))
    gate = torch.randn(n, heads, generator=g) * 2
    scale = 0.8 * dim ** -0.5
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for use_gate in (True, False):
        want = vm.attention_exact(q, k, v, pos0, chunk, scale, gate if use_gate else None)
        for code, dt, tc, tol in ((_lib.MQH_F32, torch.float32, 0, 3e-6), (_lib.MQH_BF16, torch.bfloat16, 0, 8e-3), (_lib.MQH_BF16, torch.bfloat16, 1, 1e-2)):
            a, b, c = (x.to("cuda", dt).contiguous() for x in (q, k, v))
            out, gt = torch.full((n, heads, vdim), float("nan"), dtype=dt, device="cuda"), gate.cuda()
            _lib.check(lib.mqh_launch_causal_attention(code, a.data_ptr(), None, b.data_ptr(), None, 0, c.data_ptr(), None,
                                                       gt.data_ptr() if use_gate else None, out.data_ptr(), n, pos0, heads, kv_heads, dim, 0, vdim, chunk,
                                                       scale, tc, status.data_ptr(), torch.cuda.current_stream().cuda_stream), "attention")
            err = float((out.double().cpu() - want).abs().max() / want.abs().max())
            assert err < tol and int(status.item()) == 0, (use_gate, dt, tc, err)
