"""Layer-listed models on the GPU against the plain oracle: every mechanism through
the C ABI, whole models in both compute types, and the public entry points."""
import ctypes as C
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
from oracle import hybrid_reference as ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

# rms logit error over the rms of the logits, per position.  float32 differs from the exact oracle by summation
# order only; bfloat16 by the roundings of every product's operands.  Every mistake planted in
# test_hybrid_host.py moves the logits by more than 0.1.
TOL = {"float32": 1e-5, "bfloat16": 0.04}
DTYPES = ("bfloat16", "float32")


@pytest.fixture(scope="module", autouse=True)
def built():
    from megaqwen_b200.csrc.build import build
    build(name="hybrid")


@pytest.fixture(scope="module")
def lib(built):
    from megaqwen_b200 import _lib
    return _lib.hybrid_lib()


_cache = {}


def model(name, dtype, max_seq=400, max_prefill=300):
    """(config, oracle, decoder) of a named configuration; decoders are kept over the module."""
    from megaqwen_b200.hybrid import HybridDecoder
    cfg = hm.MODELS[name] if isinstance(name, str) else name
    key = (json.dumps(cfg, sort_keys=True), dtype, max_seq, max_prefill)
    if key not in _cache:
        w = hm.weights(cfg)
        _cache[key] = (cfg, ref.HybridReference(cfg, w["tensors"]), HybridDecoder(w, max_seq, max_prefill, dtype=dtype))
    cfg, oracle, dec = _cache[key]
    oracle.reset()
    dec.reset()
    return cfg, oracle, dec


_ref_logits = {}


def oracle_logits(cfg, oracle, ids):
    key = (json.dumps(cfg, sort_keys=True), tuple(ids))
    if key not in _ref_logits:
        oracle.reset()
        _ref_logits[key] = oracle.forward(ids)
    return _ref_logits[key]


def feed(dec, ids, portions):
    """Logits at every position, the tokens cut into the given portions (the rest one by one)."""
    out, at = [], 0
    for n in list(portions) + [1] * (len(ids) - sum(portions)):
        out.append(dec.step_logits(ids[at:at + n], list(range(n))).cpu())
        at += n
    assert at == len(ids) and dec.position() == len(ids)
    return torch.cat(out)


def check(got, want, dtype, what=""):
    e = hm.errors(got, want)
    print(f"{what} {dtype}: max {float(e.max()):.2e} mean {float(e.mean()):.2e}")
    assert float(e.max()) <= TOL[dtype], (what, dtype, float(e.max()), int(e.argmax()))


# ---------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(hm.MODELS))
def test_prompt_portions_and_decoding(name, dtype):
    """A whole prompt, portions of several sizes, and token by token from the first: every position."""
    cfg, oracle, dec = model(name, dtype)
    ids = hm.tokens(cfg, 150)
    want = oracle_logits(cfg, oracle, ids)
    for portions in ([150], [], [130], [2] * 20, [17, 2, 3, 50, 2, 64], [127, 2, 15]):
        dec.reset()
        check(feed(dec, ids, portions), want, dtype, f"{name} {portions[:6]}")


ALONE = {
    "lightning": ([(hm.lightning(3, 48, 32), None)], None, 3.0),
    "latent attention": ([(hm.latent(3, 48, 20, 32, 72, scale=0.3), None)], None, 3.0),
    "one head, one pair": ([(hm.latent(1, 16, 2, 16, 16, base=2.0, scale=0.5), None)], None, 3.0),
    "feed-forward beside it": ([(hm.lightning(1, 16, 16), 176)], None, 3.0),
    # weights below 1: every pass sends the roundings of the pass before through another norm
    "loop": ([(hm.lightning(2, 32, 48), None)], hm.loop(0, 1, 4), 0.5),
    "loop in the middle": ([(hm.lightning(2, 32, 48), None)] * 3, hm.loop(1, 2, 2), 0.5),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ALONE))
def test_each_mechanism_alone(name, dtype):
    """One mechanism per model, added at a weight that lets it carry the logits."""
    layers, lp, mult = ALONE[name]
    cfg, oracle, dec = model(hm.config(layers, width=80, vocab=211, loop=lp, mult=mult, embed_scale=0.5), dtype)
    ids = hm.tokens(cfg, 140, 11)
    want = oracle_logits(cfg, oracle, ids)
    for portions in ([140], [], [2, 63, 2, 66]):
        dec.reset()
        check(feed(dec, ids, portions), want, dtype, f"{name} {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 3.0, 30.0])
def test_sink_from_negligible_to_everything(sink, dtype):
    from megaqwen_b200.hybrid import HybridDecoder
    cfg = hm.config([(hm.latent(2, 32, 16, 48, 40, scale=0.3), None)], width=64, vocab=150, mult=3.0, embed_scale=0.5)
    w = hm.weights(cfg, 12)
    w["tensors"]["l0.mix.sink"] = torch.tensor([sink, sink / 2]).bfloat16()
    ids = hm.tokens(cfg, 70, 12)
    want = ref.HybridReference(cfg, w["tensors"]).forward(ids)
    dec = HybridDecoder(w, 80, 80, dtype=dtype)
    for portions in ([70], [3], [2, 40]):
        dec.reset()
        check(feed(dec, ids, portions), want, dtype, f"sink {sink} {portions}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_sequence_over_tile_and_chunk_edges(dtype):
    """Positions around 64-key splits, 128-key tiles and 128-token chunks, in prompts and decoded."""
    cfg = hm.config([hm.latent(3, 24, 8, 40, 48, scale=0.7), hm.lightning(4, 40, 24, decay=[0.2, 0.9, 0.99, 0.9995])], width=64, vocab=257, mult=0.8)
    cfg, oracle, dec = model(cfg, dtype)
    ids = hm.tokens(cfg, 390, 1)
    want = oracle_logits(cfg, oracle, ids)
    for portions in ([300, 86], [60], [128, 128, 120], [129, 127, 129], [256, 64]):
        dec.reset()
        check(feed(dec, ids, portions), want, dtype, f"{portions}")


def loud_key_model(kind):
    """One layer whose logits follow one far token: the token LOUD has an embedding that every other token's
    query matches, so that losing (or double counting) its key changes the logits by their own size."""
    if kind == "latent":
        cfg = hm.config([(hm.latent(2, 32, 4, 48, 40, scale=1.0, base=1e9), None)], width=64, vocab=97, mult=1.0)
    else:
        cfg = hm.config([(hm.lightning(2, 24, 48, decay=[1.0, 0.9999]), None)], width=64, vocab=97, mult=1.0)
    w = hm.weights(cfg, 5)
    t = w["tensors"]
    loud = 96
    t["embed"] = t["embed"].clone()
    t["embed"][:, 0] = 0.2
    t["embed"][loud, 0] = 0.0
    t["embed"][loud, 1] = 1.6                         # the others have nothing there
    t["embed"][:loud, 1] = 0.0
    q, k = t["l0.mix.q"].clone().float(), (t["l0.mix.uk"] if kind == "latent" else t["l0.mix.k"]).clone().float()
    if kind == "latent":                              # query dimension 0 <- feature 0, latent 0 <- feature 1, key dimension 0 <- latent 0
        d = t["l0.mix.dkv"].clone().float()
        d[0], d[1:, 1] = 0, 0
        d[0, 1] = 4.0
        for h in range(2):
            q[h * 36], k[h * 32] = 0, 0
            q[h * 36, 0] = 2.0
            k[h * 32, 0] = 4.0
        t["l0.mix.dkv"], t["l0.mix.uk"] = d.bfloat16(), k.bfloat16()
    else:
        for h in range(2):
            q[h * 24], k[h * 24] = 0, 0
            q[h * 24, 0], k[h * 24, 1] = 4.0, 24.0
        t["l0.mix.k"] = k.bfloat16()
    t["l0.mix.q"] = q.bfloat16()
    return cfg, w, loud


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["latent", "lightning"])
@pytest.mark.parametrize("place", [0, 1, 63, 64, 127, 128, 191])
def test_one_loud_key_far_away(kind, place, dtype):
    """The loud token sits at tile, split and chunk edges and is read hundreds of tokens later."""
    from megaqwen_b200.hybrid import HybridDecoder
    cfg, w, loud = loud_key_model(kind)
    key = ("loud", kind, dtype)
    if key not in _cache:
        _cache[key] = HybridDecoder(w, 330, 330, dtype=dtype)
    dec = _cache[key]
    ids = [t % 96 for t in hm.tokens(cfg, 320, 2)]
    quiet = list(ids)
    ids[place] = loud
    oracle = ref.HybridReference(cfg, w["tensors"])
    tail = [0, 1, 2, place, place + 1, 62, 63, 64, 65, 126, 127, 128, 129, 254, 255, 256, 257, 258, 300, 319]
    tail = sorted({i for i in tail if i < 320})
    want = oracle_logits(dict(cfg, kind=kind), oracle, ids)
    oracle.reset()
    without = oracle_logits(dict(cfg, kind=kind), oracle, quiet)
    assert float(hm.errors(without[300:], want[300:]).min()) > 0.3          # the far key decides
    dec.reset()
    check(dec.step_logits(ids, tail).cpu(), want[tail], dtype, f"{kind} prompt {place}")
    dec.reset()
    check(feed(dec, ids, [max(place, 2), 200 - max(place, 2) + 50]), want, dtype, f"{kind} decoded {place}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_that_is_used_again(dtype):
    """A sequence after a longer one in the same decoder, after a reset: nothing of it is left, also beyond the end."""
    cfg, oracle, dec = model("mixed", dtype)
    a, b = hm.tokens(cfg, 140, 3), hm.tokens(cfg, 40, 4)
    feed(dec, a, [140])
    dec.reset()
    assert dec.position() == 0
    first = feed(dec, b, [30])
    check(first, oracle_logits(cfg, oracle, b), dtype)
    dec.reset()
    again = feed(dec, b, [30])
    assert torch.equal(first, again)                # same cut, same bits
    for buf in dec.state.buffers:                   # whatever a cache holds beyond the position is never read
        if buf.numel() and not dec.state.recurrent[[x is buf for x in dec.state.buffers].index(True)]:
            buf.view(torch.bfloat16 if dtype == "bfloat16" else torch.float32).fill_(float("nan"))
    dec.reset()
    assert torch.equal(feed(dec, b, [30]), first)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_snapshot_continues_two_ways(dtype):
    cfg, oracle, dec = model("mixed", dtype)
    ids = hm.tokens(cfg, 60, 5)
    dec.step_logits(ids[:50], [])
    saved, pos = dec.state.snapshot(), dec.position()
    one = dec.step_logits(ids[50:], list(range(10))).cpu()
    dec.state.restore(saved)
    dec.position_ = pos
    two = dec.step_logits(ids[50:], list(range(10))).cpu()
    assert torch.equal(one, two)
    check(one, oracle_logits(cfg, oracle, ids)[50:], dtype)


def test_prompt_longer_than_one_prefill_call():
    cfg, oracle, dec = model("mixed", "float32", max_seq=170, max_prefill=48)
    ids = hm.tokens(cfg, 150)
    want = oracle_logits(cfg, oracle, ids)
    places = [0, 47, 48, 49, 95, 96, 149]
    check(dec.step_logits(ids, places).cpu(), want[places], "float32")
    dec.reset()
    with pytest.raises(RuntimeError, match="Prefill sequence length exceeds maximum"):
        dec.prefill_step(ids)
    assert dec.step_logits(ids[:5], [4, 0]).shape == (2, cfg["vocab"])      # in the order they are asked for
    with pytest.raises(ValueError, match="outside"):
        dec.step_logits(ids[:5], [5])


def test_sequence_end_and_bad_tokens():
    cfg, _, dec = model("mixed", "bfloat16", max_seq=20, max_prefill=20)
    dec.prefill_step(hm.tokens(cfg, 18))
    dec.decode_step(1)
    dec.decode_step(1)
    with pytest.raises(RuntimeError, match="max_seq_len"):
        dec.decode_step(1)
    with pytest.raises(RuntimeError, match="exceeds maximum"):
        dec.prefill_append([1, 2])
    dec.reset()
    with pytest.raises(RuntimeError, match="vocabulary"):
        dec.prefill_step([3, cfg["vocab"]])
    dec.reset()
    with pytest.raises(RuntimeError, match="vocabulary"):
        dec.decode_step(-1)
    dec.reset()
    dec.decode_step(1)                              # the status word was cleared


# ---------------------------------------------------------------- generation
def same_tokens(got, tokens, margins, tie):
    for i, (g, t, m) in enumerate(zip(got, tokens, margins)):
        if g != t:
            assert m <= tie, (i, g, t, m)
            return                                  # the sequences part here
    assert len(got) == len(tokens)


@pytest.mark.parametrize("dtype, tie", [("bfloat16", 0.3), ("float32", 1e-4)])
@pytest.mark.parametrize("name", ["mixed", "latent first, loop to the end"])
def test_greedy_generation_through_the_generators(name, dtype, tie, tmp_path):
    from megaqwen_b200.generators import MegakernelGenerator, MegakernelPrefillGenerator
    cfg = hm.MODELS[name]
    w = hm.weights(cfg)
    hm.save_checkpoint(cfg, w, tmp_path)
    prompt = hm.tokens(cfg, 37, 6)
    tokens, margins = ref.HybridReference(cfg, w["tensors"]).greedy(prompt, 40)
    gen = MegakernelPrefillGenerator(str(tmp_path), max_seq_len=128, max_prefill_len=64, dtype=dtype)
    got = gen.generate_ids(prompt, 40)
    same_tokens(got, tokens, margins, tie)
    assert gen.generate_ids_fast(prompt, 40) == got                  # the device-resident chain
    one = MegakernelGenerator(str(tmp_path), max_seq_len=128, dtype=dtype)
    same_tokens(one.generate_ids(prompt, 40), tokens, margins, tie)   # the prompt token by token
    stop = got[7]
    assert gen.generate_ids(prompt, 40, stop_tokens=[stop]) == got[:got.index(stop)]


@pytest.mark.parametrize("dtype", DTYPES)
def test_chains_equal_single_steps(dtype):
    """Graph replay, eager chain, no programmatic launches, and the greedy loop with its EOS scan."""
    cfg, _, dec = model("mixed", dtype)
    prompt = hm.tokens(cfg, 20, 7)

    def start():
        dec.reset()
        return dec.prefill_step(prompt)
    t = first = start()
    steps = []
    for _ in range(70):
        t = dec.decode_step(t)
        steps.append(t)
    assert start() == first and dec.decode_steps(first, 70).tolist() == steps
    start()
    assert dec.decode_steps_cuda(first, 70).tolist() == steps
    start()
    assert dec.decode_steps_cuda_graph(first, 33).tolist() == steps[:33] and dec.decode_steps_cuda_graph(steps[32], 33).tolist() == steps[33:66]
    dec.use_pdl = False
    start()
    assert dec.decode_steps_cuda(first, 70).tolist() == steps
    dec.use_pdl = True
    start()
    out, n, reason = dec.decode_greedy_cuda(first, 60, [cfg["vocab"] + 1])
    assert (n, reason) == (60, 0) and out.tolist() == ([first] + steps)[:60]


def test_launch_counts():
    cfg, _, dec = model("mixed", "bfloat16")
    before = dec.launches
    dec.decode_step(1)
    assert dec.launches - before == dec.step_launches == 3 + 3 * (3 + 5) + 5 + 3 + 1


# ---------------------------------------------------------------- lightning attention alone
def lightning_exact(q, k, v, decay, state):
    S, out = state.double().clone(), []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t].double()[:, :, None] * v[t].double()[:, None, :]
        out.append((S * q[t].double()[:, :, None]).sum(1))
    return torch.stack(out), S


@pytest.mark.parametrize("n", [1, 2, 15, 16, 127, 128, 129, 256, 300])
@pytest.mark.parametrize("heads, dim, vdim", [(3, 32, 48), (1, 16, 16), (2, 144, 80), (2, 64, 128), (1, 256, 64)])
def test_lightning_kernels(lib, n, heads, dim, vdim):
    from megaqwen_b200 import _lib
    from megaqwen_b200.hybrid import decay_powers
    g = torch.Generator().manual_seed(n * 31 + dim)
    q, k = (torch.randn(n, heads, dim, generator=g).bfloat16() for _ in range(2))
    v = torch.randn(n, heads, vdim, generator=g).bfloat16()
    decay = torch.tensor([0.3, 0.97, 1.0][-heads:], dtype=torch.float64)
    state = torch.randn(heads, dim, vdim, generator=g)
    want, end = lightning_exact(q, k, v, decay, state)
    pw = decay_powers(decay.tolist(), _lib.MQH_CHUNK + 1).cuda()
    scratch = torch.zeros(lib.mqh_recurrence_scratch_bytes(n, heads, dim, vdim), dtype=torch.uint8, device="cuda")
    for code, dt, chunked, tol in ((_lib.MQH_F32, torch.float32, 0, 2e-6), (_lib.MQH_BF16, torch.bfloat16, 0, 2e-6), (_lib.MQH_BF16, torch.bfloat16, 1, 3e-5)):
        a, b, c = (x.to("cuda", dt).contiguous() for x in (q, k, v))
        s, o = state.cuda(), torch.full((n, heads, vdim), float("nan"), device="cuda")
        _lib.check(lib.mqh_launch_lightning(code, a.data_ptr(), b.data_ptr(), c.data_ptr(), pw.data_ptr(), s.data_ptr(), o.data_ptr(), n, heads, dim,
                                            vdim, chunked, scratch.data_ptr(), torch.cuda.current_stream().cuda_stream), "lightning")
        eo = float((o.double().cpu() - want).abs().max() / want.abs().max())
        es = float((s.double().cpu() - end).abs().max() / end.abs().max())
        assert eo < tol and es < tol, (chunked, dt, eo, es)


# ---------------------------------------------------------------- causal attention alone
@pytest.mark.parametrize("n, pos0", [(1, 0), (2, 127), (64, 64), (128, 0), (129, 128), (200, 57), (130, 255)])
@pytest.mark.parametrize("heads, dim, rot, vdim", [(3, 64, 16, 64), (2, 32, 32, 112), (2, 112, 48, 48), (1, 128, 64, 128)])
def test_causal_attention_kernels(lib, n, pos0, heads, dim, rot, vdim):
    """Both kernels, with a sink and without, one head's query aligned with one key that sits at an edge."""
    from megaqwen_b200 import _lib
    g = torch.Generator().manual_seed(n + dim)
    keys, ld = pos0 + n, rot + 32
    q, qr = torch.randn(n, heads, dim, generator=g), torch.randn(n, heads, rot, generator=g)
    k, kr, v = torch.randn(keys, heads, dim, generator=g), torch.randn(keys, ld, generator=g), torch.randn(keys, heads, vdim, generator=g)
    q, qr, k, kr, v = (x.bfloat16() for x in (q, qr, k, kr, v))
    loud = [i for i in (0, 63, 64, 127, 128, 255, 256, keys - 1) if i < keys]
    for h in range(heads):
        k[loud[h % len(loud)], h] = 3 * q[:, h].mean(0).sign()
    sink = torch.tensor([2.0, -3.0, 9.0][:heads])
    scale = 0.8 * (dim + rot) ** -0.5
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for use_sink in (True, False):
        s = (torch.einsum("thd,khd->htk", q.double(), k.double()) + torch.einsum("thr,kr->htk", qr.double(), kr[:, :rot].double())) * scale
        mask = torch.arange(keys)[None, :] > (pos0 + torch.arange(n))[:, None]
        s = s.masked_fill(mask[None], -math.inf)
        m = s.max(-1, keepdim=True).values
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(sink.double()[:, None, None] - m) if use_sink else 0)
        want = torch.einsum("htk,khv->thv", e / den, v.double())
        for code, dt, tc, tol in ((_lib.MQH_F32, torch.float32, 0, 3e-6), (_lib.MQH_BF16, torch.bfloat16, 0, 8e-3), (_lib.MQH_BF16, torch.bfloat16, 1, 1e-2)):
            dev = [x.to("cuda", dt).contiguous() for x in (q, qr, k, kr, v)]
            out = torch.full((n, heads, vdim), float("nan"), dtype=dt, device="cuda")
            sk = sink.cuda()
            _lib.check(lib.mqh_launch_causal_attention(code, *(x.data_ptr() for x in dev[:4]), ld, dev[4].data_ptr(), sk.data_ptr() if use_sink else None,
                                                       None, out.data_ptr(), n, pos0, heads, heads, dim, rot, vdim, 0, scale, tc, status.data_ptr(),
                                                       torch.cuda.current_stream().cuda_stream), "causal")
            err = float((out.double().cpu() - want).abs().max() / want.abs().max())
            assert err < tol and int(status.item()) == 0, (use_sink, dt, tc, err)


def test_causal_attention_rejects_what_it_does_not_hold(lib):
    from megaqwen_b200 import _lib
    x = torch.zeros(1 << 16, dtype=torch.bfloat16, device="cuda")
    p, st = x.data_ptr(), torch.zeros(1, dtype=torch.int32, device="cuda").data_ptr()

    def call(dtype, dim, rot, vdim, tc):
        return lib.mqh_launch_causal_attention(dtype, p, p, p, p, rot, p, None, None, p, 2, 0, 1, 1, dim, rot, vdim, 0, 1.0, tc, st, None)
    assert call(_lib.MQH_BF16, 144, 16, 16, 1) == -3 and call(_lib.MQH_F32, 16, 16, 16, 1) == -3
    assert call(_lib.MQH_BF16, 20, 16, 16, 0) == -1


def test_generate_command(tmp_path):
    cfg = hm.MODELS["mixed"]
    w = hm.weights(cfg)
    hm.save_checkpoint(cfg, w, tmp_path)
    prompt = hm.tokens(cfg, 21, 10)
    tokens, margins = ref.HybridReference(cfg, w["tensors"]).greedy(prompt, 12)
    res = subprocess.run([sys.executable, "-m", "megaqwen_b200.generate", str(tmp_path), "--ids", ",".join(map(str, prompt)), "--max-new", "12",
                          "--max-seq-len", "64", "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    same_tokens([int(t) for t in res.stdout.split()], tokens, margins, 1e-4)


# ---------------------------------------------------------------- trace runner
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_program(dtype, tmp_path):
    cfg = hm.MODELS["mixed"]
    w = hm.weights(cfg)
    hm.save_checkpoint(cfg, w, tmp_path)
    a, b = hm.tokens(cfg, 30, 8), hm.tokens(cfg, 12, 9)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:25], "want": [3, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[25:29], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[29:], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "y", "tokens": b[1:], "want": [10]}], "end": ["y"]}]
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                          "--max-tokens", "30"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not os.path.exists(tmp_path / "1.f32")
    m = ref.HybridReference(cfg, w["tensors"])
    wa = m.forward(a)
    m.reset()
    wb = m.forward(b)
    for step, rows in ((0, wa[[3, 24]]), (2, wa[[29]]), (3, wb[[0]]), (4, wb[[11]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(rows), -1))
        check(got, rows, dtype, f"step {step}")
