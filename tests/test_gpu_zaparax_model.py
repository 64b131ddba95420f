"""The Zaparax decoder end to end on the GPU: ZaparaxForCausalLM through HybridBatchEngine / HybridCacheManager (the engine a user
generates with, and the one bin/trace_run drives) against oracle/zaparax_oracle.py's float64 forward of the same seeded weights. Whole
prompts, portions down to two tokens, token-by-token decoding (also through the captured CUDA graph), mixed batches of unequal requests,
pages and state slots that are freed and handed out again, window edges in prompts and in decoding, a far token, long decoding across page
borders, other sizes, loops, both forms of the experts, greedy generation, the replayer's command line. float32 models are held to 2e-4 of
the largest logit at every position. bfloat16 ones are held to three
times what rounding alone does: the oracle is run a second time with every product's input rounded to bf16, and its largest difference sets
the limit. A router's close call may fall the other way under rounding and then moves its position by far more, so the bfloat16 models here
get corrections that lie further apart than scores can (every token chooses the same experts; the weights stay the tokens' own); the choice
itself is tested in float32 and, on inputs without rounding, in both dtypes among the mechanisms."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import zaparax_oracle as O
from tests import hybrid_util as HU
from tests import zaparax_util as U

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
FP32_TOL = 2e-4


class Ref:
    """The oracle's logits of one token sequence and, for bfloat16 models, the limit that rounding sets. `drawn`: a configuration nobody
    chose, which may amplify roundings (a norm over a few columns that cancel): its float32 limit grows with what rounding every product's
    input to float32, one of many roundings, does in the oracle."""

    def __init__(self, cfg, W, toks, dtype, fp32_tol=FP32_TOL, drawn=False):
        self.logits = O.forward(cfg, W, toks)
        self.tol = fp32_tol
        if drawn and dtype == torch.float32:
            self.tol = max(fp32_tol, 60.0 * HU.rel_err(O.forward(cfg, W, toks, rnd=lambda x: x.float().double()), self.logits))
        if dtype == torch.bfloat16:
            self.tol = max(2e-2, 3.0 * HU.rel_err(O.forward(cfg, W, toks, rnd=O.to_bf16), self.logits))


def _check(got, ref, what="", pos0=0):
    """got: logits of positions pos0 .. of the sequence ref describes."""
    e = float((got.double() - ref.logits[pos0:pos0 + got.shape[0]]).abs().max() / ref.logits.abs().max())
    assert e < ref.tol, (what, e, ref.tol)


@pytest.mark.parametrize("cfg_name", ["small", "aligned", "many_heads"])
def test_residual_stream_layer_run_by_layer_run(cfg_name):
    cfg = {"small": U.small_config, "aligned": U.aligned_config, "many_heads": U.many_heads_config}[cfg_name]()
    model, W = U.build(cfg)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(23, cfg["vocab"], 1)
    ref_res = []
    ref = O.forward(cfg, W, toks, residuals=ref_res)
    model.debug_residuals = []
    got = eng.feed([("a", toks, list(range(len(toks))))]).float().cpu()
    assert len(model.debug_residuals) == len(ref_res) == len(model.runs)
    for i, (x, r) in enumerate(zip(model.debug_residuals, ref_res)):
        assert HU.rel_err(x.cpu(), r) < 1e-4, f"layer run {i}"
    model.debug_residuals = None
    assert HU.rel_err(got, ref) < FP32_TOL


@pytest.mark.parametrize("dtype,cfg_name", [(torch.float32, "small"), (torch.float32, "aligned"), (torch.bfloat16, "aligned")])
@pytest.mark.parametrize("cuts", [[44], [2, 2, 2, 30], [1], [17, 3, 5], [33]])
def test_prompt_portions_and_decoding_agree_with_the_oracle(dtype, cfg_name, cuts):
    cfg = U.small_config() if cfg_name == "small" else U.aligned_config()
    model, W = U.build(cfg, dtype=dtype)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(44, cfg["vocab"], 2)
    _check(HU.feed_in_portions(eng, "s", toks, cuts), Ref(cfg, W, toks, dtype))


def test_cutting_changes_nothing_beyond_rounding():
    cfg = U.small_config()
    model, _ = U.build(cfg)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(48, cfg["vocab"], 3)
    whole = HU.feed_in_portions(eng, "w", toks, [48])
    for cuts in ([2] * 24, [1], [5, 9, 2, 20], [47]):
        eng.release(["p"])
        assert HU.rel_err(HU.feed_in_portions(eng, "p", toks, cuts), whole) < 5e-5, cuts


@pytest.mark.parametrize("dtype,cfg_name", [(torch.float32, "small"), (torch.bfloat16, "aligned")])
def test_mixed_batch_equals_each_request_alone(dtype, cfg_name):
    cfg = U.small_config() if cfg_name == "small" else U.aligned_config()
    model, W = U.build(cfg, dtype=dtype)
    eng, _ = HU.engine_for(model, max_seqs=1, max_tokens=16)     # pools and slots must grow under the batch
    lens = {"a": 31, "b": 3, "c": 12, "d": 1}
    toks = {k: HU.tokens(n + 6, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    ref = {k: Ref(cfg, W, t, dtype) for k, t in toks.items()}
    got = {k: [] for k in lens}
    # prompts of unequal length in one step, then decode together; "b" and "d" end early and drop out
    out = eng.feed([(k, toks[k][:n], list(range(n))) for k, n in lens.items()]).float().cpu()
    at = 0
    for k, n in lens.items():
        got[k].append(out[at:at + n])
        at += n
    live = list(lens)
    for step in range(6):
        if step == 3:
            eng.release(["b", "d"])
            live = ["a", "c"]
        out = eng.feed([(k, [toks[k][lens[k] + step]], [0]) for k in live]).float().cpu()
        for i, k in enumerate(live):
            got[k].append(out[i:i + 1])
    for k in lens:
        _check(torch.cat(got[k]), ref[k], k)


def test_prompts_beside_decoding_requests():
    """A step that holds a whole prompt, a portion and single tokens at once."""
    cfg = U.small_config()
    model, W = U.build(cfg)
    eng, _ = HU.engine_for(model)
    a, b, c = (HU.tokens(n, cfg["vocab"], s) for n, s in ((30, 16), (26, 17), (19, 18)))
    eng.feed([("a", a[:25], [])])
    eng.feed([("b", b[:9], []), ("a", a[25:26], [])])
    out = eng.feed([("a", a[26:27], [0]), ("c", c, list(range(19))), ("b", b[9:26], list(range(17)))]).float().cpu()
    _check(out[:1], Ref(cfg, W, a, torch.float32), "a", pos0=26)
    _check(out[1:20], Ref(cfg, W, c, torch.float32), "c")
    _check(out[20:], Ref(cfg, W, b, torch.float32), "b", pos0=9)


def test_pages_and_slots_freed_and_used_again():
    cfg = U.small_config()
    model, W = U.build(cfg)
    eng, mgr = HU.engine_for(model, max_tokens=64, block_size=4, max_seqs=2)
    a, b, c = (HU.tokens(n, cfg["vocab"], s) for n, s in ((37, 5), (29, 6), (41, 7)))
    eng.feed([("a", a, []), ("b", b, [])])
    used, slot = set(eng.active["a"].blocks), eng.active["a"].slot
    eng.release(["a"])
    # "c" gets a's pages and state slot back (the slot still holds a's recurrent state and convolution inputs) while "b" keeps decoding
    got_c = eng.feed([("c", c[:30], list(range(30))), ("b", [3], [])]).float().cpu()
    assert used & set(eng.active["c"].blocks) and eng.active["c"].slot == slot
    got_c = torch.cat([got_c, HU.feed_in_portions(eng, "c", c[30:], [4])])
    assert HU.rel_err(got_c, O.forward(cfg, W, c)) < FP32_TOL
    # a sequence of single tokens from its very first one in a used slot
    eng.release(["c"])
    got = HU.feed_in_portions(eng, "d", c[:9], [1])
    assert HU.rel_err(got, O.forward(cfg, W, c[:9])) < FP32_TOL


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window,block,heads", [(5, 4, 4), (16, 16, 4), (17, 4, 16), (1, 4, 4)])
def test_window_edge_inside_and_outside(window, block, heads, decode):
    """One attention layer without the hashed pairs (a pair would carry a token one position further): the last position's logits depend on
    the token window - 1 before it and not on the one before that, in a prompt and when the last tokens are decoded one by one, with the
    edge at and off a page border."""
    cfg = U.config([U.layer("attention", U.attention(heads=heads, kv_heads=2, window=window, q_temp=(0.4, 2)), None)], bigram=None)
    model, W = U.build(cfg)
    n = 3 * window + 8
    base = HU.tokens(n, cfg["vocab"], 11)

    def last_logits(toks):
        eng, _ = HU.engine_for(model, block_size=block)
        return HU.feed_in_portions(eng, "s", toks, [n - window - 2 if decode else n])[-1]

    ref = last_logits(base)
    assert HU.rel_err(ref[None], O.forward(cfg, W, base)[-1:]) < FP32_TOL
    outside, inside = list(base), list(base)
    outside[n - 1 - window] = (base[n - 1 - window] + 1) % cfg["vocab"]
    inside[n - window] = (base[n - window] + 1) % cfg["vocab"]
    assert torch.equal(last_logits(outside), ref)
    assert HU.rel_err(last_logits(inside)[None], ref[None]) > 1e-4


def test_the_previous_token_is_part_of_a_sequences_state():
    """No layers at all: logits depend on the token and the one before it, across portions, single tokens and a slot used before."""
    cfg = U.config([])
    model, W = U.build(cfg)
    toks = HU.tokens(12, cfg["vocab"], 50)
    ref = O.forward(cfg, W, toks)
    eng, _ = HU.engine_for(model, max_seqs=1)
    for cuts in ([12], [5, 1, 1, 3], [1], [2] * 6):
        assert HU.rel_err(HU.feed_in_portions(eng, "s", toks, cuts), ref) < FP32_TOL, cuts
        eng.release(["s"])
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    assert HU.rel_err(O.forward(cfg, W, other)[1:2], ref[1:2]) > 1e-2 and HU.rel_err(O.forward(cfg, W, other)[2:], ref[2:]) == 0.0


def test_a_key_far_back_reaches_through_every_mixer():
    """A change of the very first token of a long prompt must show 300 positions later through the attention without a window and
    through the recurrent states, in a whole prompt and in decoding alike."""
    cfg = U.small_config()
    model, W = U.build(cfg)
    toks = HU.tokens(300, cfg["vocab"], 21)
    ref = Ref(cfg, W, toks, torch.float32, fp32_tol=4e-4)
    for cuts in ([300], [280]):
        eng, _ = HU.engine_for(model, block_size=16, max_tokens=512)
        _check(HU.feed_in_portions(eng, "s", toks, cuts)[-20:], ref, str(cuts), pos0=280)
    changed = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    assert HU.rel_err(O.forward(cfg, W, changed)[-1:], ref.logits[-1:]) > 1e-5


def test_first_tokens_of_a_sequence():
    cfg = U.small_config()
    model, W = U.build(cfg)
    toks = HU.tokens(6, cfg["vocab"], 13)
    ref = O.forward(cfg, W, toks)
    for cuts in ([1], [2], [1, 2], [6], [3, 3]):
        eng, _ = HU.engine_for(model)
        assert HU.rel_err(HU.feed_in_portions(eng, "s", toks, cuts), ref) < FP32_TOL, cuts


@pytest.mark.parametrize("dtype,cfg_name", [(torch.float32, "small"), (torch.bfloat16, "aligned"), (torch.float32, "many_heads")])
def test_long_decoding_through_the_captured_step(dtype, cfg_name):
    """150 single-token steps (several windows, many page borders); from the third step of a shape on they replay a CUDA graph."""
    cfg = {"small": U.small_config, "aligned": U.aligned_config, "many_heads": U.many_heads_config}[cfg_name]()
    model, W = U.build(cfg, dtype=dtype)
    eng, _ = HU.engine_for(model, block_size=8, use_graph=True)
    toks = HU.tokens(160, cfg["vocab"], 14)
    got = HU.feed_in_portions(eng, "s", toks, [10])
    assert eng._graphs, "single-token steps were not captured"
    _check(got, Ref(cfg, W, toks, dtype))


def test_values_that_are_one_or_equal():
    """One head everywhere, window 1 (a token sees only itself) and a window longer than the sequence, one tap, state == vdim, one group,
    one norm group, one bucket, one expert that is always chosen, width == ff, scale 1, a loop of one pass over one layer."""
    cfg = U.config([U.layer("attention", U.attention(heads=1, kv_heads=1, dim=8, vdim=8, window=1, scale=1.0, softcap=1.0, q_temp=(1.0, 1)), U.moe(ff=16, experts=1, top=1, identity=0, shared=16)),
                    U.layer("mamba2", U.mamba(heads=1, vdim=8, state=8, groups=1, conv=1, norm_groups=1), U.moe(ff=16, experts=1, top=2, identity=1, shared=None)),
                    U.layer("attention", U.attention(heads=2, kv_heads=2, dim=8, vdim=8, window=1000), None),
                    U.layer("mamba2", U.mamba(heads=3, vdim=8, state=8, groups=3, conv=2, norm_groups=24), None)], width=16, vocab=16, loop=(3, 4, 1), bigram=(1, 1, 1), scale=1.0)
    model, W = U.build(cfg)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(30, cfg["vocab"], 15)
    assert HU.rel_err(HU.feed_in_portions(eng, "s", toks, [9, 2]), O.forward(cfg, W, toks)) < FP32_TOL


@pytest.mark.parametrize("dtype,cfg_name", [(torch.float32, "small"), (torch.bfloat16, "aligned")])
def test_experts_sorted_by_row(dtype, cfg_name):
    """Prompt steps whose experts multiply only the rows routed to them, then single tokens (all experts at once)."""
    cfg = U.small_config() if cfg_name == "small" else U.aligned_config()
    model, W = U.build(cfg, dtype=dtype, sorted_min_rows=2, force_sorted=True)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(40, cfg["vocab"], 51)
    _check(HU.feed_in_portions(eng, "s", toks, [19, 2, 14]), Ref(cfg, W, toks, dtype))


@pytest.mark.parametrize("kind", ["attention", "mamba2"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_models_of_one_mixer_and_an_odd_width(kind, dtype):
    """Only pages or only state slots to manage; rows that no 16-byte access fits."""
    cfg = U.config([U.layer(kind, U.attention() if kind == "attention" else U.mamba(), f) for f in (U.moe(), None)], width=37, vocab=61, loop=(0, 1, 2))
    model, W = U.build(cfg, dtype=dtype)
    eng, _ = HU.engine_for(model)
    toks = HU.tokens(40, cfg["vocab"], 52)
    _check(HU.feed_in_portions(eng, "s", toks, [17, 2, 9]), Ref(cfg, W, toks, dtype))


@pytest.mark.parametrize("loop", [None, (0, 2, 1), (0, 2, 2), (1, 2, 3), (0, 1, 2)])
def test_loops(loop):
    """No loop, a loop over all layers (one pass is no loop), over the last, over the first; a pass reads its own cache, so the passes of a
    decoded token differ from the prompt's only by rounding."""
    cfg = U.config([U.layer("attention", U.attention(), U.moe()), U.layer("mamba2", U.mamba(), None)], loop=loop)
    model, W = U.build(cfg)
    toks = HU.tokens(25, cfg["vocab"], 19)
    ref = O.forward(cfg, W, toks)
    for cuts in ([25], [11, 2, 1]):
        eng, _ = HU.engine_for(model)
        assert HU.rel_err(HU.feed_in_portions(eng, "s", toks, cuts), ref) < FP32_TOL
    if loop == (0, 2, 1):
        assert torch.equal(O.forward({**cfg, "loop": None}, W, toks), ref)
    elif loop is not None:
        assert HU.rel_err(O.forward({**cfg, "loop": None}, W, toks), ref) > 1e-2


@pytest.mark.parametrize("seed", range(16))
def test_configurations_drawn_at_random(seed):
    """Other layer orders, loops, head counts, channel counts, windows, constants: a prompt with decoding, portions, and two unequal
    requests in one batch, in fp32 and in bf16 (tensor-core products wherever the drawn sizes allow them) against the oracle."""
    for dtype in (torch.float32, torch.bfloat16):
        cfg = U.random_config(seed)
        toks, other = HU.tokens(70, cfg["vocab"], 40 + seed), HU.tokens(21, cfg["vocab"], 80 + seed)
        model, W = U.build(cfg, dtype=dtype, seed=seed)
        ref, ref_o = Ref(cfg, W, toks, dtype, drawn=True), Ref(cfg, W, other, dtype, drawn=True)
        eng, _ = HU.engine_for(model, block_size=16)
        _check(HU.feed_in_portions(eng, "w", toks, [40]), ref, "prompt + decoding")
        _check(HU.feed_in_portions(eng, "p", toks, [19, 2, 30, 7]), ref, "portions")
        out = eng.feed([("a", toks[:50], list(range(50))), ("b", other[:9], list(range(9)))]).float().cpu()
        _check(out[:50], ref, "batch a")
        _check(out[50:], ref_o, "batch b")
        out = eng.feed([("a", toks[50:51], [0]), ("b", other[9:10], [0])]).float().cpu()
        _check(out[:1], ref, "batch a decoded", pos0=50)
        _check(out[1:], ref_o, "batch b decoded", pos0=9)


def test_greedy_generation_through_the_engine():
    cfg = U.small_config()
    model, W = U.build(cfg)
    eng, _ = HU.engine_for(model, max_seqs=3)
    prompts = [HU.tokens(n, cfg["vocab"], 20 + n) for n in (9, 2, 17)]
    outs = eng.generate(prompts, max_new_tokens=12)
    for p, o in zip(prompts, outs):
        assert o[:len(p)] == p and len(o) == len(p) + 12
        # every generated token is the oracle's argmax given the tokens before it (ties aside: the margin is checked)
        ref = O.forward(cfg, W, o[:-1])
        for t in range(len(p), len(o)):
            row = ref[t - 1]
            top2 = torch.topk(row, 2).values
            if float(top2[0] - top2[1]) > 1e-3 * float(row.abs().max()):
                assert int(row.argmax()) == o[t], (t, o)


def test_trace_replayer_command_line(tmp_path):
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    from vyomai_b200.checkpoint import save_safetensors
    cfg = U.small_config()
    w = U.spread_corrections(ZaparaxForCausalLM.random_weights(ZaparaxConfig(cfg), seed=3))
    mdir, out = tmp_path / "model", tmp_path / "out"
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(mdir / "model.safetensors"), w)
    a, b = HU.tokens(21, cfg["vocab"], 31), HU.tokens(9, cfg["vocab"], 32)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:20], "want": [0]}, {"id": "b", "tokens": b[8:9], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[20:21], "want": [0]}], "end": ["a"]}]
    for dtype in (torch.float32, torch.bfloat16):
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", str(dtype).split(".")[1], "--out", str(out), "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        W = U.f64(w)
        ra, rb = Ref(cfg, W, a, dtype), Ref(cfg, W, b, dtype)
        V = cfg["vocab"]
        g0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V))
        g2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(-1, V))
        g3 = torch.from_numpy(np.fromfile(out / "3.f32", dtype="<f4").reshape(-1, V))
        assert not (out / "1.f32").exists()
        for got, ref, pos in ((g0[:1], ra, 0), (g0[1:2], ra, 17), (g0[2:], rb, 6), (g2[:1], ra, 19), (g2[1:], rb, 8), (g3, ra, 20)):
            assert got.shape == (1, V)
            _check(got, ref, f"position {pos}", pos0=pos)
