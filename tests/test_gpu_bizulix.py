"""GPU tests of the Bizulix engine against the CPU oracle (float64, written from the design's equations).

Small configurations and seeded random weights; fp32 engines are held to 1e-4 of the logits' spread, bf16 engines to
8e-2.  Where random weights would hide a fault the weights or the inputs are made so that it shows (one query and key
scaled until their score stands out among hundreds, retention that forgets slowly, router scores that make the choice
clear-cut, a query temperature that steps in the middle of a portion)."""
import copy

import pytest
import torch

from bizulix_util import MIXED, TOL, att, clear_routing, close_enough, config, engine_and_oracle, moe, normed, rel_err, ret, row_errs, tokens

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
both = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def run_whole(model, toks, want=None, trace=False):
    from smoltts_b200.serving import TokenBatcher

    b = TokenBatcher(model)
    want = list(range(len(toks))) if want is None else want
    out = b.feed([("w", toks, want)], end=["w"], trace=trace)
    model.check_device_errors()
    return out


def run_portions(model, toks, sizes):
    """Logits of every position, the prompt cut into portions of ``sizes`` tokens and the rest decoded one by one."""
    from smoltts_b200.serving import TokenBatcher

    b, outs, lo = TokenBatcher(model), [], 0
    for n in list(sizes) + [1] * (len(toks) - sum(sizes)):
        outs.append(b.feed([("p", toks[lo:lo + n], list(range(n)))]))
        lo += n
    b.close()
    model.check_device_errors()
    return torch.cat(outs)


# name -> (layers, loop)
LAYERS = {
    "attention": ([att()], None),
    "attention-1head": ([att(heads=1, kv_heads=1, dim=8, vdim=8)], None),
    "attention-own-kv": ([att(heads=3, kv_heads=3, dim=32, vdim=24)], None),
    "attention-12-over-1": ([att(heads=12, kv_heads=1, dim=16, vdim=40)], None),
    "attention-wide-values": ([att(heads=2, kv_heads=1, dim=12, vdim=100)], None),
    "attention-odd": ([att(heads=6, kv_heads=3, dim=10, vdim=7, scale=0.5)], None),
    "attention-96": ([att(heads=2, kv_heads=2, dim=96, vdim=72, scale=0.1)], None),
    "attention-136": ([att(heads=2, kv_heads=1, dim=136, vdim=136, scale=0.1)], None),            # beyond the tiled form
    "attention-300-values": ([att(heads=1, kv_heads=1, dim=20, vdim=300)], None),
    "attention-tight-cap": ([att(softcap=0.8, scale=2.0)], None),                                # most scores bent flat
    "attention-loose-cap": ([att(softcap=300.0, scale=1.0)], None),
    "attention-every-1": ([att(coef=1.5, every=1)], None),                                       # a temperature that grows with every position
    "attention-no-temperature": ([att(coef=0.0, every=5)], None),
    "attention-negative-temperature": ([att(coef=-0.2, every=3)], None),
    "retention": ([ret()], None),
    "retention-1head": ([ret(heads=1, dim=32, vdim=8, decay=[0.97])], None),
    "retention-64x64": ([ret(heads=2, dim=64, vdim=64)], None),
    "retention-no-rotation": ([ret(heads=2, dim=16, vdim=16, dims=0)], None),
    "retention-partly-rotated": ([ret(heads=2, dim=20, vdim=130, dims=6)], None),
    "retention-rotated-2": ([ret(heads=4, dim=12, vdim=4, dims=2, base=7.0)], None),
    "retention-160": ([ret(heads=1, dim=160, vdim=16, dims=100, base=1e5)], None),
    "retention-256": ([ret(heads=1, dim=256, vdim=24)], None),
    "retention-odd": ([ret(heads=3, dim=9, vdim=5, dims=4)], None),
    "retention-decay-1-and-0": ([ret(heads=2, dim=8, vdim=8, decay=[1.0, 0.0])], None),          # a plain running sum beside no memory at all
    "moe": ([att(mlp=moe())], None),
    "moe-top1": ([ret(mlp=moe(experts=5, top=1, ff=20))], None),
    "moe-no-shared": ([ret(mlp=moe(shared=0))], None),
    "moe-one-expert": ([att(mlp=moe(experts=1, top=1, ff=12, shared=8))], None),
    "moe-all-chosen": ([att(mlp=moe(experts=4, top=4, ff=10, shared=30))], None),
    "moe-many": ([ret(mlp=moe(experts=37, top=6, ff=12, shared=44))], None),
    "loop": ([ret(mlp=moe())], (0, 1, 3)),
    "loop-once": ([att(), ret()], (0, 2, 1)),
    "loop-tail": ([att(), ret()], (1, 2, 2)),
}


@pytest.mark.parametrize("name", list(LAYERS))
@both
def test_each_mechanism_alone(name, dtype):
    layers, loop = LAYERS[name]
    cfg = config(layers, vocab=61, width=72, loop=loop)
    model, orc, _ = engine_and_oracle(cfg, seed=1, dtype=dtype, edit=clear_routing)
    toks = tokens(37, 61)
    logits, traces = run_whole(model, toks, trace=True)
    col = []
    want = orc.forward(toks, col)
    assert traces[0].shape[0] == len(col)
    if dtype == BF16 and "mlp" in layers[0] and layers[0]["mlp"]:
        # a token's last choice can be a close call that bf16 inputs turn the other way: all rows but two
        assert int((row_errs(logits, want) > TOL[dtype]).sum()) <= 2
    else:
        for n, c in enumerate(col):
            assert rel_err(traces[0][n], c) < TOL[dtype], f"run {n}"
        assert rel_err(logits, want) < TOL[dtype]
    got = run_portions(model, toks, [9, 2, 11, 3])
    assert int((row_errs(got, want) > TOL[dtype]).sum()) <= (2 if dtype == BF16 else 0)


@both
def test_every_layer_of_a_mixed_model(dtype):
    from oracle.bizulix_oracle import Oracle

    model, orc, w = engine_and_oracle(MIXED, seed=2, dtype=dtype)
    toks = tokens(50, MIXED["vocab"], 1)
    logits, traces = run_whole(model, toks, trace=True)
    col = []
    want = orc.forward(toks, col)
    assert traces[0].shape[0] == len(col) == 7
    assert close_enough(logits, want, dtype)
    for n, c in enumerate(col):
        assert close_enough(traces[0][n], c, dtype), f"run {n}"
    if dtype == BF16:
        return

    # the test sees the constants and the small tensors: changing any of them moves the oracle far beyond the tolerance
    def moved(cfg=None, weights=None):
        return rel_err(Oracle(cfg or MIXED, weights or w).forward(toks), want)

    assert moved(dict(MIXED, residual_mult=0.8)) > 30 * TOL[F32]
    assert moved(dict(MIXED, logit_softcap=7.0)) > 30 * TOL[F32]
    assert moved(dict(MIXED, loop={"start": 1, "stop": 3, "times": 3})) > 30 * TOL[F32]
    assert moved(dict(MIXED, norm={"eps": 1e-2})) > 10 * TOL[F32]
    for li, path, value in ((1, ("mixer", "scale"), 0.4), (1, ("mixer", "softcap"), 7.0), (1, ("mixer", "q_temp", "coef"), 0.4),
                            (1, ("mixer", "q_temp", "every"), 8), (0, ("mixer", "decay"), [0.9, 0.9, 0.9]), (2, ("mixer", "rot", "dims"), 12),
                            (2, ("mixer", "rot", "base"), 500.0), (1, ("mlp", "router", "top"), 2)):
        other = copy.deepcopy(MIXED)
        d = other["layers"][li]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        assert moved(other) > 10 * TOL[F32], path
    for name in ("l0.norm1.b", "l3.norm1.b", "final.norm.b", "l1.mlp.router.b", "l0.mix.g", "l1.mlp.shared.sg", "l2.mlp.shared.down", "l4.mlp.e1.down"):
        assert moved(weights=dict(w, **{name: torch.zeros_like(w[name])})) > 10 * TOL[F32], name


@both
def test_odd_width_and_vocabulary(dtype):
    """Sizes that are multiples of nothing: no 16-byte pieces anywhere, every kernel on its element-wise form."""
    cfg = config([ret(heads=3, dim=5, vdim=7, dims=4, mlp=moe(experts=3, top=2, ff=9, shared=5)), att(heads=3, kv_heads=1, dim=6, vdim=9),
                  att(heads=2, kv_heads=2, dim=5, vdim=3, mlp=moe(experts=5, top=2, ff=11, shared=7))], vocab=37, width=50, loop=(0, 2, 2))
    model, orc, _ = engine_and_oracle(cfg, seed=14, dtype=dtype, edit=clear_routing)
    toks = tokens(45, 37, 41)
    assert int((row_errs(run_portions(model, toks, [30]), orc.forward(toks)) > TOL[dtype]).sum()) <= (0 if dtype == F32 else 2)


@pytest.mark.parametrize("width", [1030, 2104])
def test_wide_rows(width):
    """Rows wider than the norm kernels' registers (and just beyond the narrow block)."""
    cfg = config([ret(heads=1, dim=8, vdim=8, mlp=moe(experts=2, top=1, ff=8, shared=8)), att(heads=1, kv_heads=1, dim=8, vdim=8)], vocab=41, width=width, loop=(1, 2, 1))
    model, orc, _ = engine_and_oracle(cfg, seed=3, edit=clear_routing)
    toks = tokens(12, 41, 2)
    want = orc.forward(toks)
    assert rel_err(run_whole(model, toks), want) < TOL[F32] and rel_err(run_portions(model, toks, [4]), want) < TOL[F32]


@both
def test_prefill_against_token_by_token_and_portions(dtype):
    model, orc, _ = engine_and_oracle(MIXED, seed=3, edit=clear_routing, dtype=dtype)
    toks = tokens(90, MIXED["vocab"], 2)
    want = orc.forward(toks)
    whole = run_whole(model, toks)
    assert close_enough(whole, want, dtype)
    tight = 4e-5 if dtype == F32 else TOL[dtype]
    for sizes in ([], [2] * 45, [17, 2, 31, 3, 2, 16, 15, 2, 2], [15, 1, 16, 16, 1, 1, 33, 7], [64, 26], [9, 8, 8, 9, 56]):
        got = run_portions(model, toks, sizes)
        assert close_enough(got, want, dtype), sizes
        assert close_enough(got, whole, dtype, tol=tight), sizes
    assert len(model.page_pool) == model.page_pool.n and len(model.slot_pool) == model.slot_pool.n


@both
def test_unequal_batches_equal_each_alone_with_reused_pages_and_slots(dtype):
    """Four requests of different lengths share steps: portions beside single tokens, requests that pause, finish and are
    replaced.  The pool holds fewer pages than all requests together need, so pages and slots are used again, and the
    pools are filled with garbage first: nothing may depend on what a page or slot held before."""
    from smoltts_b200.serving import TokenBatcher

    model, orc, _ = engine_and_oracle(MIXED, seed=4, edit=clear_routing, max_tokens=208, max_seqs=3, dtype=dtype)
    model._kv_pool.view(dtype).fill_(1e4)
    model._state_pool.view(torch.float32).fill_(-3e3)
    V = MIXED["vocab"]
    # (requests in whose first tokens no router choice is so close that bf16 turns it)
    reqs = {"a": tokens(70, V, 14), "b": tokens(33, V, 11), "c": tokens(5, V, 12), "d": tokens(64, V, 13), "e": tokens(49, V, 17)}
    want = {k: orc.forward(v) for k, v in reqs.items()}
    plan = [[("a", 16), ("b", 2), ("c", 1)], [("a", 3), ("b", 29), ("c", 4)], [("a", 13), ("b", 1), ("d", 2)],
            [("a", 1), ("b", 1), ("d", 30)], [("a", 1), ("d", 1)], [("a", 33), ("d", 31), ("e", 17)], [("a", 1), ("e", 2)],
            [("a", 1), ("e", 30)], [("a", 1)]]
    b, at, got = TokenBatcher(model), {k: 0 for k in reqs}, {k: [] for k in reqs}
    for step in plan:
        entries, end = [], []
        for k, n in step:
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        out = b.feed(entries, end=end)
        lo = 0
        for k, n in step:
            got[k].append(out[lo:lo + n])
            lo += n
    model.check_device_errors()
    assert at == {k: len(v) for k, v in reqs.items()}
    for k in reqs:
        assert close_enough(torch.cat(got[k]), want[k], dtype), k
        # and against the engine's own answer for the request alone, whole: sharing steps changes nothing beyond rounding
        assert close_enough(torch.cat(got[k]), run_whole(model, reqs[k]), dtype, tol=4e-5 if dtype == F32 else TOL[BF16]), k
    assert len(model.page_pool) == model.page_pool.n and len(model.slot_pool) == 3


KEY, QUERY = 58, 59                                         # token ids of the key and the query that find each other


def needle(w):
    """Layer 0's attention: the query of QUERY and the key of KEY point the same way in every head, with a raw score far
    above all others (bent by the cap to nearly the cap itself), so that QUERY's result is KEY's value, however far back."""
    eps = 1e-5
    hk, hq = normed(w, KEY, eps), normed(w, QUERY, eps)
    d = 16
    u = torch.ones(d, dtype=torch.float64) / d ** 0.5
    for name, rows, h in (("l0.mix.k", w["l0.mix.k"].shape[0], hk), ("l0.mix.q", w["l0.mix.q"].shape[0], hq)):
        add = torch.outer(u.repeat(rows // d) * 12.0, h / (h @ h))
        w[name] = (w[name].double() + add).float().bfloat16().float()


@pytest.mark.parametrize("place", [0, 1, 2, 15, 16, 17, 63, 64, 65, 128, 251])
@both
def test_one_key_stands_out_wherever_it_is(place, dtype):
    """A lone key among three hundred, at the sequence's start, at page borders and ranges' edges: the rows of the query
    token follow it in a prompt, in portions and in decoding; the rows before the key do not see it."""
    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, softcap=18.0, coef=0.05, every=64)], vocab=60, mult=1.0)
    model, orc, _ = engine_and_oracle(cfg, seed=5, dtype=dtype, edit=needle, max_tokens=512)
    toks = tokens(300, 58, 3)
    queries = [3, 70, 200, 252, 260, 299]
    for q in queries:
        toks[q] = QUERY
    toks[place] = KEY
    want = orc.forward(toks)
    other = list(toks)
    other[place] = 7
    change = row_errs(orc.forward(other)[queries], want[queries])
    for q, c in zip(queries, change):
        assert (float(c) > 0.3) == (q > place), (q, float(c))
    assert rel_err(run_whole(model, toks), want) < TOL[dtype]
    assert rel_err(run_portions(model, toks, [10, 6, 47, 2, 100, 5, 80]), want) < TOL[dtype]


@both
def test_query_temperature_steps_inside_portions(dtype):
    """A temperature that steps every 13 positions and changes the attention strongly: shifting a step by one position moves
    the oracle at exactly that position; the engine agrees at every step's edge in prompts, portions and decoding."""
    from oracle.bizulix_oracle import Oracle

    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, softcap=30.0, coef=1.0, every=13)], vocab=53, mult=1.0)
    model, orc, w = engine_and_oracle(cfg, seed=6, dtype=dtype)
    toks = tokens(140, 53, 7)
    want = orc.forward(toks)
    late = copy.deepcopy(cfg)
    late["layers"][0]["mixer"]["q_temp"]["every"] = 14
    moved = row_errs(Oracle(late, w).forward(toks), want)
    assert float(moved[11]) < 1e-12 and float(moved[12]) > 0.02 and float(moved[13]) < 1e-12
    assert rel_err(run_whole(model, toks), want) < TOL[dtype]
    for sizes in ([12, 2, 24, 2, 38], [13, 13, 13, 13], [5, 20]):
        assert rel_err(run_portions(model, toks, sizes), want) < TOL[dtype], sizes


@both
def test_retention_carries_the_first_tokens_far(dtype):
    """Retention alone, forgetting slowly: logits hundreds of positions on still depend on the first token; prompt portions
    and decoding agree with the oracle."""
    cfg = config([ret(heads=4, dim=32, vdim=16, decay=[0.999, 0.9995, 1.0, 0.998], base=1e4)], vocab=59)
    model, orc, _ = engine_and_oracle(cfg, seed=6, dtype=dtype, max_tokens=512)
    toks = tokens(400, 59, 4)
    want = orc.forward(toks)
    other = [(toks[0] + 1) % 59] + toks[1:]
    assert rel_err(orc.forward(other)[-20:], want[-20:]) > 10 * TOL[F32], "the test is blind to the first token"
    assert rel_err(run_whole(model, toks), want) < TOL[dtype]
    assert rel_err(run_portions(model, toks, [1, 1, 1, 2, 3, 2, 40, 1, 2, 147]), want) < TOL[dtype]


def test_router_choice_shows():
    """Choosing fewer experts, leaving the router's bias or the shared expert's gate out would move the logits far beyond
    the tolerance; the engine agrees with the oracle in every product form (whole prompt, portions, single tokens)."""
    from oracle import bizulix_oracle as bo

    cfg = config([att(mlp=moe(experts=12, top=3, ff=20, shared=12))], vocab=41)
    model, orc, w = engine_and_oracle(cfg, seed=7, edit=clear_routing)
    toks = tokens(60, 41, 4)
    want = orc.forward(toks)
    fewer, lone = copy.deepcopy(cfg), copy.deepcopy(cfg)
    fewer["layers"][0]["mlp"]["router"]["top"] = 2
    del lone["layers"][0]["mlp"]["shared"]
    for c, ws in ((fewer, w), (lone, w), (cfg, dict(w, **{"l0.mlp.router.b": torch.zeros(12)})), (cfg, dict(w, **{"l0.mlp.shared.sg": torch.zeros(1, 64)}))):
        assert rel_err(bo.Oracle(c, ws).forward(toks), want) > 50 * TOL[F32]
    assert rel_err(run_whole(model, toks), want) < TOL[F32]
    assert rel_err(run_portions(model, toks, [3, 20, 9]), want) < TOL[F32]


def test_long_decoding_keeps_the_state():
    """300 single-token steps after a short prompt: retention states, keys and values are carried exactly through a loop."""
    cfg = config([att(coef=0.1, every=50, mlp=moe()), ret(heads=2, dim=32, vdim=24, decay=[0.999, 0.99], mlp=moe()), att(heads=2, kv_heads=1, dim=8, vdim=8)],
                 vocab=67, loop=(1, 3, 2))
    model, orc, _ = engine_and_oracle(cfg, seed=8, edit=clear_routing, max_tokens=384)
    toks = tokens(310, 67, 5)
    want = orc.forward(toks)
    got = run_portions(model, toks, [10])
    assert rel_err(got[-5:], want[-5:]) < TOL[F32] and rel_err(got, want) < TOL[F32]
    other = [(toks[0] + 1) % 67] + toks[1:]
    assert rel_err(orc.forward(other)[-20:], want[-20:]) > 3 * TOL[F32]


def test_greedy_generation_through_the_batcher():
    """The scheduler's own loop: admission, chunked prefill beside decoding, the library's sampler, retirement."""
    from smoltts_b200.serving import TokenBatcher

    model, orc, _ = engine_and_oracle(MIXED, seed=9, max_tokens=160, max_seqs=2, max_step_tokens=24)
    V = MIXED["vocab"]
    prompts = [tokens(30, V, 20), tokens(3, V, 21), tokens(41, V, 22), tokens(1, V, 23)]
    b = TokenBatcher(model, step_tokens=24)
    got = b.generate(prompts, max_new_tokens=6)
    for p, g in zip(prompts, got):
        seq = list(p)
        for tok in g:
            logits = orc.forward(seq)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(logits.std()):      # a near-tie may go either way
                assert tok == int(logits.argmax()), (p, g)
            seq.append(tok)
    assert len(model.page_pool) == model.page_pool.n and len(model.slot_pool) == 2 and b.stats["retired"] == 4


def test_generation_and_trace_through_the_registry(tmp_path):
    """A checkpoint folder on disk: the registry picks the design's class by config.json; the command line generates and
    replays a schedule of steps."""
    import json
    import subprocess
    import sys

    import numpy as np

    from smoltts_b200.registry import load_model

    model, orc, w = engine_and_oracle(MIXED, seed=9)
    ckpt = tmp_path / "ckpt"
    model.save_pretrained(str(ckpt))
    again = load_model(str(ckpt), dtype=F32, max_tokens=256, max_seqs=2, page_size=16)
    assert type(again).__name__ == "BizulixLM"
    toks = tokens(20, MIXED["vocab"], 30)
    want = orc.forward(toks)
    assert rel_err(run_whole(again, toks), want) < TOL[F32]
    out = subprocess.run([sys.executable, "-m", "smoltts_b200", "generate", "--model", str(ckpt), "--dtype", "float32",
                          "--prompt", ",".join(map(str, toks)), "--max-new-tokens", "3"], capture_output=True, text=True, check=True)
    rec = json.loads(out.stdout.strip().splitlines()[-1])
    assert rec["prompt"] == toks and len(rec["tokens"]) == 3
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:13], "want": [12, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[13:15], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[15:], "want": [4]}], "end": ["a"]}]
    run = subprocess.run([sys.executable, "-m", "smoltts_b200", "trace", "--model", str(ckpt), "--dtype", "float32", "--out", str(tmp_path / "o"),
                          "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, check=True)
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4").reshape(2, -1).copy())
    last = torch.from_numpy(np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4").reshape(1, -1).copy())
    assert rel_err(torch.cat([first, last]), want[[12, 0, 19]]) < TOL[F32]
    assert not (tmp_path / "o" / "1.f32").exists()


@both
def test_long_portions_take_the_large_tile_path(dtype):
    """Steps of several hundred tokens (the matrix products change kernels with the row count, the attention runs many
    tiles) against the oracle, against short portions of the same prompt, and beside a decoding request in the same step."""
    from smoltts_b200.serving import TokenBatcher

    cfg = config([ret(heads=4, dim=32, vdim=32, base=1e3, mlp=moe(experts=6, top=2, ff=64, shared=96)),
                  att(heads=4, kv_heads=2, dim=64, vdim=48, scale=0.15, softcap=15.0, coef=0.2, every=100, mlp=moe(experts=4, top=2, ff=96, shared=64)),
                  att(heads=2, kv_heads=1, dim=32, vdim=32, every=33)], vocab=131, width=128, loop=(0, 2, 2))
    model, orc, _ = engine_and_oracle(cfg, seed=11, dtype=dtype, edit=clear_routing, page_size=64, max_tokens=1024, max_step_tokens=512)
    toks, other = tokens(700, 131, 30), tokens(40, 131, 31)
    want, want_o = orc.forward(toks), orc.forward(other)
    b = TokenBatcher(model)
    b.feed([("o", other[:30], [])])
    got = [b.feed([("a", toks[:300], list(range(300)))])]
    out = b.feed([("a", toks[300:690], list(range(390))), ("o", other[30:31], [0])])
    got.append(out[:390])
    assert rel_err(out[390:], want_o[30:31]) < TOL[dtype]
    got.append(b.feed([("a", toks[690:], list(range(10)))], end=["a", "o"]))
    long = torch.cat(got)
    assert close_enough(long, want, dtype)
    short = torch.cat([b.feed([("s", toks[lo:lo + 100], list(range(100)))], end=["s"] if lo == 600 else []) for lo in range(0, 700, 100)])
    assert close_enough(short, want, dtype)
    assert close_enough(long, short, dtype, tol=4e-5 if dtype == F32 else TOL[dtype])
    # one entry larger than the engine's step: the batcher cuts it into engine steps itself
    once = b.feed([("w", toks, list(range(700)))], end=["w"])
    assert close_enough(once, want, dtype)
    model.check_device_errors()


@both
def test_routed_experts_on_every_grouped_product_form(dtype):
    """Experts wide enough, and steps long enough, for the grouped products' large-tile form (rows copied into sorted order,
    128-row tiles), the 32-row tile form and the few-pair form of decoding: the same prompt whole, in portions of 40 and
    token by token."""
    cfg = config([ret(heads=2, dim=32, vdim=32, mlp=moe(experts=4, top=2, ff=96, shared=104)), att(heads=2, kv_heads=1, dim=32, vdim=32, mlp=moe(experts=3, top=1, ff=128, shared=0))],
                 vocab=101, width=128)
    model, orc, _ = engine_and_oracle(cfg, seed=13, dtype=dtype, edit=clear_routing, page_size=64, max_tokens=1024, max_step_tokens=512)
    toks = tokens(420, 101, 35)
    want = orc.forward(toks)
    assert close_enough(run_whole(model, toks), want, dtype)
    assert close_enough(run_portions(model, toks, [40] * 10), want, dtype)


def test_four_decoding_requests_share_the_few_pair_form():
    """bf16: four requests decode together with 8 choices each -- exactly as many pairs as the few-pair form takes -- and
    then with a portion beside them (more pairs: sorted rows); every request's rows match its own run alone."""
    from smoltts_b200.serving import TokenBatcher

    cfg = config([ret(heads=2, dim=16, vdim=16, mlp=moe(experts=16, top=8, ff=32, shared=24)), att(mlp=moe(experts=9, top=8, ff=16, shared=16))], vocab=71)
    model, orc, _ = engine_and_oracle(cfg, seed=16, dtype=BF16, edit=clear_routing)
    reqs = {k: tokens(30, 71, 60 + i) for i, k in enumerate("abcd")}
    b, got = TokenBatcher(model), {k: [] for k in reqs}
    for lo, hi in [(0, 12)] + [(i, i + 1) for i in range(12, 25)]:
        out = b.feed([(k, v[lo:hi], list(range(hi - lo))) for k, v in reqs.items()])
        for i, k in enumerate(reqs):
            got[k].append(out[i * (hi - lo):(i + 1) * (hi - lo)])
    out = b.feed([("a", reqs["a"][25:], list(range(5)))] + [(k, reqs[k][25:26], [0]) for k in "bcd"])
    got["a"].append(out[:5])
    b.close()
    model.check_device_errors()
    for k, v in reqs.items():
        n = 30 if k == "a" else 25
        assert close_enough(torch.cat(got[k]), orc.forward(v)[:n], BF16), k
        assert close_enough(torch.cat(got[k]), run_whole(model, v)[:n], BF16), k


def random_config(seed, big=False):
    """A configuration drawn at random: kinds, sizes, counts and constants all differ from layer to layer.  ``big``: sizes
    near a small real model's."""
    import random

    r = random.Random(seed + (900 if big else 0))

    def divisor(n):
        return r.choice([d for d in range(1, n + 1) if n % d == 0])

    def feed():
        experts = r.choice([4, 8, 12, 24, 32] if big else [1, 2, 3, 6, 8, 12])
        return r.choice([None] + 3 * [moe(experts, r.randint(1, min(6, experts)), r.choice([32, 48, 80, 120] if big else [8, 16, 20, 40]),
                                          r.choice([32, 64, 136] if big else [0, 8, 24, 36]))])

    layers = []
    for _ in range(r.randint(3, 6) if big else r.randint(2, 4)):
        if r.random() < 0.5:
            heads, dim = r.choice([2, 4, 5, 8, 12] if big else [1, 2, 3, 4, 6]), r.choice([32, 64, 96, 128] if big else [8, 12, 16, 32, 64, 96])
            layers.append(ret(heads, dim, r.choice([16, 32, 64, 96, 128] if big else [8, 12, 24, 48, 64]), [r.choice([0.3, 0.9, 0.99, 0.999, 1.0]) for _ in range(heads)],
                              2 * r.randint(0, dim // 2) if r.random() < 0.4 else dim, r.choice([10.0, 1e4, 5e5]), feed()))
            continue
        heads, dim = r.choice([2, 4, 5, 8, 12, 20] if big else [1, 2, 3, 4, 6, 8]), r.choice([32, 40, 64, 72, 112, 128] if big else [8, 12, 16, 32, 48, 64])
        layers.append(att(heads, divisor(heads), dim, r.choice([32, 56, 64, 128] if big else [8, 16, 20, 48, 64]), dim ** -0.5 * r.uniform(0.7, 1.5),
                          r.choice([4.0, 15.0, 50.0]), r.uniform(-0.1, 0.6), r.choice([1, 5, 16, 33, 64, 500]), feed()))
    a = r.randint(0, len(layers) - 1)
    loop = r.choice([None, (a, r.randint(a + 1, len(layers)), r.randint(1, 3)), (0, r.randint(1, len(layers)), 2)])
    return config(layers, vocab=r.choice([300, 512, 777]) if big else r.randint(50, 400), width=r.choice([128, 192, 320, 384, 512] if big else [64, 96, 128, 200]),
                  eps=r.choice([1e-6, 1e-5]), mult=r.uniform(0.3, 1.2), cap=r.choice([5.0, 20.0, 30.0]), loop=loop)


@pytest.mark.parametrize("seed", list(range(10)))
@both
def test_random_configurations_in_mixed_steps(seed, dtype):
    """Configurations drawn at random, two requests sharing steps: a prompt in portions beside single decoded tokens."""
    from smoltts_b200.serving import TokenBatcher

    cfg = random_config(seed)
    model, orc, _ = engine_and_oracle(cfg, seed=20 + seed, dtype=dtype, edit=clear_routing, page_size=64, max_tokens=384)
    V = cfg["vocab"]
    a, b_ = tokens(150, V, 50 + seed), tokens(60, V, 70 + seed)
    tb = TokenBatcher(model)
    got_a, got_b = [tb.feed([("a", a[:37], list(range(37)))])], []
    out = tb.feed([("a", a[37:101], list(range(64))), ("b", b_[:50], list(range(50)))])
    got_a.append(out[:64]); got_b.append(out[64:])
    at = 101
    for i, n in enumerate([2, 9, 1, 17, 3, 1, 1, 1, 1, 1]):           # "b" decodes beside portions of "a", then beside its decoding
        out = tb.feed([("b", b_[50 + i:51 + i], [0]), ("a", a[at:at + n], list(range(n)))])
        got_b.append(out[:1]); got_a.append(out[1:])
        at += n
    got_a.append(tb.feed([("a", a[at:], list(range(150 - at)))], end=["a", "b"]))
    model.check_device_errors()
    for got, toks in ((torch.cat(got_a), a), (torch.cat(got_b), b_)):
        assert close_enough(got, orc.forward(toks), dtype)


@pytest.mark.parametrize("seed", list(range(4)))
@both
def test_model_sized_configurations(seed, dtype):
    """Random configurations of a small real model's sizes with the engine's default page and step sizes: a whole prompt,
    decoding, and a second request's portions beside it."""
    from smoltts_b200.serving import TokenBatcher

    cfg = random_config(seed, big=True)
    model, orc, _ = engine_and_oracle(cfg, seed=40 + seed, dtype=dtype, edit=clear_routing, page_size=64, max_tokens=640, max_step_tokens=2048)
    V = cfg["vocab"]
    a, b_ = tokens(200, V, 90 + seed), tokens(110, V, 95 + seed)
    want_a, want_b = orc.forward(a), orc.forward(b_)
    tb = TokenBatcher(model)
    whole = tb.feed([("w", a, list(range(200)))], end=["w"])
    got_a, got_b = [tb.feed([("a", a[:160], list(range(160)))])], []
    cuts = [0, 2, 33, 40, 79, 86, 87, 110]
    for i in range(40):                                   # "a" decodes; "b" arrives in portions beside it, then decodes too
        entries = [("a", a[160 + i:161 + i], [0])]
        if i < len(cuts) - 1:
            entries.append(("b", b_[cuts[i]:cuts[i + 1]], list(range(cuts[i + 1] - cuts[i]))))
        out = tb.feed(entries)
        got_a.append(out[:1]); got_b.append(out[1:])
    tb.close()
    model.check_device_errors()
    for got, want in ((whole, want_a), (torch.cat(got_a), want_a), (torch.cat(got_b), want_b)):
        assert close_enough(got, want, dtype)


@both
def test_decoding_in_a_large_pool(dtype):
    """A pool of 40 000 positions: the few-token attention cuts the keys into wider ranges than in a small pool."""
    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, softcap=18.0, coef=0.05, every=64)], vocab=60, mult=1.0)
    model, orc, _ = engine_and_oracle(cfg, seed=15, dtype=dtype, edit=needle, page_size=64, max_tokens=40000, max_step_tokens=512)
    toks = tokens(420, 58, 6)
    toks[1], toks[380], toks[419] = KEY, QUERY, QUERY
    want = orc.forward(toks)
    assert rel_err(run_portions(model, toks, [370, 7]), want) < TOL[dtype]


def test_a_step_that_only_ends_a_request():
    """A step may bring no tokens and only end requests: nothing runs, the slot and pages come back and serve the next."""
    from smoltts_b200.serving import TokenBatcher

    cfg = config([att(), ret(mlp=moe())], vocab=61)
    model, orc, _ = engine_and_oracle(cfg, seed=3, dtype=F32, page_size=16, max_tokens=64, max_seqs=1)
    toks = tokens(50, 61, 4)
    want = orc.forward(toks)
    tb = TokenBatcher(model)
    for name in ("x", "y", "x"):
        got = tb.feed([(name, toks, list(range(50)))])
        assert tb.feed([], end=[name]).shape == (0, 61)
        assert rel_err(got, want) < TOL[F32]
    assert len(model.page_pool) == 4 and len(model.slot_pool) == 1
    tb.close()
