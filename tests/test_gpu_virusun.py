"""GPU tests of the Virusun engine against the CPU oracle (float64, written from the design's equations).

Small configurations and seeded random weights; fp32 engines are held to 1e-4 of the logits' spread, bf16 engines to
8e-2.  Where random weights would hide a fault the weights or the inputs are made so that it shows (one query and key of
one map that stand out among hundreds, memories that forget slowly, a norm eps large enough for the mLSTM's denominator and
running maximum to matter)."""
import copy

import pytest
import torch

from virusun_util import MIXED, TOL, att, close_enough, config, delta, dense, engine_and_oracle, left, par, rel_err, right, row_errs, tokens

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


LAYERS = {
    "attention": [att()],
    "attention-1head": [att(heads=1, kv_heads=1, dim=8, vdim=8)],
    "attention-own-kv": [att(heads=3, kv_heads=3, dim=32, vdim=24)],
    "attention-12-over-1": [att(heads=12, kv_heads=1, dim=16, vdim=40)],
    "attention-wide-values": [att(heads=2, kv_heads=1, dim=12, vdim=100)],
    "attention-odd": [att(heads=6, kv_heads=3, dim=10, vdim=7, scale=0.5)],
    "attention-64-128": [att(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.2)],
    "attention-96": [att(heads=2, kv_heads=2, dim=96, vdim=72, scale=0.1)],
    "attention-136": [att(heads=2, kv_heads=1, dim=136, vdim=136, scale=0.1)],                  # beyond the tiled form
    "attention-300-values": [att(heads=1, kv_heads=1, dim=20, vdim=300)],
    "attention-diff-0": [att(diff=0.0)],
    "attention-diff-negative": [att(diff=-0.3)],
    "attention-lent": [att(), att(kv_from=0, scale=0.5, diff=0.1)],
    "attention-lent-past-others": [att(heads=6, kv_heads=2), delta(), att(heads=4), att(heads=6, kv_heads=2, kv_from=0), att(heads=4, kv_from=2)],
    "delta": [delta()],
    "delta-1head-1tap": [delta(heads=1, kv_heads=1, dim=16, vdim=8, conv=1)],
    "delta-2taps": [delta(conv=2)],
    "delta-9taps": [delta(conv=9)],
    "delta-6-over-1": [delta(heads=6, kv_heads=1, dim=8, vdim=12, conv=4)],
    "delta-own-keys": [delta(heads=3, kv_heads=3, dim=64, vdim=64, conv=4)],
    "delta-128x96": [delta(heads=2, kv_heads=1, dim=128, vdim=96, conv=4)],
    "delta-256": [delta(heads=1, kv_heads=1, dim=256, vdim=24)],
    "delta-odd": [delta(heads=3, kv_heads=3, dim=9, vdim=5)],
    "delta-160x130": [delta(heads=2, kv_heads=2, dim=160, vdim=130)],
    "parallel": [par()],
    "parallel-1head": [par(left(heads=1, kv_heads=1, dim=8, vdim=8), right(heads=1, dim=32, vdim=8))],
    "parallel-own-kv": [par(left(heads=3, kv_heads=3, dim=24, vdim=40), right(heads=2, dim=64, vdim=64))],
    "parallel-no-scaling": [par(left(scaling=None))],
    "parallel-no-rotation": [par(left(dims=0, scaling=None))],
    "parallel-partly-rotated": [par(left(dim=20, dims=6, base=7.0), right(heads=2, dim=20, vdim=130))],
    "parallel-step-ramp": [par(left(scaling=(16.0, 30, 2.0, 2.0)))],
    "parallel-136": [par(left(heads=2, kv_heads=1, dim=136, vdim=136, scale=0.1, dims=100), right(heads=1, dim=160, vdim=16))],
    "parallel-256-keys": [par(left(heads=2, kv_heads=1, dim=300, vdim=30, scale=0.05), right(heads=1, dim=256, vdim=24))],
    "parallel-odd": [par(left(heads=3, kv_heads=1, dim=9, vdim=7, dims=4), right(heads=3, dim=9, vdim=5))],
    "parallel-low-cap": [par(b=right(cap=0.5))],
    "parallel-scales": [par(left_scale=-0.4, right_scale=2.5)],
    "dense": [att(mlp=dense())],
    "dense-odd": [delta(mlp=dense(9))],
}


@pytest.mark.parametrize("name", list(LAYERS))
@both
def test_each_mechanism_alone(name, dtype):
    cfg = config(LAYERS[name], vocab=61, width=80)
    model, orc, _ = engine_and_oracle(cfg, seed=1, dtype=dtype)
    toks = tokens(37, 61)
    logits, traces = run_whole(model, toks, trace=True)
    col = []
    want = orc.forward(toks, col)
    assert traces[0].shape[0] == len(col)
    for n, c in enumerate(col):
        assert close_enough(traces[0][n], c, dtype), f"layer {n}"
    assert close_enough(logits, want, dtype)
    assert close_enough(run_portions(model, toks, [9, 2, 11, 3]), want, dtype)


@both
def test_every_layer_of_a_mixed_model(dtype):
    from oracle.virusun_oracle import Oracle

    model, orc, w = engine_and_oracle(MIXED, seed=2, dtype=dtype)
    toks = tokens(50, MIXED["vocab"], 1)
    logits, traces = run_whole(model, toks, trace=True)
    col = []
    want = orc.forward(toks, col)
    assert traces[0].shape[0] == len(col) == 8
    assert close_enough(logits, want, dtype)
    for n, c in enumerate(col):
        assert close_enough(traces[0][n], c, dtype), f"layer {n}"
    if dtype == BF16:
        return

    # the test sees the constants and the small tensors: changing any of them moves the oracle far beyond the tolerance
    def moved(cfg=None, weights=None):
        return rel_err(Oracle(cfg or MIXED, weights or w).forward(toks), want)

    assert moved(dict(MIXED, norm={"eps": 1e-2})) > 10 * TOL[F32]
    for li, path, value in ((1, ("mixer", "scale"), 0.4), (1, ("mixer", "diff"), 0.3), (3, ("mixer", "scale"), 0.3), (3, ("mixer", "diff"), 0.4),
                            (6, ("mixer", "diff"), 0.3), (0, ("mixer", "left_scale"), 0.9), (0, ("mixer", "right_scale"), 1.2),
                            (0, ("mixer", "left", "rot", "base"), 150.0), (0, ("mixer", "left", "rot", "scaling", "factor"), 3.0),
                            (0, ("mixer", "left", "rot", "scaling", "original"), 400), (0, ("mixer", "left", "rot", "scaling", "fast"), 3.0),
                            (0, ("mixer", "left", "rot", "scaling", "slow"), 0.1), (0, ("mixer", "left", "scale"), 0.35),
                            (7, ("mixer", "left", "rot", "dims"), 12), (7, ("mixer", "right", "gate_cap"), 6.0)):
        other = copy.deepcopy(MIXED)
        d = other["layers"][li]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        assert moved(other) > 10 * TOL[F32], path
    for name in ("l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.left.o.b", "l0.mix.right.i.b", "l0.mix.right.f.b", "l0.mix.right.g",
                 "l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l1.mix.o.b", "l1.mix.g", "l1.mix.lq1", "l3.mix.q.b", "l3.mix.lk2", "l2.mix.A_log", "l2.mix.dt_bias",
                 "l2.mix.a", "l2.mix.b", "l2.mix.g", "l5.mlp.down"):
        assert moved(weights=dict(w, **{name: torch.zeros_like(w[name])})) > 10 * TOL[F32], name
    for name in ("l0.mix.left.q.norm", "l0.mix.left.k.norm", "l0.mix.right.norm", "l1.mix.q.norm", "l1.mix.k.norm", "l2.mix.norm", "l4.norm1", "l5.norm2", "final.norm"):
        assert moved(weights=dict(w, **{name: torch.ones_like(w[name])})) > 10 * TOL[F32], name


@both
def test_odd_width_and_vocabulary(dtype):
    """Sizes that are multiples of nothing: no 16-byte pieces anywhere, every kernel on its element-wise form."""
    cfg = config([par(left(heads=3, kv_heads=1, dim=6, vdim=9, dims=4), right(heads=3, dim=5, vdim=7), mlp=dense(9)), att(heads=3, kv_heads=1, dim=7, vdim=9),
                  delta(heads=3, kv_heads=1, dim=5, vdim=3, conv=4, mlp=dense(11)), att(heads=3, kv_heads=1, dim=7, vdim=9, kv_from=1)], vocab=37, width=50)
    model, orc, _ = engine_and_oracle(cfg, seed=14, dtype=dtype)
    toks = tokens(45, 37, 41)
    assert close_enough(run_portions(model, toks, [30]), orc.forward(toks), dtype)


@pytest.mark.parametrize("width", [1030, 2104])
def test_wide_rows(width):
    """Rows wider than the norm kernels' registers (and just beyond the narrow block)."""
    cfg = config([delta(heads=1, kv_heads=1, dim=8, vdim=8, mlp=dense(8)), att(heads=1, kv_heads=1, dim=8, vdim=8)], vocab=41, width=width)
    model, orc, _ = engine_and_oracle(cfg, seed=3)
    toks = tokens(12, 41, 2)
    want = orc.forward(toks)
    assert rel_err(run_whole(model, toks), want) < TOL[F32] and rel_err(run_portions(model, toks, [4]), want) < TOL[F32]


@both
def test_prefill_against_token_by_token_and_portions(dtype):
    model, orc, _ = engine_and_oracle(MIXED, seed=3, dtype=dtype)
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

    model, orc, _ = engine_and_oracle(MIXED, seed=4, max_tokens=208, max_seqs=3, dtype=dtype)
    model._kv_pool.view(dtype).fill_(1e4)
    model._state_pool.view(torch.float32).fill_(-3e3)
    V = MIXED["vocab"]
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


def _aim(w, name, rows, token, u):
    """Adds to the given rows (head size u.numel() each) of a projection of the raw embedding a part that sends ``token`` along u."""
    x = w["embed"][token].double()
    add = torch.zeros(w[name].shape, dtype=torch.float64)
    for lo in rows:
        add[lo:lo + u.numel()] = torch.outer(u * 12.0, x / (x @ x))
    w[name] = (w[name].double() + add).float().bfloat16().float()


def needle(map_):
    """Layer 0's attention: in map ``map_`` of every head the query of QUERY and the key of KEY point the same way and the norm
    weights are large, so that their score is far above all others and QUERY's result in that map is KEY's value."""
    def edit(w):
        d = w["l0.mix.q.norm"].numel()
        u = torch.ones(d, dtype=torch.float64) / d ** 0.5
        for name, token in (("l0.mix.k", KEY), ("l0.mix.q", QUERY)):
            _aim(w, name, range(map_ * d, w[name].shape[0], 2 * d), token, u)
        w["l0.mix.q.norm"], w["l0.mix.k.norm"] = torch.full((d,), 2.5), torch.full((d,), 2.5)
        w["l0.norm1"] = torch.full_like(w["l0.norm1"], 1.5)
    edit.__name__ = f"needle{map_}"
    return edit


NEEDLES = [needle(0), needle(1)]


@pytest.mark.parametrize("place", [0, 1, 2, 15, 16, 17, 63, 64, 65, 128, 251])
@pytest.mark.parametrize("map_", [0, 1])
@both
def test_one_key_stands_out_wherever_it_is(place, map_, dtype):
    """A lone key among three hundred, at the sequence's start, at page borders and ranges' edges: the rows of the query
    token follow it in a prompt, in portions and in decoding; the rows before the key do not see it."""
    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3)], vocab=60)
    model, orc, _ = engine_and_oracle(cfg, seed=5, dtype=dtype, edit=NEEDLES[map_], max_tokens=512)
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
        assert (float(c) > 0.2) == (q > place), (q, float(c))
    got = run_whole(model, toks)
    assert close_enough(got, want, dtype) and rel_err(got[queries], want[queries]) < TOL[dtype]
    got = run_portions(model, toks, [10, 6, 47, 2, 100, 5, 80])
    assert close_enough(got, want, dtype) and rel_err(got[queries], want[queries]) < TOL[dtype]


def left_needle(w):
    """Layer 0's rotary attention: the query of QUERY and the key of KEY agree in the coordinates that are not rotated."""
    d, dims = 16, 4
    u = torch.zeros(d, dtype=torch.float64)
    u[dims:] = 1.0 / (d - dims) ** 0.5
    for name, token in (("l0.mix.left.k", KEY), ("l0.mix.left.q", QUERY)):
        _aim(w, name, range(0, w[name].shape[0], d), token, u)
        w[name + ".norm"] = torch.full_like(w[name + ".norm"], 2.5)


@pytest.mark.parametrize("place", [0, 1, 15, 16, 63, 64, 65, 200])
@both
def test_one_key_stands_out_beside_the_matrix_memory(place, dtype):
    cfg = config([par(left(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3, dims=4), right(heads=2, dim=8, vdim=8), 1.5, 0.3)], vocab=60)
    model, orc, _ = engine_and_oracle(cfg, seed=5, dtype=dtype, edit=left_needle, max_tokens=512)
    toks = tokens(300, 58, 3)
    queries = [3, 70, 201, 260, 299]
    for q in queries:
        toks[q] = QUERY
    toks[place] = KEY
    want = orc.forward(toks)
    other = list(toks)
    other[place] = 7
    change = row_errs(orc.forward(other)[queries], want[queries])
    for q, c in zip(queries, change):
        assert float(c) > 0.2 if q > place else float(c) < 1e-9, (q, float(c))
    assert rel_err(run_whole(model, toks), want) < TOL[dtype]
    assert rel_err(run_portions(model, toks, [10, 6, 47, 2, 100, 5, 80]), want) < TOL[dtype]


@both
def test_lent_keys_are_the_lenders_own(dtype):
    """A borrowing layer whose lender stands two layers back: the oracle that lets it read the nearer layer's cache, or its own
    stream through the lender's projections, gives something else; the engine follows the lender's cache in every schedule."""
    from oracle.virusun_oracle import Oracle

    layers = [att(heads=4, kv_heads=2, scale=0.5, mlp=dense()), att(heads=4, kv_heads=2, scale=0.5, mlp=dense()), delta(), att(heads=4, kv_heads=2, scale=0.5, kv_from=0)]
    cfg = config(layers, vocab=67)
    model, orc, w = engine_and_oracle(cfg, seed=6, dtype=dtype)
    toks = tokens(100, 67, 8)
    want = orc.forward(toks)
    near = copy.deepcopy(cfg)
    near["layers"][3]["mixer"]["kv_from"] = 1
    assert rel_err(Oracle(near, w).forward(toks), want) > 3 * TOL[BF16]
    own = copy.deepcopy(cfg)
    del own["layers"][3]["mixer"]["kv_from"]
    again = dict(w, **{f"l3.mix.{nm}": w[f"l0.mix.{nm}"] for nm in ("k", "k.b", "k.norm", "v", "v.b")})
    assert rel_err(Oracle(own, again).forward(toks), want) > 3 * TOL[BF16]
    assert close_enough(run_whole(model, toks), want, dtype)
    for sizes in ([2] * 10, [33, 2, 15, 16], [7]):
        assert close_enough(run_portions(model, toks, sizes), want, dtype), sizes


def slow_memory(w):
    """Recurrences that forget little: small decay rates and forget gates near one."""
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -5.0)
        if k.endswith("right.f.b"):
            w[k] = torch.full_like(w[k], 6.0)
        if k.endswith("right.f") or k.endswith("mix.b"):
            w[k] = (w[k] * 0.3).bfloat16().float()


@pytest.mark.parametrize("kind", ["delta", "mlstm"])
@both
def test_recurrences_carry_the_first_tokens_far(kind, dtype):
    """One recurrent layer that forgets slowly: logits hundreds of positions on still depend on the first token; prompt
    portions (shorter than the convolution too) and decoding agree with the oracle."""
    layer = delta(heads=4, kv_heads=2, dim=32, vdim=16, conv=4) if kind == "delta" else par(left(heads=1, kv_heads=1, dim=4, vdim=4), right(heads=4, dim=32, vdim=16, cap=12.0), 0.2, 1.5)
    cfg = config([layer], vocab=59)
    model, orc, _ = engine_and_oracle(cfg, seed=6, dtype=dtype, edit=slow_memory, max_tokens=512)
    toks = tokens(400, 59, 4)
    want = orc.forward(toks)
    other = [(toks[0] + 1) % 59] + toks[1:]
    assert rel_err(orc.forward(other)[-20:], want[-20:]) > (10 if kind == "mlstm" else 1) * TOL[F32], "the test is blind to the first token"
    assert close_enough(run_whole(model, toks), want, dtype)
    assert close_enough(run_portions(model, toks, [1, 1, 1, 2, 3, 2, 40, 1, 2, 147]), want, dtype)


def loud_gates(w):
    """Input and forget gates of the mLSTM spread over tens of units, so that the running maximum jumps and sinks."""
    for nm in ("i", "f"):
        w[f"l0.mix.right.{nm}"] = (w[f"l0.mix.right.{nm}"] * 6.0).bfloat16().float()
    w["l0.mix.right.i.b"] = torch.full_like(w["l0.mix.right.i.b"], -2.0)


@both
def test_mlstm_running_maximum_and_denominator(dtype, monkeypatch):
    """With an eps that does not vanish beside a head's values the denominator shows: an oracle without its floor or without the key
    sum gives something else.  Gates spread wide move the maximum up and down; the gate kernel's tiles (1024 tokens) are crossed by the whole prompt."""
    from oracle import virusun_oracle as vo

    cfg = config([par(left(heads=1, kv_heads=1, dim=4, vdim=4), right(heads=5, dim=8, vdim=12, cap=16.0), 0.1, 1.5)], vocab=43, eps=0.05)
    model, orc, w = engine_and_oracle(cfg, seed=8, dtype=dtype, edit=loud_gates, max_tokens=1216, max_step_tokens=2048)
    toks = tokens(1200, 43, 6)
    want = orc.forward(toks)
    for wrong in (lambda dot, m: dot.abs() + 1e-6, lambda dot, m: torch.exp(-m) + 1e-6):
        with monkeypatch.context() as mp:
            mp.setattr(vo, "memory_denominator", wrong)
            assert rel_err(orc.forward(toks), want) > 100 * TOL[F32]
    assert close_enough(run_whole(model, toks), want, dtype)
    for sizes in ([255, 2, 256, 2, 600], [1030, 1, 1, 120], [33] * 33):
        assert close_enough(run_portions(model, toks, sizes), want, dtype), sizes


@both
def test_rotation_far_out(dtype):
    """Interpolated frequencies over 700 positions (beyond the stretch's original length): prompt, portions and decoding."""
    from oracle.virusun_oracle import Oracle

    cfg = config([par(left(heads=4, kv_heads=2, dim=32, vdim=16, scale=0.4, base=500.0, scaling=(6.0, 90, 16.0, 1.0)), right(heads=1, dim=4, vdim=4), 1.5, 0.1)], vocab=53)
    model, orc, w = engine_and_oracle(cfg, seed=9, dtype=dtype, page_size=64, max_tokens=768, max_step_tokens=1024)
    toks = tokens(700, 53, 7)
    want = orc.forward(toks)
    plain = copy.deepcopy(cfg)
    plain["layers"][0]["mixer"]["left"]["rot"]["scaling"] = None
    assert rel_err(Oracle(plain, w).forward(toks)[-50:], want[-50:]) > 3 * TOL[BF16]
    tol = {F32: 2e-4, BF16: TOL[BF16]}[dtype]                     # fp32 angles of several hundred radians
    assert rel_err(run_whole(model, toks), want) < tol
    assert rel_err(run_portions(model, toks, [64, 63, 2, 300, 200, 40]), want) < tol


def test_long_decoding_keeps_the_state():
    """300 single-token steps after a short prompt: states, maxima, convolution inputs, keys and values are carried exactly."""
    cfg = config([att(mlp=dense()), delta(heads=2, kv_heads=1, dim=32, vdim=24, conv=4, mlp=dense()), par(b=right(heads=2, dim=16, vdim=8)), att(kv_from=0)], vocab=67)
    model, orc, _ = engine_and_oracle(cfg, seed=8, edit=slow_memory, max_tokens=384)
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
    assert type(again).__name__ == "VirusunLM"
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

    cfg = config([att(heads=4, kv_heads=2, dim=32, vdim=64, scale=0.2, mlp=dense(200)), delta(heads=4, kv_heads=2, dim=32, vdim=32, conv=4, mlp=dense(136)),
                  par(left(heads=4, kv_heads=2, dim=64, vdim=48, scale=0.15, base=1e3, scaling=(4.0, 300, 16.0, 1.0)), right(heads=2, dim=32, vdim=64), mlp=dense(144)),
                  att(heads=4, kv_heads=2, dim=32, vdim=64, scale=0.2, kv_from=0)], vocab=131, width=128)
    model, orc, _ = engine_and_oracle(cfg, seed=11, dtype=dtype, page_size=64, max_tokens=1024, max_step_tokens=512)
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


def test_four_decoding_requests_share_a_step():
    """bf16: four requests decode together, then with a portion beside them; every request's rows match its own run alone."""
    from smoltts_b200.serving import TokenBatcher

    model, orc, _ = engine_and_oracle(MIXED, seed=16, dtype=BF16)
    reqs = {k: tokens(30, MIXED["vocab"], 60 + i) for i, k in enumerate("abcd")}
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
        return r.choice([None] + 3 * [dense(r.choice([96, 160, 320, 512] if big else [8, 24, 40, 72]))])

    layers, lenders = [], []
    for _ in range(r.randint(4, 7) if big else r.randint(2, 5)):
        kind = r.choice(["attention", "attention", "delta", "parallel"])
        heads = r.choice([2, 4, 6, 8, 12] if big else [1, 2, 3, 4, 6])
        dim = r.choice([32, 48, 64, 96] if big else [8, 12, 16, 20, 32, 64])
        vdim = r.choice([32, 64, 96, 128] if big else [8, 12, 24, 48, 80])
        if kind == "attention":
            if lenders and r.random() < 0.5:
                j = r.choice(lenders)
                layers.append(copy.deepcopy(layers[j]))
                layers[-1]["mixer"].update(kv_from=j, diff=r.uniform(-0.2, 0.6))
                layers[-1]["mlp"] = feed()
                continue
            lenders.append(len(layers))
            layers.append(att(heads, divisor(heads), dim, vdim, dim ** -0.5 * r.uniform(0.5, 1.2), r.uniform(0.0, 0.7), mlp=feed()))
        elif kind == "delta":
            layers.append(delta(heads, divisor(heads), dim, vdim, r.choice([1, 2, 3, 4, 4, 6]), feed()))
        else:
            scaling = r.choice([None, (r.choice([2.0, 8.0, 40.0]), r.choice([20, 64, 500, 4096]), r.choice([4.0, 32.0]), r.choice([0.5, 1.0, 2.0]))])
            dims = dim if r.random() < 0.5 else 2 * r.randint(0, dim // 2)
            rh, rd = r.choice([1, 2, 3, 4]), r.choice([32, 64, 128] if big else [8, 12, 32])
            layers.append(par(left(heads, divisor(heads), dim, r.choice([16, 32, 64] if big else [8, 20, 36]), dim ** -0.5, dims, r.choice([10.0, 1e3, 1e4, 5e5]), scaling),
                              right(rh, rd, vdim, r.choice([2.0, 10.0, 20.0])), r.uniform(0.3, 1.5), r.uniform(0.3, 1.5), feed()))
    return config(layers, vocab=r.choice([300, 512, 777]) if big else r.randint(50, 400), width=r.choice([128, 192, 320, 384, 512] if big else [64, 96, 128, 200]),
                  eps=r.choice([1e-6, 1e-5, 1e-4]))


@pytest.mark.parametrize("seed", list(range(12)))
@both
def test_random_configurations_in_mixed_steps(seed, dtype):
    """Configurations drawn at random, two requests sharing steps: a prompt in portions beside single decoded tokens."""
    from smoltts_b200.serving import TokenBatcher

    cfg = random_config(seed)
    model, orc, _ = engine_and_oracle(cfg, seed=20 + seed, dtype=dtype, page_size=64, max_tokens=384)
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
    model, orc, _ = engine_and_oracle(cfg, seed=40 + seed, dtype=dtype, page_size=64, max_tokens=640, max_step_tokens=2048)
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
    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3)], vocab=60)
    model, orc, _ = engine_and_oracle(cfg, seed=15, dtype=dtype, edit=NEEDLES[0], page_size=64, max_tokens=40000, max_step_tokens=512)
    toks = tokens(420, 58, 6)
    toks[1], toks[380], toks[419] = KEY, QUERY, QUERY
    want = orc.forward(toks)
    got = run_portions(model, toks, [370, 7])
    assert close_enough(got, want, dtype) and rel_err(got[[380, 419]], want[[380, 419]]) < TOL[dtype]


def test_a_step_that_only_ends_a_request():
    """A step may bring no tokens and only end requests: nothing runs, the slot and pages come back and serve the next."""
    from smoltts_b200.serving import TokenBatcher

    cfg = config([att(), delta(mlp=dense()), par()], vocab=61)
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
