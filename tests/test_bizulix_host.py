"""CPU tests of the Bizulix design: configuration parsing and the oracle's own consistency (portions against whole prompts,
the query temperature's steps, rotation by halves, the router's choice, merged passes, retention against its unrolled sum)."""
import math

import pytest
import torch

from bizulix_util import MIXED, att, config, moe, ret, tokens
from oracle import bizulix_oracle as bo
from smoltts_b200.lm_config import BizulixConfig

F = bo.F


def test_config_round_trip_shapes_and_runs():
    cfg = BizulixConfig.from_dict(MIXED)
    assert BizulixConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert cfg.layer_runs() == [0, 1, 2, 1, 2, 3, 4] and cfg.run_merges() == [0, 1, 0, 1, 0, 0, 0]
    assert [(i, bool(a)) for i, a in zip(cfg.layer_runs(), cfg.run_merges())] == bo.layer_runs(MIXED)
    w = bo.random_weights(MIXED, 0)
    assert {k: tuple(v.shape) for k, v in w.items()} == cfg.tensor_shapes()
    assert cfg.layers[1].shared_ff == 28 and cfg.layers[3].ff == 0 and cfg.layers[2].mixer.rot.dims == 10 and cfg.layers[4].mixer.temp_every == 20
    plain = BizulixConfig.from_dict(config([att(), ret()]))
    assert plain.layer_runs() == [0, 1] and plain.run_merges() == [0, 0] and "loop.in" not in plain.tensor_shapes() and "loop" not in plain.to_dict()
    once = BizulixConfig.from_dict(config([att(), ret()], loop=(0, 2, 1)))           # a span that runs once still starts with the merge
    assert once.layer_runs() == [0, 1] and once.run_merges() == [1, 0] and once.tensor_shapes()["loop.in"] == (64, 128)
    tail = BizulixConfig.from_dict(config([att(), ret()], loop=(1, 2, 3)))
    assert tail.layer_runs() == [0, 1, 1, 1] and tail.run_merges() == [0, 1, 1, 1]
    one = config([ret(heads=3, decay=[0.75] * 3)])
    one["layers"][0]["mixer"]["decay"] = 0.75
    assert BizulixConfig.from_dict(one).layers[0].mixer.decay == [0.75] * 3
    for bad in (config([{"type": "serial", "mixer": {}, "mlp": None}]), config([att(heads=3, kv_heads=2)]), config([ret(heads=2, decay=[0.5])]),
                config([ret(dim=8, dims=10)]), config([ret(dim=8, dims=3)]), config([att()], loop=(0, 3, 2)), config([att()], loop=(0, 1, 0)),
                config([att(mlp=moe(experts=3, top=4))]), config([att(mlp={"kind": "dense", "ff": 8})])):
        with pytest.raises(ValueError):
            BizulixConfig.from_dict(bad)
    assert cfg.weight_elements(active_only=True) < cfg.weight_elements()
    # the flops of a looped layer count once per pass
    flat = config([ret(mlp=moe())])
    twice = dict(flat, loop={"start": 0, "stop": 1, "times": 2})
    a, b = BizulixConfig.from_dict(flat), BizulixConfig.from_dict(twice)
    layer = a.matmul_flops_per_token() - 2 * a.vocab * a.width
    assert b.matmul_flops_per_token() - a.matmul_flops_per_token() == layer + 2 * 2 * (2 * 64 * 64)


def test_registry_names_the_design(tmp_path):
    from smoltts_b200 import registry

    BizulixConfig.from_dict(MIXED).save(str(tmp_path / "config.json"))
    assert registry.design_of(str(tmp_path)) == "Bizulix"
    assert registry.registered()["Bizulix"] == ("smoltts_b200.lm", "BizulixLM")


def test_oracle_portions_equal_the_whole_prompt():
    orc = bo.Oracle(MIXED, bo.random_weights(MIXED, 3))
    toks = tokens(40, MIXED["vocab"])
    whole = orc.forward(toks)
    parts = [orc.step(toks[lo:hi]) for lo, hi in ((0, 7), (7, 9), (9, 10), (10, 33), (33, 40))]
    assert float((torch.cat(parts) - whole).abs().max()) < 1e-9


def test_layer_norm_by_hand():
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F)
    y = bo.layer_norm(x, torch.tensor([1.0, 2.0, 1.0, 1.0], dtype=F), torch.tensor([0.0, 0.0, 1.0, 0.0], dtype=F), 0.0)
    s = math.sqrt(5.0)
    assert [float(v) for v in y[0]] == pytest.approx([-3 / s, -2 / s, 1 / s + 1, 3 / s])


def test_query_temperature_steps():
    """The factor is 1 while p + 1 < every, and steps up where p + 1 reaches a multiple of it."""
    assert [bo.query_temperature(p, 0.5, 4) for p in (0, 1, 2)] == [1.0, 1.0, 1.0]
    assert bo.query_temperature(3, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(2)) == bo.query_temperature(6, 0.5, 4)
    assert bo.query_temperature(7, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(3))
    assert bo.query_temperature(0, 0.5, 1) == pytest.approx(1 + 0.5 * math.log(2))


def test_attention_by_hand():
    g = torch.Generator().manual_seed(0)
    n, D = 5, 6
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 2, "scale": 0.7, "softcap": 2.0, "q_temp": {"coef": 0.4, "every": 2}}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 6), ("k", 3), ("v", 2))}
    w["o"] = torch.eye(4, dtype=F)
    out = bo.attention(h, w, "", m)
    for i in range(n):
        f = 1 + 0.4 * math.log((i + 1) // 2 + 1)
        for hh in range(2):
            q = (w["q"] @ h[i])[3 * hh:3 * hh + 3] * f
            e = [math.exp(2.0 * math.tanh(0.7 * float(q @ (w["k"] @ h[j])) / 2.0)) for j in range(i + 1)]
            want = sum(e[j] / sum(e) * (w["v"] @ h[j]) for j in range(i + 1))
            assert float((out[i, 2 * hh:2 * hh + 2] - want).abs().max()) < 1e-12


def test_rotation_pairs_halves_of_the_leading_coordinates():
    x = torch.arange(1.0, 13.0, dtype=F).view(1, 1, 12)
    y = bo.rotate_halves(x, torch.tensor([3]), 8, 16.0)
    assert torch.equal(y[..., 8:], x[..., 8:])
    a = 3 * 16.0 ** (-2.0 / 8)                                        # pair 1: coordinates 1 and 5
    assert float(y[0, 0, 1]) == pytest.approx(2 * math.cos(a) - 6 * math.sin(a)) and float(y[0, 0, 5]) == pytest.approx(6 * math.cos(a) + 2 * math.sin(a))
    q, k = torch.randn(2, 1, 1, 8, dtype=F, generator=torch.Generator().manual_seed(1)).unbind(0)
    at = lambda v, p: bo.rotate_halves(v, torch.tensor([p]), 8, 16.0)
    assert float((at(q, 9) * at(k, 4)).sum()) == pytest.approx(float((at(q, 25) * at(k, 20)).sum()))      # only the distance counts


def test_retention_against_its_unrolled_sum():
    """o_t = sum_s decay^(t-s) (q_t.k_s) v_s / sqrt(dim) without rotation; divided per head, gated by silu."""
    g = torch.Generator().manual_seed(2)
    n, D = 6, 5
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 2, "dim": 3, "vdim": 2, "decay": [0.8, 0.5], "rot": {"base": 10.0, "dims": 0}}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 6), ("k", 6), ("v", 4), ("g", 4))}
    w["o"] = torch.eye(4, dtype=F)
    out = bo.retention(h, w, "", m, 1e-6)
    q, k, v = h @ w["q"].T, h @ w["k"].T, h @ w["v"].T
    for t in range(n):
        for hh in range(2):
            o = sum(m["decay"][hh] ** (t - s) * float(q[t, 3 * hh:3 * hh + 3] @ k[s, 3 * hh:3 * hh + 3]) / math.sqrt(3) * v[s, 2 * hh:2 * hh + 2] for s in range(t + 1))
            want = bo.rms_divide(o, 1e-6) * bo.silu(h[t] @ w["g"][2 * hh:2 * hh + 2].T)
            assert float((out[t, 2 * hh:2 * hh + 2] - want).abs().max()) < 1e-12


def test_router_takes_the_largest_logits_and_weighs_them_alone():
    z = torch.tensor([[1.0, 3.0, 2.0, 0.0]], dtype=F)
    ids, wts = bo.route(torch.ones(1, 1, dtype=F), z.T.contiguous(), torch.tensor([0.0, 0.0, 0.0, 2.5], dtype=F), 2)
    assert ids[0] == [1, 3] and float(wts[0, 0]) == pytest.approx(1 / (1 + math.exp(-0.5)))
    ids, wts = bo.route(torch.ones(1, 1, dtype=F), z.T.contiguous(), torch.zeros(4, dtype=F), 1)
    assert ids[0] == [1] and float(wts[0, 0]) == 1.0


def test_shared_expert_is_gated_per_token():
    mlp = moe(experts=2, top=1, ff=4, shared=3)
    cfg = config([att(mlp=mlp)], width=8)
    w = {k: v.double() for k, v in bo.random_weights(cfg, 4).items()}
    h = torch.randn(3, 8, dtype=F, generator=torch.Generator().manual_seed(3))
    both, p = bo.feed_forward(h, w, "l0.mlp.", mlp), "l0.mlp."
    alone = bo.feed_forward(h, w, p, moe(experts=2, top=1, ff=4, shared=0))
    for t in range(3):
        s = 1 / (1 + math.exp(-float(w[p + "shared.sg"][0] @ h[t])))
        assert float((both[t] - alone[t] - s * bo.gated_unit(h[t:t + 1], w, p + "shared.")[0]).abs().max()) < 1e-12


def test_both_sublayers_read_the_same_norm_and_passes_merge():
    """One layer run twice: by hand, x <- M [x; e] before each pass, then x + m (mixer(h) + ff(h)) with one h."""
    cfg = config([ret(mlp=moe())], loop=(0, 1, 2))
    w = bo.random_weights(cfg, 5)
    toks = tokens(9, cfg["vocab"], 1)
    col = []
    out = bo.Oracle(cfg, w).forward(toks, col)
    w = {k: v.double() for k, v in w.items()}
    e = w["embed"][torch.tensor(toks)]
    x = e
    for n in range(2):
        x = torch.cat([x, e], 1) @ w["loop.in"].T
        h = bo.layer_norm(x, w["l0.norm1"], w["l0.norm1.b"], 1e-5)
        x = x + 0.7 * (bo.retention(h, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5) + bo.feed_forward(h, w, "l0.mlp.", cfg["layers"][0]["mlp"]))
        assert float((x - col[n]).abs().max()) < 1e-12
    z = bo.layer_norm(x, w["final.norm"], w["final.norm.b"], 1e-5) @ w["head"].T
    assert float((6.0 * torch.tanh(z / 6.0) - out).abs().max()) < 1e-12 and float(out.abs().max()) < 6.0
