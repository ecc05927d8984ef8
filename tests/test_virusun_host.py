"""CPU tests of the Virusun design: configuration parsing and the oracle's own consistency (portions against whole prompts, every
mechanism against hand-unrolled sums)."""
import copy
import ctypes
import math

import pytest
import torch

from oracle import virusun_oracle as vo
from smoltts_b200.lm_config import RampRotarySpec, VirusunConfig
from virusun_util import MIXED, att, config, delta, dense, left, par, right, tokens

F = vo.F


def test_config_round_trip_and_shapes():
    cfg = VirusunConfig.from_dict(MIXED)
    assert cfg.to_dict() == MIXED and cfg.layer_runs() == list(range(8))
    w = vo.random_weights(MIXED, 0)
    assert {k: tuple(v.shape) for k, v in w.items()} == cfg.tensor_shapes()
    assert "l3.mix.k" not in w and "l3.mix.v.b" not in w and "l3.mix.k.norm" not in w and "l3.mix.q.norm" in w and "l4.norm2" not in w
    assert cfg.layers[0].right.gate_cap == 9.0 and cfg.layers[3].mixer.kv_from == 1 and cfg.layers[2].mixer.channels == 2 * 2 * 12 + 4 * 16
    plain = copy.deepcopy(att())
    del plain["mixer"]["kv_heads"], plain["mixer"]["vdim"]
    m = VirusunConfig.from_dict(config([plain])).layers[0].mixer
    assert (m.kv_heads, m.vdim) == (4, 16)
    nul = par()
    nul["mixer"]["left"]["rot"]["scaling"] = None
    assert VirusunConfig.from_dict(config([nul])).layers[0].left.rot.mult == 1.0
    for bad in (config([{"type": "serial", "mixer": {}, "mlp": None}]), config([att(heads=3, kv_heads=2)]), config([delta(heads=3, kv_heads=2)]),
                config([delta(conv=0)]), config([par(left(dim=8, dims=10))]), config([par(left(dims=3))]), config([par(b=right(cap=0.0))]),
                config([att(mlp={"kind": "moe", "ff": 8})]), config([att(kv_from=0)]), config([att(), att(kv_from=1)]), config([att(), att(dim=8, kv_from=0)]),
                config([att(), att(kv_from=0), att(kv_from=1)]), config([delta(), att(kv_from=0)]), config([par(), att(kv_from=0)]), config([att(), att(kv_from=-1)])):
        with pytest.raises(ValueError):
            VirusunConfig.from_dict(bad)
    assert cfg.matmul_flops_per_token() == 2 * cfg.weight_elements() > 2 * 97 * 72


def test_registry_names_the_design(tmp_path):
    from smoltts_b200 import registry

    VirusunConfig.from_dict(MIXED).save(str(tmp_path / "config.json"))
    assert registry.design_of(str(tmp_path)) == "Virusun"
    assert registry.registered()["Virusun"] == ("smoltts_b200.lm", "VirusunLM")


def test_oracle_portions_equal_the_whole_prompt():
    orc = vo.Oracle(MIXED, vo.random_weights(MIXED, 3))
    toks = tokens(40, MIXED["vocab"])
    whole = orc.forward(toks)
    parts = [orc.step(toks[lo:hi]) for lo, hi in ((0, 1), (1, 7), (7, 9), (9, 10), (10, 33), (33, 40))]
    assert float((torch.cat(parts) - whole).abs().max()) < 1e-9


def test_only_the_sublayers_outputs_are_normed():
    cfg = config([delta(mlp=dense(12))], width=24)
    w = vo.random_weights(cfg, 5)
    toks = tokens(9, cfg["vocab"], 1)
    out = vo.Oracle(cfg, w).forward(toks)
    w = {k: v.double() for k, v in w.items()}
    x = w["embed"][torch.tensor(toks)]
    y = vo.gated_delta(x, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
    x = x + y / (y.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * w["l0.norm1"]
    z = (vo.silu(x @ w["l0.mlp.gate"].T) * (x @ w["l0.mlp.up"].T)) @ w["l0.mlp.down"].T
    x = x + z / (z.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * w["l0.norm2"]
    want = (x / (x.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * w["final.norm"]) @ w["head"].T
    assert float((want - out).abs().max()) < 1e-12


def test_differential_attention_by_hand():
    g = torch.Generator().manual_seed(0)
    n, D, d, dv = 5, 6, 3, 2
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 4, "kv_heads": 2, "dim": d, "vdim": dv, "scale": 0.7, "diff": 0.4}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 24), ("k", 12), ("v", 4), ("g", 8))}
    w.update({nm: torch.randn(sz, generator=g, dtype=F) for nm, sz in (("q.b", 24), ("k.b", 12), ("v.b", 4), ("o.b", 8), ("q.norm", 3), ("k.norm", 3),
                                                                      ("lq1", 3), ("lk1", 3), ("lq2", 3), ("lk2", 3))})
    w["o"] = torch.eye(8, dtype=F)
    out, (k_all, v_all) = vo.diff_attention(h, w, "", m, 1e-3)
    lam = math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.4
    norm = lambda v, wt: v / (v.pow(2).mean() + 1e-3).sqrt() * wt
    for i in range(n):
        for hh in range(4):
            gk, maps = hh // 2, []
            for c in (0, 1):                                       # rows of a head: map 1, then map 2
                q = norm((w["q"] @ h[i] + w["q.b"])[(hh * 2 + c) * d:(hh * 2 + c + 1) * d], w["q.norm"])
                ks = [norm((w["k"] @ h[j] + w["k.b"])[(gk * 2 + c) * d:(gk * 2 + c + 1) * d], w["k.norm"]) for j in range(i + 1)]
                e = [math.exp(0.7 * float(q @ k)) for k in ks]
                maps.append(sum(e[j] / sum(e) * (w["v"] @ h[j] + w["v.b"])[gk * dv:(gk + 1) * dv] for j in range(i + 1)))
            o = maps[0] - lam * maps[1]
            o = o / (o.pow(2).mean() + 1e-3).sqrt() * 0.6 * torch.sigmoid(w["g"] @ h[i])[hh * dv:(hh + 1) * dv]
            assert float((out[i, hh * dv:(hh + 1) * dv] - o - w["o.b"][hh * dv:(hh + 1) * dv]).abs().max()) < 1e-12
    # a layer that borrows computes its own queries against those keys and values
    again, _ = vo.diff_attention(h, {k: v for k, v in w.items() if k[0] not in "kv"}, "", m, 1e-3, None, (k_all, v_all))
    assert float((again - out).abs().max()) < 1e-12


def test_ramp_frequencies_by_hand():
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 5.0, "original": 64, "fast": 4.0, "slow": 0.5}}
    f, mult = vo.ramp_frequencies(rot)
    dim = lambda t: 8 * math.log(64 / (2 * math.pi * t)) / (2 * math.log(100.0))
    lo, hi = math.floor(dim(4.0)), math.ceil(dim(0.5))
    assert (lo, hi) == (0, 3) and mult == pytest.approx(0.1 * math.log(5.0) + 1)
    plain = [100.0 ** (-2.0 * i / 8) for i in range(4)]
    assert f[0] == plain[0] and f[3] == pytest.approx(plain[3] / 5.0)
    assert f[1] == pytest.approx(plain[1] * (2 / 3 + 1 / 15)) and f[2] == pytest.approx(plain[2] * (1 / 3 + 2 / 15))
    assert vo.ramp_frequencies({"base": 100.0, "dims": 8}) == (plain, 1.0)
    # both ends on the same pair: the ramp is a step
    rot["scaling"].update(fast=1.0, slow=1.0, original=2 * math.pi * 100.0 ** 0.5)      # dim(1) = 2
    assert vo.ramp_frequencies(rot)[0] == pytest.approx([plain[0], plain[1], plain[2], plain[3] / 5.0])
    assert RampRotarySpec.from_dict(rot).mult == pytest.approx(mult)


def test_rotation_pairs_halves_and_passes_the_rest():
    rot = {"base": 16.0, "dims": 8, "scaling": {"factor": 3.0, "original": 50, "fast": 2.0, "slow": 1.0}}
    x = torch.arange(1.0, 13.0, dtype=F).view(1, 1, 12)
    y = vo.rotate_halves(x, torch.tensor([3]), rot)
    assert torch.equal(y[..., 8:], x[..., 8:])
    f, mult = vo.ramp_frequencies(rot)
    a = 3 * f[1]                                                    # pair 1: coordinates 1 and 5
    assert float(y[0, 0, 1]) == pytest.approx(mult * (2 * math.cos(a) - 6 * math.sin(a))) and float(y[0, 0, 5]) == pytest.approx(mult * (6 * math.cos(a) + 2 * math.sin(a)))
    q, k = torch.randn(2, 1, 1, 8, dtype=F, generator=torch.Generator().manual_seed(1)).unbind(0)
    at = lambda v, p: vo.rotate_halves(v, torch.tensor([p]), rot)
    assert float((at(q, 9) * at(k, 4)).sum()) == pytest.approx(float((at(q, 25) * at(k, 20)).sum()))      # only the distance counts


def test_rotary_attention_norms_all_heads_together():
    g = torch.Generator().manual_seed(3)
    n, D = 4, 5
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.6, "rot": {"base": 10.0, "dims": 2}}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 8), ("k", 4), ("v", 3))}
    w.update({nm: torch.randn(sz, generator=g, dtype=F) for nm, sz in (("q.b", 8), ("k.b", 4), ("v.b", 3), ("o.b", 6), ("q.norm", 8), ("k.norm", 4))})
    w["o"] = torch.eye(6, dtype=F)
    out = vo.rotary_attention(h, w, "", m, 1e-4)

    def vec(nm, i):
        v = w[nm] @ h[i] + w[nm + ".b"]
        v = (v / (v.pow(2).mean() + 1e-4).sqrt() * w[nm + ".norm"]).view(-1, 4).clone()
        c, s = math.cos(float(i)), math.sin(float(i))               # one pair: coordinates 0 and 1, frequency 1
        a, b = v[:, 0].clone(), v[:, 1].clone()
        v[:, 0], v[:, 1] = a * c - b * s, b * c + a * s
        return v

    for i in range(n):
        for hh in range(2):
            e = [math.exp(0.6 * float(vec("q", i)[hh] @ vec("k", j)[0])) for j in range(i + 1)]
            want = sum(e[j] / sum(e) * (w["v"] @ h[j] + w["v.b"]) for j in range(i + 1)) + w["o.b"][3 * hh:3 * hh + 3]
            assert float((out[i, 3 * hh:3 * hh + 3] - want).abs().max()) < 1e-12


def test_mlstm_against_its_unrolled_sum():
    """Without the running maximum: weights e^(i_s + f_(s+1) + ... + f_t) on k_s v_s^T, denominator max(|n.q|, 1) plus the small
    constant times e^m."""
    g = torch.Generator().manual_seed(2)
    n, D = 7, 5
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 2, "dim": 3, "vdim": 2, "gate_cap": 2.5}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 6), ("k", 6), ("v", 4), ("g", 4), ("i", 2), ("f", 2))}
    w.update({"i.b": torch.tensor([0.3, -2.0], dtype=F), "f.b": torch.tensor([1.0, 2.0], dtype=F), "norm": torch.randn(4, generator=g, dtype=F)})
    w["o"] = torch.eye(4, dtype=F)
    out = vo.mlstm(h, w, "", m, 1e-2)
    cap = lambda z: 2.5 * math.tanh(z / 2.5)
    for hh in range(2):
        ii = [cap(float(w["i"][hh] @ h[t] + w["i.b"][hh])) for t in range(n)]
        ff = [-math.log1p(math.exp(-cap(float(w["f"][hh] @ h[t] + w["f.b"][hh])))) for t in range(n)]
        mx = 0.0
        for t in range(n):
            mx = max(ff[t] + mx, ii[t])
            q = (w["q"] @ h[t])[3 * hh:3 * hh + 3] / math.sqrt(3)
            num, den = torch.zeros(2, dtype=F), 0.0
            for s in range(t + 1):
                a = math.exp(ii[s] + sum(ff[s + 1:t + 1])) * float(q @ (w["k"] @ h[s])[3 * hh:3 * hh + 3])
                num, den = num + a * (w["v"] @ h[s])[2 * hh:2 * hh + 2], den + a
            o = num / (max(abs(den), 1.0) + 1e-6 * math.exp(mx))
            o = o / (o.pow(2).mean() + 1e-2).sqrt() * w["norm"][2 * hh:2 * hh + 2] * torch.sigmoid(w["g"] @ h[t])[2 * hh:2 * hh + 2]
            assert float((out[t, 2 * hh:2 * hh + 2] - o).abs().max()) < 1e-11


def test_short_convolution_by_hand():
    z, wt = torch.tensor([[1.0], [2.0], [3.0]], dtype=F), torch.tensor([[0.5, -1.0, 2.0]], dtype=F)
    y = vo.short_conv(z, wt, torch.zeros(2, 1, dtype=F))
    raw = [2.0, 4.0 - 1.0, 6.0 - 2.0 + 0.5]
    assert [float(v) for v in y[:, 0]] == pytest.approx([r / (1 + math.exp(-r)) for r in raw])
    y = vo.short_conv(z, wt, torch.tensor([[4.0], [-2.0]], dtype=F))
    assert float(y[0, 0]) == pytest.approx(float(vo.silu(torch.tensor(2.0 + 2.0 + 2.0))))


def test_gated_delta_by_hand():
    """One head per key head and two: the state as the rule says, written out with matrices I - b k k^T."""
    g = torch.Generator().manual_seed(4)
    n, D = 6, 5
    h = torch.randn(n, D, generator=g, dtype=F)
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 2, "conv": 1}
    w = {nm: torch.randn(sz, D, generator=g, dtype=F) for nm, sz in (("q", 3), ("k", 3), ("v", 4), ("g", 4), ("a", 2), ("b", 2))}
    w.update({nm + ".conv": torch.randn(sz, 1, generator=g, dtype=F) for nm, sz in (("q", 3), ("k", 3), ("v", 4))})
    w.update({"A_log": torch.tensor([-0.5, 0.4], dtype=F), "dt_bias": torch.tensor([0.1, -0.7], dtype=F), "norm": torch.randn(2, generator=g, dtype=F)})
    w["o"] = torch.eye(4, dtype=F)
    out = vo.gated_delta(h, w, "", m, 1e-3)
    z = {nm: vo.silu((h @ w[nm].T) * w[nm + ".conv"][:, 0]) for nm in "qkv"}
    for hh in range(2):
        S = torch.zeros(3, 2, dtype=F)
        for t in range(n):
            k = z["k"][t] / math.sqrt(float(z["k"][t] @ z["k"][t]) + 1e-6)
            q = z["q"][t] / math.sqrt(float(z["q"][t] @ z["q"][t]) + 1e-6) / math.sqrt(3)
            b = 1 / (1 + math.exp(-float(w["b"][hh] @ h[t])))
            dec = math.exp(-math.exp(float(w["A_log"][hh])) * math.log1p(math.exp(float(w["a"][hh] @ h[t] + w["dt_bias"][hh]))))
            S = dec * (torch.eye(3, dtype=F) - b * torch.outer(k, k)) @ S + b * torch.outer(k, z["v"][t, 2 * hh:2 * hh + 2])
            o = S.T @ q
            o = o / (o.pow(2).mean() + 1e-3).sqrt() * w["norm"] * vo.silu(w["g"] @ h[t])[2 * hh:2 * hh + 2]
            assert float((out[t, 2 * hh:2 * hh + 2] - o).abs().max()) < 1e-12


def test_engine_create_refuses_what_it_cannot_run():
    """smol_lm_create is host code: a borrowing layer without a lender, a lender of other sizes, and sizes beyond the kernels are
    refused with a message; pages and slots are sized for what the layers keep."""
    from smoltts_b200 import _capi_lm as lm
    from smoltts_b200.lm_config import BLOCK_OUTNORM, MIXER_KINDS

    lib, one = lm.load(), ctypes.c_void_p(16)

    def layer(**kw):
        c = lm.SmolLmLayer()
        c.mixer, c.heads, c.kv_heads, c.dim, c.vdim, c.norm1, c.mix_scale = MIXER_KINDS["attention"], 4, 2, 8, 12, one, 1.0
        c.q_norm = c.k_norm = one
        c.n_maps = 2
        for k, v in kw.items():
            setattr(c, k, v)
        return c

    def create(*layers):
        arr = (lm.SmolLmLayer * len(layers))(*layers)
        cfg = lm.SmolLmConfig(dtype=lm.SMOL_LM_BF16, vocab=32, width=16, n_layers=len(layers), n_runs=len(layers), page_size=16, max_step_tokens=8,
                              max_step_seqs=2, max_want=8, max_context=64, embed_scale=1.0, norm_eps=1e-5, block=BLOCK_OUTNORM, logit_scale=1.0)
        h = ctypes.c_void_p()
        rc = lib.smol_lm_create(ctypes.byref(cfg), arr, (ctypes.c_int32 * len(layers))(*range(len(layers))), ctypes.byref(h))
        sizes = (lib.smol_lm_page_bytes(h), lib.smol_lm_slot_bytes(h)) if rc == 0 else None
        if rc == 0:
            lib.smol_lm_destroy(h)
        return rc, sizes

    page = 2 * 16 * (2 * 8 + 12) * 2
    assert create(layer()) == (0, (page, 16))
    assert create(layer(), layer(kv_from=1)) == (0, (page, 16))                       # a borrower keeps nothing of its own
    assert create(layer(), layer())[1][0] == 2 * page
    for bad in ([layer(kv_from=1)], [layer(), layer(kv_from=1, dim=16)], [layer(), layer(kv_from=1), layer(kv_from=2)], [layer(n_maps=3)],
                [layer(rot_dims=8)], [layer(norm1=None)], [layer(vdim=520)]):
        rc, _ = create(*bad)
        assert rc < 0 and lib.smol_lm_last_error()
    d = layer(mixer=MIXER_KINDS["gated_delta"], n_maps=0, conv_taps=4, conv_w=one, a_log=one, dt_bias=one, out_norm=one)
    assert create(d)[1][1] == 4 * (4 * 8 * 12 + 3 * (2 * 2 * 8 + 4 * 12))
    assert create(layer(mixer=MIXER_KINDS["gated_delta"], conv_taps=4))[0] < 0
    x = layer(mixer=MIXER_KINDS["mlstm"], n_maps=0, gate_cap=5.0, rate_bias=one, decay_bias=one, out_norm=one)
    assert create(x)[1][1] == 4 * (4 * 8 * 12 + 4 * 8 + 4)
    assert create(layer(mixer=MIXER_KINDS["mlstm"], gate_cap=0.0, rate_bias=one, decay_bias=one, out_norm=one))[0] < 0
