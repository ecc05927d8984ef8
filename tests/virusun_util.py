"""Shared helpers of the Virusun tests: small configurations, seeded weights, engine + oracle pairs."""
from __future__ import annotations

import torch

from oracle.virusun_oracle import Oracle, random_weights


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def att(heads=4, kv_heads=2, dim=16, vdim=20, scale=0.3, diff=0.35, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def delta(heads=4, kv_heads=2, dim=12, vdim=16, conv=3, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def left(heads=6, kv_heads=3, dim=16, vdim=12, scale=0.3, dims=None, base=200.0, scaling=(4.0, 100, 8.0, 1.5)):
    rot = {"base": base, "dims": dim if dims is None else dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}


def right(heads=3, dim=12, vdim=20, cap=9.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def par(a=None, b=None, left_scale=0.8, right_scale=1.3, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a or left(), "right": b or right(), "left_scale": left_scale, "right_scale": right_scale}}


def config(layers, vocab=97, width=64, eps=1e-5):
    return {"architecture": "Virusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# layers of every kind; two layers read an earlier layer's keys and values, past other layers
MIXED = config([par(mlp=dense()),
                att(mlp=dense(56)),
                delta(mlp=dense(24)),
                att(scale=0.4, diff=0.5, kv_from=1, mlp=dense()),
                delta(heads=2, kv_heads=2, dim=24, vdim=20, conv=5),
                att(heads=6, kv_heads=1, dim=10, vdim=24, mlp=dense()),
                att(diff=0.2, kv_from=1),
                par(left(heads=2, kv_heads=2, dim=20, vdim=8, dims=10, base=900.0, scaling=None), right(heads=2, dim=8, vdim=10, cap=4.0), 1.1, 0.6, mlp=dense(16))],
               width=72)


def tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(9900 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


_CACHE = {}


def engine_and_oracle(cfg, seed=0, dtype=torch.float32, edit=None, **engine):
    """(engine, oracle, weights) on identical seeded weights.  ``edit(weights)`` may change them first."""
    from smoltts_b200.lm import VirusunLM
    from smoltts_b200.lm_config import VirusunConfig

    key = (repr(cfg), seed, dtype, edit, tuple(sorted(engine.items())))
    if key not in _CACHE:
        w = random_weights(cfg, seed)
        if edit is not None:
            edit(w)
        kw = dict(max_tokens=1024, max_seqs=4, page_size=16, max_step_tokens=256)
        kw.update(engine)
        model = VirusunLM(VirusunConfig.from_dict(cfg), dtype=dtype, **kw)
        model.load_state_dict(w)
        _CACHE[key] = (model, Oracle(cfg, w), w)
    return _CACHE[key]


def row_errs(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Every row's error of ``got`` against ``want`` relative to the rows' spread (mean taken off both)."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / spread


def rel_err(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest row error."""
    return float(row_errs(got, want).max())


TOL = {torch.float32: 1e-4, torch.bfloat16: 8e-2}


def close_enough(got: torch.Tensor, want: torch.Tensor, dtype, tol=None) -> bool:
    """fp32: every row within the tolerance.  bf16: where a head's two maps nearly cancel, the division by what is left of them
    magnifies the inputs' rounding -- the bulk of the rows is held to the tolerance (the median to half of it, nineteen rows in
    twenty to all of it), not every row."""
    errs = row_errs(got, want)
    tol = tol or TOL[dtype]
    if dtype == torch.float32:
        return float(errs.max()) < tol
    return float(errs.median()) < 0.5 * tol and float((errs > tol).double().mean()) <= 0.05
