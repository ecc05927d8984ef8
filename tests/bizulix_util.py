"""Shared helpers of the Bizulix tests: small configurations, seeded weights, engine + oracle pairs."""
from __future__ import annotations

import torch

from oracle.bizulix_oracle import Oracle, random_weights


def moe(experts=6, top=2, ff=24, shared=16):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3, softcap=9.0, coef=0.5, every=7, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                      "q_temp": {"coef": coef, "every": every}}}


def ret(heads=3, dim=8, vdim=12, decay=None, dims=None, base=50.0, mlp=None):
    return {"type": "retention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.5 + 0.49 * (h + 1) / heads for h in range(heads)],
                      "rot": {"base": base, "dims": dim if dims is None else dims}}}


def config(layers, vocab=97, width=64, eps=1e-5, mult=0.7, cap=6.0, loop=None):
    cfg = {"architecture": "Bizulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_softcap": cap, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# five layers of every kind; layers 1..2 run twice
MIXED = config([ret(mlp=moe()),
                att(mlp=moe(experts=5, top=3, ff=20, shared=28)),
                ret(heads=2, dim=24, vdim=20, dims=10, base=900.0, mlp=moe(experts=4, top=1, ff=16, shared=8)),
                att(heads=3, kv_heads=3, dim=10, vdim=14, scale=0.4, softcap=5.0, coef=0.2, every=11),
                att(heads=6, kv_heads=1, dim=12, vdim=8, coef=0.8, every=20, mlp=moe(experts=3, top=3, ff=12, shared=40))],
               loop=(1, 3, 2))


def tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(9100 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


_CACHE = {}


def engine_and_oracle(cfg, seed=0, dtype=torch.float32, spread=1.0, edit=None, **engine):
    """(engine, oracle, weights) on identical seeded weights.  ``edit(weights)`` may change them first."""
    from smoltts_b200.lm import BizulixLM
    from smoltts_b200.lm_config import BizulixConfig

    key = (repr(cfg), seed, dtype, spread, edit, tuple(sorted(engine.items())))
    if key not in _CACHE:
        w = random_weights(cfg, seed, spread)
        if edit is not None:
            edit(w)
        kw = dict(max_tokens=1024, max_seqs=4, page_size=16, max_step_tokens=256)
        kw.update(engine)
        model = BizulixLM(BizulixConfig.from_dict(cfg), dtype=dtype, **kw)
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
    """fp32: every row within the tolerance.  bf16: a router's close call may go the other way, and the retention layers and
    the attention carry that row's difference on to later rows -- the bulk of the rows is held to the tolerance (the median
    to half of it, nine rows in ten to all of it), not every row."""
    errs = row_errs(got, want)
    tol = tol or TOL[dtype]
    if dtype == torch.float32:
        return float(errs.max()) < tol
    return float(errs.median()) < 0.5 * tol and float((errs > tol).double().mean()) <= 0.1


def clear_routing(w):
    """Router scores far apart, so that bf16 inputs rarely turn a choice."""
    for k in list(w):
        if k.endswith("mlp.router") or k.endswith("mlp.router.b"):
            w[k] = (w[k] * 4.0).bfloat16().float()


def normed(w, token, eps, layer=0):
    """What layer ``layer`` of an unlooped model's first run reads for ``token``: the layer norm of its embedding."""
    from oracle.bizulix_oracle import layer_norm

    return layer_norm(w["embed"][token].double(), w[f"l{layer}.norm1"].double(), w[f"l{layer}.norm1.b"].double(), eps)
