"""Plain, slow CPU oracle of the Bizulix design, one function per mechanism, written from the design's equations.

It shares no code with the engine: dense loops over tokens and heads in float64, the whole sequence at once or token by
token (``Oracle.step`` carries the caches a token-by-token run needs).  ``cfg`` is the dictionary of ``config.json``,
``w`` maps tensor names to float64 tensors.

Notation.  A layer has ONE norm whose result both sublayers read:  h = n(x),  x <- x + m (mixer(h) + ff(h)),  with the
layer norm n(x) = (x - mean) / sqrt(mean of squared deviations + eps) * weight + bias.  A span of layers may run several
times with the same weights; every pass, the first one too, starts with x <- M [x ; e], e being the embedding output and
M a [width, 2 width] matrix.  Mixers:
  * "attention": grouped-query softmax attention without biases, rotation or window; the query at position p is
    multiplied by 1 + coef ln(floor((p + 1) / every) + 1); score = q.k scale, bent to cap tanh(score / cap);
  * "retention": linear attention with one constant decay per head, S <- decay S + k v^T, o = S^T q; q and k rotated on
    their leading coordinates (coordinate i paired with i + dims / 2), k divided by sqrt(dim) after that; each head's o
    divided by its root mean square, times silu of a gate per channel.
Feed-forward: a routed mixture of down(silu(gate) * up) experts -- the `top` largest router logits (bias included) are
chosen, their weights are the softmax over the chosen logits -- plus a shared expert of the same form whose result is
multiplied by one sigmoid gate per token.  The logits are bent to cap tanh(logit / cap).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_divide(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, eps: float) -> torch.Tensor:
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * weight + bias


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def bend(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x / cap)


def query_temperature(pos: int, coef: float, every: int) -> float:
    return 1.0 + coef * math.log((pos + 1) // every + 1)


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [n, heads, d]: coordinate i < dims / 2 and coordinate i + dims / 2 turn together by pos * base^(-2i/dims)."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = float(pos[t]) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, past: Optional[dict] = None) -> torch.Tensor:
    """h [n, width] -> [n, width].  ``past``: {"k": [pos0, G, d], "v": [pos0, G, dv]}, extended in place."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = (h @ w[p + "q"].T).view(n, H, d)
    k = (h @ w[p + "k"].T).view(n, G, d)
    v = (h @ w[p + "v"].T).view(n, G, dv)
    pos0 = past["k"].shape[0] if past is not None and "k" in past else 0
    if past is not None:
        if "k" in past:
            k = torch.cat([past["k"], k], 0)
            v = torch.cat([past["v"], v], 0)
        past["k"], past["v"] = k, v
    out = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        i = pos0 + t
        warm = query_temperature(i, m["q_temp"]["coef"], m["q_temp"]["every"])
        for hh in range(H):
            g = hh // (H // G)
            s = bend((k[:i + 1, g] @ (q[t, hh] * warm)) * m["scale"], m["softcap"])
            e = torch.exp(s - s.max())
            out[t, hh] = (e / e.sum()) @ v[:i + 1, g]
    return out.reshape(n, H * dv) @ w[p + "o"].T


def retention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, past: Optional[dict] = None) -> torch.Tensor:
    """h [n, width] -> [n, width].  ``past``: {"S": [heads, d, dv], "n": positions seen}, updated in place."""
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    pos0 = past.get("n", 0) if past is not None else 0
    pos = torch.arange(pos0, pos0 + n)
    q = rotate_halves((h @ w[p + "q"].T).view(n, H, d), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves((h @ w[p + "k"].T).view(n, H, d), pos, m["rot"]["dims"], m["rot"]["base"]) / math.sqrt(d)
    v = (h @ w[p + "v"].T).view(n, H, dv)
    S = past["S"].clone() if past is not None and "S" in past else torch.zeros(H, d, dv, dtype=F)
    decay = torch.tensor(m["decay"], dtype=F)[:, None, None]
    o = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    if past is not None:
        past["S"], past["n"] = S, pos0 + n
    y = rms_divide(o, eps).reshape(n, H * dv) * silu(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h: torch.Tensor, w_router: torch.Tensor, bias: torch.Tensor, top: int):
    """-> (chosen experts, their weights), one list entry / row per token; the best choice first."""
    z = h @ w_router.T + bias
    ids, wts = [], []
    for t in range(h.shape[0]):
        pick = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:top]
        e = torch.exp(z[t, pick] - z[t, pick].max())
        ids.append(pick)
        wts.append(e / e.sum())
    return ids, torch.stack(wts)


def feed_forward(h, w, p, mlp):
    ids, wts = route(h, w[p + "router"], w[p + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k, e in enumerate(ids[t]):
            out[t] += wts[t, k] * gated_unit(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * gated_unit(h, w, p + "shared.")
    return out


def layer_runs(cfg: dict) -> List[tuple]:
    """(layer index, whether a pass of the loop starts with it) of every layer run, in execution order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(a)]
    for _ in range(times):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


class Oracle:
    def __init__(self, cfg: dict, weights: Dict[str, torch.Tensor]):
        self.cfg = cfg
        self.w = {k: v.to(F) for k, v in weights.items()}
        self.runs = layer_runs(cfg)
        self.reset()

    def reset(self) -> None:
        self.past = [dict() for _ in self.runs]

    def _run(self, tokens, past, layers_out=None) -> torch.Tensor:
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x0 = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
        x = x0.clone()
        for n, (i, opens) in enumerate(self.runs):
            L, p = cfg["layers"][i], f"l{i}."
            if opens:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T
            h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
            ps = past[n] if past is not None else None
            if L["type"] == "attention":
                y = attention(h, w, p + "mix.", L["mixer"], ps)
            elif L["type"] == "retention":
                y = retention(h, w, p + "mix.", L["mixer"], eps, ps)
            else:
                raise ValueError(L["type"])
            if L.get("mlp"):
                y = y + feed_forward(h, w, p + "mlp.", L["mlp"])
            x = x + cfg["residual_mult"] * y
            if layers_out is not None:
                layers_out.append(x.clone())
        return bend(layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T, cfg["logit_softcap"])

    def forward(self, tokens, layers_out=None) -> torch.Tensor:
        """Logits [n, vocab] of a whole sequence from position 0 (no state is kept)."""
        return self._run(tokens, None, layers_out)

    def step(self, tokens) -> torch.Tensor:
        """Logits of the next tokens of the sequence this oracle has seen so far (``reset`` starts a new one)."""
        return self._run(tokens, self.past)


def random_weights(cfg: dict, seed: int = 0, scale: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random bf16-representable weights for ``cfg`` (names and shapes of a checkpoint)."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    out: Dict[str, torch.Tensor] = {}

    def mat(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=g) * (s * scale / math.sqrt(i))

    def norm(name):
        out[name] = 1.0 + torch.randn(D, generator=g) * 0.1
        out[name + ".b"] = torch.randn(D, generator=g) * 0.1

    out["embed"] = torch.randn(V, D, generator=g)
    mat("head", V, D, 2.0)
    norm("final.norm")
    if cfg.get("loop"):
        mat("loop.in", D, 2 * D)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        kv = m["kv_heads"] if L["type"] == "attention" else m["heads"]
        mat(p + "mix.q", m["heads"] * m["dim"], D, 1.5)
        mat(p + "mix.k", kv * m["dim"], D, 1.5)
        mat(p + "mix.v", kv * m["vdim"], D)
        if L["type"] == "retention":
            mat(p + "mix.g", m["heads"] * m["vdim"], D)
        mat(p + "mix.o", D, m["heads"] * m["vdim"])
        mlp = L.get("mlp")
        if mlp:
            for e in range(mlp["router"]["experts"]):
                for nm, o, j in (("gate", mlp["expert"]["ff"], D), ("up", mlp["expert"]["ff"], D), ("down", D, mlp["expert"]["ff"])):
                    mat(f"{p}mlp.e{e}.{nm}", o, j)
            mat(p + "mlp.router", mlp["router"]["experts"], D, 2.0)
            out[p + "mlp.router.b"] = torch.randn(mlp["router"]["experts"], generator=g) * 0.5
            if mlp.get("shared"):
                ff = mlp["shared"]["ff"]
                mat(p + "mlp.shared.gate", ff, D); mat(p + "mlp.shared.up", ff, D); mat(p + "mlp.shared.down", D, ff)
                mat(p + "mlp.shared.sg", 1, D, 2.0)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in out.items()}
