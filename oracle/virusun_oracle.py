"""Plain, slow CPU oracle of the Virusun design, one function per mechanism, written from the design's equations.

It shares no code with the engine: dense loops over tokens and heads in float64, the whole sequence at once or token by
token (``Oracle.step`` carries the caches a token-by-token run needs).  ``cfg`` is the dictionary of ``config.json``,
``w`` maps tensor names to float64 tensors.

Notation.  r(x) = x / sqrt(mean x^2 + eps).  A layer norms only what its sublayers return:
x <- x + r(mixer(x)) * n1,  x <- x + r(ff(x)) * n2.  Mixers:
  * "attention": differential attention.  Every head owns two softmax maps over the same values; with a and b the maps'
    results, o = a - lam b, lam = exp(p1.q1) - exp(p2.q2) + diff from four vectors; then r(o) (1 - diff), times a sigmoid
    gate per channel.  Queries and keys are normed per head and map.  A layer may read the keys and values of an earlier one.
  * "delta": gated delta rule behind short causal convolutions with silu on q, k and v; unit queries and keys;
    S <- g S, S <- S + k (beta (v - S^T k))^T, o = S^T q; r(o) per head, times a weight, times silu of a gate.
  * "parallel": left_scale * left + right_scale * right, both on the same input.  Left: softmax attention with one norm
    over all query (key) rows and a rotation of halves whose frequencies are interpolated ramp-wise (YaRN).  Right: mLSTM,
    a matrix memory with exponential input gate, sigmoid forget gate and a running maximum m that keeps both in range.
Feed-forward: down(silu(gate) * up).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64
UNIT_EPS = 1e-6        # of the delta rule's unit vectors
DEN_EPS = 1e-6         # added to the mLSTM's denominator


def rms_divide(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def softmax_map(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """One query [d] over the visible keys [n, d] and values [n, dv]."""
    s = (k @ q) * scale
    e = torch.exp(s - s.max())
    return (e / e.sum()) @ v


def _extend(past: Optional[dict], k: torch.Tensor, v: torch.Tensor):
    """(all keys, all values, positions before this call); the cache takes the new ones."""
    pos0 = 0
    if past is not None:
        if "k" in past:
            pos0 = past["k"].shape[0]
            k, v = torch.cat([past["k"], k], 0), torch.cat([past["v"], v], 0)
        past["k"], past["v"] = k, v
    return k, v, pos0


def diff_lambda(w: Dict[str, torch.Tensor], p: str, diff: float) -> float:
    return math.exp(float((w[p + "lq1"] * w[p + "lk1"]).sum())) - math.exp(float((w[p + "lq2"] * w[p + "lk2"]).sum())) + diff


def diff_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, past: Optional[dict] = None,
                   lender: Optional[tuple] = None):
    """h [n, width] -> ([n, width], (keys [pos, G, 2, d], values [pos, G, dv])).  ``past``: {"k", "v"} of earlier tokens, extended
    in place.  ``lender``: the keys and values of another layer, up to this call's last token, instead of own ones."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = rms_divide((h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, 2, d), eps) * w[p + "q.norm"]
    if lender is None:
        k = rms_divide((h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, 2, d), eps) * w[p + "k.norm"]
        v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
        k, v, pos0 = _extend(past, k, v)
    else:
        k, v = lender
        pos0 = k.shape[0] - n
    lam = diff_lambda(w, p, m["diff"])
    out = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        i = pos0 + t
        for hh in range(H):
            g = hh // (H // G)
            a, b = (softmax_map(q[t, hh, c], k[:i + 1, g, c], v[:i + 1, g], m["scale"]) for c in (0, 1))
            out[t, hh] = rms_divide(a - lam * b, eps) * (1.0 - m["diff"])
    y = out.reshape(n, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T + w[p + "o.b"], (k, v)


def ramp_frequencies(rot: dict) -> tuple:
    """(frequency of every pair, multiplier of cosine and sine)."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    turns = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / sc["factor"] * ramp + v * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [n, heads, d]: coordinate i < dims / 2 and coordinate i + dims / 2 turn together."""
    out, half = x.clone(), rot["dims"] // 2
    freqs, mult = ramp_frequencies(rot)
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            a = float(pos[t]) * f
            c, s = math.cos(a) * mult, math.sin(a) * mult
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def rotary_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, past: Optional[dict] = None) -> torch.Tensor:
    """h [n, width] -> [n, width]."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    pos0 = past["k"].shape[0] if past is not None and "k" in past else 0
    pos = torch.arange(pos0, pos0 + n)
    q = (rms_divide(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]).view(n, H, d)
    k = (rms_divide(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]).view(n, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    q, k = rotate_halves(q, pos, m["rot"]), rotate_halves(k, pos, m["rot"])
    k, v, pos0 = _extend(past, k, v)
    out = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        i = pos0 + t
        for hh in range(H):
            g = hh // (H // G)
            out[t, hh] = softmax_map(q[t, hh], k[:i + 1, g], v[:i + 1, g], m["scale"])
    return out.reshape(n, H * dv) @ w[p + "o"].T + w[p + "o.b"]


def memory_denominator(dot: torch.Tensor, m: torch.Tensor) -> torch.Tensor:
    """dot: key sum . query, m: running maximum (the memory holds everything times e^-m)."""
    return torch.maximum(dot.abs(), torch.exp(-m)) + DEN_EPS


def mlstm(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, past: Optional[dict] = None) -> torch.Tensor:
    """h [n, width] -> [n, width].  ``past``: {"S": [heads, d, dv], "n": [heads, d], "m": [heads]}, updated in place."""
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    n = h.shape[0]
    q = (h @ w[p + "q"].T).view(n, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(n, H, d)
    v = (h @ w[p + "v"].T).view(n, H, dv)
    i_log = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f_log = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    if past is not None and "S" in past:
        S, nn, mx = past["S"].clone(), past["n"].clone(), past["m"].clone()
    else:
        S, nn, mx = torch.zeros(H, d, dv, dtype=F), torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F)
    o = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        new = torch.maximum(f_log[t] + mx, i_log[t])
        keep, write = torch.exp(f_log[t] + mx - new), torch.exp(i_log[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nn = keep[:, None] * nn + write[:, None] * k[t]
        mx = new
        o[t] = (S * q[t][:, :, None]).sum(1) / memory_denominator((nn * q[t]).sum(-1), mx)[:, None]
    if past is not None:
        past["S"], past["n"], past["m"] = S, nn, mx
    y = rms_divide(o, eps).reshape(n, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def short_conv(z: torch.Tensor, weight: torch.Tensor, before: torch.Tensor) -> torch.Tensor:
    """z [n, channels], ``before`` [taps - 1, channels] the inputs ahead of them -> silu of the causal convolution."""
    taps = weight.shape[1]
    line = torch.cat([before, z], 0)
    return silu(torch.stack([sum(weight[:, j] * line[t + j] for j in range(taps)) for t in range(z.shape[0])]))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def gated_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, past: Optional[dict] = None) -> torch.Tensor:
    """h [n, width] -> [n, width].  ``past``: {"S": [heads, d, dv], "q"/"k"/"v": last inputs of the convolutions}, updated in place."""
    H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    n = h.shape[0]
    conv = {}
    for nm in ("q", "k", "v"):
        z = h @ w[p + nm].T
        before = past[nm] if past is not None and nm in past else torch.zeros(taps - 1, z.shape[1], dtype=F)
        conv[nm] = short_conv(z, w[p + nm + ".conv"], before)
        if past is not None:
            past[nm] = torch.cat([before, z], 0)[z.shape[0]:]
    q, k = unit(conv["q"].view(n, G, d)) * d ** -0.5, unit(conv["k"].view(n, G, d))
    v = conv["v"].view(n, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * torch.nn.functional.softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    S = past["S"].clone() if past is not None and "S" in past else torch.zeros(H, d, dv, dtype=F)
    o = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        for hh in range(H):
            kk, qq = k[t, hh // (H // G)], q[t, hh // (H // G)]
            A = g[t, hh] * S[hh]
            A = A + torch.outer(kk, beta[t, hh] * (v[t, hh] - A.T @ kk))
            S[hh] = A
            o[t, hh] = A.T @ qq
    if past is not None:
        past["S"] = S
    y = rms_divide(o, eps) * w[p + "norm"]
    return (y.reshape(n, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


class Oracle:
    def __init__(self, cfg: dict, weights: Dict[str, torch.Tensor]):
        self.cfg = cfg
        self.w = {k: v.to(F) for k, v in weights.items()}
        self.reset()

    def reset(self) -> None:
        self.past = [dict() for _ in self.cfg["layers"]]

    def _run(self, tokens, past, layers_out=None) -> torch.Tensor:
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)].clone()
        lent: List[Optional[tuple]] = []                     # keys and values of every attention layer so far
        for i, L in enumerate(cfg["layers"]):
            p, m = f"l{i}.", L["mixer"]
            ps = past[i] if past is not None else None
            kv = None
            if L["type"] == "attention":
                src = m.get("kv_from")
                y, kv = diff_attention(x, w, p + "mix.", m, eps, ps, None if src is None else lent[src])
            elif L["type"] == "delta":
                y = gated_delta(x, w, p + "mix.", m, eps, ps)
            elif L["type"] == "parallel":
                a, b = (ps.setdefault("left", {}), ps.setdefault("right", {})) if ps is not None else (None, None)
                y = m["left_scale"] * rotary_attention(x, w, p + "mix.left.", m["left"], eps, a) + \
                    m["right_scale"] * mlstm(x, w, p + "mix.right.", m["right"], eps, b)
            else:
                raise ValueError(L["type"])
            lent.append(kv)
            x = x + rms_divide(y, eps) * w[p + "norm1"]
            if L.get("mlp"):
                x = x + rms_divide(feed_forward(x, w, p + "mlp."), eps) * w[p + "norm2"]
            if layers_out is not None:
                layers_out.append(x.clone())
        return (rms_divide(x, eps) * w["final.norm"]) @ w["head"].T

    def forward(self, tokens, layers_out=None) -> torch.Tensor:
        """Logits [n, vocab] of a whole sequence from position 0 (no state is kept)."""
        return self._run(tokens, None, layers_out)

    def step(self, tokens) -> torch.Tensor:
        """Logits of the next tokens of the sequence this oracle has seen so far (``reset`` starts a new one)."""
        return self._run(tokens, self.past)


def random_weights(cfg: dict, seed: int = 0, scale: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random bf16-representable weights for ``cfg`` (names and shapes of a checkpoint)."""
    gen = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    out: Dict[str, torch.Tensor] = {}

    def mat(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=gen) * (s * scale / math.sqrt(i))

    def vec(name, n, mean=0.0, s=0.3):
        out[name] = mean + torch.randn(n, generator=gen) * s

    out["embed"] = torch.randn(V, D, generator=gen)
    mat("head", V, D, 2.0)
    vec("final.norm", D, 1.0, 0.1)

    def attention_side(q, H, G, rows_q, rows_k, dv):
        for nm, rows in (("q", rows_q), ("k", rows_k), ("v", G * dv)):
            if nm == "q" or rows_k:
                mat(q + nm, rows, D, 1.0)
                vec(q + nm + ".b", rows)
        mat(q + "o", D, H * dv)
        vec(q + "o.b", D)

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        vec(p + "norm1", D, 0.6, 0.1)
        q = p + "mix."
        if L["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            own = m.get("kv_from") is None
            attention_side(q, H, G, 2 * H * d, 2 * G * d if own else 0, dv)
            vec(q + "q.norm", d, 1.2, 0.2)
            if own:
                vec(q + "k.norm", d, 1.2, 0.2)
            for nm in ("lq1", "lk1", "lq2", "lk2"):
                vec(q + nm, d, 0.0, 0.5 / d ** 0.25)
            mat(q + "g", H * dv, D)
        elif L["type"] == "delta":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for nm, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(q + nm, rows, D)
                mat(q + nm + ".conv", rows, m["conv"], 1.5)
            mat(q + "b", H, D, 1.5)
            mat(q + "a", H, D, 1.5)
            mat(q + "g", H * dv, D)
            mat(q + "o", D, H * dv)
            vec(q + "A_log", H, -1.5, 1.0)
            vec(q + "dt_bias", H, -1.0, 0.5)
            vec(q + "norm", dv, 1.0, 0.2)
        else:
            a, r = m["left"], m["right"]
            attention_side(q + "left.", a["heads"], a["kv_heads"], a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["vdim"])
            vec(q + "left.q.norm", a["heads"] * a["dim"], 1.0, 0.2)
            vec(q + "left.k.norm", a["kv_heads"] * a["dim"], 1.0, 0.2)
            t, H, d, dv = q + "right.", r["heads"], r["dim"], r["vdim"]
            for nm, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                mat(t + nm, rows, D)
            mat(t + "o", D, H * dv)
            vec(t + "norm", H * dv, 1.0, 0.2)
            for nm, mean in (("i", -1.0), ("f", 3.0)):
                mat(t + nm, H, D)
                vec(t + nm + ".b", H, mean, 1.0)
        if L.get("mlp"):
            ff = L["mlp"]["ff"]
            vec(p + "norm2", D, 0.6, 0.1)
            mat(p + "mlp.gate", ff, D); mat(p + "mlp.up", ff, D); mat(p + "mlp.down", D, ff)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in out.items()}
