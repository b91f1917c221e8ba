"""A slow float64 restatement of the Redalix design, one function per mechanism, written from its equations.  It takes a
configuration dictionary and a name -> tensor mapping and shares no code with the package: whole sequences, visibility as an
explicit matrix, a sink as one more column of the scores, every recurrence token by token, experts run token by token.

Notation: h is what a layer's sublayers read [T, W]; linear weights are [out, in] and act as W h; positions count from 0.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def _w(sd: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return sd[name].to(F64)


# ---- element-wise pieces ---------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def grouped_rms_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """The channels in ``groups`` equal neighbourhoods, each divided by its own root mean square."""
    T, C = x.shape
    return unit_rms(x.view(T, groups, C // groups), eps).reshape(T, C) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def squared_relu(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


def causal_conv(u: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y if bias is None else y + bias


# ---- rotary ----------------------------------------------------------------------------------------------------------
def rotation_angles(rot: Dict[str, Any]) -> Tuple[List[float], float]:
    """(angle per position of every pair, factor on cos and sin)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_that_turns(times: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(sc["slow"]))), dims - 1)
    out = []
    for i, v in enumerate(f):
        slowed = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(slowed * v / factor + (1.0 - slowed) * v)
    return out, 1.0 + 0.1 * math.log(factor)


def rotate_neighbours(x: torch.Tensor, positions: List[int], rot: Optional[Dict[str, Any]]) -> torch.Tensor:
    """x [T, heads, D]: coordinates 2i and 2i + 1 turn together, the coordinates past ``dims`` pass."""
    if not rot:
        return x
    f, mul = rotation_angles(rot)
    a = torch.tensor(positions, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    c, s = (torch.cos(a) * mul)[:, None, :], (torch.sin(a) * mul)[:, None, :]
    out = x.clone()
    n = 2 * len(f)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# ---- visibility and softmax ------------------------------------------------------------------------------------------
def visible(T: int, size: int, keep: int = 0) -> torch.Tensor:
    """[T, T] bool: row i sees column j -- not later, and within ``size`` positions (0: any) or among the first ``keep``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size <= 0 else (i - j < size)
    return (j <= i) & (near | (j < keep))


def softmax_rows(s: torch.Tensor, seen: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """s [T, T] -> weights; ``sink``: the score of one more column, whose weight goes nowhere."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, sink.reshape(1, 1).expand(s.shape[0], 1)], 1), -1)[:, :-1]


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int, keep: int = 0,
           sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] of one sequence -> [T, H, V]; sink [H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, size, keep)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_rows(q[:, h] @ k[:, g].T * scale, seen, None if sink is None else sink[h]) @ v[:, g]
    return out


# ---- attention mixers ------------------------------------------------------------------------------------------------
def _heads(m: Dict[str, Any]) -> Tuple[int, int, int, int]:
    H, D = int(m["heads"]), int(m["dim"])
    return H, int(m.get("kv_heads", H)), D, int(m.get("vdim", D))


def kept_window_attention(m: Dict[str, Any], sd, p: str, h: torch.Tensor) -> torch.Tensor:
    """No biases, no rotation; a window beside the first kept tokens; a learned sink per head."""
    T, (H, G, D, V) = h.shape[0], _heads(m)
    q, k, v = (h @ _w(sd, p + n).T for n in ("q", "k", "v"))
    mask = m.get("mask") or {}
    o = attend(q.view(T, H, D), k.view(T, G, D), v.view(T, G, V), float(m["scale"]), int(mask.get("size", 0) or 0),
               int(mask.get("keep_first", 0) or 0), _w(sd, p + "sink"))
    return o.reshape(T, H * V) @ _w(sd, p + "o").T


def gated_window_attention(m: Dict[str, Any], sd, p: str, h: torch.Tensor) -> torch.Tensor:
    """Biases on q, k, v; rotation; a window; every head's output times one sigmoid gate."""
    T, (H, G, D, V) = h.shape[0], _heads(m)
    q, k, v = (h @ _w(sd, p + n).T + _w(sd, p + n + ".b") for n in ("q", "k", "v"))
    at = list(range(T))
    q, k = rotate_neighbours(q.view(T, H, D), at, m.get("rot")), rotate_neighbours(k.view(T, G, D), at, m.get("rot"))
    o = attend(q, k, v.view(T, G, V), float(m["scale"]), int((m.get("mask") or {}).get("size", 0) or 0))
    o = o * sigmoid(h @ _w(sd, p + "g").T)[:, :, None]
    return o.reshape(T, H * V) @ _w(sd, p + "o").T


# ---- recurrent mixers ------------------------------------------------------------------------------------------------
def gate_blocks(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C] in w.shape[0] equal parts, each through its own square matrix and bias, then a sigmoid."""
    T, n = u.shape[0], w.shape[0]
    parts = u.view(T, n, -1)
    return sigmoid(torch.stack([parts[:, i] @ w[i].T + b[i] for i in range(n)], 1).reshape(T, -1))


def linear_recurrent_unit(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor,
                          S: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam) -> (S of every row, S after)."""
    a = torch.exp(-8.0 * r * softplus(lam))
    S = torch.zeros(u.shape[1], dtype=F64) if S is None else S.clone()
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + torch.sqrt(1.0 - a[t] * a[t]) * i[t] * u[t]
        out[t] = S
    return out, S


def recurrent_block(m: Dict[str, Any], sd, p: str, h: torch.Tensor) -> torch.Tensor:
    y = gelu_tanh(h @ _w(sd, p + "y").T + _w(sd, p + "y.b"))
    u = causal_conv(h @ _w(sd, p + "x").T + _w(sd, p + "x.b"), _w(sd, p + "conv"), _w(sd, p + "conv.b"))
    r, i = (gate_blocks(u, _w(sd, p + n), _w(sd, p + n + ".b")) for n in ("ra", "ri"))
    S, _ = linear_recurrent_unit(u, r, i, _w(sd, p + "lam"))
    return (S * y) @ _w(sd, p + "o").T


def state_space(x: torch.Tensor, dt: torch.Tensor, B: torch.Tensor, C: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor,
                S: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """x [T, H, V], dt [T, H] (after softplus), B, C [T, G, N], A_log, D [H] -> (y [T, H, V], state [H, N, V] after)."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, V, dtype=F64) if S is None else S.clone()
    y = torch.zeros_like(x)
    of = [h // (H // G) for h in range(H)]
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][of][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, C[t][of]) + D[:, None] * x[t]
    return y, S


def mamba2(m: Dict[str, Any], sd, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, V, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner, n_bc = H * V, G * N
    z, xbc, dt = (h @ _w(sd, p + "in").T).split([inner, inner + 2 * n_bc, H], 1)
    xbc = silu(causal_conv(xbc, _w(sd, p + "conv"), _w(sd, p + "conv.b")))
    x, B, C = xbc.split([inner, n_bc, n_bc], 1)
    y, _ = state_space(x.reshape(T, H, V), softplus(dt + _w(sd, p + "dt_bias")), B.reshape(T, G, N), C.reshape(T, G, N),
                       _w(sd, p + "A_log"), _w(sd, p + "D"))
    y = y.reshape(T, inner) * silu(z)
    return grouped_rms_norm(y, _w(sd, p + "norm"), int(m.get("norm_groups", 1)), eps) @ _w(sd, p + "o").T


def parallel_mixer(m: Dict[str, Any], sd, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    left = rms_norm(kept_window_attention(m["left"], sd, p + "left.", h), _w(sd, p + "left.out"), eps)
    right = rms_norm(recurrent_block(m["right"], sd, p + "right.", h), _w(sd, p + "right.out"), eps)
    return 0.5 * (left + right)


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def dense(sd, p: str, h: torch.Tensor) -> torch.Tensor:
    return gelu_tanh(h @ _w(sd, p + "up").T) @ _w(sd, p + "down").T


def expert(sd, p: str, h: torch.Tensor) -> torch.Tensor:
    return squared_relu(h @ _w(sd, p + "up").T) @ _w(sd, p + "down").T


def table_mixture(f: Dict[str, Any], sd, p: str, h: torch.Tensor, tokens: List[int]) -> torch.Tensor:
    """The token's id picks its experts from a table; all of them weigh the same."""
    top = int(f["router"]["top"])
    table = sd[p + "table"].tolist()
    y = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            y[t] += expert(sd, p + f"e{e}.", h[t:t + 1])[0] / top
    if f.get("shared"):
        y = y + sigmoid(h @ _w(sd, p + "shared.sg").T) * expert(sd, p + "shared.", h)
    return y


# ---- the model -------------------------------------------------------------------------------------------------------
def forward(cfg: Dict[str, Any], sd: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """-> logits float64 [T, vocab]; ``taps`` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = _w(sd, "embed")[tokens]
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = rms_norm(x, _w(sd, p + "norm1"), eps)
        if L["type"] == "parallel":
            y = parallel_mixer(m, sd, p + "mix.", h, eps)
        elif L["type"] == "attention":
            y = gated_window_attention(m, sd, p + "mix.", h)
        elif L["type"] == "mamba2":
            y = mamba2(m, sd, p + "mix.", h, eps)
        else:
            raise ValueError(L["type"])
        f = L.get("mlp")
        if f:
            y = y + (dense(sd, p + "mlp.", h) if f["kind"] == "dense" else table_mixture(f, sd, p + "mlp.", h, tokens))
        x = x + y
        if taps is not None:
            taps.append(x.clone())
    return rms_norm(x, _w(sd, "final.norm"), eps) @ _w(sd, "head").T


# ---- small configurations and random weights for the tests -----------------------------------------------------------
def make_config(layers=("mamba:dense", "pair:moe", "attn:moe", "pair", "mamba:moe", "attn:dense"), width=48, vocab=97, eps=1e-5,
                a_heads=4, a_kv_heads=2, a_dim=12, a_vdim=10, a_window=9, a_rot_dims=8, a_base=700.0, a_scaling=(4.0, 24.0, 2.0, 0.25),
                p_heads=6, p_kv_heads=3, p_dim=10, p_vdim=6, p_window=11, p_keep=3, r_width=40, r_blocks=5, r_conv=3,
                m_heads=6, m_vdim=7, m_state=9, m_groups=3, m_norm_groups=2, m_conv=4, ff=52, experts=5, top=2, e_ff=24,
                shared_ff=20) -> Dict[str, Any]:
    """layers: "<mixer>[:<feed-forward>]" with mixers attn, pair, mamba and feed-forwards dense, moe, or none."""
    out = []
    for spec in layers:
        kind, _, mlp = spec.partition(":")
        if kind == "attn":
            m = {"heads": a_heads, "kv_heads": a_kv_heads, "dim": a_dim, "vdim": a_vdim, "scale": 0.33, "mask": {"size": a_window}}
            if a_rot_dims:
                m["rot"] = {"base": a_base, "dims": a_rot_dims}
                if a_scaling:
                    m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), a_scaling))
            layer = {"type": "attention", "mixer": m}
        elif kind == "pair":
            left = {"heads": p_heads, "kv_heads": p_kv_heads, "dim": p_dim, "vdim": p_vdim, "scale": 0.36,
                    "mask": {"size": p_window, "keep_first": p_keep}}
            layer = {"type": "parallel", "mixer": {"left": left, "right": {"blocks": r_blocks, "conv": r_conv, "width": r_width}}}
        else:
            layer = {"type": "mamba2", "mixer": {"heads": m_heads, "vdim": m_vdim, "state": m_state, "groups": m_groups,
                                                 "norm_groups": m_norm_groups, "conv": m_conv}}
        layer["mlp"] = None
        if mlp == "dense":
            layer["mlp"] = {"kind": "dense", "ff": ff}
        elif mlp:
            layer["mlp"] = {"kind": "moe", "expert": {"ff": e_ff}, "router": {"experts": experts, "top": top}}
            if shared_ff:
                layer["mlp"]["shared"] = {"ff": shared_ff}
        out.append(layer)
    return {"architecture": "Redalix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}


def make_weights(cfg: Dict[str, Any], seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights with the checkpoint's names, scaled so that every mechanism matters in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, vocab = int(cfg["width"]), int(cfg["vocab"])

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g) * std + mean).to(torch.bfloat16)

    def lin(n, k, gain=1.0):
        return rnd(n, k, std=gain * k ** -0.5)

    sd = {"embed": rnd(vocab, W), "head": lin(vocab, W), "final.norm": rnd(W, std=0.2, mean=1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        sd[p + "norm1"] = rnd(W, std=0.2, mean=1.0)
        if L["type"] == "attention":
            H, G, D, V = _heads(m)
            for n, c in (("q", H * D), ("k", G * D), ("v", G * V)):
                sd[x + n], sd[x + n + ".b"] = lin(c, W), rnd(c, std=0.5)
            sd[x + "g"], sd[x + "o"] = lin(H, W, 1.5), lin(W, H * V)
        elif L["type"] == "parallel":
            H, G, D, V = _heads(m["left"])
            C, n = int(m["right"]["width"]), int(m["right"]["blocks"])
            for nm, c in (("q", H * D), ("k", G * D), ("v", G * V)):
                sd[x + "left." + nm] = lin(c, W)
            sd[x + "left.sink"], sd[x + "left.o"] = rnd(H, mean=1.0), lin(W, H * V)
            for nm in ("y", "x"):
                sd[x + f"right.{nm}"], sd[x + f"right.{nm}.b"] = lin(C, W), rnd(C, std=0.4)
            sd[x + "right.conv"], sd[x + "right.conv.b"] = rnd(C, int(m["right"]["conv"]), std=0.6), rnd(C, std=0.3)
            for nm in ("ra", "ri"):
                sd[x + f"right.{nm}"], sd[x + f"right.{nm}.b"] = rnd(n, C // n, C // n, std=1.5 * (C // n) ** -0.5), rnd(n, C // n, std=0.4)
            sd[x + "right.lam"], sd[x + "right.o"] = rnd(C, std=1.0, mean=-4.0), lin(W, C)
            sd[x + "left.out"], sd[x + "right.out"] = rnd(W, std=0.2, mean=0.8), rnd(W, std=0.2, mean=0.8)
        else:
            H, V, N, G, K = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv"))
            C = H * V + 2 * G * N
            sd[x + "in"], sd[x + "conv"], sd[x + "conv.b"] = lin(H * V + C + H, W, 1.3), rnd(C, K, std=0.6), rnd(C, std=0.3)
            sd[x + "dt_bias"], sd[x + "A_log"], sd[x + "D"] = rnd(H, std=0.7, mean=-2.0), rnd(H, std=0.6), rnd(H)
            sd[x + "norm"], sd[x + "o"] = rnd(H * V, std=0.2, mean=1.0), lin(W, H * V)
        f = L.get("mlp")
        if not f:
            continue
        y = p + "mlp."
        if f["kind"] == "dense":
            sd[y + "up"], sd[y + "down"] = lin(int(f["ff"]), W), lin(W, int(f["ff"]))
            continue
        E, top = int(f["router"]["experts"]), int(f["router"]["top"])
        for e in range(E):
            sd[y + f"e{e}.up"], sd[y + f"e{e}.down"] = lin(int(f["expert"]["ff"]), W), lin(W, int(f["expert"]["ff"]))
        sd[y + "table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)
        if f.get("shared"):
            sff = int(f["shared"]["ff"])
            sd[y + "shared.up"], sd[y + "shared.down"], sd[y + "shared.sg"] = lin(sff, W), lin(W, sff), lin(1, W, 2.0)
    return sd
