"""A slow float64 restatement of the Zopipel design, one function per mechanism, written from its equations.  It takes a
configuration dictionary and a name -> tensor mapping and shares no code with the package: whole sequences, keys and values
formed explicitly per head, visibility as an explicit matrix, every stream kept as a tensor of its own.

Notation: h is what a sublayer reads [T, W]; linear weights are [out, in] and act as W h; positions count from 0.
"""
from __future__ import annotations

import math
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def _w(sd: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return sd[name].to(F64)


# ---- element-wise pieces ---------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j) with zeros before the start (the last column weighs
    the current token)."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


# ---- hyper-connections -----------------------------------------------------------------------------------------------
def read_streams(xs: List[torch.Tensor], coef: torch.Tensor) -> torch.Tensor:
    """What a sublayer takes from the streams: sum_s coef[s] x_s."""
    u = torch.zeros_like(xs[0])
    for s, x in enumerate(xs):
        u = u + coef[s] * x
    return u


def write_streams(xs: List[torch.Tensor], y: torch.Tensor, mix: torch.Tensor, out: torch.Tensor) -> List[torch.Tensor]:
    """x_t <- sum_s mix[s, t] x_s + out[t] y, every new stream formed from the old ones."""
    new = []
    for t in range(len(xs)):
        v = out[t] * y
        for s, x in enumerate(xs):
            v = v + mix[s, t] * x
        new.append(v)
    return new


# ---- rotary ----------------------------------------------------------------------------------------------------------
def rotation_angles(rot: Dict[str, Any]) -> List[float]:
    """Radians per position of every pair: base^(-2i / dims), divided by the scaling's factor if there is one."""
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_halves(x: torch.Tensor, positions: List[int], rot: Dict[str, Any]) -> torch.Tensor:
    """x [T, ..., D]: coordinates (i, i + dims / 2), i < dims / 2, turn together; coordinates from dims on pass."""
    half = int(rot["dims"]) // 2
    f = rotation_angles(rot)
    out = x.clone()
    for i in range(half):
        a = torch.tensor([p * f[i] for p in positions], dtype=F64).view(-1, *([1] * (x.dim() - 2)))
        c, s = torch.cos(a), torch.sin(a)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ---- visibility ------------------------------------------------------------------------------------------------------
def visible(T: int, size: int) -> torch.Tensor:
    """[T, T] booleans: position i (row) sees j (column) when 0 <= i - j and, with a window, i - j < size."""
    i, j = torch.arange(T).view(-1, 1), torch.arange(T).view(1, -1)
    ok = j <= i
    return ok & (i - j < size) if size > 0 else ok


def softmax_rows(s: torch.Tensor, ok: torch.Tensor, sink: bool) -> torch.Tensor:
    """Weights over the visible keys of every row; sink: one is added to the denominator (a key of score 0 without a value)."""
    s = torch.where(ok, s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values
    if sink:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink:
        den = den + torch.exp(-top)
    return e / den


# ---- mixers ----------------------------------------------------------------------------------------------------------
def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale, size: int, sink: bool) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] of ONE sequence from position 0 -> [T, H, V]; scale: a number or one per head."""
    T, H, _ = q.shape
    G, V = k.shape[1], v.shape[2]
    ok = visible(T, size)
    out = torch.zeros(T, H, V, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        sc = scale[hh] if isinstance(scale, torch.Tensor) else scale
        out[:, hh] = softmax_rows((q[:, hh] @ k[:, g].T) * sc, ok, sink) @ v[:, g]
    return out


def _bias(sd, name: str):
    return _w(sd, name + ".b") if (name + ".b") in sd else 0.0


def attention(m: Dict[str, Any], sd, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Grouped heads with projection biases, rotated queries and keys, values of unit RMS per head, a number per head on the
    scores, and a softmax whose denominator has one added."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m.get("vdim", m["dim"]))
    q = (h @ _w(sd, p + "q").T + _bias(sd, p + "q")).view(T, H, D)
    k = (h @ _w(sd, p + "k").T + _bias(sd, p + "k")).view(T, G, D)
    v = unit_rms((h @ _w(sd, p + "v").T + _bias(sd, p + "v")).view(T, G, V), eps)
    if m.get("rot"):
        q, k = rotate_halves(q, list(range(T)), m["rot"]), rotate_halves(k, list(range(T)), m["rot"])
    size = int((m.get("mask") or {}).get("size", 0) or 0)
    o = attend(q, k, v, float(m["scale"]) * _w(sd, p + "temp"), size, True)
    return o.reshape(T, H * V) @ _w(sd, p + "o").T + _bias(sd, p + "o")


def latent_rows(m: Dict[str, Any], sd, p: str, h: torch.Tensor, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """(normed latent [T, kv_rank], rotated shared key part [T, rot_dim]): all that a token leaves behind."""
    R, Rd = int(m["kv_rank"]), int(m.get("rot_dim", 0) or 0)
    d = h @ _w(sd, p + "dkv").T
    c = rms_norm(d[:, :R], _w(sd, p + "dkv.norm"), eps)
    kr = d[:, R:R + Rd]
    if Rd and m.get("rot"):
        kr = rotate_halves(kr, list(range(h.shape[0])), m["rot"])
    return c, kr


def latent_attention(m: Dict[str, Any], sd, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Queries through a normed latent; per head keys [W_uk c | shared rotated part] and values W_uv c, formed explicitly; a
    window; one sigmoid gate per head."""
    T = h.shape[0]
    H, D, Rd, V = int(m["heads"]), int(m["dim"]), int(m.get("rot_dim", 0) or 0), int(m.get("vdim", m["dim"]))
    cq = rms_norm(h @ _w(sd, p + "dq").T, _w(sd, p + "dq.norm"), eps)
    q = (cq @ _w(sd, p + "uq").T).view(T, H, D + Rd)
    qu, qr = q[:, :, :D], q[:, :, D:]
    if Rd and m.get("rot"):
        qr = rotate_halves(qr, list(range(T)), m["rot"])
    c, kr = latent_rows(m, sd, p, h, eps)
    ku = (c @ _w(sd, p + "uk").T).view(T, H, D)
    vv = (c @ _w(sd, p + "uv").T).view(T, H, V)
    k = torch.cat([ku, kr.view(T, 1, Rd).expand(T, H, Rd)], -1)
    size = int((m.get("mask") or {}).get("size", 0) or 0)
    o = attend(torch.cat([qu, qr], -1), k, vv, float(m["scale"]), size, False)
    o = o * sigmoid(h @ _w(sd, p + "g").T).view(T, H, 1)
    return o.reshape(T, H * V) @ _w(sd, p + "o").T


MIXERS: Dict[str, Callable] = {"attention": attention, "latent_attention": latent_attention}


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def feed_forward(sd, p: str, h: torch.Tensor) -> torch.Tensor:
    return (gelu_tanh(h @ _w(sd, p + "gate").T) * (h @ _w(sd, p + "up").T)) @ _w(sd, p + "down").T


# ---- the model -------------------------------------------------------------------------------------------------------
def layer_order(cfg: Dict[str, Any]) -> List[int]:
    """Layer indices in the order they run (a looped span as often as the configuration says)."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or {}
    a, b = int(loop.get("start", 0)), int(loop.get("stop", 0))
    if b <= a:
        return list(range(n))
    return list(range(a)) + list(range(a, b)) * int(loop.get("times", 1)) + list(range(b, n))


def sublayer(cfg, sd, xs, p: str, q: int, norm: str, fn) -> List[torch.Tensor]:
    """One sublayer with its hyper-connection: read, norm, input convolution, fn, write."""
    eps = float(cfg["norm"]["eps"])
    h = rms_norm(read_streams(xs, _w(sd, f"{p}hc{q}.in")), _w(sd, p + norm), eps)
    if int((cfg.get("canon") or {}).get("taps", 0) or 0):
        h = h + causal_conv(h, _w(sd, f"{p}canon{q}"))
    return write_streams(xs, fn(h), _w(sd, f"{p}hc{q}.mix"), _w(sd, f"{p}hc{q}.out"))


def forward(cfg: Dict[str, Any], sd: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """-> logits float64 [T, vocab]; ``taps`` (a list) receives the sum of the streams after every layer run."""
    eps = float(cfg["norm"]["eps"])
    xs = [_w(sd, "embed")[tokens]] * int(cfg.get("streams", 1))
    for i in layer_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        xs = sublayer(cfg, sd, xs, p, 1, "norm1", lambda h: MIXERS[L["type"]](L["mixer"], sd, p + "mix.", h, eps))
        if L.get("mlp"):
            xs = sublayer(cfg, sd, xs, p, 2, "norm2", lambda h: feed_forward(sd, p + "mlp.", h))
        if taps is not None:
            taps.append(sum(xs))
    return rms_norm(sum(xs), _w(sd, "final.norm"), eps) @ _w(sd, "head").T


# ---- small configurations and random weights for the tests -----------------------------------------------------------
def make_config(layers=("latent", "attn", "latent-", "attn", "attn-"), width=48, vocab=97, eps=1e-5, streams=2, canon=3,
                loop=(1, 3, 3), l_heads=3, l_dim=8, l_rot=6, l_rot_dims=None, l_vdim=10, l_rank=12, l_q_rank=20, l_window=11,
                l_base=300.0, a_heads=4, a_kv_heads=2, a_dim=12, a_vdim=6, a_rot_dims=8, a_base=500.0, a_factor=4.0, a_window=0,
                l_scale=0.27, a_scale=0.33, ff=40) -> Dict[str, Any]:
    """layers: "latent" or "attn"; a trailing "-" leaves the feed-forward out."""
    out = []
    for spec in layers:
        if spec.startswith("attn"):
            m = {"heads": a_heads, "kv_heads": a_kv_heads, "dim": a_dim, "vdim": a_vdim, "scale": a_scale}
            if a_rot_dims:
                m["rot"] = {"base": a_base, "dims": a_rot_dims}
                if a_factor:
                    m["rot"]["scaling"] = {"factor": a_factor}
            if a_window:
                m["mask"] = {"size": a_window}
            layer = {"type": "attention", "mixer": m}
        else:
            m = {"heads": l_heads, "dim": l_dim, "rot_dim": l_rot, "vdim": l_vdim, "kv_rank": l_rank, "q_rank": l_q_rank,
                 "scale": l_scale}
            if l_window:
                m["mask"] = {"size": l_window}
            if l_rot:
                m["rot"] = {"base": l_base, "dims": l_rot if l_rot_dims is None else l_rot_dims}
            layer = {"type": "latent_attention", "mixer": m}
        layer["mlp"] = None if spec.endswith("-") else {"kind": "dense", "ff": ff}
        out.append(layer)
    cfg = {"architecture": "Zopipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": out}
    if canon:
        cfg["canon"] = {"taps": canon}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def make_weights(cfg: Dict[str, Any], seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights with the checkpoint's names, scaled so that every mechanism matters in the logits: sharp scores,
    asymmetric mixing matrices, stream coefficients far from equal."""
    g = torch.Generator().manual_seed(seed)
    W, S = int(cfg["width"]), int(cfg.get("streams", 1))
    taps = int((cfg.get("canon") or {}).get("taps", 0) or 0)
    s = W ** -0.5

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g) * std + mean).to(torch.bfloat16)

    sd = {"embed": rnd(int(cfg["vocab"]), W), "final.norm": rnd(W, std=0.2, mean=1.0), "head": rnd(int(cfg["vocab"]), W, std=s)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for q in ((1, 2) if L.get("mlp") else (1,)):
            sd[p + f"norm{q}"] = rnd(W, std=0.2, mean=1.0)
            if taps:
                sd[p + f"canon{q}"] = rnd(W, taps, std=0.4)
            sd[p + f"hc{q}.in"], sd[p + f"hc{q}.out"] = rnd(S, std=0.5, mean=1.0 / S), rnd(S, std=0.4, mean=1.0)
            sd[p + f"hc{q}.mix"] = (torch.eye(S) + torch.randn(S, S, generator=g) * 0.15).to(torch.bfloat16)
        H, V = int(m["heads"]), int(m.get("vdim", m["dim"]))
        if L["type"] == "latent_attention":
            D, Rd, R, Q = (int(m[k]) for k in ("dim", "rot_dim", "kv_rank", "q_rank"))
            sd[p + "mix.dq"], sd[p + "mix.dq.norm"] = rnd(Q, W, std=s), rnd(Q, std=0.3, mean=1.5)
            sd[p + "mix.uq"] = rnd(H * (D + Rd), Q, std=Q ** -0.5)
            sd[p + "mix.dkv"], sd[p + "mix.dkv.norm"] = rnd(R + Rd, W, std=s), rnd(R, std=0.3, mean=1.5)
            sd[p + "mix.uk"], sd[p + "mix.uv"] = rnd(H * D, R, std=R ** -0.5), rnd(H * V, R, std=R ** -0.5)
            sd[p + "mix.g"] = rnd(H, W, std=2 * s)
        else:
            G, D = int(m.get("kv_heads", m["heads"])), int(m["dim"])
            for n, r in (("q", H * D), ("k", G * D), ("v", G * V)):
                sd[p + f"mix.{n}"], sd[p + f"mix.{n}.b"] = rnd(r, W, std=1.3 * s), rnd(r, std=0.5)
            sd[p + "mix.temp"] = rnd(H, std=0.4, mean=1.0)
            sd[p + "mix.o.b"] = rnd(W, std=0.3)
        sd[p + "mix.o"] = rnd(W, H * V, std=(H * V) ** -0.5)
        f = L.get("mlp")
        if f:
            ff = int(f["ff"])
            sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"] = rnd(ff, W, std=s), rnd(ff, W, std=s), rnd(W, ff, std=ff ** -0.5)
    return sd
