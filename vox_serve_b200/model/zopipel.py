"""Zopipel adapter: a text-only decoder-only LM on ``HybridEngine`` (hybrid_engine.py) whose residual stream is several copies
tied together by hyper-connections: a sublayer reads u = sum_s in[s] x_s, takes its norm through an input convolution over time,
h + conv(h), and its output y enters every copy, x_t <- sum_s mix[s, t] x_s + out[t] y.  All copies start as the embedding; at the
end they are summed.  A span of layers may run several times in a row with the same weights (``loop``), each pass on a cache and
state of its own.

  * mixers, in any order the configuration gives:
      latent attention -- queries through a normed latent, heads of ``dim`` unrotated + ``rot_dim`` rotated dims; keys' unrotated
        parts and values are per-head expansions of one normed latent per token, the rotated key part is one vector per token
        shared by all heads ((i, i + dims/2) rotary pairs); only [latent | rotated key part] is cached; sliding window; one
        sigmoid gate per head;
      attention -- grouped key/value heads, biases on all four projections, (i, i + dims/2) rotary pairs with linearly scaled
        frequencies, values of unit root mean square per head, scores times a number per head, and a softmax whose denominator
        has one added (a sink of score 0 without a value).
  * feed-forward: none, or down(gelu(gate h) * up h) with the tanh form of gelu.
  * output: RMS norm, head.

Per request the design keeps, beside the pages of its attention layers, the last inputs of both input convolutions of every layer
run, in the request's slot of ``HybridCache``.  Everything a model of this design can vary is read from its ``config.json``;
serving (worker, scheduler, pages, slots, sampler, command lines) is what ``BobavikModel`` set up for hybrid-engine designs.
"""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from .._lib import VoxB200Error
from ..hybrid_engine import (GluMLPConfig, HybridConfig, HybridLayerConfig, LatentAttentionConfig, RotaryConfig,
                             WindowAttentionConfig)
from .bobavik import BobavikModel

SINK_SCORE = 0.0         # the softmax's further key: exp(0) = 1 joins the denominator


def _rotary(r: Optional[Dict[str, Any]], fits: int, where: str) -> Optional[RotaryConfig]:
    if not r:
        return None
    sc = r.get("scaling") or None
    rot = RotaryConfig(int(r["dims"]), float(r["base"]), float(sc["factor"]) if sc else None, layout="half", scaling="linear")
    if rot.dims > fits or rot.dims % 2:
        raise VoxB200Error(f"{where}: rotary dims {rot.dims} do not fit {fits} dims")
    return rot


def zopipel_config(c: Dict[str, Any]) -> HybridConfig:
    """config.json -> HybridConfig.  Keys: ``width``, ``vocab``, ``norm.eps``, ``streams``, ``canon.taps``, ``loop`` {start, stop,
    times} (optional) and ``layers``: per layer ``type`` (latent_attention | attention), ``mixer`` (latent_attention: heads, dim,
    rot_dim, vdim, kv_rank, q_rank, scale, mask {size}?, rot {base, dims, scaling {factor}?}?; attention: heads, kv_heads, dim,
    vdim, scale, mask {size}?, rot?) and ``mlp``: null or {kind: dense, ff}."""
    layers = []
    for i, L in enumerate(c["layers"]):
        kind, m, where = L["type"], L["mixer"], f"layer {i}"
        window = int((m.get("mask") or {}).get("size", 0) or 0)
        H, dim = int(m["heads"]), int(m["dim"])
        vdim = int(m.get("vdim", dim))
        if kind == "latent_attention":
            rot_dim = int(m.get("rot_dim", 0) or 0)
            mixer = LatentAttentionConfig(H, dim, vdim, int(m["kv_rank"]), int(m["q_rank"]), float(m["scale"]), rot_dim=rot_dim,
                                          rotary=_rotary(m.get("rot"), rot_dim, where) if rot_dim else None, head_gate=True,
                                          window=window)
            layer = HybridLayerConfig("latent", mixer)
        elif kind == "attention":
            G = int(m.get("kv_heads", H))
            if G <= 0 or H % G:
                raise VoxB200Error(f"{where}: {H} heads do not divide into {G} key/value heads")
            mixer = WindowAttentionConfig(H, G, dim, vdim, float(m["scale"]), window, _rotary(m.get("rot"), dim, where), gate=False,
                                          bias=True, value_norm=True, head_factor=True, sink=SINK_SCORE)
            layer = HybridLayerConfig("attention", mixer)
        else:
            raise VoxB200Error(f"{where}: unknown mixer type '{kind}'")
        f = L.get("mlp")
        if f:
            if f.get("kind", "dense") != "dense":
                raise VoxB200Error(f"{where}: unknown feed-forward kind '{f.get('kind')}'")
            layer.mlp = GluMLPConfig(int(f["ff"]), act="gelu_tanh")
        layers.append(layer)
    loop = c.get("loop") or {}
    a, b, times = int(loop.get("start", 0)), int(loop.get("stop", 0)), int(loop.get("times", 1))
    if not (0 <= a <= len(layers) and b <= len(layers) and times >= 0):
        raise VoxB200Error(f"loop {loop} does not fit {len(layers)} layers")
    return HybridConfig(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), 1.0, layers, block="hyper", norm="rmsnorm",
                        loop_start=a, loop_stop=b, loop_times=times, streams=int(c.get("streams", 1)),
                        input_conv=int((c.get("canon") or {}).get("taps", 0) or 0))


def synthetic_state_dict(cfg: HybridConfig, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    """Seeded random weights with the checkpoint's names (bf16), generated on ``device``."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, S = cfg.width, cfg.streams

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g, device=device) * std + mean).to(torch.bfloat16)

    s = W ** -0.5
    sd = {"embed": rnd(cfg.vocab, W), "head": rnd(cfg.vocab, W, std=s), "final.norm": rnd(W, std=0.1, mean=1.0)}
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        for q in ((1, 2) if L.mlp is not None else (1,)):
            sd[p + f"norm{q}"] = rnd(W, std=0.1, mean=1.0)
            sd[p + f"hc{q}.in"], sd[p + f"hc{q}.out"] = rnd(S, std=0.1, mean=1.0 / S), rnd(S, std=0.1, mean=1.0)
            sd[p + f"hc{q}.mix"] = (torch.eye(S, device=device) + torch.randn(S, S, generator=g, device=device) * 0.05).to(torch.bfloat16)
            if cfg.input_conv:
                sd[p + f"canon{q}"] = rnd(W, cfg.input_conv, std=0.3)
        if L.kind == "latent":
            sd[p + "mix.dq"], sd[p + "mix.dq.norm"] = rnd(m.q_rank, W, std=s), rnd(m.q_rank, std=0.1, mean=1.0)
            sd[p + "mix.uq"] = rnd(m.heads * (m.dim + m.rot_dim), m.q_rank, std=m.q_rank ** -0.5)
            sd[p + "mix.dkv"], sd[p + "mix.dkv.norm"] = rnd(m.kv_rank + m.rot_dim, W, std=s), rnd(m.kv_rank, std=0.1, mean=1.0)
            sd[p + "mix.uk"] = rnd(m.heads * m.dim, m.kv_rank, std=m.kv_rank ** -0.5)
            sd[p + "mix.uv"] = rnd(m.heads * m.vdim, m.kv_rank, std=m.kv_rank ** -0.5)
            sd[p + "mix.g"] = rnd(m.heads, W, std=s)
        else:
            for n, r in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                sd[p + f"mix.{n}"], sd[p + f"mix.{n}.b"] = rnd(r, W, std=s), rnd(r, std=0.1)
            sd[p + "mix.temp"], sd[p + "mix.o.b"] = rnd(m.heads, std=0.1, mean=1.0), rnd(W, std=0.1)
        sd[p + "mix.o"] = rnd(W, m.heads * m.vdim, std=(m.heads * m.vdim) ** -0.5)
        f = L.mlp
        if f is not None:
            sd[p + "mlp.gate"], sd[p + "mlp.up"] = rnd(f.ff, W, std=s), rnd(f.ff, W, std=s)
            sd[p + "mlp.down"] = rnd(W, f.ff, std=f.ff ** -0.5)
    return sd


class ZopipelModel(BobavikModel):
    design = "Zopipel"
    synthetic_name = "zopipel-synthetic"
    has_recurrent_state = True
    build_profile = "text_hyper"

    @staticmethod
    def read_config(config: Dict[str, Any]) -> HybridConfig:
        return zopipel_config(config)

    @staticmethod
    def synthetic_weights(cfg: HybridConfig, seed: int, device) -> Dict[str, torch.Tensor]:
        return synthetic_state_dict(cfg, seed, device)
