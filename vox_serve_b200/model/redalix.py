"""Redalix adapter: a text-only decoder-only LM on ``HybridEngine`` (hybrid_engine.py) whose layers run mixer and feed-forward side
by side on ONE RMS norm of an fp32 stream: x += mixer(norm x) + ff(norm x).

  * mixers, in any order the configuration gives:
      a pair of mixers on the same input, each with its own output projection and RMS norm, half their sum:
        left -- grouped-head attention without rotation in a sliding window outside of which a sequence's first tokens stay
          visible, with a learned sink per head in the softmax's denominator;
        right -- Griffin's recurrent block: a gelu branch times a real-gated linear recurrent unit behind a short convolution,
          gates from block-diagonal matrices, an fp32 state per request;
      attention -- grouped heads, biases on q, k and v, interleaved rotary pairs with YaRN scaling, a sliding window, one sigmoid
        gate per head;
      Mamba-2 (state-space duality) -- one decay per head and token over an fp32 state [state, vdim], B and C shared by groups of
        heads, a short convolution over x, B and C, the output gated before a grouped RMS norm.
  * feed-forward: none, dense (tanh gelu), or experts (squared relu) that a table picks by the token's id, each weighing 1 / top,
    beside a shared expert behind one sigmoid gate per token.

Per request the design keeps, beside the pages of its attention layers, the recurrent states and the last inputs of the short
convolutions in the request's slot of ``HybridCache``.  Everything a model of this design can vary is read from its
``config.json``; serving (worker, scheduler, pages, slots, sampler, command lines) is what ``BobavikModel`` set up for
hybrid-engine designs.
"""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from .._lib import VoxB200Error
from ..hybrid_engine import (DenseMLPConfig, GatedLinearRecurrenceConfig, HybridConfig, HybridLayerConfig, MoEConfig, NormedPairConfig,
                             RotaryConfig, StateSpaceConfig, WindowAttentionConfig)
from .bobavik import BobavikModel

RECURRENCE_C = 8.0       # log a = -c * r * softplus(lam)
PAIR_SCALE = 0.5


def _mask(m: Dict[str, Any], key: str) -> int:
    return int((m.get("mask") or {}).get(key, 0) or 0)


def _rotary(m: Dict[str, Any], i: int) -> Optional[RotaryConfig]:
    r = m.get("rot")
    if not r:
        return None
    dims, sc = int(r["dims"]), r.get("scaling")
    if dims > int(m["dim"]) or dims % 2:
        raise VoxB200Error(f"layer {i}: rotary dims {dims} do not fit head dim {m['dim']}")
    if dims == 0:
        return None
    rot = RotaryConfig(dims, float(r["base"]), layout="interleaved", scaling="yarn")
    if sc:
        rot.factor, rot.original = float(sc["factor"]), float(sc["original"])
        rot.fast, rot.slow = float(sc["fast"]), float(sc["slow"])
    return rot


def _attention(m: Dict[str, Any], i: int, **kw) -> WindowAttentionConfig:
    H, D = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads", H))
    if G <= 0 or H % G:
        raise VoxB200Error(f"layer {i}: {H} heads do not divide into {G} key/value heads")
    return WindowAttentionConfig(H, G, D, int(m.get("vdim", D)), float(m["scale"]), window=_mask(m, "size"), **kw)


def redalix_config(c: Dict[str, Any]) -> HybridConfig:
    """config.json -> HybridConfig.  Keys: ``width``, ``vocab``, ``norm.eps`` and ``layers``: per layer ``type`` (parallel | attention
    | mamba2), ``mixer`` (parallel: left {heads, kv_heads, dim, vdim, scale, mask {size, keep_first}}, right {width, blocks, conv};
    attention: heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims, scaling {factor, original, fast, slow}?}?; mamba2:
    heads, vdim, state, groups, conv, norm_groups) and ``mlp``: null, {kind: dense, ff} or {kind: moe, expert {ff}, router {experts,
    top}, shared {ff}?}."""
    layers = []
    for i, L in enumerate(c["layers"]):
        kind, m = L["type"], L["mixer"]
        if kind == "parallel":
            r = m["right"]
            left = _attention(m["left"], i, gate=False, learned_sink=True, keep_first=_mask(m["left"], "keep_first"))
            right = GatedLinearRecurrenceConfig(int(r["width"]), int(r["blocks"]), int(r["conv"]), RECURRENCE_C)
            if right.blocks < 1 or right.width % right.blocks:
                raise VoxB200Error(f"layer {i}: {right.width} channels do not divide into {right.blocks} blocks")
            layer = HybridLayerConfig("normed_pair", NormedPairConfig(left, right, PAIR_SCALE))
        elif kind == "attention":
            layer = HybridLayerConfig("attention", _attention(m, i, rotary=_rotary(m, i), gate=True, head_gate=True, bias=True, o_bias=False))
        elif kind == "mamba2":
            s = StateSpaceConfig(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m.get("groups", 1)), int(m["conv"]),
                                 int(m.get("norm_groups", 1)))
            if s.groups < 1 or s.heads % s.groups or s.norm_groups < 1 or s.inner % s.norm_groups:
                raise VoxB200Error(f"layer {i}: {s.heads} heads of {s.vdim} do not divide into {s.groups} groups / {s.norm_groups} norm groups")
            layer = HybridLayerConfig("state_space", s)
        else:
            raise VoxB200Error(f"layer {i}: unknown mixer type '{kind}'")
        f = L.get("mlp")
        if f:
            if f["kind"] == "dense":
                layer.mlp = DenseMLPConfig(int(f["ff"]), act="gelu_tanh")
            elif f["kind"] == "moe":
                E, top = int(f["router"]["experts"]), int(f["router"]["top"])
                if not 1 <= top <= E:
                    raise VoxB200Error(f"layer {i}: top {top} of {E} experts")
                sh = f.get("shared") or {}
                layer.mlp = MoEConfig(E, top, int(f["expert"]["ff"]), shared_ff=int(sh.get("ff", 0) or 0), act="relu2", router="table",
                                      shared_gate=True)
            else:
                raise VoxB200Error(f"layer {i}: unknown feed-forward kind '{f['kind']}'")
        layers.append(layer)
    return HybridConfig(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), 1.0, layers, block="parallel", norm="rmsnorm",
                        shared_norm=True)


def synthetic_state_dict(cfg: HybridConfig, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    """Seeded random weights with the checkpoint's names (bf16; expert tables int32), generated on ``device``."""
    g = torch.Generator(device=device).manual_seed(seed)
    W = cfg.width

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(tuple(shape), generator=g, device=device) * std + mean).to(torch.bfloat16)

    def lin(n, k):
        return rnd(n, k, std=k ** -0.5)

    sd = {"embed": rnd(cfg.vocab, W), "head": lin(cfg.vocab, W), "final.norm": rnd(W, std=0.1, mean=1.0)}
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        x = p + "mix."
        sd[p + "norm1"] = rnd(W, std=0.1, mean=1.0)
        if L.kind == "state_space":
            C = m.conv_channels
            sd[x + "in"], sd[x + "conv"], sd[x + "conv.b"] = lin(m.inner + C + m.heads, W), rnd(C, m.conv, std=0.5), rnd(C, std=0.1)
            sd[x + "dt_bias"], sd[x + "A_log"], sd[x + "D"] = rnd(m.heads, std=0.5, mean=-2.0), rnd(m.heads, std=0.5), rnd(m.heads, std=0.5)
            sd[x + "norm"], sd[x + "o"] = rnd(m.inner, std=0.1, mean=1.0), lin(W, m.inner)
        else:
            pair = L.kind == "normed_pair"
            a, q = (m.left, x + "left.") if pair else (m, x)
            for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                sd[q + n] = lin(rows, W)
                if a.bias:
                    sd[q + n + ".b"] = rnd(rows, std=0.1)
            sd[q + "o"] = lin(W, a.heads * a.vdim)
            if a.gate:
                sd[q + "g"] = lin(a.heads, W)
            if a.learned_sink:
                sd[q + "sink"] = rnd(a.heads)
            if pair:
                r, q = m.right, x + "right."
                bs = r.width // r.blocks
                for n in ("y", "x"):
                    sd[q + n], sd[q + n + ".b"] = lin(r.width, W), rnd(r.width, std=0.1)
                sd[q + "conv"], sd[q + "conv.b"] = rnd(r.width, r.conv, std=0.5), rnd(r.width, std=0.1)
                for n in ("ra", "ri"):
                    sd[q + n], sd[q + n + ".b"] = rnd(r.blocks, bs, bs, std=bs ** -0.5), rnd(r.blocks, bs, std=0.1)
                sd[q + "lam"], sd[q + "o"] = rnd(r.width, mean=-4.0), lin(W, r.width)
                sd[x + "left.out"], sd[x + "right.out"] = rnd(W, std=0.1, mean=1.0), rnd(W, std=0.1, mean=1.0)
        f = L.mlp
        if isinstance(f, DenseMLPConfig):
            sd[p + "mlp.up"], sd[p + "mlp.down"] = lin(f.ff, W), lin(W, f.ff)
        elif f is not None:
            for e in range(f.experts):
                sd[p + f"mlp.e{e}.up"], sd[p + f"mlp.e{e}.down"] = lin(f.ff, W), lin(W, f.ff)
            sd[p + "mlp.table"] = torch.argsort(torch.rand(cfg.vocab, f.experts, generator=g, device=device), 1)[:, :f.top].to(torch.int32).contiguous()
            if f.shared_ff:
                sd[p + "mlp.shared.up"], sd[p + "mlp.shared.down"] = lin(f.shared_ff, W), lin(W, f.shared_ff)
                sd[p + "mlp.shared.sg"] = lin(1, W)
    return sd


class RedalixModel(BobavikModel):
    design = "Redalix"
    synthetic_name = "redalix-synthetic"
    has_recurrent_state = True
    build_profile = "text_ssd"

    @staticmethod
    def read_config(config: Dict[str, Any]) -> HybridConfig:
        return redalix_config(config)

    @staticmethod
    def synthetic_weights(cfg: HybridConfig, seed: int, device) -> Dict[str, torch.Tensor]:
        return synthetic_state_dict(cfg, seed, device)

    def _first_attention(self):
        m = next((L.mixer for L in self.config.layers if L.kind in ("attention", "normed_pair")), None)
        return m.left if isinstance(m, NormedPairConfig) else m
