"""Redalix on the hybrid engine against the plain float64 oracle (tests/redalix_oracle.py): every mechanism alone, whole prompts
against token-by-token decoding, portions of several sizes, batches against single requests, reuse of pages and slots, keys far
away / at page borders / just inside and outside a window / among and behind the kept first tokens with inputs built so that a wrong
key (or a missing sink) shows, recurrent and convolution state on reused slots, other sizes, and greedy generation through
ModelWorker + Scheduler.  Small configurations with random weights; float32 is compared tightly, bfloat16 loosely.
"""
import json
import os
import tempfile

import pytest
import torch

from tests import redalix_oracle as O

F32, BF16, I32, F64 = torch.float32, torch.bfloat16, torch.int32, torch.float64
DEV = "cuda"


# ---- CPU: configuration, registry, cache, the oracle's own rules ------------------------------------------------------
def test_config_reader_covers_every_branch():
    from vox_serve_b200._lib import VoxB200Error
    from vox_serve_b200.hybrid_engine import DenseMLPConfig, MoEConfig, NormedPairConfig, StateSpaceConfig, WindowAttentionConfig
    from vox_serve_b200.model.redalix import redalix_config

    c = redalix_config(O.make_config())
    assert (c.block, c.norm, c.eps, c.shared_norm, c.tied_head, c.embed_scale, c.logit_scale, c.residual_mult) == (
        "parallel", "rmsnorm", 1e-5, True, False, 1.0, 1.0, 1.0)
    assert [L.kind for L in c.layers] == ["state_space", "normed_pair", "attention", "normed_pair", "state_space", "attention"]
    ssm, pair, att = (c.layers[i].mixer for i in (0, 1, 2))
    assert isinstance(ssm, StateSpaceConfig) and isinstance(pair, NormedPairConfig) and isinstance(att, WindowAttentionConfig)
    assert (ssm.heads, ssm.vdim, ssm.state, ssm.groups, ssm.conv, ssm.norm_groups, ssm.inner, ssm.conv_channels) == (6, 7, 9, 3, 4, 2, 42, 96)
    left, right = pair.left, pair.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.window, left.keep_first) == (6, 3, 10, 6, 0.36, 11, 3)
    assert left.learned_sink and not left.gate and not left.bias and left.rotary is None
    assert (right.width, right.blocks, right.conv, right.c, pair.scale) == (40, 5, 3, 8.0, 0.5)
    assert (att.heads, att.kv_heads, att.dim, att.vdim, att.scale, att.window, att.keep_first) == (4, 2, 12, 10, 0.33, 9, 0)
    assert att.bias and not att.o_bias and att.gate and att.head_gate and not att.learned_sink and att.sink is None
    r = att.rotary
    assert (r.dims, r.base, r.layout, r.scaling, r.factor, r.original, r.fast, r.slow) == (8, 700.0, "interleaved", "yarn", 4.0, 24.0, 2.0, 0.25)
    assert isinstance(c.layers[0].mlp, DenseMLPConfig) and (c.layers[0].mlp.ff, c.layers[0].mlp.act) == (52, "gelu_tanh")
    f = c.layers[1].mlp
    assert isinstance(f, MoEConfig) and (f.experts, f.top, f.ff, f.shared_ff, f.act, f.router, f.shared_gate) == (5, 2, 24, 20, "relu2", "table", True)
    assert c.layers[3].mlp is None
    # what a configuration may leave out
    c2 = redalix_config(O.make_config(a_rot_dims=0, a_window=0, p_window=0, p_keep=0, shared_ff=0))
    assert c2.layers[2].mixer.rotary is None and c2.layers[2].mixer.window == 0 and c2.layers[1].mixer.left.window == 0
    assert c2.layers[1].mixer.left.keep_first == 0 and c2.layers[1].mlp.shared_ff == 0
    assert redalix_config(O.make_config(a_scaling=None)).layers[2].mixer.rotary.factor is None
    bad = O.make_config()
    bad["layers"][0]["type"] = "convolution"
    with pytest.raises(VoxB200Error):
        redalix_config(bad)
    for kw in (dict(a_heads=3, a_kv_heads=2), dict(p_heads=5), dict(a_rot_dims=14), dict(a_rot_dims=7), dict(r_blocks=6),
               dict(m_groups=4), dict(m_norm_groups=5), dict(top=6)):
        with pytest.raises(VoxB200Error):
            redalix_config(O.make_config(**kw))
    bad = O.make_config()
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(VoxB200Error):
        redalix_config(bad)


@pytest.mark.parametrize("scaling", [None, (4.0, 24.0, 2.0, 0.25), (8.0, 300.0, 32.0, 1.0), (1.0, 64.0, 4.0, 2.0), (3.0, 9.0, 1.0, 1.0)])
def test_yarn_frequencies(scaling):
    from vox_serve_b200.model.redalix import redalix_config

    cfg = O.make_config(layers=("attn",), a_dim=20, a_rot_dims=16, a_base=900.0, a_scaling=scaling)
    rot = redalix_config(cfg).layers[0].mixer.rotary
    want, mul = O.rotation_angles(cfg["layers"][0]["mixer"]["rot"])
    assert rot.frequencies().tolist() == pytest.approx(want, rel=1e-14) and rot.multiplier() == pytest.approx(mul, rel=1e-14)


def test_registry_and_cache():
    from vox_serve_b200.build import PROFILES
    from vox_serve_b200.hybrid_engine import HybridCache
    from vox_serve_b200.model import build_profile, get_model_class
    from vox_serve_b200.model.redalix import RedalixModel, redalix_config

    cfg = O.make_config()
    with tempfile.TemporaryDirectory() as d:
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        assert get_model_class(d) is RedalixModel and build_profile(d) == "text_ssd" and "ssd.cu" in PROFILES["text_ssd"]
    assert get_model_class("redalix-synthetic:3") is RedalixModel
    cache = HybridCache(redalix_config(cfg), 5, 8, 3, torch.float32, "cpu")
    assert sorted(cache.k) == sorted(cache.v) == [1, 2, 3, 5] and sorted(cache.state) == [0, 1, 3, 4]
    assert tuple(cache.k[1].shape) == (5, 8, 3, 10) and tuple(cache.v[1].shape) == (5, 8, 3, 6)
    assert tuple(cache.k[2].shape) == (5, 8, 2, 12) and tuple(cache.v[2].shape) == (5, 8, 2, 10)
    assert tuple(cache.state[0].shape) == (3, 6, 9, 7) and tuple(cache.state[1].shape) == (3, 40)
    assert tuple(cache.conv[(0, "x")].shape) == (3, 3, 96) and tuple(cache.conv[(1, "x")].shape) == (3, 2, 40)
    assert all(t.dtype == torch.float32 for t in list(cache.state.values()) + list(cache.conv.values()))


def test_synthetic_weights_have_the_checkpoints_names_and_shapes():
    from vox_serve_b200.model.redalix import redalix_config, synthetic_state_dict

    for kw in ({}, dict(shared_ff=0, a_rot_dims=0)):
        cfg = O.make_config(**kw)
        a, b = synthetic_state_dict(redalix_config(cfg), 1), O.make_weights(cfg)
        assert {k: (tuple(v.shape), v.dtype) for k, v in a.items()} == {k: (tuple(v.shape), v.dtype) for k, v in b.items()}


def test_oracle_mechanisms_by_hand():
    t, f = True, False
    assert O.visible(4, 2).tolist() == [[t, f, f, f], [t, t, f, f], [f, t, t, f], [f, f, t, t]]
    assert O.visible(4, 1, 2).tolist() == [[t, f, f, f], [t, t, f, f], [t, t, t, f], [t, t, f, t]]
    assert O.visible(3, 0).tolist() == [[t, f, f], [t, t, f], [t, t, t]]
    s = torch.zeros(2, 2, dtype=F64)
    assert torch.allclose(O.softmax_rows(s, O.visible(2, 0), torch.tensor(0.0, dtype=F64)), torch.tensor([[0.5, 0.0], [1 / 3, 1 / 3]], dtype=F64))
    assert torch.allclose(O.softmax_rows(s, O.visible(2, 0)), torch.tensor([[1.0, 0.0], [0.5, 0.5]], dtype=F64))
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64)
    assert O.causal_conv(u, torch.tensor([[10.0, 1.0]], dtype=F64), torch.tensor([100.0], dtype=F64)).view(-1).tolist() == [101.0, 112.0, 124.0]
    x = O.grouped_rms_norm(torch.tensor([[3.0, 3.0, 5.0, -5.0]], dtype=F64), torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=F64), 2, 0.0)
    assert x.view(-1).tolist() == [1.0, 2.0, 3.0, -4.0]
    S, last = O.linear_recurrent_unit(torch.ones(2, 1, dtype=F64), torch.ones(2, 1, dtype=F64), torch.full((2, 1), 2.0, dtype=F64),
                                      torch.tensor([-40.0], dtype=F64) * 0 + torch.log(torch.expm1(torch.log(torch.tensor(2.0, dtype=F64)) / 8)))
    b = (0.75 ** 0.5) * 2.0                                # a = 1/2
    assert S.view(-1).tolist() == pytest.approx([b, b / 2 + b]) and float(last) == pytest.approx(1.5 * b)
    y, S = O.state_space(torch.tensor([[[2.0]], [[3.0]]], dtype=F64), torch.tensor([[1.0], [2.0]], dtype=F64), torch.ones(2, 1, 1, dtype=F64),
                         torch.tensor([[[1.0]], [[10.0]]], dtype=F64), torch.log(torch.log(torch.tensor([2.0], dtype=F64))), torch.tensor([5.0], dtype=F64))
    assert y.view(-1).tolist() == pytest.approx([2.0 + 10.0, 10 * (0.25 * 2.0 + 6.0) + 15.0]) and float(S) == pytest.approx(6.5)


# ---- helpers ---------------------------------------------------------------------------------------------------------
def _worker(cfg, sd, dtype, slots=3, pages=24, page_size=8, max_rows=256, **kw):
    from vox_serve_b200.model.redalix import RedalixModel
    from vox_serve_b200.worker import ModelWorker

    model = RedalixModel("redalix-test", dtype=dtype, device="cuda:0", state_dict=sd, config=cfg, max_tokens=512, **kw)
    return ModelWorker("redalix-test", max_batch_size=slots, max_num_pages=pages, page_size=page_size, model=model,
                       max_prefill_tokens=max_rows, max_logit_rows=max_rows)


def _replay(worker, seqs, steps, free=True):
    """steps: [[(id, count), ...], ...]; every token's logits are tapped.  Returns id -> [len, vocab] fp32 (CPU)."""
    from vox_serve_b200.requests import Request

    live, at, out = {}, {k: 0 for k in seqs}, {k: [] for k in seqs}
    for step in steps:
        reqs = []
        for rid, n in step:
            toks = seqs[rid][at[rid]:at[rid] + n]
            if rid not in live:
                live[rid] = Request(request_id=rid, prompt=list(toks))
            else:
                live[rid].pending_tokens = (live[rid].pending_tokens or []) + list(toks)
            live[rid].step_tokens, live[rid].logit_rows = n, list(range(n))
            at[rid] += n
            reqs.append(live[rid])
        inp = worker.prepare_lm_inputs(reqs, [])
        assert inp is not None and len(reqs) == len(step), [r.finish_reason for r in live.values()]
        task = (worker.run_lm_prefill if inp["is_prefill"] else worker.run_lm_decode)(reqs, inp)
        try:
            while True:
                task.send(None)
        except StopIteration:
            pass
        for rid, _ in step:
            out[rid].append(worker.step_logits(rid))
        for rid, _ in step:
            if free and at[rid] == len(seqs[rid]):
                live[rid].done_all = True
                worker.free_kv_cache(live.pop(rid))
    return {k: torch.cat(v, 0) for k, v in out.items() if v}


def _err(got, ref):
    """difference over the vocabulary (mean removed), rms, relative to the rms of the reference logits; the worst position"""
    d = got.double() - ref
    d = d - d.mean(-1, keepdim=True)
    r = ref - ref.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / r.pow(2).mean().sqrt()).max().item()


TOL = {F32: 1e-4, BF16: 8e-2}


def _tokens(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


# ---- whole models ----------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_layers_and_logits_whole_prompt(dtype):
    cfg = O.make_config()
    sd = O.make_weights(cfg, 3)
    toks = _tokens(45, cfg["vocab"], 5)
    w = _worker(cfg, sd, dtype)
    w.engine.layer_tap = []
    got = _replay(w, {"a": toks}, [[("a", 45)]])["a"]
    taps, w.engine.layer_tap = w.engine.layer_tap, None
    layers = []
    ref = O.forward(cfg, sd, toks, layers)
    assert len(taps) == len(layers) == 6
    for i, (x, r) in enumerate(zip(taps, layers)):
        rel = (x.cpu().double() - r).pow(2).mean(-1).sqrt() / r.pow(2).mean().sqrt()        # per token
        assert rel.max().item() < (1e-5 if dtype == F32 else 5e-2), (i, rel.max().item())
    assert _err(got, ref) < TOL[dtype]


@pytest.mark.gpu
@pytest.mark.parametrize("layers", [("mamba",), ("pair",), ("attn",), ("mamba:dense",), ("pair:dense",), ("attn:moe",), ("mamba:moe", "mamba:moe"),
                                    ("pair:moe", "pair"), ("attn", "attn:dense"), ("attn", "pair:moe", "mamba")])
def test_each_mixer_alone(layers):
    cfg = O.make_config(layers=layers)
    sd = O.make_weights(cfg, 11)
    toks = _tokens(30, cfg["vocab"], 2)
    got = _replay(_worker(cfg, sd, F32), {"a": toks}, [[("a", 30)]])["a"]
    assert _err(got, O.forward(cfg, sd, toks)) < TOL[F32]


OTHER_SIZES = [
    dict(a_heads=1, a_kv_heads=1, p_heads=1, p_kv_heads=1, m_heads=1, m_groups=1, m_norm_groups=1, r_blocks=1, experts=1, top=1),
    dict(a_heads=6, a_kv_heads=6, a_dim=5, a_vdim=9, a_rot_dims=4, p_heads=5, p_kv_heads=5, p_dim=3, p_vdim=7, m_heads=4, m_groups=4, top=5),
    dict(a_heads=6, a_kv_heads=1, a_dim=16, a_vdim=16, a_rot_dims=16, p_heads=8, p_kv_heads=1, p_dim=16, p_vdim=32, width=44, ff=20, e_ff=9),
    dict(a_window=1, p_window=1, p_keep=1, m_conv=1, r_conv=1, a_rot_dims=0, ff=3, m_state=1, m_vdim=1, m_norm_groups=1, e_ff=1, shared_ff=1),
    dict(a_window=0, p_window=0, p_keep=0, a_scaling=None, shared_ff=0, r_blocks=40, r_width=40),
    dict(a_window=5, p_window=6, p_keep=20, m_conv=6, r_conv=5, width=50, eps=1e-2, m_state=17, m_vdim=5),
    dict(a_heads=34, a_kv_heads=2, a_dim=4, a_vdim=3, a_rot_dims=2, p_heads=36, p_kv_heads=2, p_dim=4, p_vdim=5, p_keep=9, m_heads=24, m_groups=2),
    dict(width=37, vocab=31, a_dim=2, a_vdim=1, a_rot_dims=2, r_width=33, r_blocks=11, m_heads=3, m_vdim=5, m_norm_groups=5, experts=3, top=3),
    dict(a_dim=256, a_vdim=256, a_heads=2, p_dim=192, p_vdim=256, p_heads=3, p_kv_heads=1, a_rot_dims=64, m_heads=2, m_groups=1, m_state=130,
         m_vdim=72, r_width=96, r_blocks=2),
    dict(a_base=12.0, a_scaling=(1.0, 16.0, 2.0, 1.0), a_window=40, p_window=33, p_keep=33, m_heads=8, m_groups=2, m_state=16, m_vdim=16,
         m_norm_groups=8, r_width=128, r_blocks=4, width=64, experts=16, top=1),
    dict(m_heads=2, m_groups=2, m_state=64, m_vdim=80, m_norm_groups=4, r_width=48, r_blocks=1, width=64, p_keep=2, p_window=3),
]


@pytest.mark.gpu
@pytest.mark.parametrize("kw", OTHER_SIZES)
def test_other_sizes(kw):
    """head counts of one and many, key/value heads = heads and = 1, key size != value size, sizes of one and odd sizes that rule
    tensor-core kernels and 16-byte rows out and sizes that take them, the largest heads, windows of one / none, kept tokens of none /
    one / more than the window / all of it, no rotation and rotation on a slice, scaling by one and none, convolutions of one to six
    taps, one group and a group per head, one block and a block per channel, one expert, all experts, more experts than the stacked
    form takes, no shared expert, a large eps."""
    cfg = O.make_config(layers=("mamba:moe", "pair:dense", "attn:moe", "pair:moe"), **kw)
    sd = O.make_weights(cfg, 7)
    toks = _tokens(41, cfg["vocab"], 3)
    ref = O.forward(cfg, sd, toks)
    cuts = [[("a", 17)], [("a", 2)], [("a", 9)]] + [[("a", 1)]] * 13
    w = _worker(cfg, sd, F32)
    assert _err(_replay(w, {"a": toks}, [[("a", 41)]])["a"], ref) < TOL[F32]
    assert _err(_replay(w, {"a": toks}, cuts)["a"], ref) < TOL[F32]
    w = _worker(cfg, sd, BF16)
    assert _err(_replay(w, {"a": toks}, [[("a", 41)]])["a"], ref) < TOL[BF16]
    assert _err(_replay(w, {"a": toks}, cuts)["a"], ref) < TOL[BF16]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prefill_decode_portions_and_batches(dtype):
    """whole prompt = token by token from the first token = portions of 1 ... 64 tokens cut inside pages and windows = batches of
    five unequal requests on three slots with requests left out of steps and reused pages and slots."""
    cfg = O.make_config()
    sd = O.make_weights(cfg, 5)
    V = cfg["vocab"]
    seqs = {k: _tokens(n, V, i) for i, (k, n) in enumerate((("a", 140), ("b", 9), ("c", 33), ("d", 1), ("e", 26)))}
    ref = {k: O.forward(cfg, sd, t) for k, t in seqs.items()}
    w = _worker(cfg, sd, dtype, pages=40)
    same = (lambda k: 3e-5 * ref[k].abs().max().item()) if dtype == F32 else (lambda k: 0.15 * ref[k].abs().max().item())
    whole = _replay(w, seqs, [[(k, len(t))] for k, t in seqs.items()])
    for k in seqs:
        assert _err(whole[k], ref[k]) < TOL[dtype], k
    one = _replay(w, {"a": seqs["a"]}, [[("a", 1)]] * 140)["a"]
    assert _err(one, ref["a"]) < TOL[dtype] and (one - whole["a"]).abs().max().item() < same("a")
    for cuts in ([2] * 70, [2, 2, 3, 1, 5, 7, 11, 13, 2, 94], [64, 2, 74], [3, 128, 9], [8] * 17 + [4], [65, 63, 12], [127, 1, 12]):
        assert sum(cuts) == 140
        got = _replay(w, {"a": seqs["a"]}, [[("a", n)] for n in cuts])["a"]
        assert _err(got, ref["a"]) < TOL[dtype] and (got - whole["a"]).abs().max().item() < same("a"), cuts
    # five requests on three slots: portions beside single tokens, requests left out of steps, slots and pages taken again
    steps = [[("a", 5), ("b", 2)], [("a", 1), ("b", 1), ("c", 20)], [("b", 6), ("c", 1)], [("a", 30), ("c", 12)],
             [("a", 1)], [("d", 1), ("a", 72)], [("e", 3), ("a", 31)], [("e", 1)], [("e", 22)]]
    got = _replay(w, seqs, steps)
    for k in seqs:
        assert _err(got[k], ref[k]) < TOL[dtype] and (got[k] - whole[k]).abs().max().item() < same(k), k
    assert w.empty_pages.qsize() == 40 and len(w.free_slots) == 3


@pytest.mark.gpu
@pytest.mark.parametrize("graph", [True, False])
def test_long_decoding_across_pages_and_windows(graph):
    cfg = O.make_config(layers=("mamba:moe", "pair:moe", "attn"))
    sd = O.make_weights(cfg, 9)
    toks = _tokens(250, cfg["vocab"], 4)
    ref = O.forward(cfg, sd, toks)
    w = _worker(cfg, sd, F32, pages=40)
    w.use_cuda_graph = graph
    got = _replay(w, {"a": toks}, [[("a", 10)]] + [[("a", 1)]] * 240)["a"]
    assert _err(got, ref) < TOL[F32]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_decoding_batches_on_reused_slots(dtype):
    """steps of single tokens only, four requests on two slots one after the other, beside ones that stay: what a slot's states,
    convolutions and pages held before never shows (they hold NaNs at first)"""
    cfg = O.make_config(layers=("mamba", "pair", "attn"), r_width=64, r_blocks=2)
    sd = O.make_weights(cfg, 15)
    seqs = {k: _tokens(n, cfg["vocab"], 20 + i) for i, (k, n) in enumerate((("a", 40), ("b", 3), ("c", 17), ("d", 2), ("e", 9)))}
    w = _worker(cfg, sd, dtype, slots=2, pages=9)
    for t in list(w.cache.state.values()) + list(w.cache.conv.values()):
        t.fill_(float("nan"))
    steps = [[("a", 1), ("b", 1)]] * 3 + [[("c", 1), ("a", 1)]] * 17 + [[("a", 1), ("d", 1)]] * 2 + [[("e", 1), ("a", 1)]] * 9 + [[("a", 1)]] * 9
    got = _replay(w, seqs, steps)
    for k in seqs:
        assert _err(got[k], O.forward(cfg, sd, seqs[k])) < TOL[dtype], k
    assert w.empty_pages.qsize() == 9 and len(w.free_slots) == 2


TC = dict(width=128, vocab=160, a_heads=4, a_kv_heads=2, a_dim=32, a_vdim=48, a_rot_dims=32, a_window=100, p_heads=4, p_kv_heads=2, p_dim=32,
          p_vdim=32, p_window=70, p_keep=5, r_width=192, r_blocks=3, r_conv=4, m_heads=8, m_vdim=32, m_state=48, m_groups=2, m_norm_groups=4,
          ff=192, experts=4, top=2, e_ff=64, shared_ff=128)


@pytest.mark.gpu
@pytest.mark.parametrize("kw", [{}, dict(shared_ff=96), dict(shared_ff=0, top=1), dict(e_ff=96, top=1), dict(experts=20, top=1)])
def test_bfloat16_tensor_core_sizes(kw):
    """sizes whose projections, attention, recurrence gates and state-space tiles run on the tensor-core kernels: a 600-token prompt
    whole (grouped experts, tiles) against portions (single rows among them), against the plain projection kernel with the recurrences
    row by row, and against the oracle; expert widths and counts that take the grouped and the stacked form and neither"""
    cfg = O.make_config(layers=("mamba:moe", "pair:moe", "attn:moe", "pair:dense"), **{**TC, **kw})
    sd = O.make_weights(cfg, 21)
    toks = _tokens(600, cfg["vocab"], 6)
    ref = O.forward(cfg, sd, toks)
    kw = dict(slots=2, pages=24, page_size=64, max_rows=1024)          # (the worker's)
    cuts = [[("a", 130)], [("a", 1)], [("a", 300)], [("a", 2)], [("a", 167)]]
    w = _worker(cfg, sd, BF16, **kw)
    whole, parts = _replay(w, {"a": toks}, [[("a", 600)]])["a"], _replay(w, {"a": toks}, cuts)["a"]
    w = _worker(cfg, sd, BF16, tensor_core_projections=False, **kw)
    w.engine.use_tiled_recurrence = False
    plain = _replay(w, {"a": toks}, [[("a", 600)]])["a"]
    for got in (whole, parts, plain):
        assert _err(got, ref) < TOL[BF16]
    w32 = _worker(cfg, sd, F32, **kw)
    assert _err(_replay(w32, {"a": toks}, [[("a", 600)]])["a"], ref) < TOL[F32]
    w32.engine.use_tiled_attention = w32.engine.use_tiled_recurrence = False
    assert _err(_replay(w32, {"a": toks}, [[("a", 333)], [("a", 267)]])["a"], ref) < TOL[F32]


# ---- single mechanisms -----------------------------------------------------------------------------------------------
def _paged(n_req_tokens, page_size, seed=0, spare=3):
    """scattered pages for requests of the given lengths -> (page_indptr, page_indices, number of pages)"""
    need = [(n + page_size - 1) // page_size for n in n_req_tokens]
    total = sum(need) + spare
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    indptr, idx = [0], []
    for n in need:
        idx += perm[len(idx):len(idx) + n]
        indptr.append(len(idx))
    return torch.tensor(indptr, dtype=I32, device=DEV), torch.tensor(idx, dtype=I32, device=DEV), total


def _step_tables(spans):
    """spans: per request (first position, rows) -> qo_indptr, row_req, pos (device int32)"""
    qo, row_req, pos = [0], [], []
    for b, (p0, n) in enumerate(spans):
        row_req += [b] * n
        pos += list(range(p0, p0 + n))
        qo.append(qo[-1] + n)
    mk = lambda v: torch.tensor(v, dtype=I32, device=DEV)
    return mk(qo), mk(row_req), mk(pos)


def _gather(cache, indptr, pages, b, n):
    """the first n cached rows of request b -> float64 [n, heads, dims] (CPU)"""
    ps = cache.shape[1]
    pg = pages[int(indptr[b]):int(indptr[b + 1])].tolist()
    return torch.stack([cache[pg[t // ps], t % ps] for t in range(n)]).double().cpu()


def _attend(q, k, v, dtype, page, window, keep, sink, gate, mode, lens=None, seed=6):
    """one or several sequences through the attention kernels: "tiles" (prompt portions), "rows" (single rows, keys split over
    CTAs where there are few), "heads" (single rows as tiles over the heads).  q [T, H, D] float64 in the operand type's values."""
    from vox_serve_b200 import ops

    lens = lens or [q.shape[0]]
    T, H, D = q.shape
    G, V = k.shape[1], v.shape[2]
    indptr, pages, n_pages = _paged(lens, page, seed=seed)
    kc = torch.full((n_pages, page, G, D), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((n_pages, page, G, V), float("nan"), dtype=dtype, device=DEV)
    t0 = 0
    for b, n in enumerate(lens):
        pg = pages[int(indptr[b]):int(indptr[b + 1])].tolist()
        for t in range(n):
            kc[pg[t // page], t % page], vc[pg[t // page], t % page] = k[t0 + t].to(dtype), v[t0 + t].to(dtype)
        t0 += n
    qo, row_req, pos = _step_tables([(0, n) for n in lens])
    out = torch.zeros(T, H * V, dtype=dtype, device=DEV)
    qd = q.reshape(T, -1).to(dtype).to(DEV).contiguous()
    gd = gate.to(F32).to(DEV) if gate is not None else None
    kw = dict(sink=sink.to(F32).to(DEV) if sink is not None else None, keep_first=keep, head_gate=gate is not None)
    args = (qd, kc, vc, out, gd, row_req, pos, indptr, pages, T, H, G, D, V, window, 1.0)
    if mode == "tiles":
        R = ops.window_attn_tile_rows()
        tl = [(b, r) for b, n in enumerate(lens) for r in range(int(qo[b]), int(qo[b]) + n, R)]
        ops.window_attn(*args, tiles=(qo, torch.tensor([b for b, _ in tl], dtype=I32, device=DEV),
                                      torch.tensor([r for _, r in tl], dtype=I32, device=DEV), len(tl)), **kw)
    else:
        # a few rows at a time: their keys are dealt to several CTAs and merged
        scratch = torch.zeros(256 * 8 * H * (V + 2), dtype=F32, device=DEV)
        for r0 in range(0, T, 16):
            idx = torch.arange(r0, min(r0 + 16, T), dtype=I32, device=DEV)
            ops.window_attn(*args, scratch=scratch, rows=(idx, idx.numel()), head_rows=mode == "heads", **kw)
        o2 = torch.zeros_like(out)
        ops.window_attn(*args[:3], o2, *args[4:], head_rows=mode == "heads", **kw)          # and all at once, unsplit
        assert (o2.double() - out.double()).abs().max().item() < (1e-5 if dtype == F32 else 3e-2)
    return out.double().cpu().view(T, H, V)


@pytest.mark.gpu
@pytest.mark.parametrize("mode", ["tiles", "rows", "heads"])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window,keep,page", [(1, 0, 8), (1, 1, 8), (7, 3, 8), (64, 5, 16), (65, 64, 8), (30, 70, 8), (100, 33, 16), (0, 4, 8),
                                              (40, 300, 8)])
def test_window_and_kept_token_edges_with_a_sink(mode, dtype, window, keep, page):
    """Hot keys among the kept tokens, right behind them, at both ends of a page, of a tile of 64 rows and of the sequence: kept ones
    are seen from everywhere, the others to distance window - 1 and by nothing further; where no hot key is seen only the sink is left
    (all other scores lie far below it).  Unused cache rows hold NaNs."""
    H, G, D, V, T = 4, 2, 16, 16, 230
    g = torch.Generator().manual_seed(window * 7 + keep)
    v = torch.randn(T, G, V, generator=g, dtype=F64)
    sink = torch.linspace(-1.0, 1.0, H, dtype=F64)
    for hots in ([0], [min(max(keep - 1, 0), T - 1)], [keep] if keep < T else [T - 1], [63, 64], [127, 128, T - 1]):
        q, k = torch.randn(T, H, D, generator=g, dtype=F64) * 0.05, torch.randn(T, G, D, generator=g, dtype=F64) * 0.05
        q[:, :, 1], k[:, :, 1] = 4.0, -5.0
        k[hots, :, 1] = 4.0
        q, k, v = (t.to(dtype).to(F64) for t in (q, k, v))
        ref = O.attend(q, k, v, 1.0, window, keep, sink)
        if window and len(hots) == 1 and hots[0] + window < T:
            hp = hots[0]
            assert ref[hp + window - 1].abs().max() > 0.1
            assert (ref[hp + window].abs().max() > 0.1) if hp < keep else (ref[hp + window].abs().max() < 1e-3)
        got = _attend(q, k, v, dtype, page, window, keep, sink, None, mode)
        assert (got - ref).abs().max().item() < (2e-5 if dtype == F32 else 4e-2), hots


@pytest.mark.gpu
@pytest.mark.parametrize("mode", ["tiles", "rows", "heads"])
@pytest.mark.parametrize("dtype,H,G,D,V", [(F32, 4, 2, 12, 6), (BF16, 8, 2, 64, 32), (BF16, 6, 1, 16, 128), (F32, 34, 2, 8, 5), (BF16, 3, 3, 10, 7),
                                           (BF16, 4, 4, 144, 16), (F32, 2, 1, 256, 256)])
def test_requests_beside_each_other_with_head_gates_and_sinks(mode, dtype, H, G, D, V):
    """three requests (one of a single token) in one launch, a far kept key that stands out, sinks from -4 to 6 per head and none, a
    gate per head and none"""
    g = torch.Generator().manual_seed(H * D)
    lens, T, window, keep = [200, 1, 67], 268, 21, 4
    q = torch.randn(T, H, D, generator=g, dtype=F64) * 0.05
    k = torch.randn(T, G, D, generator=g, dtype=F64) * 0.05
    v = torch.randn(T, G, V, generator=g, dtype=F64)
    q[:, :, 0] = 3.0
    k[3, :, 0] = 5.0                                    # request 0: a kept hot key, 196 positions away at its end
    k[200:, :, 0] = -6.0                                # requests 1, 2: every score ~ -18: the sink wins
    k[201 + 30, :, 0] = 4.0                             # request 2: a hot key at position 30, not kept
    q, k, v = (t.to(dtype).to(F64) for t in (q, k, v))
    gate = torch.randn(T, H, generator=g, dtype=F32).to(F64)
    for sink, gt in ((torch.linspace(-4.0, 6.0, H, dtype=F64), gate), (None, gate), (torch.zeros(H, dtype=F64), None)):
        ref = torch.cat([O.attend(q[a:a + n], k[a:a + n], v[a:a + n], 1.0, window, keep, sink) for a, n in ((0, 200), (200, 1), (201, 67))], 0)
        if sink is not None:
            assert ref[200].abs().max() < 1e-4 and (ref[199] - v[3].repeat_interleave(H // G, 0)).abs().max() < 0.05
            assert ref[201 + 30 + window - 1].abs().max() > 0.1 and ref[201 + 30 + window].abs().max() < 1e-4
        if gt is not None:
            ref = ref * O.sigmoid(gt)[:, :, None]
        got = _attend(q, k, v, dtype, 8, window, keep, sink, gt, mode, lens=lens)
        assert (got - ref).abs().max().item() < (2e-5 if dtype == F32 else 4e-2) * max(1.0, ref.abs().max().item())


CUTS = ([1000], [1, 1000], [64, 2, 1000], [3, 61, 65, 1, 1000], [17, 1, 1, 130, 1000])


def _walk(lens, cuts, run):
    """requests of ``lens`` rows cut into steps, each a batch: run(live = [(request, first position, rows)], tables) for every step"""
    from vox_serve_b200 import ops

    at = [0] * len(lens)
    slots_all = [5, 1, 3, 0, 6][:len(lens)]
    R = ops.window_attn_tile_rows()
    mk = lambda v: torch.tensor(v, dtype=I32, device=DEV)
    for c in cuts:
        live = [(b, at[b], min(c, lens[b] - at[b])) for b in range(len(lens)) if at[b] < lens[b]]
        if not live:
            break
        qo, row_req, pos = _step_tables([(p0, n) for _, p0, n in live])
        tl = [(i, r) for i, (_, _, n) in enumerate(live) if n > 1 for r in range(int(qo[i]), int(qo[i]) + n, R)]
        tiles = (mk([b for b, _ in tl]), mk([r for _, r in tl]), len(tl)) if tl else None
        run(live, qo, row_req, pos, mk([slots_all[b] for b, _, _ in live]), tiles, any(n == 1 for _, _, n in live))
        for b, _, n in live:
            at[b] += n
    assert at == lens


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tiled", [True, False])
@pytest.mark.parametrize("C,blocks", [(40, 5), (96, 2), (128, 8), (33, 1), (320, 2), (144, 1)])
def test_gated_linear_recurrence(dtype, tiled, C, blocks):
    """five requests on scattered slots that hold NaNs, cut five ways: block sizes that run on tensor cores (with several chunks of
    inputs, and with a last one that is not full) and that do not, both ways through a portion's rows; decays near 0 and near 1"""
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(C + blocks)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F32)
    lens, bs, wt = [150, 1, 67, 2, 64], C // blocks, dtype
    us, ys = [r(n, C) * 1.5 for n in lens], [r(n, C) for n in lens]
    ra, ri = ((r(blocks, bs, bs) * 2 * bs ** -0.5).to(BF16).to(F32) for _ in range(2))
    rb, ib, lam, yb = r(blocks, bs), r(blocks, bs), r(C) * 3 - 4.0, r(C)
    ref = []
    for u, y in zip(us, ys):
        u, y = u.double(), y.double()
        S, _ = O.linear_recurrent_unit(u, O.gate_blocks(u, ra.double(), rb.double()), O.gate_blocks(u, ri.double(), ib.double()), lam.double())
        ref.append(S * O.gelu_tanh(y + yb.double()))
    w = torch.cat([ra, ri], 1).to(wt).to(DEV).contiguous()
    bias, rate = torch.cat([rb, ib], 1).to(DEV).contiguous(), (8.0 * O.softplus(lam.double())).to(F32).to(DEV)
    for cuts in CUTS:
        state = torch.full((7, C), float("nan"), dtype=F32, device=DEV)
        outs = [[] for _ in lens]

        def run(live, qo, row_req, pos, slots, tiles, single):
            T = int(qo[-1])
            u, y = (torch.cat([x[b][p0:p0 + n] for b, p0, n in live], 0).to(DEV) for x in (us, ys))
            wide = torch.zeros(T, 2 * C + 4, device=DEV)
            wide[:, :C], wide[:, C + 4:] = u, y
            out = torch.zeros(T, C, dtype=dtype, device=DEV)
            ops.rglru(wide[:, :C], w, bias, rate, wide[:, C + 4:], yb.to(DEV), state, out, torch.zeros(2 * T * C, device=DEV), qo,
                      row_req, pos, slots, len(live), multi_rows=tiles is not None, tiles=(*tiles, 64) if (tiles and tiled) else None,
                      scratch=torch.zeros(ops.mingru_scratch_floats(tiles[2], 64, C) if tiles else 1, device=DEV))
            for i, (b, _, n) in enumerate(live):
                outs[b].append(out[int(qo[i]):int(qo[i]) + n].double().cpu())

        _walk(lens, cuts, run)
        for b in range(len(lens)):
            big = max(1.0, ref[b].abs().max().item())
            assert (torch.cat(outs[b], 0) - ref[b]).abs().max().item() < (2e-5 if dtype == F32 else 1e-2) * big, (cuts, b)


@pytest.mark.gpu
def test_split_products_of_the_gates_keep_fp32_accuracy():
    """bf16 matrices on tensor cores against fp32 FMAs on the same values: the decays and scaled inputs agree far below bf16 rounding"""
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(3)
    T, C, blocks = 70, 256, 2
    u, y = torch.randn(T, C, generator=g).to(DEV) * 2, torch.randn(T, C, generator=g).to(DEV)
    w = (torch.randn(blocks, 2 * C // blocks, C // blocks, generator=g) * 0.15).to(BF16).to(DEV)
    bias, rate = torch.randn(blocks, 2 * C // blocks, generator=g).to(DEV), 8.0 * O.softplus(torch.randn(C, generator=g) - 4).to(DEV)
    qo, row_req, pos = _step_tables([(0, T)])
    got = []
    for wt in (BF16, F32):
        ab = torch.zeros(2 * T * C, device=DEV)
        ops.rglru(u, w.to(wt), bias, rate, y, None, torch.zeros(1, C, device=DEV), torch.zeros(T, C, device=DEV), ab, qo, row_req, pos,
                  torch.zeros(1, dtype=I32, device=DEV), 1)
        got.append(ab)
    assert (got[0] - got[1]).abs().max().item() < 1e-4 and (got[0] - got[1]).pow(2).mean().sqrt().item() < 5e-6


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tiled", [True, False])
@pytest.mark.parametrize("H,V,N,G", [(6, 7, 9, 3), (4, 16, 16, 2), (8, 64, 128, 1), (2, 80, 48, 2), (3, 32, 64, 1), (1, 1, 1, 1), (2, 20, 130, 1)])
def test_state_space_duality(dtype, tiled, H, V, N, G):
    """five requests on scattered slots that hold NaNs, cut five ways: sizes on tensor cores (value dims in one block, in two of
    unequal size, fewer than a block) and not, tiles and row by row; step sizes from tiny to those that forget everything at once"""
    from vox_serve_b200 import ops

    if tiled and ops.ssd_tile_rows(V, N) == 0:
        pytest.skip("sizes of the row-by-row form only")
    g = torch.Generator().manual_seed(H * V + N)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F32)
    lens = [150, 1, 67, 2, 64]
    xbc = [(r(n, H * V + 2 * G * N) * 0.7).to(dtype) for n in lens]
    dts, zs = [r(n, H) * 2 for n in lens], [r(n, H * V) for n in lens]
    dt_b, A_log, D = r(H) - 1.0, r(H) * 1.5, r(H)
    ref = []
    for x, dt, z in zip(xbc, dts, zs):
        x, n = x.double(), x.shape[0]
        y, _ = O.state_space(x[:, :H * V].reshape(n, H, V), O.softplus(dt.double() + dt_b.double()), x[:, H * V:H * V + G * N].reshape(n, G, N),
                             x[:, H * V + G * N:].reshape(n, G, N), A_log.double(), D.double())
        ref.append(y.reshape(n, H * V) * O.silu(z.double()))
    for cuts in CUTS:
        state = torch.full((7, H, N, V), float("nan"), dtype=F32, device=DEV)
        outs = [[] for _ in lens]

        def run(live, qo, row_req, pos, slots, tiles, single):
            T = int(qo[-1])
            cat = lambda v: torch.cat([v[b][p0:p0 + n] for b, p0, n in live], 0).to(DEV)
            zdt = torch.cat([cat(zs), cat(dts)], 1).contiguous()
            out = torch.zeros(T, H * V, device=DEV)
            args = (cat(xbc).contiguous(), zdt[:, H * V:], dt_b.to(DEV), A_log.to(DEV), D.to(DEV), zdt[:, :H * V], state, out, qo, pos, slots,
                    len(live), G)
            if single or (tiles and not tiled):
                ops.ssd(*args, single_rows=single, multi_rows=bool(tiles and not tiled))
            if tiles and tiled:
                ops.ssd(*args, tiles=tiles, scratch=torch.full((ops.ssd_scratch_floats(tiles[2], H, V, N),), float("nan"), device=DEV))
            for i, (b, _, n) in enumerate(live):
                outs[b].append(out[int(qo[i]):int(qo[i]) + n].double().cpu())

        _walk(lens, cuts, run)
        for b in range(len(lens)):
            err = (torch.cat(outs[b], 0) - ref[b]).abs().max().item() / max(1.0, ref[b].abs().max().item())
            assert err < (2e-5 if dtype == F32 else 1e-4), (cuts, b, err)       # (bf16 rows are exact inputs here: the sums stay fp32)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,C,groups", [(3, 42, 2), (40, 512, 1), (17, 4096, 8), (5, 48, 12), (2, 9000, 2), (4, 30, 10)])
def test_grouped_norm(dtype, T, C, groups):
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(C)
    x, w = torch.randn(T, C, generator=g) * torch.linspace(0.01, 30, C), torch.randn(C, generator=g)
    out = torch.zeros(T, C, dtype=dtype, device=DEV)
    ops.group_rmsnorm(x.to(DEV), w.to(DEV), groups, 1e-3, out)
    ref = O.grouped_rms_norm(x.double(), w.double(), groups, 1e-3)
    assert (out.double().cpu() - ref).abs().max().item() < (1e-5 if dtype == F32 else 2e-2) * ref.abs().max().item()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [1, 37, 256, 1030, 2048, 3072, 4100, 6000])
def test_branch_tail(dtype, W):
    """one to three branches, normed or not, widths in and out of 16-byte pieces and past the register form, with and without a next norm"""
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(W)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F32)
    T, eps = 7, 1e-2
    for pattern in ([(True, 0.5), (True, 0.5), (False, 1.0)], [(False, 1.0)], [(False, 1.0), (False, 1.0)], [(True, 0.5), (True, 0.25)],
                    [(False, 0.3), (True, 2.0), (True, 1.0)]):
        for nxt in (True, False):
            x, wn = r(T, W), r(W)
            br = [(r(T, W) * 3, r(W) if normed else None, s) for normed, s in pattern]
            ref = x.double()
            for y, w, s in br:
                ref = ref + s * (O.rms_norm(y.double(), w.double(), eps) if w is not None else y.double())
            xd, out = x.to(DEV), torch.zeros(T, W, dtype=dtype, device=DEV)
            ops.branch_residual_norm_f32(xd, [(y.to(DEV), w.to(DEV) if w is not None else None, s) for y, w, s in br], eps,
                                         out=out if nxt else None, w=wn.to(DEV) if nxt else None)
            assert (xd.double().cpu() - ref).abs().max().item() < 1e-5 * max(1.0, ref.abs().max().item())
            if nxt:
                want = O.rms_norm(ref, wn.double(), eps)
                assert (out.double().cpu() - want).abs().max().item() < (2e-5 if dtype == F32 else 2e-2) * max(1.0, want.abs().max().item())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,E,top", [(48, 5, 2), (37, 1, 1), (2048, 64, 8), (1030, 40, 32)])
def test_table_router(dtype, W, E, top):
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(W)
    vocab, T = 50, 70
    table = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(I32)
    ids, h, sg = torch.randint(0, vocab, (T,), generator=g).to(I32), torch.randn(T, W, generator=g).to(dtype), torch.randn(W, generator=g) * 0.1
    idx, wts, gate = torch.full((T * top,), -1, dtype=I32, device=DEV), torch.zeros(T * top, device=DEV), torch.zeros(T, device=DEV)
    ops.moe_route_table(ids.to(DEV), table.to(DEV), E, idx, wts, h.to(DEV), sg.to(DEV), gate)
    assert idx.view(T, top).cpu().tolist() == table[ids.long()].tolist() and (wts - 1.0 / top).abs().max().item() < 1e-7
    assert (gate.double().cpu() - O.sigmoid(h.double() @ sg.double())).abs().max().item() < 1e-5
    gate.fill_(7.0)
    ops.moe_route_table(ids.to(DEV), table.to(DEV), E, idx, wts)
    assert (gate == 7.0).all() and idx.view(T, top).cpu().tolist() == table[ids.long()].tolist()


@pytest.mark.gpu
@pytest.mark.parametrize("top,W", [(1, 64), (3, 48), (8, 36), (9, 40), (2, 37)])
def test_expert_combine(top, W):
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(W)
    T = 29
    eo, sh, wts, ss = (torch.randn(*s, generator=g) for s in ((T * top, W), (T, W), (T * top,), (T,)))
    rows = torch.randperm(T * top, generator=g).to(I32)
    ref = (wts.double().view(T, top, 1) * eo.double()[rows.long()].view(T, top, W)).sum(1)
    for shared, scale in ((None, None), (sh, None), (sh, ss)):
        want = ref + (0.0 if shared is None else shared.double() * (1.0 if scale is None else scale.double()[:, None]))
        out = torch.zeros(T, W, device=DEV)
        ops.moe_combine(eo.to(DEV), shared.to(DEV) if shared is not None else None, wts.to(DEV), rows.to(DEV), top, out,
                        shared_scale=scale.to(DEV) if scale is not None else None)
        assert (out.double().cpu() - want).abs().max().item() < 1e-5


@pytest.mark.gpu
@pytest.mark.parametrize("taps,C", [(1, 20), (2, 64), (3, 33), (4, 520), (4, 21), (7, 40)])
def test_convolution_adds_its_inputs_bias_but_not_before_the_start(taps, C):
    from vox_serve_b200 import ops

    g = torch.Generator().manual_seed(taps * C)
    w, bv, ib = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g) * 3
    lens = [131, 1, 96, 2, 45]
    xs = [torch.randn(n, C, generator=g) for n in lens]
    for cuts in CUTS:
        state = torch.full((7, max(taps - 1, 1), C), float("nan"), dtype=F32, device=DEV)
        outs = [[] for _ in lens]

        def run(live, qo, row_req, pos, slots, tiles, single):
            x = torch.cat([xs[b][p0:p0 + n] for b, p0, n in live], 0).to(DEV)
            out = torch.zeros_like(x)
            ops.short_conv(x, w.to(DEV), bv.to(DEV), state, qo, row_req, pos, slots, len(live), out_f32=out, in_bias=ib.to(DEV))
            for i, (b, _, n) in enumerate(live):
                outs[b].append(out[int(qo[i]):int(qo[i]) + n].double().cpu())

        _walk(lens, cuts, run)
        for b in range(len(lens)):
            ref = O.causal_conv(xs[b].double() + ib.double(), w.double(), bv.double())
            assert (torch.cat(outs[b], 0) - ref).abs().max().item() < 1e-5 * max(1.0, ref.abs().max().item()), (cuts, b)


@pytest.mark.gpu
@pytest.mark.parametrize("at", [2, 4, 5, 40])
@pytest.mark.parametrize("kind", ["attn", "pair"])
def test_far_kept_and_edge_tokens_show_in_a_models_logits(kind, at):
    """One token id gets a key that every query scores high: positions just inside and just outside its window differ from a sequence
    without that token exactly where the oracle's do -- everywhere after it when it is among the kept tokens."""
    cfg = O.make_config(layers=(kind,), a_window=24, p_window=24, p_keep=5, width=64, a_rot_dims=0, a_heads=2, p_heads=2, p_kv_heads=1)
    sd = O.make_weights(cfg, 41)
    hot_id, T, p = 96, 150, "l0.mix." if kind == "attn" else "l0.mix.left."
    sd["embed"][:, 0], sd["embed"][:, 1] = 0.0, 1.0
    sd["embed"][hot_id, 0] = 40.0
    sd[p + "k"][:, 0], sd[p + "q"][:, 1] = 3.0, 3.0
    if kind == "pair":
        sd["l0.mix.right.x"].zero_()                   # (the recurrence would carry the token everywhere)
        sd["l0.mix.right.conv"].zero_()
    base = [t % 90 for t in _tokens(T, 90, 8)]
    with_hot = base[:at] + [hot_id] + base[at + 1:]
    ref = {n: O.forward(cfg, sd, t) for n, t in (("b", base), ("h", with_hot))}
    diff = (ref["h"] - ref["b"]).abs().max(-1).values
    assert diff[at + 23] > 1e-2
    if kind == "pair" and at < 5:
        assert diff[T - 1] > 1e-2
    else:
        assert diff[at + 24:].max() < 1e-9
    w = _worker(cfg, sd, F32, pages=60)
    for steps in ([[("h", T)]], [[("h", 50)]] + [[("h", 1)]] * 100, [[("h", 63)], [("h", 1)], [("h", 2)], [("h", 84)]]):
        got = _replay(w, {"h": with_hot}, steps)["h"]
        assert _err(got, ref["h"]) < TOL[F32]
        d = (got.double() - ref["b"]).abs().max(-1).values
        assert ((d > 5e-3) == (diff > 5e-3)).all()


# ---- serving ---------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_generation_through_scheduler(dtype):
    """ModelWorker + Scheduler: three requests of unequal prompts, prompts fed in portions of 16 beside decoding requests,
    more requests than slots.  Tokens equal the oracle's greedy tokens wherever the oracle's top-2 margin is clear."""
    from vox_serve_b200.requests import Request
    from vox_serve_b200.sampling import SamplingConfig
    from vox_serve_b200.scheduler import Scheduler

    cfg = O.make_config()
    sd = O.make_weights(cfg, 13)
    prompts = {"r0": _tokens(41, cfg["vocab"], 1), "r1": _tokens(5, cfg["vocab"], 2), "r2": _tokens(23, cfg["vocab"], 3)}
    n_new = 12
    w = _worker(cfg, sd, dtype, slots=2, pages=40, page_size=8)
    sch = Scheduler(w, prefill_chunk_tokens=16)
    reqs = {}
    for rid, p in prompts.items():
        reqs[rid] = Request(request_id=rid, prompt=p, sampling_config=SamplingConfig(greedy=True, max_tokens=n_new))
        sch.submit(reqs[rid])
    sch.run_until_done(max_steps=400)
    assert len(sch.finished) == 3 and w.empty_pages.qsize() == 40 and len(w.free_slots) == 2
    margin = 0.05 if dtype == F32 else 0.25
    wrong = clear = 0
    for rid, p in prompts.items():
        got = [int.from_bytes(c, "little", signed=True) for c in sch.audio[rid]]
        assert len(got) == n_new and reqs[rid].finish_reason == "max_tokens_reached"
        toks = list(p)
        for t in got:                       # teacher-forced comparison: every step is judged on the framework's own prefix
            z = O.forward(cfg, sd, toks)[-1]
            top = torch.topk(z, 2)
            if float(top.values[0] - top.values[1]) > margin:
                clear += 1
                wrong += t != int(top.indices[0])
            toks.append(t)
    assert wrong == 0 and clear > n_new, (wrong, clear)


def _write_model_dir(d, cfg, sd):
    """config.json + model.safetensors (8-byte length, JSON header, raw little-endian data) of a bfloat16 checkpoint with int32 tables"""
    import struct

    meta, blobs, off = {}, [], 0
    for k, v in sd.items():
        raw = v.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        meta[k] = {"dtype": "I32" if v.dtype == I32 else "BF16", "shape": list(v.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(meta).encode()
    with open(os.path.join(d, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)


@pytest.mark.gpu
def test_command_lines_on_a_model_directory(capsys):
    """a checkpoint directory through the trace replay tool (a subprocess: portions, two requests, a request ended and its
    slot taken again) and through the generate command (in process)."""
    import subprocess
    import sys

    import numpy as np

    from vox_serve_b200 import generate

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = O.make_config()
    sd = O.make_weights(cfg, 17)
    V = cfg["vocab"]
    a, b, c = _tokens(30, V, 1), _tokens(12, V, 2), _tokens(9, V, 3)
    with tempfile.TemporaryDirectory() as d:
        _write_model_dir(d, cfg, sd)
        out = os.path.join(d, "out")
        steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
                 {"step": 1, "entries": [{"id": "a", "tokens": a[20:21], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [9]}], "end": ["b"]},
                 {"step": 2, "entries": [{"id": "c", "tokens": c, "want": [8]}, {"id": "a", "tokens": a[21:], "want": [8]}], "end": ["a", "c"]}]
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out,
                            "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                           text=True, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
        ra, rb, rc = (O.forward(cfg, sd, t) for t in (a, b, c))
        want = {0: torch.stack([ra[0], ra[19]]), 1: torch.stack([ra[20], rb[11]]), 2: torch.stack([rc[8], ra[29]])}
        for s_, ref in want.items():
            got = torch.from_numpy(np.fromfile(os.path.join(out, f"{s_}.f32"), dtype="<f4").reshape(2, V).copy())
            assert _err(got, ref) < TOL[F32], s_
        capsys.readouterr()
        assert generate.main(["--model", d, "--prompt", " ".join(map(str, a)), "--prompt", " ".join(map(str, b)), "--max-new", "6",
                              "--dtype", "float32", "--prefill-chunk", "16", "--page-size", "8"]) == 0
        lines = capsys.readouterr().out.strip().splitlines()[-2:]
        for line, prompt in zip(lines, (a, b)):
            toks = list(prompt)
            for t in (int(x) for x in line.split()):
                z = O.forward(cfg, sd, toks)[-1]
                top = torch.topk(z, 2)
                assert float(top.values[0] - top.values[1]) < 0.05 or t == int(top.indices[0])
                toks.append(t)
            assert len(toks) == len(prompt) + 6
