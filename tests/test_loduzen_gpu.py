"""GPU parity of the Loduzen language model against the plain restatement in ``oracle/loduzen_oracle.py``.

Small made-up configurations and random weights; the product runs through ``CausalLM`` / ``LMEngine`` (state records,
scheduler, CUDA kernels), the oracle recomputes whole sequences in float64 on the CPU without cache or carried state.
"""

import copy
import json

import pytest
import torch

from oracle import loduzen_oracle as O

pytestmark = pytest.mark.gpu

YARN = {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 0.5}
PAIR = {"left": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 24, "scale": 0.25, "mask": {"size": 21},
                 "rot": {"base": 700.0, "dims": 16, "scaling": YARN}},
        "right": {"heads": 3, "dim": 16, "vdim": 20, "tau": 8.0}, "left_scale": 0.9, "right_scale": 0.7}
SSM = {"heads": 4, "vdim": 12, "state": 20, "groups": 2, "conv": 4, "norm_groups": 3}
DENSE = {"kind": "dense", "ff": 72}


def layer(kind, mixer, mlp=DENSE):
    return {"type": kind, "mixer": copy.deepcopy(mixer), "mlp": copy.deepcopy(mlp)}


def small_config(**over):
    cfg = {"architecture": "Loduzen", "vocab": 130, "width": 96, "norm": {"eps": 1e-5}, "token_side": {"dim": 12},
           "layers": [layer("mamba2", SSM), layer("parallel", PAIR), layer("parallel", PAIR), layer("mamba2", SSM), layer("parallel", PAIR)]}
    cfg.update(over)
    return cfg


def pair(heads, kv_heads, dim, lin_heads, lin_dim, lin_vdim, window=None, rot=None, scale=0.3, tau=16.0, ls=1.0, rs=1.0):
    left = {"heads": heads, "dim": dim, "vdim": dim, "scale": scale}
    if kv_heads:
        left["kv_heads"] = kv_heads
    if window:
        left["mask"] = {"size": window}
    if rot:
        left["rot"] = rot
    return {"left": left, "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": tau}, "left_scale": ls, "right_scale": rs}


def ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def odd_config():
    """Sizes that share nothing and are multiples of nothing: one head and several, as many key heads as heads and fewer, head
    sizes off every vector width, windows of 1, beyond the prompt and none, rotation of a part of the channels, of all and of
    none, with and without rescaling, 1 and 6 taps, one group and one per head, one norm part and one per head, layers without
    feed-forward, a token input of 5 channels."""
    plain = {"base": 10000.0, "dims": 10}
    return {"architecture": "Loduzen", "vocab": 77, "width": 74, "norm": {"eps": 1e-6}, "token_side": {"dim": 5},
            "layers": [layer("parallel", pair(5, None, 10, 1, 37, 9, window=1, rot=plain, ls=-0.6, rs=1.3), None),
                       layer("mamba2", ssm(3, 7, 38, 3, 1, 1)),
                       layer("parallel", pair(6, 1, 7, 2, 9, 33, window=500, rot={"base": 90.0, "dims": 6, "scaling": YARN}, tau=1.0)),
                       layer("mamba2", ssm(6, 5, 3, 1, 6, 6), None),
                       layer("parallel", pair(1, 1, 34, 5, 6, 3, rot={"base": 5e5, "dims": 34, "scaling": dict(YARN, factor=8.0)}, rs=0.0)),
                       layer("parallel", pair(2, 2, 9, 3, 5, 4, window=33))]}


def build(cfg, seed=1, dtype="float32", weights=None, rank=12, **kw):
    from dia_tts_prune_b200.lm_config import LoduzenConfig
    from dia_tts_prune_b200.lm_model import CausalLM
    w = O.random_weights(cfg, seed, rank=rank) if weights is None else weights
    kw.setdefault("max_tokens", 640)
    kw.setdefault("page_size", 8)
    return CausalLM(LoduzenConfig.model_validate(cfg), w, dtype=dtype, device="cuda:0", **kw), w


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def close(got, ref, tol=2e-4, slack=0.0):
    got, ref = got.detach().cpu().double(), ref.double()
    err = (got - ref).abs().max().item()
    assert err <= tol * max(1.0, ref.abs().max().item()) + 2.0 * slack, err


def mixer_ref(kind, h, p, m, eps):
    """The float64 reference of a mixer and how far the same plain code lands from it in float32 arithmetic."""
    ref = O.MIXERS[kind](h.double(), p, m, eps)
    ref32 = O.MIXERS[kind](h.float(), {k: v.float() for k, v in p.items()}, m, eps)
    return ref, (ref32.double() - ref).abs().max().item()


def whole(model, name, toks, want=None, **kw):
    want = list(range(len(toks))) if want is None else want
    return model.run_step([{"id": name, "tokens": toks, "want": want}], [name], **kw)


def part(w, prefix):
    return {k[len(prefix):]: v.double() for k, v in w.items() if k.startswith(prefix)}


def run_mixer(model, record, h, cuts):
    """The mixer of one layer record alone on given inputs, fed in portions ``cuts`` to a fresh sequence."""
    T = h.shape[0]
    assert sum(cuts) == T
    seq = model.state.open("t")
    model.state.reserve(seq, T)
    out, at = [], 0
    for n in cuts:
        out.append(model.engine.op_mixer(record, h[at:at + n].cuda(), [(seq, n, at)]))
        at += n
    model.state.close("t")
    return torch.cat(out)


def inputs(cfg, T, seed, gain=1.0):
    return torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(seed)) * gain


# ---- each mechanism alone -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("make", [small_config, odd_config])
@pytest.mark.parametrize("cuts", [[75], [40] + [1] * 35, [17, 15, 1, 2, 16, 3, 21], [2] * 37 + [1]])
def test_every_mixer_alone_whole_in_portions_and_decoded(make, cuts):
    cfg = make()
    model, w = build(cfg, 4)
    h = inputs(cfg, 75, 6)
    for i, lc in enumerate(cfg["layers"]):
        ref, slack = mixer_ref(lc["type"], h, part(w, f"l{i}.mix."), lc["mixer"], cfg["norm"]["eps"])
        close(run_mixer(model, i, h, cuts), ref, 2e-5, slack)


def test_mixer_kernels_between_the_projections():
    """The mixer kernels alone on given stacked projections: a pair's columns are the left mixer's, then the right's, each times
    its weight; the oracle gets the same numbers through identity projections."""
    cfg = small_config(layers=[layer("parallel", PAIR, None)])
    model, w = build(cfg, 5)
    m, p = cfg["layers"][0]["mixer"], part(w, "l0.mix.")
    h = inputs(cfg, 40, 2)
    rows = torch.cat([p["left.q"], p["left.k"], p["right.q"], p["right.k"], p["right.v"], p["right.g"], p["right.a1"]])
    seq = model.state.open("k")
    model.state.reserve(seq, 40)
    got = model.engine.op_mixer_kernels(0, (h.double() @ rows.T).float(), [(seq, 40, 0)])
    for side, cols, scale in (("left", slice(0, 96), 0.9), ("right", slice(96, 156), 0.7)):
        n = got[:, cols].shape[1]
        q = dict(part(p, side + "."), o=torch.eye(n, dtype=torch.float64))
        fn = O.window_attention if side == "left" else O.gated_linear_attention
        close(got[:, cols], scale * fn(h.double(), q, m[side], 1e-5), 2e-5)


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 40])
def test_gated_unit_with_the_tanh_form_of_gelu(rows):
    cfg = small_config()
    model, w = build(cfg, 5)
    h = inputs(cfg, rows, rows, 2.0)
    p = part(w, "l1.mlp.")
    ref = O.dense_ff(h.double(), p)
    g, u = h.double() @ p["gate"].T, h.double() @ p["up"].T
    assert (g > 1).any() and (g < -1).any()
    exact = (torch.nn.functional.gelu(g) * u) @ p["down"].T       # the error-function form is another function
    assert (exact - ref).abs().max() > 1e-4
    close(model.engine.op_ff(1, h.cuda()), ref, 1e-6)


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 40, 70])
@pytest.mark.parametrize("make", [small_config, odd_config])
def test_token_input_alone(make, rows):
    cfg = make()
    model, w = build(cfg, 6)
    x, toks = inputs(cfg, rows, rows, 3.0), tokens(cfg, rows, 9)
    n, eps = cfg["token_side"]["dim"], cfg["norm"]["eps"]
    table = w["side.embed"].double()[toks]
    for i in (0, 2, 4):
        p = part(w, f"l{i}.side.")
        ref = x.double() + O.token_input(x.double(), table[:, i * n:(i + 1) * n], p, eps)
        other = x.double() + O.token_input(x.double(), table[:, (i - 1) * n:i * n] if i else table[:, n:2 * n], p, eps)
        assert (other - ref).abs().max() > 1e-2                 # another layer's slice of the table shows
        close(model.engine.op_token_input(i, x, toks), ref, 1e-5)


def test_token_input_of_a_small_output_is_normed_with_eps_inside_the_root():
    cfg = small_config(norm={"eps": 1e-3})
    w = O.random_weights(cfg, 8)
    w["l1.side.proj"] = w["l1.side.proj"] * 2.0 ** -6            # an output about as large as the root of eps
    model, _ = build(cfg, weights=w)
    x, toks = inputs(cfg, 20, 3), tokens(cfg, 20, 4)
    p, e = part(w, "l1.side."), w["side.embed"].double()[toks][:, 12:24]
    ref = x.double() + O.token_input(x.double(), e, p, 1e-3)
    assert (x.double() + O.token_input(x.double(), e, p, 0.0) - ref).abs().max() > 1e-2
    close(model.engine.op_token_input(1, x, toks), ref, 1e-5)


ATTENTIONS = [(4, 2, 64, 50), (16, 16, 32, 7), (3, 1, 100, 64), (2, 2, 200, 65), (12, 4, 40, 33), (5, 5, 9, 3), (1, 1, 256, 90), (6, 2, 18, None),
              (8, 1, 130, 16)]


@pytest.mark.parametrize("heads,kv_heads,dim,window", ATTENTIONS)
def test_attention_with_other_shapes(heads, kv_heads, dim, window):
    cfg = small_config(layers=[layer("parallel", pair(heads, kv_heads, dim, 1, 4, 4, window=window, scale=dim ** -0.5,
                                                      rot={"base": 300.0, "dims": dim - dim % 2, "scaling": YARN}, rs=0.0), None)])
    model, w = build(cfg, 48)
    h = inputs(cfg, 100, dim)
    ref, slack = mixer_ref("parallel", h, part(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5)
    close(run_mixer(model, 0, h, [70] + [1] * 30), ref, 2e-5, slack)


def test_values_are_the_keys_before_norm_and_rotation_and_the_denominator_has_one_more_unit():
    cfg = small_config(layers=[layer("parallel", pair(4, 2, 24, 1, 4, 4, window=30, rot={"base": 50.0, "dims": 24}, rs=0.0), None)])
    model, w = build(cfg, 50)
    h = inputs(cfg, 60, 3)
    p, m = part(w, "l0.mix.left."), cfg["layers"][0]["mixer"]["left"]
    ref = O.window_attention(h.double(), p, m, 1e-5)
    assert (O.window_attention(h.double(), p, m, 1e-5, sink=False) - ref).abs().max() > 1e-2
    k_raw = (h.double() @ p["k"].T).reshape(60, 2, 24)
    normed = O.rotate(O.rms_unit(k_raw, 1e-5) * p["k.norm"], torch.arange(60), m["rot"])
    real = O.rms_unit
    assert (normed - k_raw).abs().max() > 0.1
    try:                                                        # q without its norm, for contrast
        O.rms_unit = lambda x, eps: x if x.shape[-2] == 4 else real(x, eps)
        assert (O.window_attention(h.double(), p, m, 1e-5) - ref).abs().max() > 1e-2
    finally:
        O.rms_unit = real
    close(run_mixer(model, 0, h, [45] + [1] * 15), ref, 2e-5)
    # the very first token: its own key is the value, times e^s / (1 + e^s)
    q = O.rotate(real((h[:1].double() @ p["q"].T).reshape(1, 4, 24), 1e-5) * p["q.norm"], torch.arange(1), m["rot"])
    s = (q * normed[:1].repeat_interleave(2, dim=1)).sum(-1) * m["scale"]
    first = (torch.sigmoid(s)[..., None] * k_raw[:1].repeat_interleave(2, dim=1)).reshape(1, -1) @ p["o"].T
    close(run_mixer(model, 0, h[:1], [1]), first, 1e-5)


def test_rotary_rescaling_ramp_and_amplitude_far_from_the_start():
    """Positions where the angles differ: against the oracle without the rescaling, without the amplitude, and with the ramp over
    other pairs the oracle itself differs; the product follows the full rule.  Factors and originals on both sides of the ramp's
    clamps."""
    for k, sc in enumerate([YARN, {"factor": 4.0, "original": 4000, "fast": 30.0, "slow": 1.0}, {"factor": 2.0, "original": 7, "fast": 2.0, "slow": 1.0},
                            {"factor": 16.0, "original": 100, "fast": 3.0, "slow": 3.0}, {"factor": 1.0, "original": 100, "fast": 32.0, "slow": 1.0}]):
        rot = {"base": 2000.0, "dims": 20, "scaling": sc}
        cfg = small_config(layers=[layer("parallel", pair(2, 1, 24, 1, 4, 4, rot=rot, scale=0.4, rs=0.0), None)])
        model, w = build(cfg, 51)
        h = inputs(cfg, 150, 5)
        p, m = part(w, "l0.mix.left."), cfg["layers"][0]["mixer"]["left"]
        ref = O.window_attention(h.double(), p, m, 1e-5)
        if sc["factor"] != 1.0:
            assert (O.window_attention(h.double(), p, dict(m, rot={"base": 2000.0, "dims": 20}), 1e-5) - ref).abs().max() > 1e-2
            real = O.frequencies
            try:
                O.frequencies = lambda r: (real(r)[0], 1.0)
                assert (O.window_attention(h.double(), p, m, 1e-5) - ref).abs().max() > 1e-3, k
            finally:
                O.frequencies = real
        close(run_mixer(model, 0, h, [120] + [1] * 30), ref, 3e-5)


@pytest.mark.parametrize("heads,dim,vdim,tau,rank", [(4, 128, 128, 16.0, 16), (2, 200, 20, 4.0, 3), (5, 72, 130, 16.0, 40), (1, 3, 15, 1.0, 1),
                                                     (9, 32, 16, 0.5, 8), (2, 64, 8, 30.0, 24)])
def test_gated_linear_attention_with_other_state_shapes(heads, dim, vdim, tau, rank):
    cfg = small_config(layers=[layer("parallel", pair(1, 1, 4, heads, dim, vdim, tau=tau, ls=0.0), None)])
    model, w = build(cfg, 49, rank=rank)
    h = inputs(cfg, 50, vdim)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref, slack = mixer_ref("parallel", h, p, m, 1e-5)
    flat = dict(m, right=dict(m["right"], tau=2.0 * tau))
    assert (O.parallel(h.double(), p, flat, 1e-5) - ref).abs().max() > 1e-4       # the root of the decay shows
    close(run_mixer(model, 0, h, [33, 1, 1, 15]), ref, 2e-5, slack)


@pytest.mark.parametrize("heads,vdim,state,groups,conv,norm_groups", [(8, 64, 128, 2, 4, 8), (2, 20, 200, 1, 4, 1), (5, 130, 72, 5, 3, 2),
                                                                      (1, 15, 3, 1, 2, 5), (9, 16, 32, 3, 7, 9), (4, 6, 64, 4, 1, 12)])
def test_state_space_mixer_with_other_shapes(heads, vdim, state, groups, conv, norm_groups):
    cfg = small_config(layers=[layer("mamba2", ssm(heads, vdim, state, groups, conv, norm_groups), None)])
    model, w = build(cfg, 47)
    h = inputs(cfg, 50, state)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref, slack = mixer_ref("mamba2", h, p, m, 1e-5)
    if norm_groups > 1:
        assert (O.mamba2(h.double(), p, dict(m, norm_groups=1), 1e-5) - ref).abs().max() > 1e-3
    close(run_mixer(model, 0, h, [33, 1, 1, 15]), ref, 2e-5, slack)


def test_state_space_mixer_each_term_shows():
    """The skip term, the convolution's bias, the step size's bias and the gate-before-norm order each change the oracle's result
    by far more than the product's distance from it."""
    cfg = small_config(layers=[layer("mamba2", SSM, None)])
    model, w = build(cfg, 46)
    h = inputs(cfg, 40, 1)
    p = part(w, "l0.mix.")
    ref = O.mamba2(h.double(), p, SSM, 1e-5)
    for name in ("D", "conv.b", "dt_bias", "A_log"):
        assert (O.mamba2(h.double(), dict(p, **{name: torch.zeros_like(p[name])}), SSM, 1e-5) - ref).abs().max() > 1e-2, name
    close(run_mixer(model, 0, h, [25] + [1] * 15), ref, 2e-5)
    # step sizes far beyond the exponential's comfortable range: softplus is the identity there and has no upper clamp
    w2 = dict(w, **{"l0.mix.dt_bias": torch.tensor([-30.0, 0.0, 25.0, 60.0]), "l0.mix.A_log": torch.tensor([0.0, -4.0, -6.0, -8.0])})
    model2, _ = build(cfg, weights=w2)
    ref, slack = mixer_ref("mamba2", h, part(w2, "l0.mix."), SSM, 1e-5)
    close(run_mixer(model2, 0, h, [25] + [1] * 15), ref, 2e-5, slack)


def test_pair_weights_and_parts():
    cfg = small_config(layers=[layer("parallel", dict(PAIR, left_scale=ls, right_scale=rs), None) for ls, rs in
                               ((1.0, 0.0), (0.0, 1.0), (-0.5, 2.0), (1.0, 1.0))])
    w = O.random_weights(cfg, 45)
    for name in [k for k in w if k.startswith("l0.mix.")]:      # the same weights under four pairs of scales
        for i in (1, 2, 3):
            w[name.replace("l0.", f"l{i}.", 1)] = w[name]
    model, _ = build(cfg, weights=w)
    h = inputs(cfg, 30, 2)
    out = [run_mixer(model, i, h, [20] + [1] * 10) for i in range(4)]
    p = part(w, "l0.mix.")
    left, right = (O.window_attention(h.double(), part(p, "left."), PAIR["left"], 1e-5),
                   O.gated_linear_attention(h.double(), part(p, "right."), PAIR["right"], 1e-5))
    for got, ref in zip(out, (left, right, 2.0 * right - 0.5 * left, left + right)):
        close(got, ref, 2e-5)


def test_any_two_stream_mixers_form_a_pair():
    """Mixers of other designs side by side (their own kernels write at an offset, with a weight): latent attention with gate,
    matrix memory, retention, the gated delta rule, and an attention with values of its own and no sink."""
    from dia_tts_prune_b200.lm_engine import LMEngine
    from dia_tts_prune_b200.lm_layers import (GatedDelta, HyperConnection, LatentAttention, MLstm, PairMixer, Retention, RmsNorm,
                                              RotaryAttention, StreamLayer, rotary_angles)
    from dia_tts_prune_b200.lm_state import PagedState
    from oracle import fipadra_oracle as FO
    from oracle import luketar_oracle as LO
    dev, D, eps = torch.device("cuda:0"), 48, 1e-5
    res = HyperConnection.residual(dev)
    base = {"vocab": 20, "width": D, "norm": {"eps": eps}}
    lat = {"heads": 3, "dim": 8, "vdim": 12, "q_rank": 16, "kv_rank": 20, "scale": 0.3}
    mls = {"heads": 2, "dim": 8, "vdim": 10, "gate_cap": 15.0}
    ret = {"heads": 3, "dim": 8, "vdim": 6, "decay": [0.9, 0.95, 0.99], "rot": {"base": 100.0, "dims": 8}}
    dlt = {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 12, "conv": 3}
    lw = LO.random_weights(dict(base, architecture="Luketar", layers=[{"type": "latent_attention", "mixer": lat, "mlp": None},
                                                                      {"type": "mlstm", "mixer": mls, "mlp": None}]), 3)
    fw = FO.random_weights(dict(base, architecture="Fipadra", layers=[{"type": "retention", "mixer": ret, "mlp": None},
                                                                      {"type": "delta", "mixer": dlt, "mlp": None}]), 4)
    a, b, r, d = part(lw, "l0.mix."), part(lw, "l1.mix."), part(fw, "l0.mix."), part(fw, "l1.mix.")
    latent = LatentAttention(a["dq"], a["dq.norm"], a["uq"], a["dkv"], a["dkv.norm"], a["uk"], a["uv"], a["g"], a["o"], heads=3, dim=8, vdim=12,
                             scale=0.3, sink=a["sink"], device=dev)
    mlstm = MLstm(b["q"], b["k"], b["v"], b["i"], b["f"], b["g"], b["o"], b["norm"], heads=2, dim=8, vdim=10, gate_cap=15.0, b_i=b["i.b"],
                  b_f=b["f.b"], device=dev)
    keep = Retention(r["q"], r["k"], r["v"], r["g"], r["o"], ret["decay"], heads=3, dim=8, vdim=6, rot_angles=rotary_angles(100.0, 8), device=dev)
    delta = GatedDelta(d["q"], d["k"], d["v"], d["b"], d["a"], d["g"], d["o"], d["q.conv"], d["k.conv"], d["v.conv"], d["A_log"], d["dt_bias"],
                       d["norm"], heads=2, kv_heads=1, dim=8, vdim=12, device=dev)
    g = torch.Generator().manual_seed(8)
    mat = lambda n, k: (torch.randn(n, k, generator=g) * k ** -0.5).to(torch.bfloat16).double()      # noqa: E731
    wq, wk, wv, wo, one = mat(32, D), mat(16, D), mat(16, D), mat(D, 32), torch.ones(8, dtype=torch.float64)
    attn = RotaryAttention(wq, wk, wv, wo, one, one, heads=4, kv_heads=2, dim=8, scale=0.5, window=9, device=dev)

    def attention(h):
        q, k = (O.rms_unit((h @ m.T).reshape(len(h), -1, 8), eps) for m in (wq, wk))
        v, gap = (h @ wv.T).reshape(len(h), 2, 8), torch.arange(len(h))[:, None] - torch.arange(len(h))[None, :]
        s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(2, 1)) * 0.5
        s = s.masked_fill((gap < 0) | (gap >= 9), -float("inf"))
        return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v.repeat_interleave(2, 1)).reshape(len(h), 32) @ wo.T

    refs = {latent: lambda h: LO.latent_attention(h, a, lat, eps), mlstm: lambda h: LO.mlstm(h, b, mls, eps),
            keep: lambda h: FO.retention(h, r, ret, eps), delta: lambda h: FO.gated_delta(h, d, dict(dlt), eps), attn: attention}
    pairs = [(latent, mlstm, 0.5, 2.0), (keep, latent, 1.5, -1.0), (delta, keep, 0.25, 1.0), (mlstm, attn, 1.0, 3.0), (attn, delta, 2.0, 0.5)]
    layers = [StreamLayer(torch.ones(D), res, PairMixer(x, y, s, t, device=dev), device=dev, rms=True) for x, y, s, t in pairs]
    state = PagedState([ly.state_spec() for ly in layers], D, 0, 128, dev, page_size=8, max_sequences=2)
    embed = torch.randn(20, D)
    eng = LMEngine(layers, embed, embed, RmsNorm(torch.ones(D), dev), width=D, vocab=20, taps=0, eps=eps, state=state, precision="float32")
    h = torch.randn(50, D, generator=g)
    for i, (x, y, s, t) in enumerate(pairs):
        ref = s * refs[x](h.double()) + t * refs[y](h.double())
        seq = state.open(f"s{i}")
        state.reserve(seq, 50)
        got, at = [], 0
        for n in [30, 3] + [1] * 17:
            got.append(eng.op_mixer(i, h[at:at + n].cuda(), [(seq, n, at)]))
            at += n
        state.close(f"s{i}")
        close(torch.cat(got), ref, 5e-5)
