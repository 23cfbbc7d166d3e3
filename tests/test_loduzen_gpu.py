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


# ---- the whole model ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("make", [small_config, odd_config])
def test_whole_prompt_logits_and_residual_after_every_layer(make):
    cfg = make()
    model, w = build(cfg, 11)
    toks = tokens(cfg, 61, 2)
    ref, streams = O.forward(cfg, w, toks, keep_layers=True)
    got, got_streams = whole(model, "a", toks, keep_layers=True)
    assert got_streams.shape[0] == len(cfg["layers"])
    slack = (O.forward(cfg, w, toks, keep_layers=True, dtype=torch.float32)[1].double() - streams).abs().max().item()
    close(got_streams, streams, 2e-5, slack)
    close(got, ref, 2e-4, slack)
    for n in (1, 2, 3):                                         # the first tokens of a sequence
        close(whole(model, "b", toks[:n]), ref[:n], 2e-4, slack)


def test_layers_without_token_input_or_feed_forward():
    cfg = small_config(layers=[layer("mamba2", SSM), layer("parallel", PAIR, None), layer("mamba2", SSM, None)], token_side=None)
    model, w = build(cfg, 9)
    toks = tokens(cfg, 40, 5)
    got = [model.run_step([{"id": "d", "tokens": toks[:30], "want": list(range(30))}])]
    got += [model.run_step([{"id": "d", "tokens": [t], "want": [0]}]) for t in toks[30:]]
    close(torch.cat(got), O.forward(cfg, w, toks))


def test_sublayers_run_one_after_the_other_and_the_token_input_reads_their_sum():
    """With the feed-forward or the token input reading the residual from before the layer's mixer, the oracle differs."""
    cfg = small_config()
    model, w = build(cfg, 10)
    toks = tokens(cfg, 33, 5)
    ref = O.forward(cfg, w, toks)
    wd = {k: v.double() for k, v in w.items()}
    for early_ff in (True, False):
        x = wd["embed"][toks]
        for i, lc in enumerate(cfg["layers"]):
            p, old = f"l{i}.", x
            x = x + O.MIXERS[lc["type"]](O.rms_unit(x, 1e-5) * wd[p + "norm1"], O.part(wd, p + "mix."), lc["mixer"], 1e-5)
            x = x + O.dense_ff(O.rms_unit(old if early_ff else x, 1e-5) * wd[p + "norm2"], O.part(wd, p + "mlp."))
            x = x + O.token_input(x if early_ff else old, wd["side.embed"][toks][:, 12 * i:12 * i + 12], O.part(wd, p + "side."), 1e-5)
        assert ((O.rms_unit(x, 1e-5) * wd["final.norm"]) @ wd["embed"].T - ref).abs().max() > 1e-2
    close(whole(model, "a", toks), ref)


@pytest.mark.parametrize("make", [small_config, odd_config])
def test_prefill_then_long_token_by_token_decoding(make):
    cfg = make()
    model, w = build(cfg, 12)
    toks = tokens(cfg, 150, 3)
    ref = O.forward(cfg, w, toks)
    got = [model.run_step([{"id": "d", "tokens": toks[:9], "want": list(range(9))}])]
    for t in range(9, 150):                                     # the windows pass over decoded tokens
        got.append(model.run_step([{"id": "d", "tokens": [toks[t]], "want": [0]}], ["d"] if t == 149 else []))
    close(torch.cat(got), ref)


@pytest.mark.parametrize("make", [small_config, odd_config])
@pytest.mark.parametrize("cuts", [[2] * 40, [1, 2, 3, 5, 8, 13, 21, 27], [19, 1, 20, 21, 2, 17], [79, 1], [3, 77]])
def test_portions_of_any_size_give_the_same_logits(make, cuts):
    cfg = make()
    model, w = build(cfg, 13, max_rows=32)                      # long portions are also split by the engine itself
    toks = tokens(cfg, 80, 4)
    ref = O.forward(cfg, w, toks)
    assert sum(cuts) == 80
    got, at = [], 0
    for n in cuts:
        got.append(model.run_step([{"id": "p", "tokens": toks[at:at + n], "want": list(range(n))}]))
        at += n
    model.run_step([], ["p"])
    close(torch.cat(got), ref)
    close(torch.cat(got), whole(model, "q", toks).cpu(), 2e-5)   # how the rows were cut changes rounding at most


@pytest.mark.parametrize("make", [small_config, odd_config])
def test_mixed_batch_of_unequal_requests_equals_each_alone(make):
    cfg = make()
    model, w = build(cfg, 15, max_sequences=4)
    A, B, C = tokens(cfg, 50, 6), tokens(cfg, 31, 7), tokens(cfg, 12, 8)
    alone = {n: whole(model, n, t) for n, t in (("A", A), ("B", B), ("C", C))}
    out = {"A": [], "B": [], "C": []}

    def run(parts, end=()):
        lg = model.run_step([{"id": n, "tokens": t, "want": list(range(len(t)))} for n, t in parts], list(end))
        at = 0
        for n, t in parts:
            out[n].append(lg[at:at + len(t)])
            at += len(t)

    run([("A", A[:23]), ("C", C)], end=["C"])                   # a portion beside a whole prompt
    run([("A", A[23:40]), ("B", B[:25])])
    for k in range(6):                                          # two requests decode side by side
        run([("B", [B[25 + k]]), ("A", [A[40 + k]])])
    run([("A", A[46:])], end=["A", "B"])
    for n in "ABC":
        got = torch.cat(out[n])
        close(got, alone[n][:got.shape[0]].cpu(), 2e-5)
    close(alone["A"], O.forward(cfg, w, A))
    both = model.run_step([{"id": "A", "tokens": A, "want": list(range(50))},
                           {"id": "B", "tokens": B, "want": list(range(31))}], ["A", "B"])
    assert torch.equal(both[:50], alone["A"]) and torch.equal(both[50:], alone["B"])


def test_freed_pages_slots_states_and_tails_are_used_again():
    cfg = small_config()
    model, w = build(cfg, 16, max_tokens=96, max_sequences=2, page_size=8)
    st = model.state
    X, Y, Z = tokens(cfg, 70, 9), tokens(cfg, 26, 10), tokens(cfg, 64, 11)
    ref = {n: O.forward(cfg, w, t) for n, t in (("X", X), ("Y", Y), ("Z", Z))}
    gx = model.run_step([{"id": "X", "tokens": X, "want": list(range(70))}])
    gy = model.run_step([{"id": "Y", "tokens": Y, "want": list(range(26))}])
    pages_x, slot_x = list(st.sequences["X"].pages), st.sequences["X"].slot
    assert st.free_slots == 0
    model.run_step([], ["X"])
    # Z takes X's slot and pages - dirty with X's keys, matrix states and convolution tails - and starts with two tokens (fewer
    # than the convolution has taps), while Y's state stays as it is
    gz = model.run_step([{"id": "Z", "tokens": Z[:2], "want": [0, 1]}])
    assert st.sequences["Z"].slot == slot_x and set(st.sequences["Z"].pages) <= set(pages_x)
    gz1 = model.run_step([{"id": "Z", "tokens": Z[2:40], "want": list(range(38))}])
    gz2 = model.run_step([{"id": "Z", "tokens": Z[40:], "want": list(range(24))}], ["Z", "Y"])
    close(gx, ref["X"]); close(gy, ref["Y"]); close(torch.cat([gz, gz1, gz2]), ref["Z"])
    assert st.free_pages == st.n_pages and st.free_slots == 2
    from dia_tts_prune_b200.lm_state import OutOfPages
    with pytest.raises(OutOfPages):
        model.run_step([{"id": "big", "tokens": tokens(cfg, 200, 1), "want": []}])


# ---- inputs and weights made so that one thing stands out -----------------------------------------------------------------
def standout_attention(page_size, window):
    """One layer whose queries equal its keys (no rotation), so that a position whose input points the way the query's input does
    gets a score far above all others; the other half of the pair is off."""
    cfg = small_config(layers=[layer("parallel", pair(2, 2, 32, 1, 4, 4, window=window, scale=0.6, rs=0.0), None)])
    w = O.random_weights(cfg, 21)
    w["l0.mix.left.q"], w["l0.mix.left.q.norm"] = w["l0.mix.left.k"], w["l0.mix.left.k.norm"]
    model, _ = build(cfg, weights=w, max_tokens=512, page_size=page_size)
    return cfg, w, model


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [None, 130, 75, 64])
def test_standout_key_far_away_at_page_tile_and_window_borders(decode, window):
    P = 16
    cfg, w, model = standout_attention(P, window)
    T = 300
    g = torch.Generator().manual_seed(2)
    base = torch.randn(T, 96, generator=g) * 0.3
    mark, near = torch.randn(96, generator=g) * 3, torch.randn(96, generator=g) * 0.5
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    i = T - 1
    blank = base.clone()
    blank[i] = mark
    ref_blank = O.parallel(blank.double(), p, m, 1e-5)
    span = window or T + 1
    # the first token, far back among hundreds, both sides of page borders and of the 64-key tile border, the neighbour,
    # and the last key inside and the first outside the window
    for j in (0, 3, 63, 64, 127, 128, (i // P) * P, (i // P) * P - 1, i - 1, i - span + 1, i - span, i - span + 2):
        if j < 0:
            continue
        h = base.clone()
        h[j] = 2 * mark + near                                  # nearly the query's direction, a value of its own
        h[i] = mark
        ref = O.parallel(h.double(), p, m, 1e-5)
        carried = (ref[i] - ref_blank[i]).abs().max() > 1e-2
        assert carried == (i - j < span), j                     # the marked key carries the row exactly when it is seen
        n0 = T - 60 if decode else T
        close(run_mixer(model, 0, h, [n0] + [1] * (T - n0)), ref, 2e-5)


@pytest.mark.parametrize("cuts", [[200], [150] + [1] * 50, [3, 61, 2, 64, 70]])
def test_window_edge_moves_with_every_row_of_a_portion(cuts):
    """Every row of a portion has its own first visible key: a key made to stand out is seen by exactly the rows that are
    less than `window` tokens on."""
    window = 40
    cfg, w, model = standout_attention(8, window)
    T = 200
    g = torch.Generator().manual_seed(4)
    h = torch.randn(T, 96, generator=g) * 0.3
    mark = torch.randn(96, generator=g) * 3
    plain = h.clone()
    h[100] = 2 * mark
    h[101:] += mark * 0.5                                        # every later query leans towards the marked key
    plain[101:] += mark * 0.5
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    m = dict(m, right_scale=0.0)
    ref = O.parallel(h.double(), p, m, 1e-5)
    gap = (O.parallel(plain.double(), p, m, 1e-5) - ref).abs().amax(dim=-1)
    assert gap[100 + window - 1] > 1e-2 and gap[100 + window:].max() == 0    # seen up to row 139, gone from row 140 on
    close(run_mixer(model, 0, h, cuts), ref, 2e-5)


def test_the_unit_in_the_denominator_shows_where_all_scores_are_low():
    """Queries that point away from every key: nearly all of the softmax's weight falls on the unit."""
    cfg, w, _ = standout_attention(8, 30)
    w["l0.mix.left.q"] = -w["l0.mix.left.q"]
    model, _ = build(cfg, weights=w, max_tokens=256)
    mark = torch.randn(96, generator=torch.Generator().manual_seed(3))
    h = mark + 0.1 * inputs(cfg, 80, 7)
    p, m = part(w, "l0.mix.left."), cfg["layers"][0]["mixer"]["left"]
    ref = O.window_attention(h.double(), p, m, 1e-5)
    bare = O.window_attention(h.double(), p, m, 1e-5, sink=False)
    assert ref[40:].abs().max() < 0.3 * bare[40:].abs().max()
    close(run_mixer(model, 0, h, [50] + [1] * 30), ref, 1e-5)


def long_memory(kind):
    """A recurrence that forgets almost nothing, so that the first tokens still carry the read-out hundreds of tokens on."""
    mixer = pair(1, 1, 4, 2, 16, 16, tau=16.0, ls=0.0) if kind == "parallel" else ssm(2, 16, 16, 1, 4, 1)
    cfg = small_config(layers=[layer(kind, mixer, None)])
    w = O.random_weights(cfg, 23)
    if kind == "parallel":
        w["l0.mix.right.a2.b"] = torch.full((32,), 9.0)         # sigmoid ~ 1: decay ~ 1
    else:
        w["l0.mix.A_log"], w["l0.mix.D"] = torch.full((2,), -9.0), torch.zeros(2)
    model, _ = build(cfg, weights=w, max_tokens=512, page_size=16)
    return cfg, w, model


@pytest.mark.parametrize("kind", ["parallel", "mamba2"])
@pytest.mark.parametrize("cuts", [[400], [340] + [1] * 60, [2, 14, 16, 1, 31, 64, 272]])
def test_recurrent_state_keeps_the_first_tokens_over_hundreds_of_steps(kind, cuts):
    cfg, w, model = long_memory(kind)
    h = inputs(cfg, 400, 5, 0.5)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref, slack = mixer_ref(kind, h, p, m, 1e-5)
    h2 = h.clone()
    h2[1] = h2[1] * -3.0                                        # what the second token wrote is still read at the end
    assert (O.MIXERS[kind](h2.double(), p, m, 1e-5)[-1] - ref[-1]).abs().max() > 1e-3
    close(run_mixer(model, 0, h, cuts), ref, 5e-5, slack)


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_convolution_portions_shorter_than_equal_to_and_beyond_its_taps(taps):
    mixer = dict(SSM, conv=taps)
    cfg = small_config(layers=[layer("mamba2", mixer, None)])
    model, w = build(cfg, 27)
    h = inputs(cfg, 40, 8)
    p = part(w, "l0.mix.")
    ref = O.mamba2(h.double(), p, mixer, 1e-5)
    if taps > 1:
        last = dict(p, conv=torch.cat([torch.zeros_like(p["conv"][:, :-1]), p["conv"][:, -1:]], dim=1))
        assert (O.mamba2(h.double(), last, mixer, 1e-5) - ref).abs().max() > 1e-3      # the earlier tokens' taps matter
    for cuts in ([25] + [1] * 15, [1, 1, 1, 37], [2, 2, 36], [3, 37], [4, 36], [5, 35], [16, 24], [40]):
        close(run_mixer(model, 0, h, cuts), ref, 2e-5)


# ---- precisions, replayed steps, drawn sizes ------------------------------------------------------------------------------
def wide_config():
    """Sizes the tensor-core kernel takes: every product of a 64-row step runs with bfloat16 operands."""
    mixer = pair(4, 2, 32, 4, 32, 48, window=30, scale=0.18, rot={"base": 10000.0, "dims": 32, "scaling": YARN}, ls=0.7, rs=0.8)
    return small_config(width=128, vocab=256, token_side={"dim": 24},
                        layers=[layer("parallel", mixer, {"kind": "dense", "ff": 160}), layer("mamba2", ssm(8, 32, 64, 2, 4, 4), {"kind": "dense", "ff": 128}),
                                layer("parallel", mixer, {"kind": "dense", "ff": 128})])


@pytest.mark.parametrize("make", [wide_config, small_config])
def test_bfloat16_products_stay_within_bfloat16_rounding_of_the_oracle(make):
    cfg = make()
    lo, w = build(cfg, 31, dtype="bfloat16")
    toks = tokens(cfg, 70, 13)
    ref = O.forward(cfg, w, toks)
    got = whole(lo, "a", toks).cpu().double()
    err = (got - ref).abs().amax(dim=-1) / ref.abs().max()
    assert err.max() < 4e-2 and err.median() < 2e-2, (err.max(), err.median())
    dec = torch.cat([lo.run_step([{"id": "d", "tokens": toks[:40], "want": list(range(40))}])] +
                    [lo.run_step([{"id": "d", "tokens": [t], "want": [0]}]) for t in toks[40:]]).cpu().double()
    lo.run_step([], ["d"])
    err = (dec - ref).abs().amax(dim=-1) / ref.abs().max()
    assert err.max() < 4e-2 and err.median() < 2e-2, (err.max(), err.median())


def test_replayed_step_graphs_give_the_same_bits_as_plain_launches():
    cfg = small_config()
    a, w = build(cfg, 32, step_graphs=True)
    b, _ = build(cfg, 32, step_graphs=False)
    toks = tokens(cfg, 30, 14)
    for m in (a, b):
        m.run_step([{"id": "s", "tokens": toks[:20], "want": []}])
    for t in toks[20:]:
        ga = a.run_step([{"id": "s", "tokens": [t], "want": [0]}])
        gb = b.run_step([{"id": "s", "tokens": [t], "want": [0]}])
        assert torch.equal(ga, gb)


def drawn_config(seed):
    g = torch.Generator().manual_seed(4000 + seed)
    r = lambda lo, hi: int(torch.randint(lo, hi + 1, (1,), generator=g))          # noqa: E731
    layers = []
    for _ in range(r(2, 5)):
        H = r(1, 6)
        groups = [k for k in range(1, H + 1) if H % k == 0]
        if r(0, 1):
            kind, dim = "parallel", r(3, 40)
            rot = None
            if r(0, 3):
                rot = {"base": float(10 ** r(1, 6)), "dims": 2 * r(0, dim // 2)}
                if r(0, 1):
                    rot["scaling"] = {"factor": float(r(1, 8)), "original": r(20, 5000), "fast": 2.0 ** r(1, 6), "slow": 2.0 ** -r(0, 3)}
            m = pair(H, groups[r(0, len(groups) - 1)], dim, r(1, 6), r(2, 40), r(2, 40), window=r(1, 70) if r(0, 3) else None, rot=rot,
                     scale=0.05 + 0.05 * r(0, 8), tau=2.0 ** r(-1, 5), ls=0.25 * r(1, 8), rs=0.25 * r(1, 8))
        else:
            kind, vdim = "mamba2", r(2, 40)
            parts = [k for k in range(1, H * vdim + 1) if H * vdim % k == 0]
            m = ssm(H, vdim, r(2, 70), groups[r(0, len(groups) - 1)], r(1, 6), parts[r(0, len(parts) - 1)])
        layers.append(layer(kind, m, {"kind": "dense", "ff": r(5, 70)} if r(0, 3) else None))
    return {"architecture": "Loduzen", "vocab": r(20, 200), "width": r(16, 120), "norm": {"eps": 10.0 ** -r(4, 7)},
            "token_side": {"dim": r(1, 30)}, "layers": layers}


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations_whole_portioned_and_decoded(seed):
    cfg = drawn_config(seed)
    model, w = build(cfg, 40 + seed, page_size=(4, 8, 16)[seed % 3], rank=1 + 3 * seed)
    toks = tokens(cfg, 75, seed)
    ref = O.forward(cfg, w, toks)
    slack = (O.forward(cfg, w, toks, dtype=torch.float32).double() - ref).abs().max().item()
    close(whole(model, "a", toks), ref, 2e-4, slack)
    got, at = [], 0
    for n in (7, 2, 19, 1, 1, 12):
        got.append(model.run_step([{"id": "p", "tokens": toks[at:at + n], "want": list(range(n))}]))
        at += n
    got += [model.run_step([{"id": "p", "tokens": [t], "want": [0]}]) for t in toks[at:]]
    model.run_step([], ["p"])
    close(torch.cat(got), ref, 2e-4, slack)


# ---- generation through the scheduler, the registry and the command line ---------------------------------------------------
def test_greedy_generation_through_the_scheduler():
    cfg = small_config()
    model, w = build(cfg, 17, max_tokens=400, max_sequences=3, max_rows=24)
    prompts = [tokens(cfg, 37, 20), tokens(cfg, 5, 21), tokens(cfg, 1, 22), tokens(cfg, 50, 23), tokens(cfg, 18, 24)]
    outs = model.generate(prompts, max_new_tokens=10, max_step_tokens=24)      # 5 requests over 3 slots, portioned prompts
    assert model.state.free_slots == 3 and model.state.free_pages == model.state.n_pages
    for p, o in zip(prompts, outs):
        assert len(o) == 10
        ref = O.forward(cfg, w, p + o[:-1])[len(p) - 1:]
        top2 = torch.topk(ref, 2, dim=-1)
        for t, tok in enumerate(o):
            if tok != int(top2.indices[t, 0]):                 # only an exact near-tie may go the other way
                assert tok == int(top2.indices[t, 1]) and float(top2.values[t, 0] - top2.values[t, 1]) < 1e-4
    assert model.generate(prompts[:2], max_new_tokens=10) == outs[:2]


def test_registry_loads_a_model_folder_and_the_trace_command_replays_steps(tmp_path):
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    from dia_tts_prune_b200.checkpoint import save_safetensors
    from dia_tts_prune_b200.registry import load_model
    cfg = odd_config()
    w = O.random_weights(cfg, 30)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tmp_path / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in w.items()})
    model = load_model(tmp_path, dtype="float32", max_tokens=128)
    toks = tokens(cfg, 40, 31)
    ref = O.forward(cfg, w, toks)
    close(whole(model, "r", toks), ref)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[33:35], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[35:], "want": [4, 1]}], "end": ["x"]}]
    root = Path(__file__).resolve().parents[1]
    r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "out" / "1.f32").exists()
    got0 = torch.from_numpy(np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").reshape(2, -1))
    got2 = torch.from_numpy(np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(2, -1))
    close(got0, ref[[0, 32]])
    close(got2, ref[[39, 36]])
