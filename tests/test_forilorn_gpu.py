"""GPU parity of the Forilorn language model against the plain restatement in ``oracle/forilorn_oracle.py``.

Small made-up configurations and random weights; the product runs through ``CausalLM`` / ``LMEngine`` (state records,
scheduler, CUDA kernels), the oracle recomputes whole sequences in float64 on the CPU without cache or carried state.
"""

import copy
import json

import pytest
import torch

from oracle import forilorn_oracle as O

pytestmark = pytest.mark.gpu

ATT = {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 20, "scale": 0.4, "mask": {"size": 22}, "rot": {"base": 700.0, "dims": 16}}
LAT = {"heads": 5, "dim": 12, "rot_dim": 8, "vdim": 16, "q_rank": 28, "kv_rank": 36, "scale": 0.25, "mask": {"size": 19},
       "rot": {"base": 300.0, "dims": 8}}
DENSE = {"kind": "dense", "ff": 72}
BIGRAM = {"buckets": 53, "mul_prev": 7, "mul_cur": 11}


def layer(kind, mixer, mlp=DENSE):
    return {"type": kind, "mixer": copy.deepcopy(mixer), "mlp": copy.deepcopy(mlp)}


def small_config(**over):
    cfg = {"architecture": "Forilorn", "vocab": 130, "width": 96, "norm": {"eps": 1e-5}, "residual_mult": 0.45,
           "embedding": {"scale": 9.5, "bigram": dict(BIGRAM)},
           "layers": [layer("latent_attention", LAT), layer("attention", ATT), layer("attention", ATT), layer("latent_attention", LAT),
                      layer("attention", ATT)]}
    cfg.update(over)
    return cfg


def att(heads, kv_heads, dim, chunk=None, rot=None, scale=0.3):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = rot
    return m


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, window=None, base=1000.0, scale=0.25):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        m["mask"] = {"size": window}
    return m


def odd_config():
    """Sizes that share nothing and are multiples of nothing: one head and several, as many key heads as heads and fewer, odd head
    sizes, chunks and windows of 1, beyond the prompt and none, rotation of a part of the channels, of all and of none, ranks
    above and below the width, value sizes apart from the key sizes, layers without feed-forward, multipliers beyond the buckets,
    a negative residual multiplier."""
    return {"architecture": "Forilorn", "vocab": 77, "width": 74, "norm": {"eps": 1e-6}, "residual_mult": -1.3,
            "embedding": {"scale": 0.7, "bigram": {"buckets": 10, "mul_prev": 1000003, "mul_cur": 3}},
            "layers": [layer("attention", att(5, 5, 11, chunk=1, rot={"base": 10000.0, "dims": 10}), None),
                       layer("latent_attention", lat(3, 9, 6, 7, 85, 33, window=1)),
                       layer("attention", att(6, 1, 7, chunk=500)),
                       layer("latent_attention", lat(1, 34, 10, 1, 5, 91, window=500, base=20.0), None),
                       layer("attention", att(1, 1, 34, rot={"base": 5e5, "dims": 34})),
                       layer("latent_attention", lat(4, 3, 2, 30, 17, 12)),
                       layer("attention", att(2, 2, 9, chunk=33))]}


def build(cfg, seed=1, dtype="float32", weights=None, **kw):
    from dia_tts_prune_b200.lm_config import ForilornConfig
    from dia_tts_prune_b200.lm_model import CausalLM
    w = O.random_weights(cfg, seed) if weights is None else weights
    kw.setdefault("max_tokens", 640)
    kw.setdefault("page_size", 8)
    return CausalLM(ForilornConfig.model_validate(cfg), w, dtype=dtype, device="cuda:0", **kw), w


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
    """The attention kernels alone on given stacked projections q | k | gate: the oracle gets the same numbers through an identity
    output projection."""
    cfg = small_config(layers=[layer("attention", ATT, None)])
    model, w = build(cfg, 5)
    p = part(w, "l0.mix.")
    h = inputs(cfg, 40, 2)
    rows = torch.cat([p["q"], p["k"], p["g"]])
    for n in (40, 5):
        seq = model.state.open(f"k{n}")
        model.state.reserve(seq, n)
        got = model.engine.op_mixer_kernels(0, (h[:n].double() @ rows.T).float(), [(seq, n, 0)])
        close(got, O.attention(h[:n].double(), dict(p, o=torch.eye(120, dtype=torch.float64)), ATT, 1e-5), 2e-5)


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 40])
def test_dense_unit_with_the_tanh_form_of_gelu(rows):
    cfg = small_config()
    model, w = build(cfg, 5)
    h = inputs(cfg, rows, rows, 2.0)
    p = part(w, "l1.mlp.")
    ref = O.dense_ff(h.double(), p)
    z = h.double() @ p["up"].T
    assert (z > 1).any() and (z < -1).any()
    exact = torch.nn.functional.gelu(z) @ p["down"].T             # the error-function form is another function
    assert (exact - ref).abs().max() > 1e-4
    close(model.engine.op_ff(1, h.cuda()), ref, 1e-6)


@pytest.mark.parametrize("rows,width,ff", [(32, 96, 72), (70, 128, 160), (300, 64, 520)])
def test_gelu_in_the_tensor_core_products_epilogue(rows, width, ff):
    """bfloat16 products: the activated operand leaves the first product as bfloat16; large negative and positive pre-activations
    stay finite."""
    cfg = small_config(width=width, layers=[layer("attention", ATT, {"kind": "dense", "ff": ff})])
    w = O.random_weights(cfg, 5)
    w["l0.mlp.up"][:7] *= 512.0                                   # pre-activations in the thousands, either sign
    model, _ = build(cfg, weights=w, dtype="bfloat16")
    h = inputs(cfg, rows, rows, 2.0)
    p = part(w, "l0.mlp.")
    hb = h.to(torch.bfloat16).double()
    z = hb @ p["up"].T
    assert z[:, :7].max() > 500 and z[:, :7].min() < -500
    mid = O.gelu(z).to(torch.bfloat16).double()
    ref = mid @ p["down"].T
    got = model.engine.op_ff(0, h.cuda()).cpu().double()
    slack = (O.gelu(z) @ p["down"].T - ref).abs().max().item()    # a few operands may round the other way
    assert torch.isfinite(got).all() and (got - ref).abs().max() <= slack + 1e-4 * ref.abs().max(), (got - ref).abs().max()


ATTENTIONS = [(4, 2, 64, 50), (16, 16, 32, 7), (3, 1, 100, 64), (2, 2, 200, 65), (12, 4, 40, 33), (5, 5, 9, 3), (1, 1, 256, 90), (6, 2, 18, None),
              (8, 1, 130, 16), (7, 7, 1, 40), (32, 1, 48, 63), (9, 3, 2, 128)]


@pytest.mark.parametrize("heads,kv_heads,dim,chunk", ATTENTIONS)
def test_chunked_attention_with_other_shapes(heads, kv_heads, dim, chunk):
    cfg = small_config(layers=[layer("attention", att(heads, kv_heads, dim, chunk=chunk, scale=1.3 * dim ** -0.5,
                                                      rot={"base": 300.0, "dims": dim - dim % 2} if dim > 1 else None), None)])
    model, w = build(cfg, 48)
    h = inputs(cfg, 140, dim)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref, slack = mixer_ref("attention", h, p, m, 1e-5)
    if chunk:
        as_window = O.in_chunk
        try:
            O.in_chunk = O.in_window                              # a sliding window of the same size is another thing
            assert (O.attention(h.double(), p, m, 1e-5) - ref).abs().max() > 1e-2
        finally:
            O.in_chunk = as_window
    close(run_mixer(model, 0, h, [100] + [1] * 40), ref, 2e-5, slack)
    close(run_mixer(model, 0, h, [5, 2, 60, 9, 64]), ref, 2e-5, slack)


LATENTS = [(4, 64, 32, 64, 96, 128, 50), (16, 8, 16, 12, 20, 24, 7), (3, 20, 2, 100, 64, 200, 64), (2, 128, 64, 64, 300, 256, 65), (9, 5, 6, 9, 11, 13, 33),
           (1, 1, 2, 1, 1, 1, 40), (6, 18, 0, 10, 30, 40, None), (70, 4, 4, 6, 16, 48, 16), (3, 16, 32, 16, 24, 300, 21), (5, 24, 26, 40, 50, 600, None)]


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,q_rank,kv_rank,window", LATENTS)
def test_latent_attention_with_other_shapes(heads, dim, rot_dim, vdim, q_rank, kv_rank, window):
    """Ranks beyond what the tiled kernel takes and more heads than it holds among them."""
    cfg = small_config(layers=[layer("latent_attention", lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, scale=(dim + rot_dim) ** -0.5), None)])
    model, w = build(cfg, 49)
    h = inputs(cfg, 100, vdim)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref, slack = mixer_ref("latent_attention", h, p, m, 1e-5)
    close(run_mixer(model, 0, h, [70] + [1] * 30), ref, 2e-5, slack)


def without(name):
    """The oracle with one piece of its arithmetic taken out, for contrast."""
    real = {"rms_unit": O.rms_unit, "rotate": O.rotate}
    swap = {"rms_unit": lambda x, eps: x if x.dim() == 3 else real["rms_unit"](x, eps), "rotate": lambda x, pos, rot: x}

    class Ctx:
        def __enter__(self):
            setattr(O, name, swap[name])

        def __exit__(self, *a):
            setattr(O, name, real[name])
    return Ctx()


def test_values_are_the_raw_keys_norms_have_no_weight_and_the_gate_is_elementwise():
    cfg = small_config(layers=[layer("attention", att(4, 2, 24, chunk=30, rot={"base": 50.0, "dims": 16}, scale=0.4), None)])
    model, w = build(cfg, 50)
    h = inputs(cfg, 80, 3, 0.6)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref = O.attention(h.double(), p, m, 1e-5)
    for name in ("rms_unit", "rotate"):
        with without(name):
            assert (O.attention(h.double(), p, m, 1e-5) - ref).abs().max() > 1e-2
    per_head = p["g"].reshape(4, 24, 96)[:, :1].expand(4, 24, 96).reshape(96, 96)      # one gate row per head is another thing
    assert (O.attention(h.double(), dict(p, g=per_head), m, 1e-5) - ref).abs().max() > 1e-2
    close(run_mixer(model, 0, h, [65] + [1] * 15), ref, 2e-5)
    # the first token of a chunk sees itself alone: its own key, as projected, gated
    for i in (0, 30, 60):
        k = (h[i].double() @ p["k"].T).reshape(2, 24).repeat_interleave(2, dim=0).reshape(-1)
        own = (k * torch.sigmoid(h[i].double() @ p["g"].T)) @ p["o"].T
        assert (own - ref[i]).abs().max() < 1e-12
        close(run_mixer(model, 0, h[:i + 1], [i + 1])[i], own, 1e-5)


def test_small_queries_and_keys_are_normed_with_eps_inside_the_root():
    cfg = small_config(norm={"eps": 1e-2}, layers=[layer("attention", ATT, None), layer("latent_attention", LAT, None)])
    w = O.random_weights(cfg, 8)
    for name in ("l0.mix.q", "l0.mix.k", "l1.mix.dq", "l1.mix.dkv"):
        w[name] = w[name] * 2.0 ** -4
    model, _ = build(cfg, weights=w)
    h = inputs(cfg, 50, 3)
    for i, lc in enumerate(cfg["layers"]):
        p = part(w, f"l{i}.mix.")
        ref = O.MIXERS[lc["type"]](h.double(), p, lc["mixer"], 1e-2)
        assert (O.MIXERS[lc["type"]](h.double(), p, lc["mixer"], 0.0) - ref).abs().max() > 1e-3
        close(run_mixer(model, i, h, [35] + [1] * 15), ref, 1e-5)


def test_one_gate_number_per_head_and_the_shared_turned_key_part():
    cfg = small_config(layers=[layer("latent_attention", dict(LAT, scale=0.5), None)])
    model, w = build(cfg, 51)
    h = inputs(cfg, 60, 4)
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref = O.latent_attention(h.double(), p, m, 1e-5)
    assert (O.latent_attention(h.double(), dict(p, g=p["g"].roll(1, 0)), m, 1e-5) - ref).abs().max() > 1e-2      # another head's number
    with without("rotate"):
        assert (O.latent_attention(h.double(), p, m, 1e-5) - ref).abs().max() > 1e-3
    no_turned = dict(p, dkv=torch.cat([p["dkv"][:36], 0 * p["dkv"][36:]]))
    assert (O.latent_attention(h.double(), no_turned, m, 1e-5) - ref).abs().max() > 1e-2
    close(run_mixer(model, 0, h, [45] + [1] * 15), ref, 2e-5)


@pytest.mark.parametrize("width", [96, 74, 1028, 2052, 4100])
@pytest.mark.parametrize("rows", [1, 8, 33])
def test_outputs_are_normed_around_one_and_weighed(width, rows):
    """A layer with a dense unit alone behind a mixer that gives nothing (zero output rows: its normed output is zero): the
    residual takes mult x norm(unit(x)), for widths of one and of several vector loads per thread and off every vector width."""
    cfg = small_config(width=width, residual_mult=-0.7, layers=[layer("attention", att(1, 1, 4), {"kind": "dense", "ff": 24})])
    w = O.random_weights(cfg, 6)
    w["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])
    for dtype in ("float32", "bfloat16"):
        model, _ = build(cfg, weights=w, dtype=dtype)
        toks = tokens(cfg, rows, 3)
        ref, streams = O.forward(cfg, w, toks, keep_layers=True)
        x = O.embedding(cfg, {k: v.double() for k, v in w.items()}, toks)
        plain = x - 0.7 * O.rms_unit(O.dense_ff(x, part(w, "l0.mlp.")), 1e-5) * w["l0.norm2"].double()      # a weight around zero
        assert (plain - streams[0]).abs().max() > 1e-1
        got, got_streams = whole(model, "a", toks, keep_layers=True)
        close(got_streams, streams, 1e-5 if dtype == "float32" else 2e-2)
        close(got, ref, 1e-4 if dtype == "float32" else 2e-2)


# ---- the embedding --------------------------------------------------------------------------------------------------------
def embedding_only(**over):
    """One layer whose sublayer gives nothing, so that the kept residual is the embedding itself."""
    cfg = small_config(layers=[layer("attention", att(1, 1, 4), None)], **over)
    w = O.random_weights(cfg, 7)
    w["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])
    return cfg, w


@pytest.mark.parametrize("cuts", [[40], [1] * 40, [2] * 20, [7, 1, 8, 1, 1, 22], [39, 1]])
def test_pair_table_rows_follow_the_previous_token_through_every_cut(cuts):
    cfg, w = embedding_only()
    model, _ = build(cfg, weights=w, page_size=4)
    toks = tokens(cfg, 40, 5)
    ref = O.embedding(cfg, {k: v.double() for k, v in w.items()}, toks)
    got, at = [], 0
    for n in cuts:
        got.append(model.run_step([{"id": "e", "tokens": toks[at:at + n], "want": []}], keep_layers=True)[1][0])
        at += n
    close(torch.cat(got), ref, 1e-6)


def test_pair_table_multipliers_first_row_and_scale():
    big = {"buckets": 97, "mul_prev": 10 ** 12 + 39, "mul_cur": 2 ** 40 + 15}
    for bigram, scale in ((big, 3.0), ({"buckets": 1, "mul_prev": 5, "mul_cur": 0}, 1.0), ({"buckets": 12, "mul_prev": 0, "mul_cur": 1}, -2.0),
                          (None, 0.25)):
        emb = {"scale": scale}
        if bigram:
            emb["bigram"] = bigram
        cfg, w = embedding_only(embedding=emb)
        model, _ = build(cfg, weights=w)
        toks = tokens(cfg, 30, 6)
        wd = {k: v.double() for k, v in w.items()}
        ref = O.embedding(cfg, wd, toks)
        if bigram:
            assert (ref[0] - (wd["embed"][toks[0]] * scale + wd["bigram"][-1])).abs().max() == 0
            swapped = dict(bigram, mul_prev=bigram["mul_cur"], mul_cur=bigram["mul_prev"])
            if bigram["buckets"] > 1:
                assert (O.embedding(dict(cfg, embedding={"scale": scale, "bigram": swapped}), wd, toks) - ref).abs().max() > 0.1
        got = model.run_step([{"id": "e", "tokens": toks, "want": []}], ["e"], keep_layers=True)[1][0]
        close(got, ref, 1e-6)


def test_kept_tokens_of_a_freed_page_do_not_reach_the_next_sequence():
    cfg, w = embedding_only()
    model, _ = build(cfg, weights=w, page_size=4, max_tokens=24, max_sequences=2)
    wd = {k: v.double() for k, v in w.items()}
    A, B = tokens(cfg, 20, 1), tokens(cfg, 18, 2)
    model.run_step([{"id": "A", "tokens": A, "want": []}])
    pages = list(model.state.sequences["A"].pages)
    model.run_step([], ["A"])
    first = model.run_step([{"id": "B", "tokens": B[:1], "want": []}], keep_layers=True)[1][0]
    rest = [model.run_step([{"id": "B", "tokens": [t], "want": []}], keep_layers=True)[1][0] for t in B[1:]]
    assert set(model.state.sequences["B"].pages) <= set(pages)
    close(torch.cat([first] + rest), O.embedding(cfg, wd, B), 1e-6)


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


def test_layers_without_feed_forward_and_without_pair_table():
    cfg = small_config(layers=[layer("attention", ATT, None), layer("latent_attention", LAT), layer("latent_attention", LAT, None)],
                       embedding={"scale": 4.0})
    model, w = build(cfg, 9)
    assert model.state.token_pages is None
    toks = tokens(cfg, 40, 5)
    got = [model.run_step([{"id": "d", "tokens": toks[:30], "want": list(range(30))}])]
    got += [model.run_step([{"id": "d", "tokens": [t], "want": [0]}]) for t in toks[30:]]
    close(torch.cat(got), O.forward(cfg, w, toks))


def test_sublayers_run_one_after_the_other_on_the_stream_itself():
    """With the feed-forward reading the residual from before the mixer, or with input norms, the oracle differs."""
    cfg = small_config()
    model, w = build(cfg, 10)
    toks = tokens(cfg, 33, 5)
    ref = O.forward(cfg, w, toks)
    wd = {k: v.double() for k, v in w.items()}
    for early_ff in (True, False):
        x = O.embedding(cfg, wd, toks)
        read = (lambda v: v) if early_ff else (lambda v: O.rms_unit(v, 1e-5))
        for i, lc in enumerate(cfg["layers"]):
            p, old = f"l{i}.", x
            x = x + 0.45 * O.zero_norm(O.MIXERS[lc["type"]](read(x), O.part(wd, p + "mix."), lc["mixer"], 1e-5), wd[p + "norm1"], 1e-5)
            x = x + 0.45 * O.zero_norm(O.dense_ff(old if early_ff else read(x), O.part(wd, p + "mlp.")), wd[p + "norm2"], 1e-5)
        assert (O.zero_norm(x, wd["final.norm"], 1e-5) @ wd["embed"].T - ref).abs().max() > 1e-2
    close(whole(model, "a", toks), ref)


@pytest.mark.parametrize("make", [small_config, odd_config])
def test_prefill_then_long_token_by_token_decoding(make):
    cfg = make()
    model, w = build(cfg, 12)
    toks = tokens(cfg, 150, 3)
    ref = O.forward(cfg, w, toks)
    slack = (O.forward(cfg, w, toks, dtype=torch.float32).double() - ref).abs().max().item()
    got = [model.run_step([{"id": "d", "tokens": toks[:9], "want": list(range(9))}])]
    for t in range(9, 150):                                     # windows and chunks pass over decoded tokens
        got.append(model.run_step([{"id": "d", "tokens": [toks[t]], "want": [0]}], ["d"] if t == 149 else []))
    close(torch.cat(got), ref, slack=slack)


@pytest.mark.parametrize("make", [small_config, odd_config])
@pytest.mark.parametrize("cuts", [[2] * 40, [1, 2, 3, 5, 8, 13, 21, 27], [19, 1, 20, 21, 2, 17], [21, 1, 1, 21, 22, 14], [79, 1], [3, 77]])
def test_portions_of_any_size_give_the_same_logits(make, cuts):
    cfg = make()
    model, w = build(cfg, 13, max_rows=32)                      # long portions are also split by the engine itself
    toks = tokens(cfg, 80, 4)
    ref = O.forward(cfg, w, toks)
    slack = (O.forward(cfg, w, toks, dtype=torch.float32).double() - ref).abs().max().item()
    assert sum(cuts) == 80
    got, at = [], 0
    for n in cuts:
        got.append(model.run_step([{"id": "p", "tokens": toks[at:at + n], "want": list(range(n))}]))
        at += n
    model.run_step([], ["p"])
    close(torch.cat(got), ref, slack=slack)
    close(torch.cat(got), whole(model, "q", toks).cpu(), 2e-5, slack)   # how the rows were cut changes rounding at most


@pytest.mark.parametrize("make", [small_config, odd_config])
def test_mixed_batch_of_unequal_requests_equals_each_alone(make):
    cfg = make()
    model, w = build(cfg, 15, max_sequences=4)
    A, B, C = tokens(cfg, 50, 6), tokens(cfg, 31, 7), tokens(cfg, 12, 8)
    alone = {n: whole(model, n, t) for n, t in (("A", A), ("B", B), ("C", C))}
    ref = O.forward(cfg, w, A)
    slack = (O.forward(cfg, w, A, dtype=torch.float32).double() - ref).abs().max().item()
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
        close(got, alone[n][:got.shape[0]].cpu(), 2e-5, slack)
    close(alone["A"], ref, slack=slack)
    both = model.run_step([{"id": "A", "tokens": A, "want": list(range(50))},
                           {"id": "B", "tokens": B, "want": list(range(31))}], ["A", "B"])
    assert torch.equal(both[:50], alone["A"]) and torch.equal(both[50:], alone["B"])


def test_freed_pages_and_slots_are_used_again():
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
    # Z takes X's slot and pages - dirty with X's keys, latents and tokens - and starts with two tokens, while Y's stay
    gz = model.run_step([{"id": "Z", "tokens": Z[:2], "want": [0, 1]}])
    assert st.sequences["Z"].slot == slot_x and set(st.sequences["Z"].pages) <= set(pages_x)
    gz1 = model.run_step([{"id": "Z", "tokens": Z[2:40], "want": list(range(38))}])
    gz2 = model.run_step([{"id": "Z", "tokens": Z[40:], "want": list(range(24))}], ["Z", "Y"])
    close(gx, ref["X"])
    close(gy, ref["Y"])
    close(torch.cat([gz, gz1, gz2]), ref["Z"])
    assert st.free_pages == st.n_pages and st.free_slots == 2
    from dia_tts_prune_b200.lm_state import OutOfPages
    with pytest.raises(OutOfPages):
        model.run_step([{"id": "big", "tokens": tokens(cfg, 200, 1), "want": []}])


# ---- inputs and weights made so that one key stands out -------------------------------------------------------------------
def standout(kind, page_size, size):
    """One layer in which a position whose input points the way the query's input does gets a score far above all others (no
    rotation to speak of: queries equal keys in the attention, and the latent attention's turned part is off)."""
    if kind == "attention":
        cfg = small_config(layers=[layer(kind, att(2, 2, 32, chunk=size, scale=0.6), None)])
        w = O.random_weights(cfg, 21)
        w["l0.mix.q"] = w["l0.mix.k"]
    else:
        cfg = small_config(layers=[layer(kind, lat(2, 32, 2, 16, 40, 40, window=size, scale=0.2), None)])
        w = O.random_weights(cfg, 21)
        w["l0.mix.dq"], w["l0.mix.dq.norm"] = w["l0.mix.dkv"][:40], w["l0.mix.dkv.norm"]
        up = torch.zeros(2, 34, 40)
        up[:, :32] = w["l0.mix.uk"].reshape(2, 32, 40)
        w["l0.mix.uq"] = up.reshape(68, 40)
    model, _ = build(cfg, weights=w, max_tokens=512, page_size=page_size)
    return cfg, w, model


def is_seen(kind, i, j, size):
    rule = O.in_chunk if kind == "attention" else O.in_window
    return j <= i and (size is None or rule(i, j, size))


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("size", [None, 130, 75, 64, 160])
def test_standout_key_far_away_at_page_tile_window_and_chunk_borders(kind, decode, size):
    P = 16
    cfg, w, model = standout(kind, P, size)
    T = 300
    g = torch.Generator().manual_seed(2)
    base = torch.randn(T, 96, generator=g) * 0.3
    mark, near = torch.randn(96, generator=g) * 3, torch.randn(96, generator=g) * 0.5
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    i = T - 1
    blank = base.clone()
    blank[i] = mark
    ref_blank = O.MIXERS[kind](blank.double(), p, m, 1e-5)
    span = size or T + 1
    lo = (i // span) * span if kind == "attention" else i - span + 1      # the first key the last row sees
    # the first token, far back among hundreds, both sides of page borders and of the 64-key tile border, the neighbour, and the
    # first key inside and the last outside the window or chunk
    for j in sorted({0, 3, 63, 64, 127, 128, (i // P) * P, (i // P) * P - 1, i - 1, lo - 1, lo, lo + 1} & set(range(T - 1))):
        h = base.clone()
        h[j] = 2 * mark + near                                  # nearly the query's direction, a value of its own
        h[i] = mark
        ref = O.MIXERS[kind](h.double(), p, m, 1e-5)
        carried = (ref[i] - ref_blank[i]).abs().max() > 1e-2
        assert carried == is_seen(kind, i, j, size), j          # the marked key carries the row exactly when it is seen
        n0 = T - 60 if decode else T
        close(run_mixer(model, 0, h, [n0] + [1] * (T - n0)), ref, 3e-5)


@pytest.mark.parametrize("cuts", [[200], [150] + [1] * 50, [3, 61, 2, 64, 70], [95, 2, 2, 3, 98]])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_edge_moves_with_every_row_of_a_portion(kind, cuts):
    """Every row of a portion has its own first visible key: a key made to stand out is seen by exactly the rows of its window or
    its chunk (chunks counted from the sequence's start, wherever the portions are cut)."""
    size = 40
    cfg, w, model = standout(kind, 8, size)
    T = 200
    g = torch.Generator().manual_seed(4)
    h = torch.randn(T, 96, generator=g) * 0.3
    mark, near = torch.randn(96, generator=g) * 3, torch.randn(96, generator=g)
    plain = h.clone()
    h[100] = 2 * mark + 2 * near                                 # (of its own direction: a normed latent has no length)
    h[101:] += mark * 0.5                                        # every later query leans towards the marked key
    plain[101:] += mark * 0.5
    p, m = part(w, "l0.mix."), cfg["layers"][0]["mixer"]
    ref = O.MIXERS[kind](h.double(), p, m, 1e-5)
    gap = (O.MIXERS[kind](plain.double(), p, m, 1e-5) - ref).abs().amax(dim=-1)
    last = 119 if kind == "attention" else 139                  # chunk 80 .. 119; window 100 .. 139
    assert gap[last] > 2e-3 and gap[last + 1:].max() == 0, gap[last]
    close(run_mixer(model, 0, h, cuts), ref, 3e-5)


def test_batches_of_sequences_at_different_places_in_their_chunks():
    """Decoding rows of several sequences in one step, and rows of several sequences in one tile, each with its own chunk and
    window."""
    cfg = small_config(layers=[layer("attention", dict(ATT, mask={"size": 12})), layer("latent_attention", dict(LAT, mask={"size": 7}))])
    model, w = build(cfg, 18, max_sequences=6)
    lens = [11, 12, 13, 24, 1, 35]
    toks = [tokens(cfg, n + 15, 60 + n) for n in lens]
    refs = [O.forward(cfg, w, t) for t in toks]
    got = [[] for _ in lens]

    def run(cut):
        lg = model.run_step([{"id": str(b), "tokens": t[a:z], "want": list(range(z - a))} for b, (t, (a, z)) in enumerate(zip(toks, cut))])
        at = 0
        for b, (a, z) in enumerate(cut):
            got[b].append(lg[at:at + z - a])
            at += z - a
    run([(0, n) for n in lens])
    for k in range(13):
        run([(n + k, n + k + 1) for n in lens])
    run([(n + 13, n + 15) for n in lens])
    for b in range(6):
        close(torch.cat(got[b]), refs[b])


# ---- precisions, replayed steps, drawn sizes ------------------------------------------------------------------------------
def wide_config():
    """Sizes the tensor-core kernel takes: every product of a 64-row step runs with bfloat16 operands."""
    a = att(4, 2, 32, chunk=30, scale=0.9, rot={"base": 10000.0, "dims": 32})
    m = lat(4, 24, 16, 32, 64, 80, window=25, scale=0.16)
    return small_config(width=128, vocab=256, embedding={"scale": 11.3, "bigram": {"buckets": 200, "mul_prev": 31, "mul_cur": 5}},
                        layers=[layer("attention", a, {"kind": "dense", "ff": 160}), layer("latent_attention", m, {"kind": "dense", "ff": 128}),
                                layer("attention", a, {"kind": "dense", "ff": 128})])


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
    g = torch.Generator().manual_seed(5000 + seed)
    r = lambda lo, hi: int(torch.randint(lo, hi + 1, (1,), generator=g))          # noqa: E731
    layers = []
    for _ in range(r(2, 5)):
        H = r(1, 9)
        groups = [k for k in range(1, H + 1) if H % k == 0]
        size = r(1, 70) if r(0, 3) else None
        if r(0, 1):
            dim = r(3, 60)
            rot = {"base": float(10 ** r(1, 6)), "dims": 2 * r(0, dim // 2)} if r(0, 3) else None
            kind, m = "attention", att(H, groups[r(0, len(groups) - 1)], dim, chunk=size, rot=rot, scale=0.1 * r(1, 8))
        else:
            kind, m = "latent_attention", lat(H, r(1, 50), 2 * r(1, 20), r(1, 50), r(2, 90), r(2, 120), window=size, base=float(10 ** r(1, 6)),
                                              scale=0.04 * r(1, 8))
        layers.append(layer(kind, m, {"kind": "dense", "ff": r(5, 90)} if r(0, 3) else None))
    vocab = r(20, 200)
    emb = {"scale": 0.5 * r(1, 30)}
    if r(0, 4):
        emb["bigram"] = {"buckets": r(1, 300), "mul_prev": r(0, 10 ** 6), "mul_cur": r(0, 10 ** 6)}
    return {"architecture": "Forilorn", "vocab": vocab, "width": r(16, 150), "norm": {"eps": 10.0 ** -r(4, 7)}, "residual_mult": 0.1 * r(1, 12),
            "embedding": emb, "layers": layers}


@pytest.mark.parametrize("seed", range(14))
def test_drawn_configurations_whole_portioned_and_decoded(seed):
    cfg = drawn_config(seed)
    model, w = build(cfg, 40 + seed, page_size=(4, 8, 16)[seed % 3])
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
    # a small embedding beside large sublayer outputs: logits against the table itself would otherwise repeat the last token
    cfg = small_config(residual_mult=1.6, embedding={"scale": 0.8, "bigram": dict(BIGRAM)})
    model, w = build(cfg, 17, max_tokens=400, max_sequences=3, max_rows=24)
    prompts = [tokens(cfg, 37, 20), tokens(cfg, 5, 21), tokens(cfg, 1, 22), tokens(cfg, 50, 23), tokens(cfg, 18, 24)]
    outs = model.generate(prompts, max_new_tokens=10, max_step_tokens=24)      # 5 requests over 3 slots, portioned prompts
    assert model.state.free_slots == 3 and model.state.free_pages == model.state.n_pages
    for p, o in zip(prompts, outs):
        assert len(o) == 10 and len(set(o)) >= 2
        ref = O.forward(cfg, w, p + o[:-1])[len(p) - 1:]
        top2 = torch.topk(ref, 2, dim=-1)
        for t, tok in enumerate(o):
            if tok != int(top2.indices[t, 0]):                 # only an exact near-tie may go the other way
                assert tok == int(top2.indices[t, 1]) and float(top2.values[t, 0] - top2.values[t, 1]) < 1e-4
    assert len({t for o in outs for t in o}) >= 8
    assert model.generate(prompts[:2], max_new_tokens=10) == outs[:2]


def test_registry_command_line_and_trace_replay(tmp_path):
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
    slack = (O.forward(cfg, w, toks, dtype=torch.float32).double() - ref).abs().max().item()
    close(whole(model, "r", toks), ref, slack=slack)
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
    close(got0, ref[[0, 32]], slack=slack)
    close(got2, ref[[39, 36]], slack=slack)
    r = subprocess.run([sys.executable, "-m", "dia_tts_prune_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                        " ".join(map(str, toks[:7])), "--max-new-tokens", "5"], capture_output=True, text=True, timeout=600, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == model.generate([toks[:7]], max_new_tokens=5)[0]
