"""The Sezopel design in the engine against the plain numpy statement of it (tests/plain/sezopel_plain.py).

Every test makes its own small configuration and random weights.  Each body runs twice: with the PyTorch stand-ins
for the kernels on the CPU (the parts, the cache manager, the batching), and on the GPU with the real kernels (marked
``gpu``).  The configurations differ from one another in everything a configuration can say: the order of the two kinds of
mixers, keys and values read by one, two or no later layer, key sizes unlike value sizes, part or all or none of a head
rotated, layers without a feed-forward, a model without the tokens' vectors or without caps.
"""

import json
import os

import numpy as np
import pytest
import torch

import sllm_b200.models  # noqa: F401  (registers the parts and the architecture)
from tests import traces
from tests.plain import sezopel_plain as plain
from tests.test_kidolorn import CUTS, _bf16_exact, _portions, _requests, _step, _to, dev, dtypes_on, make_model  # noqa: F401


def _att(heads, kv, dim, vdim, scale, softcap, rot=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
         "rot": {"base": rot[0], "dims": rot[1]} if rot else None}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _ret(decay, dim, vdim, rot=None):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": rot[0], "dims": rot[1]} if rot else None}


def _layer(mixer, ff):
    return {"type": "retention" if "decay" in mixer else "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _config(vocab, width, layers, side=None, scale=1.0, cap=None, eps=1e-5):
    c = {"architecture": "Sezopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if side is not None:
        c["token_side"] = {"dim": side}
    if cap is not None:
        c["logit_softcap"] = cap
    return c


CONFIG_A = _config(300, 96, [                         # keys and values read one and three layers on; a layer without a feed-forward
    _layer(_att(6, 2, 24, 40, 0.4, 6.0, (1000.0, 8)), 120),
    _layer(_att(4, 2, 24, 40, 0.3, 3.0, (1000.0, 8), kv_from=0), None),
    _layer(_ret([0.6, 0.95, 0.998], 16, 24, (500.0, 12)), 72),
    _layer(_att(2, 2, 24, 40, 0.5, None, (1000.0, 8), kv_from=0), 40),
], side=20, scale=8.0, cap=9.0)
CONFIG_B = _config(210, 128, [                        # cached heads of 64 and 128 on pages of 16: the tensor-core attention forms on the GPU (bfloat16)
    _layer(_ret([0.9, 0.9995], 64, 64, (10000.0, 64)), 256),
    _layer(_att(8, 2, 64, 48, 0.25, 10.0, (10000.0, 32)), 192),
    _layer(_att(4, 1, 96, 128, 0.2, 15.0, (300.0, 96)), 128),
    _layer(_ret([0.97, 0.8, 0.99], 32, 48, (10000.0, 16)), None),
    _layer(_att(16, 2, 64, 48, 0.3, 5.0, (10000.0, 32), kv_from=1), 64),
    _layer(_att(3, 1, 96, 128, 0.1, 15.0, (300.0, 96), kv_from=2), 320),
], side=64, scale=11.0, cap=20.0, eps=1e-6)
ODD = _config(77, 50, [                               # sizes that are multiples of nothing; one head; nothing rotated
    _layer(_att(3, 3, 10, 7, 0.6, 4.0, (50.0, 6)), 33),
    _layer(_ret([0.7], 22, 9), 19),
    _layer(_att(1, 1, 13, 18, 0.5, 2.0), None),
    _layer(_ret([0.3, 0.9, 0.5, 0.97, 0.99], 6, 10, (20.0, 2)), 51),
    _layer(_att(6, 3, 10, 7, 0.8, 8.0, (50.0, 6), kv_from=0), 14),
], side=5, scale=5.0, cap=3.0, eps=1e-4)
BARE = _config(90, 64, [                              # no vectors of the tokens, no caps, no feed-forwards; heads of 32 and of 16
    _layer(_att(4, 4, 32, 32, 0.3, None, (10.0, 32)), None),
    _layer(_ret([0.9, 0.99], 16, 16, (100.0, 16)), None),
    _layer(_att(5, 1, 16, 16, 0.4, None), None)], scale=6.0)
RETENTION_ONLY = _config(120, 72, [_layer(_ret([0.5, 0.9, 0.99, 0.999], 32, 16, (10000.0, 32)), 100),
                                   _layer(_ret([0.95, 0.9], 40, 64), None)], side=8, scale=4.0, cap=30.0)
MID = _config(1000, 352, [                            # a few hundred channels, no power of two: the products' tensor-core forms between tiny and real
    _layer(_att(12, 3, 64, 64, 0.2, 12.0, (20000.0, 24)), 1024),
    _layer(_ret([0.6, 0.99, 0.999, 0.9999, 0.9], 64, 48, (20000.0, 48)), 768),
    _layer(_att(6, 3, 64, 64, 0.15, 20.0, (20000.0, 24), kv_from=0), 512),
    _layer(_ret([0.97, 0.9997], 96, 160, (20000.0, 96)), 640),
], side=32, scale=10.0, cap=12.0)
CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 16), "odd": (ODD, 8), "bare": (BARE, 4), "retention": (RETENTION_ONLY, 32), "mid": (MID, 16)}


def plain_logits(d, reqs):
    cfg, w = plain.load_model(d)
    return {r: plain.forward(ids, cfg, w).astype(np.float32) for r, ids in reqs.items()}


def models_for(tmp_path, config, dev, reqs, seed=5, edit=None):
    """(dtype, model folder, plain logits) for every dtype the device runs."""
    d = make_model(tmp_path, config, seed=seed, edit=edit)
    want = plain_logits(d, reqs)
    for dtype in dtypes_on(dev):
        yield dtype, d, want


def compare(tr, out, want, dtype, what):
    """float32: every logit to 3e-4.  bfloat16: the difference of a row (mean taken off, root mean square over the vocabulary)
    relative to the row's own spread is rounding's: under 4 % for 19 rows in 20, under 15 % for 99 in 100.  (Every sublayer's output
    is divided by its own size, a head's too: where terms all but cancel, their rounding is divided as well, so the odd row may
    lie further out, and is then held to 40 %.)"""
    if dtype == "float32":
        return traces.compare(tr, out, want, what=what, rtol=3e-4, atol=3e-4)
    errs = []
    for s in tr.steps:
        for row, (req, pos) in enumerate(s["expect"]):
            ref, got = want[req][pos], out[s["step"]][row]
            d, r = got - ref, ref - ref.mean()
            errs.append(float(np.sqrt(((d - d.mean()) ** 2).mean()) / np.sqrt((r ** 2).mean())))
            assert errs[-1] < 0.4, f"{what}: step {s['step']}, request {req!r}, position {pos}: relative difference {errs[-1]:.3g}"
    for q, limit in ((0.95, 0.04), (0.99, 0.15)):
        assert np.quantile(errs, q) < limit, f"{what}: quantile {q} of the rows' relative difference {np.quantile(errs, q):.3g}"


def _term(t):
    return (t.sum(0) if t.dim() == 3 else t).float().cpu().numpy()


def _relative(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.maximum(np.sqrt((want ** 2).mean(-1)), 0.01 * np.sqrt((want ** 2).mean()))


# ---- configuration, plan, weights ---------------------------------------------------------------------------

def test_config_plan_and_cache_needs():
    from sllm_b200.config import ConfigError, architecture_of
    from sllm_b200.models.causal_lm import CausalLM
    from sllm_b200.parts import PagedKV, SlotState
    arch = architecture_of(CONFIG_A)
    cfg = arch.config_cls.from_dict(CONFIG_A)
    assert cfg.to_dict() == CONFIG_A
    p = arch.plan(cfg)
    assert len(p.layers) == 4 and [e.layer for e in p.run_list] == [0, 1, 2, 3] and p.position is None
    assert [e.cache_from for e in p.run_list] == [None, 0, None, 0]
    assert p.embedding_scale == 8.0 and p.logit_softcap == 9.0 and p.token_table_width == 4 * 20 and p.ignored_names == ("l1.norm2",)
    assert "ffn" not in p.layers[1].parts and "side" in p.layers[1].parts
    m = CausalLM(p, dtype=torch.float32, device="cpu")
    assert m.cache_needs() == [("own", PagedKV(2, 40, None)), ("borrow", 0), ("own", SlotState((3, 16, 24), "retention")), ("borrow", 0)]
    assert CausalLM(p, dtype=torch.bfloat16, device="cpu").cache_needs()[0] == ("own", PagedKV(2, 64, None))     # a size the tensor-core forms take
    shapes = {s.name: tuple(s.shape) for s in m.tensor_specs()}
    assert set(n for n in shapes if n.startswith("l1.")) == {"l1.norm1", "l1.mix.q", "l1.mix.g", "l1.mix.o", "l1.side.gate", "l1.side.proj",
                                                            "l1.side.norm"}
    assert shapes["embed"] == shapes["head"] == (300, 96) and shapes["side.embed"] == (300, 80) and shapes["final.norm"] == (96,)
    assert shapes["l0.mix.q"] == (144, 96) and shapes["l0.mix.k"] == (48, 96) and shapes["l0.mix.v"] == (80, 96) and shapes["l0.mix.g"] == (6, 96)
    assert shapes["l0.mix.o"] == (96, 240) and shapes["l0.mlp.up"] == (120, 96) and shapes["l0.mlp.down"] == (96, 120)
    assert shapes["l2.mix.g"] == (72, 96) and shapes["l2.mix.o"] == (96, 72) and shapes["l2.side.proj"] == (96, 20)

    bare = architecture_of(BARE)
    q = bare.plan(bare.config_cls.from_dict(BARE))
    assert q.token_table_name is None and q.logit_softcap is None and set(q.layers[0].parts) == {"mixer", "mixer_post"}

    def edited(path, value):
        c = json.loads(json.dumps(CONFIG_A))
        at = c
        for k in path[:-1]:
            at = at[k]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return c
    for bad in (edited(("layers", 2, "mixer", "decay"), [0.5, 0.6]),              # one decay per head
                edited(("layers", 0, "mixer", "kv_heads"), 4),                    # 6 heads on 4
                edited(("layers", 0, "mixer", "rot", "dims"), 7), edited(("layers", 0, "mixer", "rot", "dims"), 26),
                edited(("layers", 3, "mixer", "kv_from"), 2),                     # layer 2 holds no keys and values
                edited(("layers", 3, "mixer", "kv_from"), 1),                     # layer 1 borrows itself
                edited(("layers", 3, "mixer", "kv_from"), 3),
                edited(("layers", 3, "mixer", "dim"), 32), edited(("layers", 3, "mixer", "vdim"), 24), edited(("layers", 1, "mixer", "kv_heads"), 1),
                edited(("layers", 0, "type"), "other"), edited(("layers", 0, "mlp", "kind"), "other"), edited(("layers", 0, "mixer", "scale"), None),
                edited(("norm",), None), edited(("layers",), []), edited(("layers", 2, "mixer", "vdim"), None), edited(("token_side", "dim"), None)):
        with pytest.raises(ConfigError):
            arch.config_cls.from_dict(bad)


# ---- each mechanism alone: an operation or a part against the plain function ------------------------------------------

@pytest.mark.parametrize("W", [50, 96, 1000, 1500, 3000, 4500])     # the kernel keeps rows of up to 1,024, 2,048 and 4,096 channels in registers
def test_norm_of_a_term_and_the_stream_for_the_next_reader(dev, W):
    """The sublayer's term (whole, and as a stack of partial sums) is normed, joins the stream, and the stream comes back in the
    reader's dtype; each half alone too."""
    import sllm_b200.ops as ops
    rng = np.random.default_rng(W)
    T, eps = 7, 1e-3
    x, y, g = rng.standard_normal((T, W)) * 3, rng.standard_normal((3, T, W)) * 0.02, 1 + rng.standard_normal(W)       # (a small term: eps counts)
    to = _to(dev)
    want = x + plain.norm(y.sum(0), g, eps)
    for term in (to(y.sum(0)), to(y)):
        for dtype in (torch.float32, torch.bfloat16, None):
            stream = to(x)
            h = ops.post_add_copy(stream, term, to(g), eps, dtype)
            np.testing.assert_allclose(stream.cpu().numpy(), want, rtol=2e-5, atol=2e-5)
            if dtype is None:
                assert h is None
            else:
                assert h.dtype == dtype
                np.testing.assert_array_equal(h.float().cpu().numpy(), stream.to(dtype).float().cpu().numpy())
    stream = to(x)
    h = ops.post_add_copy(stream, None, None, 0.0, torch.bfloat16)
    np.testing.assert_array_equal(h.float().cpu().numpy(), stream.to(torch.bfloat16).float().cpu().numpy())
    np.testing.assert_array_equal(stream.cpu().numpy(), x.astype(np.float32))


def test_caps_bend_values_into_their_range(dev):
    import sllm_b200.ops as ops
    rng = np.random.default_rng(0)
    for n, cap in ((1, 0.5), (77 * 3, 3.0), (1001, 30.0), (4096, 15.0)):
        z = rng.standard_normal(n) * 20.0 * np.exp(rng.standard_normal(n))
        z[0] = 1e6
        got = ops.softcap_(_to(dev)(z), cap).cpu().numpy()
        np.testing.assert_allclose(got, plain.cap(z, cap), rtol=3e-6, atol=1e-6)
        assert np.abs(got).max() <= cap
    np.testing.assert_array_equal(plain.cap(z, None), z)


def _paged(dev, nkv, D, ps, lens, rng, spare=3):
    """Scattered pages for requests of ``lens`` tokens: random keys and values [pages, nkv, ps, D], tables, the group's view."""
    from sllm_b200.parts import GroupView
    per = [-(-n // ps) for n in lens]
    order = rng.permutation(sum(per) + spare)
    tables = np.full((len(lens), max(per) + 1), -1, dtype=np.int32)
    at = 0
    for s, n in enumerate(per):
        tables[s, :n] = order[at:at + n]
        at += n
    k, v = (rng.standard_normal((sum(per) + spare, nkv, ps, D)).astype(np.float32) for _ in range(2))
    return k, v, tables, GroupView(ps, torch.from_numpy(tables).to(dev), torch.zeros(1, dtype=torch.int32, device=dev))


@pytest.mark.parametrize("D,ps,dtype,nq,nkv,cap", [
    (27, 4, "float32", 3, 1, 4.0), (64, 16, "bfloat16", 8, 2, 6.0), (64, 16, "bfloat16", 24, 1, 30.0), (128, 32, "bfloat16", 6, 3, 5.0),
    (32, 8, "bfloat16", 2, 2, 7.0), (56, 16, "float32", 4, 4, 50.0), (16, 16, "bfloat16", 5, 1, 3.0), (128, 64, "bfloat16", 16, 2, 0.0),
    (64, 8, "bfloat16", 3, 3, 1.5), (80, 16, "bfloat16", 4, 2, 8.0)])
def test_capped_scores_and_gated_heads_over_keys_near_and_far(dev, D, ps, dtype, nq, nkv, cap):
    """Every attention form (single tokens and portions in one step, contexts cut into ranges, scattered pages) with capped
    scores and a sigmoid gate per head.  For every query one key stands out in its first head: the sequence's first token,
    the one a page back, the query's own; the cap decides how much weight it takes, so scores that are not capped, or
    capped after the maximum is taken off, give another output.  Masked keys must weigh nothing although a capped score cannot
    be -inf.  One gate is all but shut, one all but open."""
    import sllm_b200.ops as ops
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(D + nq)
    scale = 0.3
    cases = [(1, 1), (1, 2), (1, 700), (1, 3 * ps), (1, 3 * ps + 1), (2, 2), (5, 5), (2, 2 * ps + 1), (ps + 3, 4 * ps + 2), (3, 333), (150, 150),
             (130, 400), (1, 64), (1, 65)]
    q_lens, ctx = [c[0] for c in cases], [c[1] for c in cases]
    k, v, tables, g = _paged(dev, nkv, D, ps, ctx, rng)
    T = sum(q_lens)
    q = rng.standard_normal((T, nq, D)).astype(np.float32)
    step = _step(dev, q_lens, list(range(len(cases))), ctx, g)
    pos, seq = step.positions.cpu().numpy(), step.seq_of_token.cpu().numpy()
    for t in range(T):
        j = (0, max(pos[t] - ps, 0), pos[t])[t % 3]
        k[tables[seq[t], j // ps], 0, j % ps] = q[t, 0] * (20.0 / np.sqrt(D))
    gates = rng.standard_normal((T, nq + 3)).astype(np.float32)
    gates[:, 2], gates[:, 2 + nq - 1] = -6.0, 5.0
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    qd, kd, vd = (torch.from_numpy(a).to(dev).to(td).contiguous() for a in (q.reshape(T, nq * D), k, v))
    gd = torch.from_numpy(gates).to(dev)
    got = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, None, softcap=cap, gate=(gd, 2)).float().cpu().numpy().reshape(T, nq, D)
    ungated = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, None, softcap=cap).float().cpu().numpy().reshape(T, nq, D)
    qf, kf, vf = (a.float().cpu().numpy().astype(np.float64) for a in (qd, kd, vd))
    qf = qf.reshape(T, nq, D)
    tol = 3e-5 if dtype == "float32" else 3e-2
    for t in range(T):
        js = np.arange(pos[t] + 1)
        kk, vv = kf[tables[seq[t], js // ps], :, js % ps], vf[tables[seq[t], js // ps], :, js % ps]
        for h in range(nq):
            s = plain.cap(kk[:, h // (nq // nkv)] @ qf[t, h] * scale, cap or None)
            e = np.exp(s - s.max())
            o = (e / e.sum()) @ vv[:, h // (nq // nkv)]
            where = f"token {t} (position {pos[t]}), head {h}"
            np.testing.assert_allclose(ungated[t, h], o, rtol=tol, atol=tol, err_msg=where)
            np.testing.assert_allclose(got[t, h], o * plain.sigmoid(gates[t, 2 + h]), rtol=tol, atol=tol, err_msg=where)


@pytest.mark.gpu
@pytest.mark.parametrize("D,nq,nkv,q_len,ctx", [(64, 4, 1, 40, 2500), (128, 8, 2, 33, 2304), (64, 4, 4, 1, 5000), (128, 4, 2, 1, 3001), (32, 4, 2, 1, 2100)])
def test_capped_scores_over_a_context_cut_into_ranges(D, nq, nkv, q_len, ctx):
    """Few rows over thousands of keys: the context is cut into ranges that CTAs of their own walk, the gate is applied where
    they are merged.  A key far back that stands out, and beside it one request's single token."""
    import sllm_b200.ops as ops
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    dev, ps, cap, scale = "cuda:0", 16, 9.0, 0.4
    rng = np.random.default_rng(ctx)
    k, v, tables, g = _paged(dev, nkv, D, ps, [ctx, 70], rng)
    q_lens = [q_len, 1]
    T = q_len + 1
    q = rng.standard_normal((T, nq, D)).astype(np.float32)
    step = _step(dev, q_lens, [0, 1], [ctx, 70], g)
    pos, seq = step.positions.cpu().numpy(), step.seq_of_token.cpu().numpy()
    for t in range(q_len):
        j = 7 + 31 * t
        k[tables[0, j // ps], 0, j % ps] = q[t, 0] * (16.0 / np.sqrt(D))
    gates = rng.standard_normal((T, nq)).astype(np.float32)
    qd, kd, vd = (torch.from_numpy(a).to(dev).bfloat16().contiguous() for a in (q.reshape(T, nq * D), k, v))
    got = ops.paged_attention(qd, kd, vd, step, 0, nq, nkv, D, scale, None, softcap=cap,
                              gate=(torch.from_numpy(gates).to(dev), 0)).float().cpu().numpy().reshape(T, nq, D)
    qf, kf, vf = (a.float().cpu().numpy().astype(np.float64) for a in (qd, kd, vd))
    qf = qf.reshape(T, nq, D)
    for t in range(T):
        js = np.arange(pos[t] + 1)
        kk, vv = kf[tables[seq[t], js // ps], :, js % ps], vf[tables[seq[t], js // ps], :, js % ps]
        for h in range(nq):
            s = plain.cap(kk[:, h // (nq // nkv)] @ qf[t, h] * scale, cap)
            e = np.exp(s - s.max())
            np.testing.assert_allclose(got[t, h], (e / e.sum()) @ vv[:, h // (nq // nkv)] * plain.sigmoid(gates[t, h]), rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("H,G,dk,dv,rot,H2,ps,dtype", [
    (6, 2, 24, 40, 8, 4, 4, "float32"), (3, 3, 10, 7, 6, 3, 8, "float32"), (8, 2, 64, 48, 32, 2, 16, "bfloat16"), (4, 1, 96, 128, 96, 16, 16, "bfloat16"),
    (2, 2, 16, 16, 0, 6, 16, "bfloat16"), (1, 1, 33, 12, 32, 1, 16, "float32"), (4, 4, 32, 16, 2, 8, 16, "bfloat16"), (4, 2, 144, 100, 16, 2, 16, "bfloat16")])
def test_attention_and_a_second_layer_on_the_same_keys_and_values(dev, H, G, dk, dv, rot, H2, ps, dtype):
    """The whole mixer through its part: heads rotated over part of their channels and normed without a gain, the cache holding
    them so, capped scores, a gate per head, value sizes unlike key sizes; then a second mixer without keys and values that
    reads what the first one cached, with heads, scale and cap of its own.  Two requests in portions down to one token on
    scattered pages.  eps is large beside some heads' channels, so that it counts."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, GroupView, LayerCache
    if dev == "cpu" and dtype != "float32":
        pytest.skip("the stand-ins are float32")
    rng = np.random.default_rng(dk + H)
    W, eps, base = 72, 0.05, 300.0
    td = torch.float32 if dtype == "float32" else torch.bfloat16

    def weights(H, own):
        w = {"m.q": rng.standard_normal((H * dk, W)) * 0.1, "m.g": rng.standard_normal((H, W)) * 0.3, "m.o": rng.standard_normal((W, H * dv)) * 0.2}
        if own:
            w.update({"m.k": rng.standard_normal((G * dk, W)) * 0.1, "m.v": rng.standard_normal((G * dv, W)) * 0.3})
        return _bf16_exact(w)

    def build(H, scale, cap, w, shared):
        m = MIXERS.build(PartSpec("normed_attention", {
            "hidden_size": W, "heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "eps": eps, "softcap": cap, "head_gain": False,
            "head_gate": True, "shared_kv": shared, "max_positions": 512,
            "rotary": {"theta": base, "rotary_dim": rot, "max_positions": 512} if rot else None}), dtype=td, device=dev)
        m.bind(lambda rel: torch.from_numpy(w["m." + rel].astype(np.float32)))
        return m
    w1, w2 = weights(H, True), weights(H2, False)
    first, second = build(H, 0.5, 6.0, w1, False), build(H2, 0.2, 2.0, w2, True)
    assert first.cache_need() == second.cache_need() and first.cache_need().head_dim >= max(dk, dv)
    lens = {0: 110, 1: 37}
    xs = {s: _bf16_exact({"x": rng.standard_normal((n, W))})["x"] for s, n in lens.items()}
    m1 = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 0.5, "softcap": 6.0, "rot": {"base": base, "dims": rot} if rot else None}
    m2 = dict(m1, heads=H2, scale=0.2, softcap=2.0)
    want = {}
    for s, x in xs.items():
        kv = plain.keys_values(x, w1, "m.", m1, eps)
        want[s] = np.concatenate([plain.attention(x, w1, "m.", m1, eps, kv), plain.attention(x, w2, "m.", m2, eps, kv)], axis=1)
    D = first.cache_need().head_dim
    _, _, tables, _ = _paged(dev, G, D, ps, list(lens.values()), rng)
    kc, vc = (torch.full((int(tables.max()) + 1, G, ps, D), 3.0, dtype=td, device=dev) for _ in range(2))
    cache = LayerCache(group=0, k=kc, v=vc)
    to = _to(dev)
    row = {s: i for i, s in enumerate(lens)}

    def run(rows, step):
        slot_map = np.concatenate([[tables[row[s], p // ps] * ps + p % ps for p in range(a, b)] for s, a, b in rows]).astype(np.int32)
        step.groups = [GroupView(ps, torch.from_numpy(tables[[row[s] for s, _, _ in rows]]).to(dev), torch.from_numpy(slot_map).to(dev))]
        x = to(np.concatenate([xs[s][a:b] for s, a, b in rows])).to(td)
        return np.concatenate([_term(first.forward(x, step, cache, None)), _term(second.forward(x, step, cache, None, write_cache=False))], axis=1)
    got = _portions(dev, lens, {0: 0, 1: 1}, CUTS, run)
    for s in lens:
        for part in (slice(0, W), slice(W, 2 * W)):
            if dtype == "float32":
                np.testing.assert_allclose(got[s][:, part], want[s][:, part], rtol=5e-4, atol=5e-4)
            else:
                e = _relative(got[s][:, part], want[s][:, part])
                assert e.max() < 0.05 and np.quantile(e, 0.9) < 0.02, (s, float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("heads,dk,dv,rot", [(1, 64, 64, 64), (3, 16, 24, 12), (5, 6, 10, 2), (2, 130, 12, 66), (80, 16, 16, 16), (4, 32, 16, 0), (2, 128, 128, 128),
                                             (1, 256, 80, 40), (3, 96, 160, 96), (4, 48, 70, 32)])
def test_retention_in_portions_and_slots(dev, heads, dk, dv, rot):
    """S <- decay_h S + k v^T on rotated queries and keys, through the part with its norm per head, gate and projection.  The last
    head all but never forgets (0.9999) and the first forgets within a few tokens; portions start at every kind of position,
    one state row was used before, one stays untouched."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, LayerCache
    rng = np.random.default_rng(dk + heads)
    W, eps = 40, 1e-3
    K, V = heads * dk, heads * dv
    decay = [float(np.float32(1.0 - 0.8 * (1e-4 / 0.8) ** (i / max(heads - 1, 1)))) for i in range(heads)] if heads > 1 else [0.97]
    w = _bf16_exact({"m.q": rng.standard_normal((K, W)) * 0.3, "m.k": rng.standard_normal((K, W)) * 0.3, "m.v": rng.standard_normal((V, W)) * 0.3,
                     "m.g": rng.standard_normal((V, W)) * 0.3, "m.o": rng.standard_normal((W, V)) * 0.2})
    mixer = MIXERS.build(PartSpec("retention", {"hidden_size": W, "heads": heads, "dim": dk, "vdim": dv, "decay": decay, "eps": eps,
                                                "rotary": {"theta": 90.0, "rotary_dim": rot, "max_positions": 256} if rot else None}),
                         dtype=torch.float32, device=dev)
    mixer.bind(lambda rel: torch.from_numpy(w["m." + rel].astype(np.float32)))
    lens, slots = {0: 110, 1: 21}, {0: 1, 1: 2}
    xs = {s: rng.standard_normal((n, W)) for s, n in lens.items()}
    m = {"heads": heads, "dim": dk, "vdim": dv, "decay": [float(np.float32(d)) for d in decay], "rot": {"base": 90.0, "dims": rot} if rot else None}
    want = {s: plain.retention(x, w, "m.", m, eps) for s, x in xs.items()}
    cache = LayerCache(states={"retention": torch.zeros((3, heads, dk, dv), dtype=torch.float32, device=dev)})
    to = _to(dev)
    run = lambda rows, step: _term(mixer.forward(to(np.concatenate([xs[s][a:b] for s, a, b in rows])), step, cache, None))
    got = _portions(dev, lens, slots, CUTS, run)
    for s in lens:
        np.testing.assert_allclose(got[s], want[s], rtol=5e-4, atol=5e-4)
    assert float(cache.states["retention"][0].abs().max()) == 0.0


@pytest.mark.parametrize("heads,dk,dv,rot", [(2, 64, 64, 64), (3, 48, 30, 16), (1, 128, 128, 128), (5, 16, 100, 8), (2, 100, 64, 50), (2, 33, 7, 0), (1, 200, 24, 40)])
def test_retention_over_long_portions_beside_short_ones(dev, heads, dk, dv, rot):
    """Long portions run in chunks on the GPU, short ones and single tokens token by token: portions that end beside a chunk's
    border (64, 65, 127 to 129 tokens, 192, 200) and on either side of where chunks begin to be used (95 to 97), alone and beside others in one step, each going on from its state row,
    against the whole sequences token by token.  One head all but never forgets, one forgets at once."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import MIXERS, LayerCache
    rng = np.random.default_rng(dk + dv)
    W, eps = 40, 1e-3
    K, V = heads * dk, heads * dv
    decay = [0.9998, 0.0, 0.5, 0.97, 1.0][:heads] if heads > 1 else [0.995]
    w = _bf16_exact({"m.q": rng.standard_normal((K, W)) * 0.3, "m.k": rng.standard_normal((K, W)) * 0.3, "m.v": rng.standard_normal((V, W)) * 0.3,
                     "m.g": rng.standard_normal((V, W)) * 0.3, "m.o": rng.standard_normal((W, V)) * 0.2})
    mixer = MIXERS.build(PartSpec("retention", {"hidden_size": W, "heads": heads, "dim": dk, "vdim": dv, "decay": decay, "eps": eps,
                                                "rotary": {"theta": 700.0, "rotary_dim": rot, "max_positions": 1024} if rot else None}),
                         dtype=torch.float32, device=dev)
    mixer.bind(lambda rel: torch.from_numpy(w["m." + rel].astype(np.float32)))
    cuts = [(200, 1, 64), (1, 129, 95), (97, 1, 96), (1, 2, 65), (127, 128, 1), (95, 192, 1)]
    lens, slots = {s: sum(c[s] for c in cuts) for s in range(3)}, {0: 2, 1: 0, 2: 3}
    xs = {s: rng.standard_normal((n, W)) for s, n in lens.items()}
    m = {"heads": heads, "dim": dk, "vdim": dv, "decay": [float(np.float32(d)) for d in decay], "rot": {"base": 700.0, "dims": rot} if rot else None}
    cache = LayerCache(states={"retention": torch.zeros((4, heads, dk, dv), dtype=torch.float32, device=dev)})
    to = _to(dev)
    run = lambda rows, step: _term(mixer.forward(to(np.concatenate([xs[s][a:b] for s, a, b in rows])), step, cache, None))
    got = _portions(dev, lens, slots, cuts, run)
    for s in lens:
        np.testing.assert_allclose(got[s], plain.retention(xs[s], w, "m.", m, eps), rtol=5e-4, atol=5e-4)
    assert float(cache.states["retention"][1].abs().max()) == 0.0


@pytest.mark.parametrize("W,ff,T", [(36, 20, 41), (64, 72, 9), (40, 17, 30), (128, 256, 70)])
def test_two_matrices_with_a_squared_relu(dev, W, ff, T):
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import FEED_FORWARDS
    rng = np.random.default_rng(ff)
    w = _bf16_exact({"up": rng.standard_normal((ff, W)) * 0.3, "down": rng.standard_normal((W, ff)) * 0.3})
    h = rng.standard_normal((T, W))
    part = FEED_FORWARDS.build(PartSpec("plain_dense", {"hidden_size": W, "intermediate_size": ff}), dtype=torch.float32, device=dev)
    part.bind(lambda rel: torch.from_numpy(w[rel].astype(np.float32)))
    want = plain.feed_forward(h, w, "")
    np.testing.assert_allclose(_term(part.forward(_to(dev)(h), None)), want, rtol=3e-4, atol=3e-4)
    assert np.abs(want - np.maximum(h @ w["up"].T, 0) @ w["down"].T).max() > 0.1


@pytest.mark.parametrize("W,dim,layer,layers", [(36, 8, 0, 3), (64, 5, 2, 3), (40, 32, 1, 2), (48, 1, 3, 4)])
def test_the_tokens_own_vector(dev, W, dim, layer, layers):
    """The layer's columns of the table at the tokens' ids (the first and the last row among them), through gate, gelu,
    product and projection; the norm is the block's."""
    from sllm_b200.config.plan import PartSpec
    from sllm_b200.parts import FEED_FORWARDS
    rng = np.random.default_rng(W + dim)
    V, ids = 19, [0, 18, 3, 3, 7, 0, 11]
    w = _bf16_exact({f"l{layer}.side.gate": rng.standard_normal((dim, W)) * 0.4, f"l{layer}.side.proj": rng.standard_normal((W, dim)) * 0.4,
                     f"l{layer}.side.norm": 1 + 0.3 * rng.standard_normal(W), "side.embed": rng.standard_normal((V, dim * layers))})
    h = rng.standard_normal((len(ids), W))
    part = FEED_FORWARDS.build(PartSpec("token_side", {"hidden_size": W, "dim": dim, "offset": layer * dim}), dtype=torch.float32, device=dev)
    part.bind(lambda rel: torch.from_numpy(w[f"l{layer}.side.{rel}"].astype(np.float32)))
    part.adopt_token_table(_to(dev)(w["side.embed"]))
    step = _step(dev, [len(ids)], [0])
    step.token_ids = torch.tensor(ids, dtype=torch.int32, device=dev)
    got = plain.norm(_term(part.forward(_to(dev)(h), step)), w[f"l{layer}.side.norm"], 1e-5)
    np.testing.assert_allclose(got, plain.token_side(h, ids, w, layer, dim, 1e-5), rtol=3e-4, atol=3e-4)
    with pytest.raises(ValueError):
        part.adopt_token_table(_to(dev)(w["side.embed"][:, :layer * dim]))


@pytest.mark.gpu
@pytest.mark.parametrize("M", [1, 8, 12, 30, 40, 64, 100, 128, 200, 300])
@pytest.mark.parametrize("N,K", [(384, 256), (24, 328), (8448, 2048), (9000, 512), (30, 64), (33, 44)])
def test_activations_that_leave_with_the_products_tile(M, N, K):
    """Squared relu and the tokens' table behind every form of the bfloat16 product (warp-split, streaming, tensor memory, CTA
    pairs, and the activation kernel behind a plain product where no form has it) against float32 arithmetic on the same
    operands."""
    import sllm_b200.ops as ops
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    gen = torch.Generator(device="cuda:0")
    gen.manual_seed(M * 7 + N)
    x = torch.randn(M, K, device="cuda:0", generator=gen).bfloat16()
    w = (torch.randn(N, K, device="cuda:0", generator=gen) * K ** -0.5).bfloat16()
    z = x.double() @ w.double().t()
    got = ops.linear_plain_act(x, w, torch.bfloat16, "relu2").double()
    want = torch.relu(z).square()
    assert float(((got - want).abs() - 2 ** -7 * want).max()) < 1e-3 and float((got - want).norm() / want.norm()) < 4e-3
    V, off = 13, 5
    table = torch.randn(V, off + N + 2, device="cuda:0", generator=gen).bfloat16()
    ids = torch.randint(0, V, (M,), device="cuda:0", generator=gen).int()
    got = ops.linear_plain_act(x, w, torch.bfloat16, "token", ops.TokenColumns(table, ids, off)).double()
    want = torch.nn.functional.gelu(z, approximate="tanh") * table[ids.long(), off:off + N].double()
    assert float(((got - want).abs() - 2 ** -7 * want.abs()).max()) < 1e-3 and float((got - want).norm() / want.norm()) < 4e-3
    ops.check_tcgen05_status()


# ---- the whole model through the engine: every cutting against the plain implementation ---------------------------

@pytest.mark.parametrize("which", ["A", "odd"])
def test_residual_stream_after_every_layer(tmp_path, dev, which):
    """The stream after each layer (float32), taken where the engine's own blocks leave it."""
    from sllm_b200.engine import Engine, StepEntry, build_model
    config = CONFIGS[which][0]
    d = make_model(tmp_path, config)
    cfg, w = plain.load_model(d)
    ids = _requests(config["vocab"], (19,))["r0"]
    streams = []
    want = plain.forward(ids, cfg, w, streams)
    model, _ = build_model(d, "float32", dev)
    seen = []
    for layer in model.layers:
        inner = layer.block.forward

        def forward(residual, *a, _inner=inner, **kw):
            out = _inner(residual, *a, **kw)
            seen.append(residual.cpu().numpy().copy())
            return out
        layer.block.forward = forward
    eng = Engine(model, page_size=8, num_pages=8, max_requests=1)
    got = eng.step([StepEntry("a", ids, list(range(len(ids))))]).cpu().numpy()
    np.testing.assert_allclose(got, want, rtol=3e-4, atol=3e-4)
    assert len(seen) == len(streams) == len(config["layers"])
    for i, (a, b) in enumerate(zip(seen, streams)):
        np.testing.assert_allclose(a, b, rtol=2e-4, atol=2e-4, err_msg=f"after layer {i}")


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_every_cutting_against_plain(tmp_path, dev, which):
    """Whole prompts; most of a prompt and the rest token by token; portions of changing size down to two tokens; up to
    four requests at a time, portions beside single tokens.  The pools hold the trace's peak only and freed pages are
    poisoned, so pages and state slots are used again and a read of a page no longer held would show."""
    from sllm_b200.engine import Engine, build_model
    config, page = CONFIGS[which]
    reqs = _requests(config["vocab"], (70, 37, 100, 1, 45, 64, 23))
    for dtype, d, want in models_for(tmp_path, config, dev, reqs):
        model, _ = build_model(d, dtype, dev)
        for mode in ("whole", "tail_decode", "portions", "mixed"):
            tr = getattr(traces, mode)(reqs)
            eng = Engine(model, page_size=page, num_pages=max(tr.max_tokens // page, 1), max_requests=4, poison_freed=True)
            out = traces.replay_engine(tr, eng)
            compare(tr, out, want, dtype, f"{which}/{dtype}/{mode}")
            eng.cache.check()
            assert not eng.cache.requests and all(g.pool.used_count == 0 for g in eng.cache.groups)
            if mode == "mixed" and eng.cache.groups:
                assert eng.cache.reuse_count > 0


def test_batch_of_unequal_requests_equals_each_alone(tmp_path, dev):
    from sllm_b200.engine import Engine, StepEntry, build_model
    d = make_model(tmp_path, CONFIG_A)
    reqs = _requests(CONFIG_A["vocab"], (33, 2, 19, 50), seed=8)
    model, _ = build_model(d, "float32", dev)
    alone = {}
    for r, ids in reqs.items():
        eng = Engine(model, page_size=16, num_pages=8, max_requests=2)
        a = eng.step([StepEntry(r, ids[:-1], [len(ids) - 2])])
        b = eng.step([StepEntry(r, ids[-1:], [0])])
        alone[r] = torch.cat([a, b]).cpu().numpy()
    eng = Engine(model, page_size=16, num_pages=16, max_requests=5)
    eng.step([StepEntry("warm", [1, 2, 3], [])])            # takes slot 0 and the first page, then leaves
    eng.finish("warm")
    order = ["r3", "r1", "r0", "r2"]
    a = eng.step([StepEntry(r, reqs[r][:-1], [len(reqs[r]) - 2]) for r in order]).cpu().numpy()
    b = eng.step([StepEntry(r, reqs[r][-1:], [0]) for r in order]).cpu().numpy()
    for i, r in enumerate(order):
        np.testing.assert_allclose(np.stack([a[i], b[i]]), alone[r], rtol=2e-5, atol=2e-5)


def test_a_slot_that_is_used_again_starts_from_nothing(tmp_path, dev):
    """Four state slots, nine requests one after another and side by side: a request that gets a slot and pages another
    one left behind must not see that one's states, keys or values."""
    from sllm_b200.engine import Engine, StepEntry, build_model
    d = make_model(tmp_path, ODD)
    reqs = _requests(ODD["vocab"], (12, 30, 7, 18, 3, 25, 9, 14, 2), seed=17)
    want = plain_logits(d, reqs)
    model, _ = build_model(d, "float32", dev)
    eng = Engine(model, page_size=8, num_pages=16, max_requests=4, poison_freed=True)
    names = list(reqs)
    for a in range(0, len(names), 3):
        group = names[a:a + 3]
        first = eng.step([StepEntry(r, reqs[r][:-1], [len(reqs[r]) - 2]) for r in group]).cpu().numpy()
        last = eng.step([StepEntry(r, reqs[r][-1:], [0]) for r in group]).cpu().numpy()
        for i, r in enumerate(group):
            np.testing.assert_allclose(first[i], want[r][-2], rtol=3e-4, atol=3e-4)
            np.testing.assert_allclose(last[i], want[r][-1], rtol=3e-4, atol=3e-4)
            eng.finish(r)
    assert eng.cache.reuse_count > 0


LONG_MEMORY = _config(150, 128, [                     # both mixers can hold on to the sequence's first tokens
    _layer(_att(4, 2, 32, 32, 0.6, 15.0, (10000.0, 8)), 96),
    _layer(_ret([0.95, 0.99995], 64, 32, (10000.0, 32)), None),
    _layer(_att(2, 2, 32, 32, 0.5, 18.0, (10000.0, 8), kv_from=0), 64),
    _layer(_att(4, 1, 64, 64, 0.3, 12.0, (10000.0, 16)), None),
], side=16, scale=6.0, cap=10.0)


def _sharp(t):
    """Outputs of the mixers that weigh more than the other terms (attention with scores of up to +-15 all but picks one key): a lost
    key or a dropped state changes the logits by far more than the tolerance."""
    for n in list(t):
        if n.endswith("norm1"):
            t[n] *= 2.0
        if n.endswith(("norm2", "side.norm")):
            t[n] *= 0.5


def test_keys_far_back_at_page_borders_and_a_long_memory(tmp_path, dev):
    """Sharpened weights (`_sharp`): a prompt of several hundred tokens, cut at and beside page borders, then decoded
    token by token across more of them; every position wanted."""
    from sllm_b200.engine import Engine, build_model
    config, page = LONG_MEMORY, 16
    reqs = _requests(config["vocab"], (260,), seed=12)
    ids = reqs["r0"]
    for dtype, d, want in models_for(tmp_path, config, dev, reqs, seed=11, edit=_sharp):
        cfg, w = plain.load_model(d)
        cut = plain.forward(ids[150:], cfg, w)              # the memory matters: without the first 150 tokens the end differs
        assert np.abs(cut[-1] - want["r0"][-1]).max() > 0.05
        model, _ = build_model(d, dtype, dev)
        tr = traces.Trace()
        at = 0
        for n in (15, 1, 1, 16, 14, 1, 1, 2, 45, 1, 2, 3, 25):     # up to, onto and over page borders
            tr.step([("r0", at, ids[at:at + n], range(n))])
            at += n
        while at < len(ids):
            tr.step([("r0", at, ids[at:at + 1], [0])], end=["r0"] if at == len(ids) - 1 else [])
            at += 1
        eng = Engine(model, page_size=page, num_pages=tr.max_tokens // page, max_requests=1, poison_freed=True)
        compare(tr, traces.replay_engine(tr, eng), want, dtype, f"far/{dtype}")


def test_long_decoding_from_a_short_prompt(tmp_path, dev):
    """Three tokens of prompt, then 150 tokens one at a time: the states and the cache carry everything, across many
    pages; every step's logits against the plain implementation.  The first tokens of the sequence are wanted too (the
    empty states, a softmax over one key)."""
    from sllm_b200.engine import Engine, build_model
    reqs = _requests(CONFIG_A["vocab"], (153,), seed=42)
    for dtype, d, want in models_for(tmp_path, CONFIG_A, dev, reqs, seed=41):
        model, _ = build_model(d, dtype, dev)
        tr = traces.tail_decode(reqs, tail=150)
        eng = Engine(model, page_size=8, num_pages=tr.max_tokens // 8, max_requests=1)
        compare(tr, traces.replay_engine(tr, eng), want, dtype, f"long/{dtype}")
        tr = traces.Trace()
        tr.step([("r0", 0, reqs["r0"][:1], [0])])
        tr.step([("r0", 1, reqs["r0"][1:2], [0])])
        tr.step([("r0", 2, reqs["r0"][2:5], [0, 1, 2])], end=["r0"])
        eng = Engine(model, page_size=8, num_pages=8, max_requests=1)
        compare(tr, traces.replay_engine(tr, eng), want, dtype, f"first/{dtype}")


def test_greedy_generation_through_the_entry_point(tmp_path, dev):
    """`LLM.generate`: admission, the token budget, prompts in portions, decoding (from captured graphs on the GPU),
    sampling on the device; against greedy decoding with the plain implementation."""
    from sllm_b200.engine import build_model
    from sllm_b200.engine.llm import LLM
    from sllm_b200.sampling import SamplingParams
    d = make_model(tmp_path, CONFIG_A, seed=21)
    cfg, w = plain.load_model(d)
    prompts = list(_requests(CONFIG_A["vocab"], (9, 40, 17, 3, 26), seed=22).values())
    new = 10
    model, _ = build_model(d, "float32", dev)
    llm = LLM(model=model, block_size=16, num_pages=40, max_num_seqs=3, chunk_size=16, max_batch_tokens=48, max_model_len=128)
    res = llm.generate(prompts, SamplingParams(max_new=new))
    for pr, r in zip(prompts, res):
        ids, out = list(pr), []
        for _ in range(new):
            logits = plain.forward(ids, cfg, w)[-1]
            top = np.sort(logits)[-2:]
            out.append(int(np.argmax(logits)))
            ids.append(out[-1])
            if top[1] - top[0] < 1e-3:      # a tie the rounding may break either way: compare up to here
                break
        assert r.ids[:len(out)] == out, (len(pr), r.ids, out)
    llm.engine.cache.check()
    assert not llm.engine.cache.requests


def test_command_line_with_random_weights(tmp_path, capsys, dev, monkeypatch):
    import sllm_b200.engine.llm as llm_mod
    from sllm_b200.serving import main as cli
    recipe = "tiny-sezopel"
    if dev == "cpu":
        import yaml
        real = llm_mod.LLM
        monkeypatch.setattr(llm_mod, "LLM", lambda model_dir, **kw: real(model_dir, **dict(kw, device="cpu")))
        with open(os.path.join(cli.RECIPES_DIR, "tiny-sezopel.yaml")) as f:
            raw = yaml.safe_load(f)
        raw["memory"] = {"kv_device_bytes": 1 << 20}
        recipe = os.path.join(str(tmp_path), "tiny-sezopel.yaml")
        with open(recipe, "w") as f:
            yaml.safe_dump(raw, f)
    assert cli.main([recipe]) == 0
    out = capsys.readouterr().out
    assert "Sezopel: 4 layers" in out
    assert cli.main([recipe, "--mode", "run", "--random-weights", "4", "--prompt-ids", "5,17,3,150,42", "--max-new", "5",
                     "--dtype", "float32", "--log-level", "ERROR"]) == 0
    got = [int(t) for t in capsys.readouterr().out.strip().split(",")]
    assert len(got) == 5 and all(0 <= t < 260 for t in got)


@pytest.mark.gpu
def test_replay_program_on_a_model_folder(tmp_path):
    """bin/trace_run as a user runs it: the model class chosen by config.json, all four cuttings in one trace, four state slots."""
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    reqs = _requests(CONFIG_B["vocab"], (40, 75, 9, 120, 51), seed=32)
    tr = traces.all_modes(reqs)
    for dtype, d, want in models_for(tmp_path, CONFIG_B, "cuda:0", reqs, seed=31):
        want = traces.tagged(want)
        out = traces.replay_subprocess(tr, d, dtype, os.path.join(str(tmp_path), f"out_{dtype}"), 16)
        compare(tr, out, want, dtype, f"replay/{dtype}")
