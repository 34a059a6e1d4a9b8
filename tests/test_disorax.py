"""Disorax in the engine against the plain implementation (tests/plain_disorax.py): each mechanism's kernel alone, then
whole models through bin/trace_run (whole prompts, decoding, portions down to two tokens, mixed batches with pages and
slots used again) and greedy generation through the engine's entry point, on small configurations of its own."""
import json
import math

import numpy as np
import pytest
import torch

import plain_disorax as P
import replay_util as R
from conftest import random_tokens

gpu = pytest.mark.gpu
F64 = torch.float64


def configs():
    from vllm_cpp_b200.config.disorax import AttentionSpec as A, DisoraxConfig, DisoraxLayer as L, DisoraxMlp as F, LatentSpec as Lat
    moe = lambda *a: F("moe", *a)       # (an expert's size, experts, chosen, the shared expert's size)
    return {
        # a window of 9 that keeps five tokens over pages of 4, values narrower than keys, half of the lanes turning; two
        # layers that mix values and one between that does not; windows of 10 over latent rows; a layer without a feed-forward
        "A": (DisoraxConfig(vocab=150, width=48, norm_eps=1e-5, residual_mult=0.7, layers=(
            L("attention", A(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.35, rope_base=100.0, rope_dims=4, window=9, keep_first=5, v_mix=True),
              moe(16, 5, 2, 24)),
            L("latent_attention", Lat(heads=3, dim=5, vdim=7, kv_rank=9, scale=0.4), moe(8, 3, 1, 40)),
            L("attention", A(heads=2, kv_heads=1, dim=6, vdim=10, scale=0.4, rope_base=30.0, rope_dims=6, window=14, keep_first=2), moe(24, 4, 3, 8)),
            L("latent_attention_2", Lat(heads=2, dim=6, vdim=4, kv_rank=12, scale=0.5, window=10)),
            L("attention", A(heads=6, kv_heads=2, dim=8, vdim=6, scale=0.3, rope_base=500.0, rope_dims=8, window=6, keep_first=11, v_mix=True),
              moe(16, 6, 2, 16)))), 4),
        # sizes that bfloat16 runs on the tensor cores, padded to 64 and 128 lanes
        "B": (DisoraxConfig(vocab=260, width=64, norm_eps=1e-6, residual_mult=0.4, layers=(
            L("latent_attention_2", Lat(heads=3, dim=16, vdim=20, kv_rank=72, scale=0.25, window=33), moe(24, 4, 2, 32)),
            L("attention", A(heads=6, kv_heads=2, dim=48, vdim=64, scale=0.14, rope_base=10000.0, rope_dims=32, window=40, keep_first=19, v_mix=True),
              moe(40, 6, 3, 24)),
            L("attention", A(heads=2, kv_heads=2, dim=64, vdim=64, scale=0.11, rope_base=1e6, rope_dims=64, window=70, keep_first=3, v_mix=True),
              moe(32, 3, 1, 48)),
            L("latent_attention", Lat(heads=5, dim=24, vdim=40, kv_rank=48, scale=0.2), moe(16, 8, 4, 16)))), 16),
        # a width that is no multiple of 4, no factor on the results; one layer alone that says its values are mixed; all keys
        # seen, a window of one token, more kept tokens than the window; latent rows of three blocks; no shared expert; pages of 8
        "C": (DisoraxConfig(vocab=97, width=50, norm_eps=1e-4, residual_mult=1.0, layers=(
            L("attention", A(heads=5, kv_heads=1, dim=6, vdim=10, scale=1.0, rope_base=50.0, rope_dims=2, window=1, keep_first=7), moe(9, 7, 1)),
            L("latent_attention", Lat(heads=2, dim=7, vdim=3, kv_rank=290, scale=0.3), moe(11, 2, 2, 5)),
            L("attention", A(heads=3, kv_heads=3, dim=10, vdim=14, scale=0.3, rope_base=30.0, rope_dims=0, v_mix=True)),
            L("latent_attention_2", Lat(heads=1, dim=3, vdim=1, kv_rank=5, scale=0.6), moe(13, 5, 3, 7)))), 8),
        # heads of 128 lanes with values of 96; latent rows of two blocks, with and without a window; 20 heads over one row
        "D": (DisoraxConfig(vocab=210, width=96, norm_eps=1e-5, residual_mult=0.55, layers=(
            L("attention", A(heads=4, kv_heads=4, dim=128, vdim=96, scale=0.09, rope_base=1e5, rope_dims=96, window=56, keep_first=30, v_mix=True),
              moe(48, 3, 3, 64)),
            L("latent_attention", Lat(heads=20, dim=24, vdim=16, kv_rank=136, scale=0.15), moe(32, 6, 2, 40)),
            L("latent_attention_2", Lat(heads=4, dim=20, vdim=24, kv_rank=200, scale=0.15, window=70), moe(40, 4, 1, 24)),
            L("attention", A(heads=8, kv_heads=4, dim=80, vdim=96, scale=0.1, rope_base=2000.0, rope_dims=16, window=25, keep_first=64, v_mix=True)))), 16),
    }


LENGTHS = {"A": [40, 75, 150, 33, 2, 17, 64], "B": [1, 7, 33, 64, 170, 97, 3], "C": [50, 3, 77, 31, 9], "D": [120, 2, 230, 57, 33]}
REL_TOL = {"float32": 2e-5, "bfloat16": 3e-2}
HOT = 2                 # lanes of the stream that tell the routers where a token goes
MIN_MARGIN = 0.03       # no routing decision of the test models is closer than this share of the logits' spread


def decisive_routers(cfg, out, g):
    """Random routers have a close call every hundred tokens or so, which 16-bit activations settle differently from the
    64-bit oracle, and one token sent elsewhere moves every later row.  So two lanes of every token's embedding are a
    direction in the plane; no sublayer writes to them, the routers read nothing else, each expert a direction of its own,
    and a token's direction is drawn again until every router settles it by a wide margin however the norms scale it."""
    H, W = HOT, cfg.width
    routers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        out[p + "mix.o"][:H] = 0.0
        if layer.mlp is None:
            continue
        E = layer.mlp.experts
        angle = 2 * math.pi * (torch.arange(E, dtype=F64) + 0.3 * torch.rand(E, generator=g, dtype=F64)) / E
        out[p + "mlp.router"] = torch.zeros(E, W)
        out[p + "mlp.router"][:, :H] = torch.stack([angle.cos(), angle.sin()], 1).float()
        out[p + "mlp.router.b"] = (torch.rand(E, generator=g) - 0.5) * 0.8
        out[p + "norm2"][:H] = 1.0
        for e in [f"e{j}." for j in range(E)] + (["shared."] if layer.mlp.shared_ff else []):
            out[p + "mlp." + e + "down"][:H] = 0.0
        routers.append((out[p + "mlp.router"][:, :H].to(torch.bfloat16).double(), out[p + "mlp.router.b"].to(torch.bfloat16).double(), layer.mlp.top))
    # the direction's length: most of the row's, so that the norm leaves it between these two
    lo, hi = 0.45 * W ** 0.5, W ** 0.5
    for t in range(cfg.vocab):
        for _ in range(10000):
            a = 2 * math.pi * float(torch.rand(1, generator=g))
            d = torch.tensor([math.cos(a), math.sin(a)])
            if all(margin(s * (r @ d.double()) + b, top) > 2 * MIN_MARGIN for r, b, top in routers for s in (lo, 0.7 * hi, hi)):
                break
        else:
            raise AssertionError("no direction that every router settles")
        out["embed"][t, :H] = d * 8.0
        out["embed"][t, H:] *= 40.0
    out["final.norm"][:H] = 0.0


def margin(z, top):
    """How far the last chosen logit is above the first one left out, as a share of the logits' spread."""
    if top >= z.shape[-1]:
        return 1.0
    s = z.sort(-1, descending=True).values
    return float(((s[..., top - 1] - s[..., top]) / (s[..., 0] - s[..., -1])).min())


def hand_made(cfg, tensors, seed):
    """The random tensors, changed so that a fault shows: sharp softmaxes (single keys, often far ones or ones at the edge
    of a window, carry the rows), sinks of the size of the scores, gates that matter, values mixed in very different shares,
    routers that decide by a margin."""
    g = torch.Generator().manual_seed(seed)
    out = dict(tensors)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}.mix."
        if layer.type == "attention":
            for n in ("q", "k"):       # (heads of many lanes have larger scores by themselves)
                out[p + n] = tensors[p + n] * 12.0 * min(1.0, 48.0 / layer.mixer.dim) ** 0.5
            out[p + "v"] = tensors[p + "v"] * 5.0
            if layer.mixer.v_mix:
                out[p + "vmix"] = torch.tensor(0.35 + 0.17 * i)
        else:
            for n in ("q", "dkv"):
                out[p + n] = tensors[p + n] * 12.0
            out[p + "uk"] = tensors[p + "uk"] * 10.0
            out[p + "uv"] = tensors[p + "uv"] * 5.0
            if layer.type == "latent_attention_2":
                out[p + "sink"] = torch.linspace(-1.0, 3.0, layer.mixer.heads)
        out[p + "g"] = tensors[p + "g"] * 10.0
        out[p + "o"] = tensors[p + "o"] * 6.0
        if layer.mlp is not None:
            for n in [f"e{j}." for j in range(layer.mlp.experts)] + (["shared."] if layer.mlp.shared_ff else []):
                for m, f in (("gate", 6.0), ("up", 6.0), ("down", 6.0)):
                    out[f"l{i}.mlp.{n}{m}"] = tensors[f"l{i}.mlp.{n}{m}"] * f
            if layer.mlp.shared_ff:
                out[f"l{i}.mlp.shared.sg"] = tensors[f"l{i}.mlp.shared.sg"] * 10.0
    decisive_routers(cfg, out, g)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def write_models(tmp_path_factory):
    from vllm_cpp_b200 import write_random_model
    from vllm_cpp_b200.weights.safetensors_io import read_safetensors, write_safetensors
    out = {}
    for i, (name, (cfg, _)) in enumerate(configs().items()):
        d = tmp_path_factory.mktemp(f"disorax_{name}")
        write_random_model(cfg, 71 + i, d, dtype="bfloat16")
        tensors = {k: v.float() for k, v in read_safetensors(d / "model.safetensors").items()}
        write_safetensors(d / "model.safetensors", hand_made(cfg, tensors, 25 + i), {"format": "pt"})
        out[name] = d
    return out


@pytest.fixture(scope="module")
def disorax_dirs(tmp_path_factory):
    return write_models(tmp_path_factory)


class Oracle:
    def __init__(self, dirs):
        self.models = {n: P.read_model(d) for n, d in dirs.items()}
        self.cache = {}

    def __call__(self, name, tokens):
        key = (name, tuple(tokens))
        if key not in self.cache:
            self.cache[key] = P.forward(*self.models[name], list(tokens)).numpy()
        return self.cache[key]


@pytest.fixture(scope="module")
def oracle(disorax_dirs):
    return Oracle(disorax_dirs)


def requests_of(name):
    vocab = configs()[name][0].vocab
    return {f"r{i}": random_tokens(vocab, n, 11 * i + ord(name)) for i, n in enumerate(LENGTHS[name])}


# -------------------------------------------------------------------------- without a GPU


def small_config():
    moe = {"kind": "moe", "expert": {"ff": 7}, "router": {"experts": 9, "top": 4}, "shared": {"ff": 13}}
    return {"architecture": "Disorax", "vocab": 31, "width": 24, "norm": {"eps": 3e-5}, "residual_mult": 0.25, "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.5, "v_mix": True,
                                        "mask": {"size": 7, "keep_first": 3}, "rot": {"base": 777.0, "dims": 6}}, "mlp": moe},
        {"type": "latent_attention", "mixer": {"heads": 3, "dim": 4, "vdim": 5, "kv_rank": 11, "scale": 0.9},
         "mlp": dict(moe, shared=None)},
        {"type": "latent_attention_2", "mixer": {"heads": 2, "dim": 3, "vdim": 8, "kv_rank": 6, "scale": 0.8, "mask": {"size": 17}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 1, "dim": 2, "vdim": 2, "scale": 1.5, "rot": {"base": 5.0, "dims": 0}}}]}


def test_config_reads_every_size_and_constant():
    from vllm_cpp_b200.config import ConfigError, DisoraxConfig
    c = small_config()
    cfg = DisoraxConfig.from_dict(c)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.residual_mult, len(cfg.layers)) == (31, 24, 3e-5, 0.25, 4)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.window, m.keep_first, m.rope_base, m.rope_dims, m.v_mix) == (
        6, 2, 10, 14, 0.5, 7, 3, 777.0, 6, True)
    f = cfg.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.shared_ff, cfg.layers[1].mlp.shared_ff, cfg.layers[2].mlp, cfg.layers[3].mlp) == (7, 9, 4, 13, 0, None, None)
    m = cfg.layers[2].mixer
    assert (m.heads, m.dim, m.vdim, m.kv_rank, m.scale, m.window, cfg.layers[1].mixer.window) == (2, 3, 8, 6, 0.8, 17, 0)
    m = cfg.layers[3].mixer
    assert (m.kv_heads, m.window, m.keep_first, m.v_mix) == (1, 0, 0, False)        # what is left out
    assert DisoraxConfig.from_dict(cfg.to_dict()) == cfg
    layer = c["layers"]
    change = lambda i, key, **kw: {"layers": [dict(l, **{key: dict(l[key], **kw)}) if j == i else l for j, l in enumerate(layer)]}
    for bad in ({"layers": []}, {"vocab": None}, {"norm": {"eps": 0}}, {"layers": [dict(layer[0], type="mamba")]},
                change(0, "mixer", kv_heads=4), change(0, "mixer", rot={"base": 10.0, "dims": 3}), change(0, "mixer", rot={"base": 10.0, "dims": 12}),
                change(0, "mixer", mask={"size": 0}), change(0, "mixer", v_mix=1), change(1, "mixer", kv_rank=None),
                change(2, "mixer", mask={"size": 4, "keep_first": 1}), change(0, "mlp", router={"experts": 2, "top": 3}),
                change(0, "mlp", kind="dense"), change(3, "mixer", v_mix=True)):      # (mixed values of two sizes)
        with pytest.raises(ConfigError):
            DisoraxConfig.from_dict(dict(c, **bad))


def test_model_folder_is_recognised_and_names_its_tensors(tmp_path):
    from vllm_cpp_b200.config import DisoraxConfig
    from vllm_cpp_b200.models import expected_tensors, load_config
    c = small_config()
    (tmp_path / "config.json").write_text(json.dumps(c))
    assert load_config(tmp_path) == DisoraxConfig.from_dict(c)
    s = {t.name: tuple(t.shape) for t in expected_tensors(DisoraxConfig.from_dict(c))}
    want = {"embed": (31, 24), "head": (31, 24), "final.norm": (24,), "l0.norm1": (24,), "l0.norm2": (24,), "l0.mix.q": (60, 24),
            "l0.mix.k": (20, 24), "l0.mix.v": (28, 24), "l0.mix.g": (84, 24), "l0.mix.o": (24, 84), "l0.mix.vmix": (),
            "l0.mlp.router": (9, 24), "l0.mlp.router.b": (9,), "l0.mlp.e8.gate": (7, 24), "l0.mlp.e8.up": (7, 24), "l0.mlp.e8.down": (24, 7),
            "l0.mlp.shared.gate": (13, 24), "l0.mlp.shared.up": (13, 24), "l0.mlp.shared.down": (24, 13), "l0.mlp.shared.sg": (1, 24),
            "l1.mix.q": (12, 24), "l1.mix.dkv": (11, 24), "l1.mix.dkv.norm": (11,), "l1.mix.uk": (12, 11), "l1.mix.uv": (15, 11),
            "l1.mix.g": (3, 24), "l1.mix.o": (24, 15), "l2.mix.sink": (2,), "l2.mix.g": (2, 24), "l3.mix.g": (2, 24)}
    assert {k: s.get(k) for k in want} == want
    # a layer without a feed-forward needs no second norm, and is not refused one
    assert {t.name: t.optional for t in expected_tensors(DisoraxConfig.from_dict(c)) if "norm2" in t.name} == {
        "l0.norm2": False, "l1.norm2": False, "l2.norm2": True, "l3.norm2": True}
    for absent in ("l1.mix.sink", "l1.mlp.shared.up", "l1.mlp.shared.sg", "l2.mlp.router", "l3.mix.vmix", "l0.mlp.e9.up"):
        assert absent not in s


def test_what_a_layer_keeps_per_request():
    import vllm_cpp_b200.models as models
    from vllm_cpp_b200.cache.device_cache import CacheLayout
    cfg = configs()["B"][0]
    for dtype, latent, latent2, dims in ((torch.float32, (1, 48), (1, 72), (48, 64)), (torch.bfloat16, (1, 64), (1, 128), (64, 0))):
        s = models.build_model(cfg, dtype, "cpu").cache_specs()
        assert (s[0].num_kv_heads, s[0].head_dim) == latent2 and (s[0].window, s[0].one_row) == (33, True)
        assert (s[3].num_kv_heads, s[3].head_dim) == latent and (s[3].window, s[3].one_row) == (0, True)
        assert (s[1].num_kv_heads, s[1].head_dim, s[1].v_head_dim, s[1].window, s[1].keep_first) == (2, *dims, 40, 19)
        # a latent row is kept once, and only what is kept is counted
        lay = CacheLayout({3: s[3]})
        assert lay.bytes_per_token(2) == 2 * latent[1]
    # a row wider than the kernels' tiles is kept in blocks
    s = models.build_model(configs()["C"][0], torch.bfloat16, "cpu").cache_specs()
    assert (s[1].num_kv_heads, s[1].head_dim) == (3, 128)
    assert models.build_model(configs()["C"][0], torch.float32, "cpu").cache_specs()[1].head_dim == 290


def test_oracle_mechanisms_by_hand():
    # a window that keeps first tokens
    assert P.window_mask(6, 2, 1).int().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0],
                                                     [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    assert int(P.window_mask(4, 0, 0).sum()) == 10 and torch.equal(P.window_mask(4, 2, 9), P.window_mask(4, 0))
    # a sink is a term of the denominator that no key has
    s = torch.tensor([[[0.0, 1.0], [2.0, 3.0]]], dtype=F64)
    w = P.masked_softmax(s, torch.tensor([[True, False], [True, True]]), torch.tensor([0.5], dtype=F64))
    e = math.exp
    torch.testing.assert_close(w, torch.tensor([[[1 / (1 + e(0.5)), 0.0], [e(2) / (e(2) + e(3) + e(0.5)), e(3) / (e(2) + e(3) + e(0.5))]]], dtype=F64))
    # rotation in halves, the lanes behind them left alone
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]], [[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    h = P.turn_halves(x, torch.tensor([0, 3]), 10.0, 4)
    a0, a1 = 3.0, 3.0 * 10.0 ** -0.5
    assert torch.equal(h[0], x[0])
    torch.testing.assert_close(h[1, 0], torch.tensor([math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1),
                                                      3 * math.cos(a0) + math.sin(a0), 4 * math.cos(a1) + 2 * math.sin(a1), 5.0], dtype=F64))
    # the softmax goes over the chosen logits only
    idx, weight = P.route(torch.tensor([[1.0, 5.0, 3.0, -2.0]], dtype=F64), 2)
    assert idx.tolist() == [[1, 2]]
    torch.testing.assert_close(weight, torch.tensor([[1 / (1 + e(-2)), 1 / (1 + e(2))]], dtype=F64))
    torch.testing.assert_close(P.mixed_values(torch.tensor(4.0), 0.25, torch.tensor(8.0)), torch.tensor(5.0))


def test_the_test_models_route_by_a_margin(disorax_dirs):
    """What makes the bfloat16 engine comparable row by row: every router settles every token of the tests' requests by a
    margin, tokens differ in whom they choose, and the biases have a say."""
    for name, d in disorax_dirs.items():
        cfg, w = P.read_model(d)
        worst, seen, swayed = 1.0, {}, 0
        real = P.feed_forward

        def watched(h, mw, mlp):
            nonlocal worst, swayed
            z = h @ mw["router"].T
            top = int(mlp["router"]["top"])
            worst = min(worst, margin(z + mw["router.b"], top))
            chosen = P.route(z + mw["router.b"], top)[0].sort(-1).values
            swayed += int((chosen != P.route(z, top)[0].sort(-1).values).any(-1).sum())
            seen.setdefault(id(mlp), set()).update(map(tuple, chosen.tolist()))
            return real(h, mw, mlp)
        P.feed_forward = watched
        try:
            for toks in requests_of(name).values():
                P.forward(cfg, w, toks)
        finally:
            P.feed_forward = real
        assert worst > MIN_MARGIN, (name, worst)
        assert max(len(s) for s in seen.values()) >= 3, (name, seen)


# -------------------------------------------------------------------------- on the GPU: each kernel alone


def dev():
    return torch.device("cuda:0")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=dev())


def f32(x):
    return None if x is None else x.float().contiguous().to(dev())


def freqs(base, dims):
    return f32(torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64))


def entries_of(lengths):
    starts = np.concatenate([[0], np.cumsum(lengths)])[:-1]
    return i32(starts.tolist()), i32(list(lengths))


def partial_sums(x, S, g):
    """x [T, C] (64-bit) as S 32-bit partial sums that add up to it (to 32-bit rounding)."""
    if S == 1:
        return x.float().to(dev())
    parts = torch.randn(S - 1, *x.shape, generator=g, dtype=F64)
    return torch.cat([parts, (x - parts.sum(0))[None]]).float().to(dev())


TOL32 = dict(atol=3e-5, rtol=3e-5)
TOL16 = dict(atol=3e-2, rtol=2e-2)


def tol_of(dtype):
    return TOL32 if dtype == torch.float32 else TOL16


@gpu
@pytest.mark.parametrize("W,n_terms,S,dtype", [(6, 2, 1, torch.float32), (50, 1, 2, torch.bfloat16), (320, 2, 3, torch.float32),
                                               (2500, 4, 1, torch.bfloat16), (64, 0, 1, torch.float32), (8192, 2, 2, torch.bfloat16)])
def test_results_enter_times_a_constant_and_two_norms_follow(W, n_terms, S, dtype):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(W + n_terms)
    T, eps, m = 7, 1e-5, 0.37
    x = torch.randn(T, W, generator=g, dtype=F64)
    terms = [torch.randn(T, W, generator=g, dtype=F64) for _ in range(n_terms)]
    first, vec, g1, g2 = torch.randn(T, W, generator=g, dtype=F64), *(torch.randn(W, generator=g, dtype=F64) for _ in range(3))
    want = x + m * sum(terms) + first + vec         # (what is added beside the results is not scaled)
    resid, out1, out2 = f32(x), *(torch.empty(T, W, dtype=dtype, device=dev()) for _ in range(2))
    ops.sum_add_rmsnorm(resid, [partial_sums(t, S, g) for t in terms], f32(g1), eps, out1, row_extra=f32(first), vec_extra=f32(vec), scale=m,
                        gain2=f32(g2), out2=out2)
    torch.testing.assert_close(resid.double().cpu(), want, **TOL32)
    torch.testing.assert_close(out1.double().cpu(), P.rms(want, eps) * g1, **tol_of(dtype))
    torch.testing.assert_close(out2.double().cpu(), P.rms(want, eps) * g2, **tol_of(dtype))
    # on a list of rows, one norm; the stream stays
    resid, out = f32(x), torch.empty(3, W, dtype=dtype, device=dev())
    ops.sum_add_rmsnorm(resid, [f32(t) for t in terms], f32(g1), eps, out, i32([5, 0, 5]), scale=m)
    torch.testing.assert_close(out.double().cpu(), (P.rms(x + m * sum(terms), eps) * g1)[[5, 0, 5]], **tol_of(dtype))
    assert torch.equal(resid.cpu(), x.float())
    ops.sum_add_rmsnorm(resid, [f32(t) for t in terms], None, 0.0, None, scale=m)
    torch.testing.assert_close(resid.double().cpu(), x + m * sum(terms), **TOL32)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd,rot,S", [(4, 2, 8, 6, 4, 1), (6, 2, 64, 64, 32, 2), (5, 1, 10, 14, 0, 3), (3, 3, 7, 5, 6, 1), (8, 4, 128, 96, 96, 2)])
def test_lane_gates_and_mixed_values(dtype, nh, nkv, hd, vd, rot, S):
    """The first layer of a kind leaves its values as projected; a later one mixes them into its own before they are
    cached; the gates' sigmoids lie lane by lane."""
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(nh * hd)
    T, n_pages, ps, base = 6, 4, 8, 50.0
    pos, slots = [0, 1, 700, 6, 31, 8], [2, -1, ps * 3 + 1, 0, ps + 3, 5]
    n = nh * hd + nkv * hd + nkv * vd
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    v_first = torch.randn(T, nkv * vd, generator=g, dtype=F64)
    for keep, share in ((True, None), (False, 0.3), (False, 1.0), (False, None)):
        u = torch.randn(T, n + nh * vd, generator=g, dtype=F64)
        pages = torch.full((n_pages, nkv * ps * (hd + vd)) if vd != hd else (n_pages, 2, nkv, ps, hd), float("nan"), dtype=dtype, device=dev())
        q_out = torch.empty(T, nh * hd, dtype=dtype, device=dev())
        gate = torch.full((T, nh * vd), float("nan"), device=dev())
        kept = torch.full((T, nkv * vd), float("nan"), device=dev()) if keep else None
        ops.qkv_rope_store(partial_sums(u, S, g), None, None, 1e-6, i32(pos), freqs(base, rot) if rot else None, None, i32(slots), q_out, pages,
                           nh, nkv, hd, vd, status, rot=rot, gate_out=gate, v_keep=kept, v_first=f32(v_first) if share is not None else None,
                           v_share=f32(torch.tensor([share])) if share is not None else None)
        assert int(status.item()) == 0
        q = P.turn_halves(u[:, :nh * hd].view(T, nh, hd), torch.tensor(pos), base, rot)
        k = P.turn_halves(u[:, nh * hd:(nh + nkv) * hd].view(T, nkv, hd), torch.tensor(pos), base, rot)
        v = u[:, (nh + nkv) * hd:n]
        tol = dict(atol=2e-4, rtol=2e-4) if dtype == torch.float32 else TOL16
        torch.testing.assert_close(q_out.double().cpu(), q.reshape(T, -1), **tol)
        torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(u[:, n:]), **TOL32)
        if keep:
            torch.testing.assert_close(kept.double().cpu(), v, **TOL32)
        if share is not None:
            v = P.mixed_values(v, share, v_first)
        flat = pages.view(n_pages, -1).double().cpu()
        keys, vals = flat[:, :nkv * ps * hd].view(n_pages, nkv, ps, hd), flat[:, nkv * ps * hd:].view(n_pages, nkv, ps, vd)
        for t, s in enumerate(slots):
            if s >= 0:
                torch.testing.assert_close(keys[s // ps, :, s % ps], k[t], **tol)
                torch.testing.assert_close(vals[s // ps, :, s % ps], v[t].view(nkv, vd), **tol)
        assert int((~torch.isnan(flat)).sum()) == 5 * nkv * (hd + vd)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kv_rank,rot,width,block,nh,S", [(9, 0, 9, 9, 3, 1), (48, 0, 64, 64, 5, 2), (290, 0, 384, 128, 2, 1), (200, 30, 256, 128, 4, 3),
                                                          (100, 16, 128, 128, 1, 1)])
def test_latent_rows_kept_once_padded_and_in_blocks(dtype, kv_rank, rot, width, block, nh, S):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(kv_rank)
    T, n_pages, ps, eps, base, d = 5, 4, 8, 1e-4, 21.0, 6
    pos, slots = [0, 1, 900, 6, 31], [2, -1, ps * 3 + 1, 0, ps + 3]
    q_cols = nh * (d + rot)
    u = torch.randn(T, q_cols + kv_rank + rot + nh, generator=g, dtype=F64)
    gain = 1 + 0.3 * torch.randn(kv_rank, generator=g, dtype=F64)
    pages = torch.full((n_pages, 1, width // block, ps, block), float("nan"), dtype=dtype, device=dev())
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    freq = freqs(base, rot) if rot else f32(torch.zeros(1))
    gate = torch.full((T, nh), float("nan"), device=dev())
    dev_u = partial_sums(u, S, g)
    ops.latent_norm_rope_store(dev_u[..., q_cols:], None, f32(gain), eps, i32(pos), freq, 1.0, i32(slots), None, pages, ps, 0, kv_rank, rot,
                               status, v_width=0, k_width=width, k_block=block, gate_out=gate)
    assert int(status.item()) == 0
    torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(u[:, q_cols + kv_rank + rot:]), **TOL32)
    c = P.rms(u[:, q_cols:q_cols + kv_rank], eps) * gain
    kr = P.turn_halves(u[:, None, q_cols + kv_rank:q_cols + kv_rank + rot], torch.tensor(pos), base, rot)[:, 0]
    row = torch.cat([c, kr, torch.zeros(T, width - kv_rank - rot, dtype=F64)], 1)
    tol = dict(atol=1e-3, rtol=1e-4) if dtype == torch.float32 else TOL16
    got = pages.double().cpu()
    for t, s in enumerate(slots):
        if s >= 0:
            torch.testing.assert_close(got[s // ps, 0, :, s % ps].reshape(-1), row[t], **tol)
    assert int((~torch.isnan(got)).sum()) == 4 * width
    if rot:     # the queries' turned part with the zeros behind it
        out = torch.full((T, nh * width), float("nan"), dtype=dtype, device=dev())
        ops.rope_rows(dev_u[..., :q_cols], i32(pos), freq, 1.0, out, heads=nh, dims=rot, width=rot, in_head_stride=d + rot, in_off=d,
                      out_head_stride=width, out_off=kv_rank, pad=width - kv_rank - rot)
        q = P.turn_halves(u[:, :q_cols].view(T, nh, d + rot)[..., d:], torch.tensor(pos), base, rot)
        got = out.double().cpu().view(T, nh, width)
        torch.testing.assert_close(got[..., kv_rank:kv_rank + rot], q, **tol)
        assert bool((got[..., kv_rank + rot:] == 0).all())


@gpu
@pytest.mark.parametrize("T,I,ld,S,dtype", [(3, 5, 13, 1, torch.float32), (70, 24, 64, 2, torch.bfloat16), (9, 12, 27, 3, torch.bfloat16), (300, 40, 80, 1, torch.bfloat16)])
def test_silu_gate_on_the_first_columns_of_a_product(T, I, ld, S, dtype):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(T)
    u = torch.randn(T, ld, generator=g, dtype=F64)
    out = torch.empty(T, I, dtype=dtype, device=dev())
    ops.swiglu(partial_sums(u, S, g)[..., :2 * I], out)
    torch.testing.assert_close(out.double().cpu(), P.silu(u[:, :2 * I:2]) * u[:, 1:2 * I:2], **tol_of(dtype))


# -------------------------------------------------------------------------- the experts


class _MoeCtx:
    def __init__(self, lengths):
        self.q_start, self.q_len = entries_of(lengths)
        self.E = len(lengths)
        self.status = torch.zeros(1, dtype=torch.int32, device=dev())


class _Store:
    """What a part asks of a weight store, for tensors at hand."""

    def __init__(self, tensors, dtype):
        self.t, self.dtype = tensors, dtype

    def matrix(self, name):
        return self.t[name].to(self.dtype).to(dev()).contiguous()

    def matrices(self, names, interleave=False):
        parts = [self.matrix(n) for n in names]
        return torch.stack(parts, 1).reshape(-1, parts[0].shape[1]).contiguous() if interleave else torch.cat(parts).contiguous()

    def vector(self, name):
        return self.t[name].float().to(dev())


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,E,top,ff,sff", [(1, 16, 4, 1, 8, 16), (37, 48, 5, 2, 24, 40), (150, 64, 3, 3, 16, 8), (64, 50, 7, 4, 9, 11), (9, 32, 70, 2, 72, 0),
                                              (700, 128, 6, 2, 136, 200), (2, 64, 9, 9, 200, 72)])
def test_experts_beside_a_gated_shared_one(dtype, T, H, E, top, ff, sff):
    """Biased choice, softmax over the chosen, gated experts (on the tensor cores the gate runs in the product's epilogue, at
    every tile size the step's length asks for), a gated shared expert behind a sigmoid of its own; rows of padding."""
    from vllm_cpp_b200.parts import BuildContext, RoutedExperts
    g = torch.Generator().manual_seed(T + E)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    w = {"router": rnd(E, H) * 2.0, "router.b": rnd(E) * 3.0, "shared.sg": rnd(1, H) * H ** -0.5}
    for e in [f"e{i}." for i in range(E)] + ["shared."]:
        n = sff if e == "shared." else ff
        w[e + "gate"], w[e + "up"], w[e + "down"] = rnd(n, H) * H ** -0.5, rnd(n, H) * H ** -0.5, rnd(H, n) * max(n, 1) ** -0.5
    w = {k: v.to(torch.bfloat16).double() for k, v in w.items()}
    # rows whose choice is not a close call
    x = rnd(8 * T + 80, H).to(torch.bfloat16).double()
    z = (x @ w["router"].T + w["router.b"]).sort(-1, descending=True).values
    x = x[torch.ones(len(x), dtype=torch.bool) if top == E else z[:, top - 1] - z[:, top] > 0.05][:T]
    assert len(x) == T
    mlp = {"router": {"top": top, "experts": E}, "shared": {"ff": sff} if sff else None}
    want = P.feed_forward(x, w, mlp)
    part = RoutedExperts({"hidden_size": H, "num_experts": E, "top": top, "expert_size": ff, "shared_size": sff, "activation": "silu", "gated": True,
                          "shared_gated": True, "shared_gate": True, "router_weights": "softmax", "router_bias": True, "weight_on": "output"},
                         "", BuildContext(dtype, dev()))
    names = {s.name for s in part.tensor_specs()}
    assert ("shared.sg" in names) == ("shared.gate" in names) == (sff > 0) and "router.b" in names
    part.bind(_Store({k: v for k, v in w.items() if k in names}, dtype))
    ctx = _MoeCtx([T // 2, 0, T - T // 2])
    rows = torch.cat([x, torch.full((2, H), 9.0, dtype=F64)]).to(dtype).to(dev())      # the last two rows belong to no entry
    got = part.forward(rows, ctx)
    assert int(ctx.status.item()) == 0
    torch.testing.assert_close(got.double().cpu()[:T], want, **(dict(atol=1e-4, rtol=1e-4) if dtype == torch.float32 else dict(atol=5e-2, rtol=3e-2)))


@gpu
@pytest.mark.parametrize("tile_rows", [16, 32, 64, 128, 256])
@pytest.mark.parametrize("E,I,K,tiles", [(5, 12, 48, 7), (3, 64, 64, 4), (4, 100, 128, 5), (2, 200, 72, 3)])
def test_silu_gate_in_the_grouped_products_epilogue(tile_rows, E, I, K, tiles):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(E * I)
    w = (torch.randn(E, 2 * I, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    x = torch.randn(tiles * tile_rows, K, generator=g).to(torch.bfloat16)
    expert = sorted(int(e) for e in torch.randint(0, E, (tiles - 1,), generator=g)) + [-1]
    out = torch.full((tiles * tile_rows, I), 7.0, dtype=torch.bfloat16, device=dev())
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    ops.gemm_bf16_grouped(w.to(dev()), x.to(dev()), i32(expert), tile_rows, out, status, act="swiglu")
    assert int(status.item()) == 0
    got = out.double().cpu().view(tiles, tile_rows, I)
    for t, e in enumerate(expert):
        if e < 0:
            assert bool((got[t] == 7.0).all())
            continue
        u = x.double().view(tiles, tile_rows, K)[t] @ w[e].double().T
        torch.testing.assert_close(got[t], P.silu(u[:, ::2]) * u[:, 1::2], **TOL16)


# -------------------------------------------------------------------------- attention alone


class _Group:
    def __init__(self, table):
        self.block_table = table


class _Ctx:
    """What paged_attention asks of a step, for entries laid out by hand."""

    def __init__(self, lens, ctxs, table):
        self.device = dev()
        self.host_q_len, self.host_ctx_len = list(lens), list(ctxs)
        self.host_q_start = np.concatenate([[0], np.cumsum(lens)])[:-1].tolist()
        self.q_start, self.q_len, self.ctx_len = i32(self.host_q_start), i32(lens), i32(ctxs)
        self.slots = i32(list(range(len(lens))))
        self.status = torch.zeros(1, dtype=torch.int32, device=dev())
        self.groups = [_Group(table)]
        self.T, self.E = int(sum(lens)), len(lens)
        self._plans = {}

    def plan(self, key, make):
        if key not in self._plans:
            self._plans[key] = make()
        return self._plans[key]


class _Kv:
    group = 0

    def __init__(self, pages):
        self.pages = pages


def attention_by_hand(kind, H, nkv, hd, vd, dtype, ctxs, lens, *, size=0, keep=0, sink=False, gate="", make_hot=None, ps=16, seed=0, scale=0.2):
    """Entries of ``lens`` new tokens whose contexts end at ``ctxs``: random keys and values laid into pages in a scrambled
    order, pages that no new token may read left out of the block table; the engine's attention and the plain one.
    kind "heads": H query heads on nkv KV heads; "row": all H heads share one row of nkv blocks of hd lanes, whose first
    nkv * vd lanes are the values too (nkv 1, or vd = hd)."""
    from vllm_cpp_b200.parts.window_attention import paged_attention
    row = kind == "row"
    kh, kw, vw = (1, nkv * hd, nkv * vd) if row else (nkv, hd, vd)      # KV heads and their lanes as the plain one sees them
    g = torch.Generator().manual_seed(seed + H * 7 + hd)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    E, max_blocks = len(lens), max(-(-c // ps) for c in ctxs)
    n_pages = E * max_blocks + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((E, max_blocks), -1, dtype=torch.int32)
    keys = torch.full((n_pages, nkv, ps, hd), float("nan"), dtype=F64)
    vals = torch.full((n_pages, nkv, ps, vd), float("nan"), dtype=F64)
    of = torch.arange(H) // (H // kh)
    sinks = rnd(H) * 2.0 if sink else None
    qs, wants, gates = [], [], []
    for e in range(E):
        n, first = ctxs[e], ctxs[e] - lens[e]
        q, k = rnd(n, H, kw), rnd(n, kh, kw)
        v = k[..., :vw].clone() if row else rnd(n, kh, vw)
        if make_hot is not None:
            make_hot(e, q, k, v)
            v = k[..., :vw].clone() if row else v
        q, k, v = (t.to(dtype).double() for t in (q, k, v))         # what the cache and the query buffer hold
        gt = torch.rand(n, H * vw if gate == "lane" else H, generator=g, dtype=F64) * 1.5
        lo = max(0, first - size + 1) if size else 0
        for b in range(-(-n // ps)):
            if b * ps + ps <= lo and b * ps >= (keep if size else 0):
                continue            # given back: no new token reads it
            page = order.pop()
            table[e, b] = page
            m = min(ps, n - b * ps)
            keys[page, :, :m] = k[b * ps:b * ps + m].reshape(m, nkv, hd).transpose(0, 1)
            if not row:
                vals[page, :, :m] = v[b * ps:b * ps + m].transpose(0, 1)
        s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
        o = torch.einsum("hij,jhe->ihe", P.masked_softmax(s, P.window_mask(n, size, keep), sinks), v[:, of])
        o = o * (gt.view(n, H, vw) if gate == "lane" else gt[:, :, None] if gate else 1.0)
        wants.append(o[first:])
        qs.append(q.reshape(n, -1)[first:])
        gates.append(gt[first:])
    if row:
        pages = keys[:, None]
    else:
        pages = torch.stack([keys, vals], 1) if vd == hd else torch.cat([keys.reshape(n_pages, -1), vals.reshape(n_pages, -1)], 1)
    ctx = _Ctx(lens, ctxs, table.to(dev()))
    out = torch.full((ctx.T, H * vw), float("nan"), dtype=dtype, device=dev())
    blocks = row and nkv > 1
    paged_attention(ctx, _Kv(pages.to(dtype).to(dev())), torch.cat(qs).to(dtype).to(dev()), out, nh=H * nkv if blocks else H, nkv=nkv, hd=hd, vd=vd,
                    scale=scale, window=size, keep_first=keep if size else 0, sink=f32(sinks) if sink else False,
                    out_gate=f32(torch.cat(gates)) if gate else None, blocks=blocks)
    assert int(ctx.status.item()) == 0
    return out.double().cpu().view(-1, H, vw), torch.cat(wants)


ATTN_TOL = {torch.float32: dict(atol=3e-5, rtol=3e-5), torch.bfloat16: dict(atol=3e-2, rtol=2e-2)}
MIXED_LENS = [1, 1, 1, 7, 40, 1, 130, 2]
MIXED_CTXS = [1, 17, 700, 7, 95, 64, 200, 50]
HEADS = [("heads", 4, 2, 8, 6, dict(size=9, keep=5, gate="lane")), ("heads", 6, 2, 64, 64, dict(size=40, keep=19, gate="lane")),
         ("heads", 4, 4, 128, 128, dict(size=56, keep=70, gate="lane")), ("heads", 5, 1, 64, 64, dict(size=1, keep=3, gate="lane")),
         ("heads", 8, 2, 128, 128, dict(gate="lane")), ("heads", 3, 3, 16, 10, dict(size=20, keep=0, gate="lane")),
         ("heads", 40, 2, 64, 64, dict(size=100, keep=1, gate="lane"))]
ROWS = [("row", 3, 1, 9, 9, dict(gate="head")), ("row", 5, 1, 64, 64, dict(gate="head")), ("row", 8, 1, 128, 128, dict(size=40, sink=True, gate="head")),
        ("row", 2, 1, 24, 20, dict(size=7, sink=True, gate="head")), ("row", 6, 2, 128, 128, dict(gate="head")), ("row", 4, 3, 128, 128, dict(size=33, sink=True, gate="head")),
        ("row", 20, 2, 128, 128, dict(size=90, sink=True)), ("row", 16, 4, 128, 128, dict(sink=True, gate="head")), ("row", 40, 2, 128, 128, dict(gate="head")),
        ("row", 33, 4, 128, 128, dict(size=300, sink=True, gate="head")), ("row", 7, 8, 128, 128, dict(size=64, gate="head")), ("row", 12, 5, 128, 128, dict(gate="lane")),
        ("row", 140, 1, 128, 128, dict(sink=True, gate="head")), ("row", 4, 1, 300, 290, dict(gate="head"))]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,H,nkv,hd,vd,opt", HEADS + ROWS)
def test_attention_on_a_mixed_batch(dtype, kind, H, nkv, hd, vd, opt):
    """First tokens, single tokens behind short and long contexts, portions that cross borders of pages and windows: heads
    and shared rows of sizes that each of the kernels takes, and some that only the plain one does."""
    got, want = attention_by_hand(kind, H, nkv, hd, vd, dtype, MIXED_CTXS, MIXED_LENS, scale=0.5 * (hd * (nkv if kind == "row" else 1)) ** -0.5, **opt)
    torch.testing.assert_close(got, want, **ATTN_TOL[dtype])


@gpu
@pytest.mark.parametrize("kind,H,nkv,hd,opt", [("heads", 8, 2, 64, dict(size=300, keep=40, gate="lane")), ("row", 8, 1, 128, dict(size=300, sink=True, gate="head")),
                                               ("row", 10, 2, 128, dict(size=300, sink=True, gate="head")), ("row", 32, 4, 128, dict(gate="head")),
                                               ("row", 48, 3, 128, dict(sink=True, gate="head"))])
def test_single_tokens_of_many_lengths(kind, H, nkv, hd, opt):
    """Many tokens (one slice each) and few (sliced keys, merged); contexts that end at the first key of a page and of a tile."""
    scale = 0.5 * (hd * (nkv if kind == "row" else 1)) ** -0.5
    for ctxs in ([1, 2, 16, 17, 64, 65, 128, 129, 300, 301, 500, 600, 601, 899], [900], [899, 601, 640], list(range(5, 5 + 160))):
        got, want = attention_by_hand(kind, H, nkv, hd, hd, torch.bfloat16, ctxs, [1] * len(ctxs), scale=scale, **opt)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("ps", [8, 12, 32, 64])
def test_attention_on_other_page_sizes(ps):
    """Pages that the tensor cores' loaders bring in whole, and one size (12) that they do not."""
    for kind, H, nkv, hd, opt in (("heads", 4, 2, 64, dict(size=45, keep=21, gate="lane")), ("row", 5, 1, 64, dict(gate="head")),
                                  ("row", 6, 3, 128, dict(size=100, sink=True, gate="head"))):
        got, want = attention_by_hand(kind, H, nkv, hd, hd, torch.bfloat16, MIXED_CTXS, MIXED_LENS, ps=ps, scale=0.5 * hd ** -0.5, **opt)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("env", [{"TCGEN05_SPANS": False}, {"WIDE_DECODE": False}, {"MMA_ATTENTION": False}, {"CLUSTER_MERGE": False}])
def test_every_kernel_takes_the_options(env, monkeypatch):
    """The kernels that serve what the preferred ones do not: forced onto sizes that those take."""
    import vllm_cpp_b200.parts.window_attention as wa
    for k, v in env.items():
        monkeypatch.setattr(wa, k, v)
    for kind, H, nkv, hd, vd, opt in (HEADS[1], HEADS[2], ROWS[1], ROWS[2], ROWS[4], ROWS[5], ROWS[6]):
        got, want = attention_by_hand(kind, H, nkv, hd, vd, torch.bfloat16, MIXED_CTXS, MIXED_LENS, scale=0.5 * hd ** -0.5, **opt)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,hd,nkv", [("heads", 16, 2), ("heads", 64, 1), ("heads", 128, 2), ("row", 20, 1), ("row", 64, 1), ("row", 128, 1), ("row", 128, 3)])
def test_one_key_decides_the_row(dtype, kind, hd, nkv):
    """A key whose score stands out, placed just inside and just outside the query's window, at the last first token that
    the window keeps and at the next one, and far back among hundreds, in a prompt portion and behind a single token."""
    H, size, length, keep = 2 * nkv if kind == "heads" else 3, 70, 300, 13 if kind == "heads" else 0
    edge = length - size            # the last query, 299, sees keys from 230 on
    lanes = hd * (nkv if kind == "row" else 1)
    for n_new in (1, 60):
        for at, window in ((length - 1, size), (edge, size), (edge - 1, size), (keep - 1, size), (keep, size), (3, 0)):
            if at < 0:
                continue

            def hot(e, q, k, v, at=at):
                q *= 0.05
                k[:, 0, -1] *= 0.1
                q[-1, 0] = 0.0
                q[-1, 0, -1] = 8.0 if kind == "row" else 20.0
                k[at, 0, -1] = 8.0 if kind == "row" else 10.0
                v[at, 0] = 5.0
                k[at, 0, 0] = 5.0
                k[:at, 0, 0] *= 0.1
                k[at + 1:, 0, 0] *= 0.1
            got, want = attention_by_hand(kind, H, nkv, hd, hd, dtype, [length], [n_new], size=window, keep=keep, make_hot=hot)
            torch.testing.assert_close(got, want, **(ATTN_TOL[dtype]))
            seen = at >= edge or window == 0 or at < keep
            assert (abs(float(want[-1, 0, 0]) - 5.0) < 0.5) == seen, (at, window, want[-1, 0, 0])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd,nkv", [(20, 1), (64, 1), (128, 1), (128, 2)])
def test_a_sink_that_outweighs_the_keys(dtype, hd, nkv):
    """Scores far below the sink leave a head nearly nothing, scores far above it everything, and the sink counts once however
    the keys are sliced."""
    def low(e, q, k, v):
        q *= 0.01
        q[:, 1] *= 1000.0
    for n_new, ctx in ((1, 900), (40, 200), (1, 1)):
        got, want = attention_by_hand("row", 4, nkv, hd, hd, dtype, [ctx], [n_new], size=500, sink=True, make_hot=low, seed=4)
        # (scores of some tens: their 32-bit rounding shows in the weights)
        torch.testing.assert_close(got, want, **(dict(atol=2e-4, rtol=2e-4) if dtype == torch.float32 else ATTN_TOL[dtype]))


# -------------------------------------------------------------------------- whole models through bin/trace_run


def compare(name, dtype, trace, out_dir, requests, oracle):
    vocab = configs()[name][0].vocab
    worst = 0.0
    for step, want in enumerate(trace.wanted):
        got = R.read_step(out_dir, step, vocab)
        if not want:
            assert got is None
            continue
        assert got is not None and got.shape == (len(want), vocab), f"step {step}: {None if got is None else got.shape}"
        ref = np.stack([oracle(name, requests[rid])[pos] for rid, pos in want])
        err = np.abs(got - ref).max(axis=1) / np.abs(ref).max()
        bad = np.nonzero(~(err <= REL_TOL[dtype]))[0]
        assert len(bad) == 0, (f"{name} {dtype}: step {step}, first wrong row {want[bad[0]]} (request, position): "
                               f"relative error {err[bad[0]]:.3e} > {REL_TOL[dtype]}")
        worst = max(worst, err.max())
    return worst


MODES = {"whole": R.whole, "tail": R.tail_one_by_one, "portions": R.portions, "portions_last": R.portions_last, "mixed": R.mixed,
         "mixed_last": R.mixed_last}
REPLAYS = ([("A", "float32", m) for m in MODES]
           + [(n, "float32", m) for n, ms in (("B", "portions mixed_last"), ("C", "whole portions mixed"), ("D", "mixed")) for m in ms.split()]
           + [(n, "bfloat16", m) for n, ms in (("A", "mixed"), ("B", "whole tail portions mixed"), ("C", "portions mixed_last"),
                                               ("D", "whole tail mixed mixed_last")) for m in ms.split()])


@gpu
@pytest.mark.parametrize("name,dtype,mode", REPLAYS)
def test_replay(name, dtype, mode, disorax_dirs, oracle, tmp_path):
    """Whole prompts; the last 32 tokens one by one; portions of changing size down to two tokens; up to four live
    requests with pages and slots used again -- the last two also as serving asks (logits of an entry's last token
    only: captured steps), all over a NaN-filled cache."""
    requests = requests_of(name)
    trace = MODES[mode](requests)
    out = R.run_trace(disorax_dirs[name], dtype, trace, tmp_path / "out", configs()[name][1], extra_args=["--poison"])
    worst = compare(name, dtype, trace, out, requests, oracle)
    print(f"{name} {dtype} {mode}: worst relative error {worst:.3e}, pool {trace.max_tokens} tokens, {len(trace.steps)} steps")


@gpu
def test_replay_modes_agree_with_each_other(disorax_dirs, tmp_path):
    """Cutting and batching change the logits by rounding only."""
    for name in ("A", "B"):
        requests = requests_of(name)
        vocab = configs()[name][0].vocab
        rows = {}
        for mode in ("whole", "mixed"):
            trace = MODES[mode](requests)
            out = R.run_trace(disorax_dirs[name], "float32", trace, tmp_path / (name + mode), configs()[name][1])
            for step, want in enumerate(trace.wanted):
                got = R.read_step(out, step, vocab)
                for i, key in enumerate(want):
                    rows.setdefault(key, {})[mode] = got[i]
        worst = max(np.abs(v["whole"] - v["mixed"]).max() / np.abs(v["whole"]).max() for v in rows.values())
        assert worst < 2e-5, (name, worst)


@gpu
def test_long_decoding(disorax_dirs, oracle, tmp_path):
    """A short prompt, then 250 tokens one by one: windows passing over decoded tokens and pages' borders, pages given back as
    they pass, the first tokens kept."""
    for name, dtype in (("A", "float32"), ("B", "float32"), ("D", "bfloat16")):
        toks = random_tokens(configs()[name][0].vocab, 260, 99)
        trace = R.tail_one_by_one({"long": toks}, tail=250)
        out = R.run_trace(disorax_dirs[name], dtype, trace, tmp_path / name, configs()[name][1], extra_args=["--poison"])
        compare(name, dtype, trace, out, {"long": toks}, oracle)


# -------------------------------------------------------------------------- generation through the engine's entry point


@gpu
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(name, disorax_dirs):
    """Several prompts at once through LLM.generate (scheduler, portions under a small token budget, captured decoding
    steps, device-side sampling at temperature 0) against the plain implementation's greedy continuation."""
    from vllm_cpp_b200 import LLM
    cfg, w = P.read_model(disorax_dirs[name])
    vocab, page = configs()[name][0].vocab, configs()[name][1]
    prompts = [random_tokens(vocab, n, 3 + n) for n in (5, 41, 18, 70, 2)]
    llm = LLM(str(disorax_dirs[name]), dtype="float32", page_size=page, max_tokens=page * 64, max_num_seqs=3, max_step_tokens=32,
              max_model_len=256)
    got = llm.generate(prompts, max_new_tokens=24, temperature=0.0, top_p=1.0, repeat_penalty=1.0, ignore_eos=True)
    for prompt, g in zip(prompts, got):
        want = P.greedy(cfg, w, prompt, 24)
        # a near tie between two logits may fall the other way in 32-bit: compare up to the first such place
        for i, (a, b) in enumerate(zip(g, want)):
            if a != b:
                logits = P.forward(cfg, w, prompt + want[:i])[-1]
                assert abs(float(logits[a] - logits[b])) < 1e-4 * float(logits.abs().max()), (i, a, b)
                break
        assert len(g) == 24
