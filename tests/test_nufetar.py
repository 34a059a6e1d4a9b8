"""Nufetar in the engine against the plain implementation (tests/plain_nufetar.py): each mechanism's kernel alone, then
whole models through bin/trace_run (whole prompts, decoding, portions down to two tokens, mixed batches with pages and
slots used again) and greedy generation through the engine's entry point, on small configurations of its own."""
import json
import math

import numpy as np
import pytest
import torch

import plain_nufetar as P
import replay_util as R
from conftest import random_tokens

gpu = pytest.mark.gpu
F64 = torch.float64


def configs():
    from vllm_cpp_b200.config.nufetar import (ChunkAttentionSpec as A, LatentSpec as Lat, NufetarConfig, NufetarLayer as L,
                                              NufetarMlp as F, Rotation as Rot, WkvSpec as W)
    return {
        # chunks of 10 and a window of 9 over pages of 4; values narrower than keys, half of the lanes turning; a wkv layer
        # without a feed-forward
        "A": (NufetarConfig(vocab=150, width=48, norm_eps=1e-5, layers=(
            L("wkv", W(heads=3, dim=6, rank=5), F("dense", ff=40)),
            L("attention", A(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.35, chunk=10, rot=Rot(100.0, 4)), F("dense", ff=24)),
            L("latent_attention", Lat(heads=3, dim=5, rot_dim=4, vdim=7, kv_rank=9, scale=0.4, window=9, rot=Rot(50.0, 4)), F("dense", ff=16)),
            L("wkv", W(heads=2, dim=12, rank=3)))), 4),
        # sizes that bfloat16 runs on the tensor cores: heads of 64 lanes in chunks of 48 on two KV heads, latent rows of
        # 48 + 16 lanes under a window of 21, heads of 64 lanes on one KV head that see every earlier token; state rows of 64
        "B": (NufetarConfig(vocab=260, width=64, norm_eps=1e-6, layers=(
            L("attention", A(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, chunk=48, rot=Rot(10000.0, 64)), F("dense", ff=48)),
            L("latent_attention", Lat(heads=2, dim=24, rot_dim=16, vdim=40, kv_rank=48, scale=0.2, window=21, rot=Rot(500.0, 16)), F("dense", ff=32)),
            L("wkv", W(heads=1, dim=64, rank=16), F("dense", ff=24)),
            L("attention", A(heads=2, kv_heads=1, dim=64, vdim=64, scale=0.11, chunk=0, rot=Rot(1e6, 32)), F("dense", ff=40)))), 16),
        # a width that is no multiple of 4; five heads on one KV head in chunks of one token; a latent wider than a block's
        # threads hold, all keys seen; three heads with KV heads of their own in chunks of 7 whose lanes do not turn; one
        # head of 33 state rows; pages of 8
        "C": (NufetarConfig(vocab=97, width=50, norm_eps=1e-4, layers=(
            L("attention", A(heads=5, kv_heads=1, dim=6, vdim=10, scale=1.0, chunk=1, rot=Rot(50.0, 2)), F("dense", ff=11)),
            L("latent_attention", Lat(heads=2, dim=7, rot_dim=6, vdim=3, kv_rank=290, scale=0.3, window=0, rot=Rot(30.0, 6)), F("dense", ff=9)),
            L("attention", A(heads=3, kv_heads=3, dim=10, vdim=14, scale=0.3, chunk=7, rot=Rot(30.0, 0))),
            L("wkv", W(heads=1, dim=33, rank=2), F("dense", ff=13)))), 8),
        # heads of 128 lanes: query rows of 512 and of 384 lanes once mixed; latent rows of 112 + 16 lanes
        "D": (NufetarConfig(vocab=210, width=96, norm_eps=1e-5, layers=(
            L("attention", A(heads=8, kv_heads=4, dim=128, vdim=128, scale=0.09, chunk=56, rot=Rot(1e5, 128)), F("dense", ff=64)),
            L("latent_attention", Lat(heads=4, dim=20, rot_dim=16, vdim=24, kv_rank=112, scale=0.15, window=70, rot=Rot(2000.0, 16)), F("dense", ff=56)),
            L("attention", A(heads=3, kv_heads=3, dim=128, vdim=128, scale=0.09, chunk=33, rot=Rot(1e4, 96)), F("dense", ff=72)),
            L("wkv", W(heads=3, dim=32, rank=8), F("dense", ff=48)))), 16),
    }


LENGTHS = {"A": [40, 75, 150, 33, 2, 17, 64], "B": [1, 7, 33, 64, 170, 97, 3], "C": [50, 3, 77, 31, 9], "D": [120, 2, 230, 57, 33]}
REL_TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def hand_made(cfg, tensors, seed):
    """The random tensors, changed so that a fault shows: sharp softmaxes (single keys, often far ones or ones at the edge
    of a window or a chunk, carry the rows), heads that really read one another's scores, gates and biases that matter,
    decays spread from fast to slow and a bonus of the size of the state."""
    g = torch.Generator().manual_seed(seed)
    out = dict(tensors)
    rnd = lambda *shape: torch.randn(*shape, generator=g)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}.mix."
        if layer.type == "attention":
            H = layer.mixer.heads
            for n in ("q", "k"):
                out[p + n] = tensors[p + n] * 9.0
            for n in ("q.b", "k.b", "v.b", "o.b"):
                out[p + n] = tensors[p + n] * 4.0
            out[p + "talk"] = 0.6 * torch.eye(H) + rnd(H, H) * 0.8 / H ** 0.5
            out[p + "g"] = tensors[p + "g"] * 25.0
        elif layer.type == "latent_attention":
            for n in ("q", "dkv"):
                out[p + n] = tensors[p + n] * 12.0
            out[p + "uk"] = tensors[p + "uk"] * 10.0
        else:
            n = tensors[p + "w0"].numel()
            out[p + "w0"] = torch.linspace(-7.0, 1.0, n)[torch.randperm(n, generator=g)]
            out[p + "w2"] = tensors[p + "w2"] * 30.0
            out[p + "w1"] = tensors[p + "w1"] * 10.0
            out[p + "u"] = tensors[p + "u"] * 8.0
            for m in "rkvgw":
                out[p + "mu." + m] = torch.rand(cfg.width, generator=g)
        # sublayers whose results outweigh the embedding they are added to: what is generated depends on all that came before
        out[p + "o"] = tensors[p + "o"] * 3.0
        if layer.mlp is not None:
            out[f"l{i}.mlp.down"] = tensors[f"l{i}.mlp.down"] * 3.0
            out[f"l{i}.mlp.act"] = torch.tensor([0.7, -0.9]) + 0.3 * i
            out[f"l{i}.mlp.up"] = tensors[f"l{i}.mlp.up"] * 8.0
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


@pytest.fixture(scope="module")
def nufetar_dirs(tmp_path_factory):
    from vllm_cpp_b200 import write_random_model
    from vllm_cpp_b200.weights.safetensors_io import read_safetensors, write_safetensors
    out = {}
    for i, (name, (cfg, _)) in enumerate(configs().items()):
        d = tmp_path_factory.mktemp(f"nufetar_{name}")
        write_random_model(cfg, 61 + i, d, dtype="bfloat16")
        tensors = {k: v.float() for k, v in read_safetensors(d / "model.safetensors").items()}
        write_safetensors(d / "model.safetensors", hand_made(cfg, tensors, 15 + i), {"format": "pt"})
        # the rank of the decay's projection is not a key of a model folder's configuration: the tensors say it
        c = json.loads((d / "config.json").read_text())
        for layer in c["layers"]:
            layer["mixer"].pop("rank", None)
        (d / "config.json").write_text(json.dumps(c))
        out[name] = d
    return out


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
def oracle(nufetar_dirs):
    return Oracle(nufetar_dirs)


def requests_of(name):
    vocab = configs()[name][0].vocab
    return {f"r{i}": random_tokens(vocab, n, 11 * i + ord(name)) for i, n in enumerate(LENGTHS[name])}


# -------------------------------------------------------------------------- without a GPU


def test_config_reads_every_size_and_constant():
    from vllm_cpp_b200 import ConfigError
    from vllm_cpp_b200.config.nufetar import NufetarConfig
    d = {"architecture": "Nufetar", "vocab": 51, "width": 24, "norm": {"eps": 3e-4},
         "layers": [{"type": "attention", "mlp": None,
                     "mixer": {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.5, "mask": {"size": 7},
                               "rot": {"base": 777.0, "dims": 6}}},
                    {"type": "wkv", "mlp": {"kind": "dense", "ff": 31}, "mixer": {"heads": 4, "dim": 6}},
                    {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 5},
                     "mixer": {"heads": 2, "dim": 8, "rot_dim": 4, "vdim": 9, "kv_rank": 11, "scale": 0.25, "mask": {"size": 3},
                               "rot": {"base": 9.0, "dims": 4}}}]}
    cfg = NufetarConfig.from_dict(d)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (51, 24, 3e-4)
    a, b, c = cfg.layers
    m = a.mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.chunk, m.rot.base, m.rot.dims, a.mlp) == (6, 2, 10, 14, 0.5, 7, 777.0, 6, None)
    assert (b.mixer.heads, b.mixer.dim, b.mixer.rank, b.mlp.kind, b.mlp.ff) == (4, 6, 0, "dense", 31)
    m = c.mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.window, m.rot.base, m.rot.dims) == (2, 8, 4, 9, 11, 0.25, 3, 9.0, 4)
    assert NufetarConfig.from_dict(cfg.to_dict()) == cfg
    # a mask left out or null: every earlier token is seen
    layer = d["layers"]
    for k, attr in ((0, "chunk"), (2, "window")):
        for mixer in ({n: v for n, v in layer[k]["mixer"].items() if n != "mask"}, dict(layer[k]["mixer"], mask=None)):
            assert getattr(NufetarConfig.from_dict(dict(d, layers=[dict(layer[k], mixer=mixer)])).layers[0].mixer, attr) == 0
    for bad in ({"layers": []}, {"layers": [dict(layer[0], type="other")]}, {"layers": [{"type": "wkv", "mlp": None}]},
                {"layers": [dict(layer[0], mixer=dict(layer[0]["mixer"], kv_heads=4))]},
                {"layers": [dict(layer[0], mixer=dict(layer[0]["mixer"], rot={"base": 5.0, "dims": 3}))]},
                {"layers": [dict(layer[0], mixer=dict(layer[0]["mixer"], rot={"base": 5.0, "dims": 12}))]},
                {"layers": [dict(layer[0], mixer=dict(layer[0]["mixer"], mask={"size": 0}))]},
                {"layers": [dict(layer[2], mixer=dict(layer[2]["mixer"], rot={"base": 9.0, "dims": 2}))]},
                {"layers": [dict(layer[1], mlp={"kind": "routed", "ff": 3})]}, {"vocab": None}):
        with pytest.raises(ConfigError):
            NufetarConfig.from_dict(dict(d, **bad))


def test_model_folder_is_recognised_and_names_its_tensors(tmp_path):
    from vllm_cpp_b200.config.nufetar import NufetarConfig
    from vllm_cpp_b200.models import expected_tensors, load_config
    cfg, _ = configs()["A"]
    (tmp_path / "config.json").write_text(json.dumps(cfg.to_dict()))
    assert load_config(tmp_path) == cfg
    s = {t.name: tuple(t.shape) for t in expected_tensors(cfg)}
    assert s["embed"] == (150, 48) and s["final.norm"] == (48,) and "head" not in s       # the head is the embedding table
    assert all(s[f"l0.mix.mu.{m}"] == (48,) for m in "rkvgw") and all(s[f"l0.mix.{m}"] == (18, 48) for m in "rkvg")
    assert s["l0.mix.w1"] == (5, 48) and s["l0.mix.w2"] == (18, 5) and s["l0.mix.w0"] == s["l0.mix.norm"] == (18,)
    assert s["l0.mix.u"] == (3, 6) and s["l0.mix.o"] == (48, 18)
    assert s["l0.norm1"] == s["l0.norm2"] == (48,) and s["l0.mlp.up"] == (40, 48) and s["l0.mlp.down"] == (48, 40) and s["l0.mlp.act"] == (2,)
    assert s["l1.mix.q"] == (32, 48) and s["l1.mix.k"] == (16, 48) and s["l1.mix.v"] == (12, 48) and s["l1.mix.o"] == (48, 24)
    assert s["l1.mix.q.b"] == (32,) and s["l1.mix.k.b"] == (16,) and s["l1.mix.v.b"] == (12,) and s["l1.mix.o.b"] == (48,)
    assert s["l1.mix.talk"] == (4, 4) and s["l1.mix.g"] == (4, 48) and "l1.mix.g.b" not in s
    assert s["l2.mix.q"] == (27, 48) and s["l2.mix.dkv"] == (13, 48) and s["l2.mix.dkv.norm"] == (9,)
    assert s["l2.mix.uk"] == (15, 9) and s["l2.mix.uv"] == (21, 9) and s["l2.mix.o"] == (48, 21) and "l2.mix.dq" not in s
    assert not any(k.startswith(("l3.mlp", "l3.norm2")) for k in s)                       # a layer without a feed-forward
    c = cfg.to_dict()
    del c["layers"][0]["mixer"]["rank"]
    s = {t.name: tuple(t.shape) for t in expected_tensors(NufetarConfig.from_dict(c))}
    assert s["l0.mix.w1"] == (-1, 48) and s["l0.mix.w2"] == (18, -1)


def test_what_a_layer_keeps_per_request():
    import vllm_cpp_b200.models as models
    cfg, _ = configs()["A"]
    specs = models.build_model(cfg, torch.float32, "cpu").cache_specs()
    assert (specs[(0, 0)].kind, specs[(0, 0)].shape, specs[(0, 0)].dtype) == ("state", (3, 6, 6), "float32")
    assert (specs[(0, 1)].kind, specs[(0, 1)].shape, specs[(0, 1)].dtype) == ("state", (48,), "float32")
    kv = specs[1]
    assert (kv.kind, kv.num_kv_heads, kv.head_dim, kv.v_head_dim, kv.window, kv.chunked) == ("kv", 2, 8, 6, 10, True)
    kv = specs[2]
    assert (kv.kind, kv.num_kv_heads, kv.head_dim, kv.one_row, kv.window, kv.chunked) == ("kv", 1, 13, True, 9, False)
    from vllm_cpp_b200.cache.device_cache import CacheLayout
    lay = CacheLayout(specs)
    assert len(lay.paged) == 2       # a standing and a sliding window are different pools
    # an attention over all earlier tokens has no chunks to give back
    b = models.build_model(configs()["B"][0], torch.float32, "cpu").cache_specs()
    assert (b[3].window, b[3].chunked) == (0, False)


def test_pages_of_a_chunk_are_given_back_when_it_is_through():
    from vllm_cpp_b200.runtime import runtime
    rt = runtime()
    g = rt.GroupSpec(4, 64, 10, 0, True)
    assert [g.first_read(p) for p in (0, 9, 10, 19, 20, 25)] == [0, 0, 10, 10, 20, 20]
    assert [rt.GroupSpec(4, 64, 10).first_read(p) for p in (0, 9, 10, 19)] == [0, 0, 1, 10]
    m = rt.CacheManager([g, rt.GroupSpec(4, 64, 10)], 2)
    m.open(7)
    assert m.reserve(7, 40)
    dead = lambda grp: sum(p < 0 for p in m.block_table(7, grp))
    m.commit(7, 9)
    assert (dead(0), dead(1)) == (0, 0)
    m.commit(7, 10)                 # the next token opens chunk [10, 20): pages 0 and 1 are through, page 2 holds tokens 10, 11
    assert (dead(0), dead(1)) == (2, 0)
    m.commit(7, 19)
    assert (dead(0), dead(1)) == (2, 2)
    m.commit(7, 20)
    assert (dead(0), dead(1)) == (5, 2)
    m.commit(7, 33)
    assert (dead(0), dead(1)) == (7, 6)
    m.check_invariants()
    m.close(7)
    m.check_invariants()
    # the first positions that are kept for good stay, whatever the chunks do
    m = rt.CacheManager([rt.GroupSpec(4, 64, 10, 6, True)], 1)
    m.open(1)
    assert m.reserve(1, 40)
    m.commit(1, 40)
    assert [p < 0 for p in m.block_table(1, 0)] == [False, False] + [True] * 8


def test_oracle_mechanisms_by_hand():
    # chunks stand still, windows slide
    assert P.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    assert P.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert torch.equal(P.chunk_mask(4, 0), P.window_mask(4, 0)) and int(P.chunk_mask(4, 0).sum()) == 10
    # rotation: halves and neighbours
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]], [[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    pos = torch.tensor([0, 3])
    a0, a1 = 3.0, 3.0 * 10.0 ** -0.5
    h = P.turn(x, pos, 10.0, 4, False)
    assert torch.equal(h[0], x[0])
    torch.testing.assert_close(h[1, 0], torch.tensor([math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1),
                                                      3 * math.cos(a0) + math.sin(a0), 4 * math.cos(a1) + 2 * math.sin(a1), 5.0], dtype=F64))
    n = P.turn(x, pos, 10.0, 4, True)
    torch.testing.assert_close(n[1, 0], torch.tensor([math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + math.sin(a0),
                                                      3 * math.cos(a1) - 4 * math.sin(a1), 4 * math.cos(a1) + 3 * math.sin(a1), 5.0], dtype=F64))
    # xIELU at its joint, above it and below
    z = torch.tensor([0.0, 2.0, -1.0], dtype=F64)
    sp, sq = math.log(1 + math.exp(0.3)), math.log(1 + math.exp(-1.2))
    torch.testing.assert_close(P.xielu(z, 0.3, -1.2), torch.tensor([0.0, 4 * sp + 1, (0.5 + sq) * math.exp(-1.0) - 0.5], dtype=F64))
    # wkv: the state as it was, plus the current token with its bonus; then decay and write
    out, S = P.wkv_scan(torch.tensor([[1.0, 1.0], [1.0, 2.0]], dtype=F64), torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64),
                        torch.tensor([[1.0], [10.0]], dtype=F64), torch.tensor([[0.5, 0.25], [0.5, 0.25]], dtype=F64),
                        torch.tensor([3.0, -1.0], dtype=F64))
    torch.testing.assert_close(out, torch.tensor([[3.0 - 2.0], [1.0 + 4.0 + 90.0 - 80.0]], dtype=F64))
    torch.testing.assert_close(S, torch.tensor([[0.5 + 30.0], [0.5 + 40.0]], dtype=F64))
    h = torch.tensor([[1.0, 2.0], [5.0, 0.0]], dtype=F64)
    torch.testing.assert_close(P.shifted(h, torch.tensor([0.25, 1.0], dtype=F64)), torch.tensor([[0.75, 0.0], [4.0, 2.0]], dtype=F64))
    # mixing the scores of the heads is the same as mixing their queries, one block per KV head
    g = torch.Generator().manual_seed(1)
    q, k, talk = (torch.randn(*s, generator=g, dtype=F64) for s in ((5, 4, 3), (5, 2, 3), (4, 4)))
    raw = torch.einsum("ihd,jhd->hij", q, k[:, [0, 0, 1, 1]])
    torch.testing.assert_close(torch.einsum("ihgd,jgd->hij", wide_queries(q, talk, 2), k), P.mixed_scores(raw, talk))


def wide_queries(q, talk, nkv):
    """q [T, H, d] -> [T, H, nkv, d]: block G of head h is the sum over the heads g of KV head G of talk[h, g] q_g."""
    T, H, d = q.shape
    return torch.einsum("hGg,tGgd->thGd", talk.view(H, nkv, H // nkv), q.view(T, nkv, H // nkv, d))


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


@gpu
@pytest.mark.parametrize("F,S,dtype", [(5, 1, torch.float32), (40, 2, torch.bfloat16), (260, 1, torch.float32), (3001, 3, torch.float32)])
def test_xielu_and_tanh(F, S, dtype):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(F)
    z = torch.randn(6, F, generator=g, dtype=F64) * 2.5
    z[1] *= 1e-3
    z[2, 0], z[2, 1], z[2, 2] = 0.0, -30.0, 15.0
    coef = torch.tensor([P.softplus(0.6), 0.5 + P.softplus(-1.1)], dtype=F64)
    tol = dict(atol=1e-4, rtol=3e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=1e-2)
    for kind, want in (("xielu", P.xielu(z, 0.6, -1.1)), ("tanh", torch.tanh(z))):
        out = torch.full((6, F), float("nan"), dtype=dtype, device=dev())
        ops.bias_act(partial_sums(z, S, g), out, kind, coef=f32(coef))
        torch.testing.assert_close(out.double().cpu(), want, **tol)


@gpu
@pytest.mark.parametrize("M,K,T", [(96, 64, 5), (300, 128, 70), (512, 200, 129), (1024, 72, 300)])
def test_xielu_in_the_products_epilogue(M, K, T):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(M)
    w = torch.randn(M, K, generator=g, dtype=F64).to(torch.bfloat16)
    x = (torch.randn(T, K, generator=g, dtype=F64) * 2.0 * K ** -0.5).to(torch.bfloat16)
    x[1] *= 1e-3        # sums near zero, where the branches meet
    coef = torch.tensor([P.softplus(0.6), 0.5 + P.softplus(-1.1)], dtype=F64)
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    want = P.xielu(x.double() @ w.double().T, 0.6, -1.1)
    for shape in [-1] + ([i for i, n in enumerate(ops.GEMM_SHAPES) if n in ("n256", "m256_n192", "pair")] if M >= 256 and T > 128 else []):
        out = torch.full((T, M), float("nan"), dtype=torch.bfloat16, device=dev())
        ops.gemm_bf16_xielu(w.to(dev()), x.to(dev()), f32(coef), out, status, shape=shape)
        assert int(status.item()) == 0
        torch.testing.assert_close(out.double().cpu(), want, atol=2e-5, rtol=6e-3)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd,rot,S,talks", [(4, 2, 8, 6, 4, 1, True), (2, 1, 64, 64, 64, 2, True), (6, 3, 10, 14, 0, 3, True),
                                                      (5, 1, 7, 3, 6, 1, True), (8, 4, 128, 128, 96, 1, True), (3, 3, 5, 5, 2, 1, False),
                                                      (10, 5, 16, 20, 16, 1, True)])
def test_bias_rotation_unit_values_mixed_queries_and_gates(dtype, nh, nkv, hd, vd, rot, S, talks):
    """Everything between the stacked projection and the attention kernels, in both page layouts, at near and far positions,
    with rows that are stored nowhere."""
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(nh * 31 + hd)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    T, ps, n_pages, eps, base = 6, 4, 5, 1e-3, 37.0
    pos, slots = [0, 1, 5, 5000, 33, 2], [3, 17, -1, 8, 0, 19]
    C = nh * hd + nkv * (hd + vd)
    u, bias, talk = rnd(T, C + nh), rnd(C), (rnd(nh, nh) if talks else None)
    u[1, nh * hd + nkv * hd:C] *= 1e-2          # values so small that eps has its part
    q_out = torch.full((T, nh * hd * (nkv if talks else 1)), float("nan"), dtype=dtype, device=dev())
    gate = torch.full((T, nh), float("nan"), device=dev())
    shape = (n_pages, 2, nkv, ps, hd) if vd == hd else (n_pages, nkv * ps * (hd + vd))
    pages = torch.full(shape, float("nan"), dtype=dtype, device=dev())
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    ops.qkv_rope_store(partial_sums(u, S, g), None, None, eps, i32(pos), freqs(base, rot) if rot else None, None, i32(slots), q_out, pages,
                       nh, nkv, hd, vd, status, rot=rot, bias=f32(bias), unit_values=True, talk=f32(talk), gate_out=gate)
    assert int(status.item()) == 0
    x = u[:, :C] + bias
    q = P.turn(x[:, :nh * hd].reshape(T, nh, hd), torch.tensor(pos), base, rot, False)
    k = P.turn(x[:, nh * hd:nh * hd + nkv * hd].reshape(T, nkv, hd), torch.tensor(pos), base, rot, False)
    v = P.unit_values(x[:, nh * hd + nkv * hd:].reshape(T, nkv, vd), eps)
    want_q = wide_queries(q, talk, nkv) if talks else q
    tol = dict(atol=5e-3, rtol=1e-4) if dtype == torch.float32 else dict(atol=5e-2, rtol=2e-2)   # (the angle at position 5,000 is a 32-bit product)
    torch.testing.assert_close(q_out.double().cpu().view(want_q.shape), want_q, **tol)
    torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(u[:, C:]), **TOL32)
    flat = pages.double().cpu().view(n_pages, -1)
    keys = flat[:, :nkv * ps * hd].view(n_pages, nkv, ps, hd)
    vals = flat[:, nkv * ps * hd:].view(n_pages, nkv, ps, vd)
    written = torch.zeros(n_pages, ps, dtype=torch.bool)
    for t, s in enumerate(slots):
        if s >= 0:
            written[s // ps, s % ps] = True
            torch.testing.assert_close(keys[s // ps, :, s % ps], k[t], **tol)
            torch.testing.assert_close(vals[s // ps, :, s % ps], v[t], **(dict(atol=2e-4, rtol=2e-4) if dtype == torch.float32 else TOL16))
    assert bool(torch.isnan(keys[~written[:, None, :].expand(-1, nkv, -1)]).all())       # nothing else was touched


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kv_rank,rot,ps,v_width,S", [(9, 4, 4, 9, 1), (48, 16, 16, 64, 2), (290, 6, 8, 290, 1), (5, 0, 4, 5, 3)])
def test_latent_rows_without_a_query_latent(dtype, kv_rank, rot, ps, v_width, S):
    """The normed latent and the shared key part turned in neighbouring pairs into their cache row, from a slice of the
    stacked product; and the queries' turning part alone."""
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(kv_rank)
    T, n_pages, eps, base, nh, d = 5, 4, 1e-4, 21.0, 3, 7
    pos, slots = [0, 1, 900, 6, 31], [2, -1, ps * 3 + 1, 0, ps + 3]
    q_cols = nh * (d + rot)
    u = torch.randn(T, q_cols + kv_rank + rot, generator=g, dtype=F64)
    gain = 1 + 0.3 * torch.randn(kv_rank, generator=g, dtype=F64)
    pages = torch.full((n_pages, ps * (kv_rank + rot + v_width)), float("nan"), dtype=dtype, device=dev())
    status = torch.zeros(1, dtype=torch.int32, device=dev())
    freq = freqs(base, rot) if rot else f32(torch.zeros(1))
    dev_u = partial_sums(u, S, g)
    ops.latent_norm_rope_store(dev_u[..., q_cols:], None, f32(gain), eps, i32(pos), freq, 1.0, i32(slots), None, pages, ps, 0, kv_rank, rot,
                               status, v_width=v_width, interleaved=True)
    assert int(status.item()) == 0
    c = P.rms(u[:, q_cols:q_cols + kv_rank], eps) * gain
    kr = P.turn(u[:, None, q_cols + kv_rank:], torch.tensor(pos), base, rot, True)[:, 0]
    tol = dict(atol=1e-3, rtol=1e-4) if dtype == torch.float32 else TOL16
    flat = pages.double().cpu()
    for t, s in enumerate(slots):
        if s >= 0:
            row, off = flat[s // ps], s % ps
            torch.testing.assert_close(row[off * (kv_rank + rot):(off + 1) * (kv_rank + rot)], torch.cat([c[t], kr[t]]), **tol)
            at = ps * (kv_rank + rot) + off * v_width
            torch.testing.assert_close(row[at:at + v_width], torch.cat([c[t], torch.zeros(v_width - kv_rank, dtype=F64)]), **tol)
    assert int((~torch.isnan(flat)).sum()) == 4 * (kv_rank + rot + v_width)
    if rot:
        out = torch.zeros(T, nh * (kv_rank + rot), dtype=dtype, device=dev())
        ops.rope_rows(dev_u[..., :q_cols], i32(pos), freq, 1.0, out, heads=nh, dims=rot, width=rot, in_head_stride=d + rot, in_off=d,
                      out_head_stride=kv_rank + rot, out_off=kv_rank, interleaved=True)
        want = P.turn(u[:, :q_cols].view(T, nh, d + rot)[..., d:], torch.tensor(pos), base, rot, True)
        torch.testing.assert_close(out.double().cpu().view(T, nh, -1)[..., kv_rank:], want, **tol)


@gpu
@pytest.mark.parametrize("T", [3, 40, 64, 200])
@pytest.mark.parametrize("H,n_in,n_out,S", [(3, 96, 128, 1), (2, 40, 33, 2), (5, 7, 70, 1), (1, 16, 300, 3), (2, 250, 24, 1)])
def test_a_small_matrix_per_head_on_steps_of_every_length(T, H, n_in, n_out, S):
    from vllm_cpp_b200 import ops
    g = torch.Generator().manual_seed(T + n_in)
    stride_in, in_off, stride_out, out_off = n_in + 6, 2, n_out + 4, 3
    x = torch.randn(T, H * stride_in, generator=g, dtype=F64)
    m = (torch.randn(H, n_out, n_in, generator=g, dtype=F64) * n_in ** -0.5).to(torch.bfloat16)
    heads = lambda t: torch.einsum("hjc,thc->thj", m.double(), t.view(T, H, stride_in)[..., in_off:in_off + n_in])
    for sums in (True, False):
        src = partial_sums(x, S, g) if sums else x.to(torch.bfloat16).to(dev())
        want = heads(x if sums else x.to(torch.bfloat16).double())
        out = torch.full((T, H * stride_out), 7.0, dtype=torch.bfloat16, device=dev())
        ops.head_linear(src, m.to(dev()), out, heads=H, n_in=n_in, n_out=n_out, in_head_stride=stride_in, in_off=in_off,
                        out_head_stride=stride_out, out_off=out_off)
        got = out.double().cpu().view(T, H, stride_out)
        torch.testing.assert_close(got[..., out_off:out_off + n_out], want, atol=1e-3, rtol=6e-3)     # rounded once, on the way out
        assert bool((got[..., :out_off] == 7.0).all()) and bool((got[..., out_off + n_out:] == 7.0).all())


PORTION_STEPS = [(3, 1), (1, 1), (2, 7), (1, 2), (9, 1), (1, 0), (2, 2), (1, 1), (1, 1), (1, 1), (16, 1), (1, 17)]
DECODE_STEPS = [(4, 2)] + [(1, 1)] * 45
# portions of several staged batches each (the kernels stage 8 or 16 tokens at a time), ending on, before and behind a batch's edge
LONG_STEPS = [(37, 16), (1, 33), (48, 5), (17, 32), (8, 9), (70, 1)]


def run_in_steps(W, steps, one_step, seed):
    """Two requests (in slots 2 and 0 of three) cut as ``steps`` says, two rows of padding behind every step;
    ``one_step(rows, qs, ql, slots, gen)`` -> that step's result rows [..., T, n].  Returns the requests' inputs and results."""
    g = torch.Generator().manual_seed(seed)
    total = [sum(s[0] for s in steps), sum(s[1] for s in steps)]
    seqs = [torch.randn(n, W, generator=g, dtype=F64) for n in total]
    got, at = [[], []], [0, 0]
    for n0, n1 in steps:
        lens = [n0, n1]
        rows = torch.cat([seqs[r][at[r]:at[r] + lens[r]] for r in range(2)] + [torch.full((2, W), float("nan"), dtype=F64)])
        qs, ql = entries_of(lens)
        o = one_step(rows, qs, ql, i32([2, 0]), g).double().cpu()
        got[0].append(o[..., :n0, :]); got[1].append(o[..., n0:n0 + n1, :])
        at = [at[0] + n0, at[1] + n1]
    return seqs, [torch.cat(x, -2) for x in got]


@gpu
@pytest.mark.parametrize("W,n_mix,dtype", [(7, 1, torch.float32), (48, 5, torch.float32), (50, 5, torch.bfloat16), (1028, 3, torch.bfloat16)])
def test_mixes_with_the_previous_token_in_portions(W, n_mix, dtype):
    from vllm_cpp_b200 import ops
    mu = torch.rand(n_mix, W, generator=torch.Generator().manual_seed(W), dtype=F64)
    state = torch.zeros(3, W, device=dev())
    state[1] = float("nan")

    def one_step(rows, qs, ql, slots, gen):
        T = rows.shape[0]
        out = torch.full((n_mix, T + 3, W), float("nan"), dtype=dtype, device=dev())
        ops.token_shift(f32(rows), f32(mu), state, qs, ql, slots, 2, out)
        assert bool(torch.isnan(out[:, T - 2:]).all())       # rows of no entry are left alone
        return out[:, :T]

    seqs, got = run_in_steps(W, PORTION_STEPS, one_step, W)
    for r in range(2):
        want = torch.stack([P.shifted(seqs[r], mu[m]) for m in range(n_mix)])
        torch.testing.assert_close(got[r], want, **(TOL32 if dtype == torch.float32 else TOL16))
        torch.testing.assert_close(state[(2, 0)[r]].double().cpu(), seqs[r][-1], **TOL32)
    assert bool(torch.isnan(state[1]).all())


def check_wkv(H, d, S, steps, dtype=torch.float32, dv=None, blocks=False):
    """``blocks``: r, k and v as row blocks of one buffer (products of their own), else columns of one stacked product."""
    from vllm_cpp_b200 import ops
    dv = dv or d
    W, eps = 24, 1e-5
    g = torch.Generator().manual_seed(H * 100 + d)
    rnd = lambda *shape: torch.randn(*shape, generator=g, dtype=F64)
    qk, inner = H * d, H * dv
    w = {"r": rnd(qk, W), "k": rnd(qk, W) * 0.3, "v": rnd(inner, W), "g": rnd(inner, W) * 0.5, "z": rnd(qk, W) * 0.3}
    w0 = torch.linspace(-7.0, 1.0, qk, dtype=F64)[torch.randperm(qk, generator=g)]
    bonus, gain = rnd(H, d), 1 + 0.2 * rnd(inner)
    state = torch.zeros(3, H, dv, d, device=dev())
    state[1] = float("nan")

    def one_step(rows, qs, ql, slots, gen):
        T = rows.shape[0]
        z = partial_sums(rows @ w["z"].T, min(S, 2), gen)
        o = torch.full((T, inner), float("nan"), device=dev())
        out = torch.empty(T, inner, device=dev(), dtype=dtype)
        if blocks:
            pad = T + 5
            u = torch.full((4, pad, qk), float("nan"), device=dev())
            for i, n in enumerate("rkvg"):
                u[i, :T] = f32(rows @ w[n].T)
            cols, first, gate, gate_col = (0, pad * qk, 2 * pad * qk), u[0, :T], u[3, :T], 0
        else:
            first = gate = partial_sums(torch.cat([rows @ w[n].T for n in "rkvg"], 1), S, gen)
            cols, gate_col = (0, qk, 2 * qk), 2 * qk + inner
        ops.matrix_rnn("wkv", first, state, qs, ql, slots, 2, o, heads=H, d=d, dv=dv, q_col=cols[0], k_col=cols[1], v_col=cols[2], z=z,
                       f_bias=f32(w0), bonus=f32(bonus))
        ops.head_norm_gate(o, f32(gain), eps, qs, ql, 2, H, dv, out, gate=gate, gate_col=gate_col)
        return out

    seqs, got = run_in_steps(W, steps, one_step, d * 7 + dv)
    tol = dict(atol=2e-4, rtol=1e-4) if dtype == torch.float32 else TOL16
    for r in range(2):
        h, T = seqs[r], seqs[r].shape[0]
        heads = lambda n, size: (h @ w[n].T).view(T, H, size)
        decay = torch.exp(-torch.exp(h @ w["z"].T + w0)).view(T, H, d)
        o = [P.wkv_scan(heads("r", d)[:, i], heads("k", d)[:, i], heads("v", dv)[:, i], decay[:, i], bonus[i]) for i in range(H)]
        want = P.rms(torch.stack([x[0] for x in o], 1), eps).reshape(T, inner) * gain * P.silu(h @ w["g"].T)
        torch.testing.assert_close(got[r], want, **tol)
        torch.testing.assert_close(state[(2, 0)[r]].double().cpu(), torch.stack([x[1].T for x in o]), atol=2e-4, rtol=1e-4)
    assert bool(torch.isnan(state[1]).all())        # the neighbour's slot is untouched


@gpu
@pytest.mark.parametrize("H,d,S,dv,blocks", [(3, 6, 1, None, False), (1, 33, 2, None, False), (2, 64, 1, None, True), (4, 16, 3, 10, False),
                                             (1, 128, 1, 40, False), (2, 1, 2, None, False), (1, 270, 1, 12, False), (2, 12, 1, None, True)])
def test_wkv_recurrence_in_portions_equals_the_whole(H, d, S, dv, blocks):
    check_wkv(H, d, S, PORTION_STEPS, dv=dv, blocks=blocks)


@gpu
@pytest.mark.parametrize("H,d,S,dv,blocks", [(2, 64, 1, None, True), (1, 128, 1, 48, False), (1, 270, 1, 11, False), (3, 20, 2, None, False),
                                             (2, 3, 1, 280, False)])
def test_wkv_recurrence_in_long_portions(H, d, S, dv, blocks):
    check_wkv(H, d, S, LONG_STEPS, dv=dv, blocks=blocks)


@gpu
def test_wkv_recurrence_decoding_token_by_token_and_in_bfloat16():
    check_wkv(3, 40, 2, DECODE_STEPS)
    check_wkv(2, 64, 1, DECODE_STEPS, blocks=True)
    check_wkv(2, 16, 1, PORTION_STEPS, dtype=torch.bfloat16)


# -------------------------------------------------------------------------- attention alone: chunks, mixed scores, gates


class _Group:
    def __init__(self, table):
        self.block_table = table


class _Ctx:
    """What paged_attention asks of a step, for entries laid out by hand."""

    def __init__(self, lens, ctxs, table):
        import vllm_cpp_b200.workspace  # noqa: F401
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


def attention_by_hand(nh, nkv, hd, dtype, size, chunked, ctxs, lens, *, talks=True, gated=True, make_hot=None, ps=16, seed=0, vd=None,
                      scale=0.2):
    """Entries of ``lens`` new tokens whose contexts end at ``ctxs``: random keys and values laid into pages in a scrambled
    order, pages that no new token may read left out of the block table; the engine's attention and the plain one."""
    from vllm_cpp_b200.parts.window_attention import paged_attention
    vd = vd or hd
    g = torch.Generator().manual_seed(seed + nh * 7 + hd)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    E, max_blocks = len(lens), max(-(-c // ps) for c in ctxs)
    n_pages = E * max_blocks + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((E, max_blocks), -1, dtype=torch.int32)
    keys = torch.full((n_pages, nkv, ps, hd), float("nan"), dtype=F64)
    vals = torch.full((n_pages, nkv, ps, vd), float("nan"), dtype=F64)
    talk = 0.6 * torch.eye(nh, dtype=F64) + rnd(nh, nh) * 0.8 / nh ** 0.5 if talks else None
    of = torch.arange(nh) // (nh // nkv)
    qs, wants, gates = [], [], []
    for e in range(E):
        n, first = ctxs[e], ctxs[e] - lens[e]
        q, k, v, gate = rnd(n, nh, hd), rnd(n, nkv, hd), rnd(n, nkv, vd), torch.rand(n, nh, generator=g, dtype=F64) * 1.5
        if make_hot is not None:
            make_hot(e, q, k, v, talk)
        k, v = k.to(dtype).double(), v.to(dtype).double()       # what the cache and the query buffer hold
        rows = (wide_queries(q, talk, nkv) if talks else q).to(dtype).double()
        lo = 0 if not size else (first - first % size if chunked else max(0, first - size + 1))
        for b in range(lo // ps, -(-n // ps)):
            page = order.pop()
            table[e, b] = page
            m = min(ps, n - b * ps)
            keys[page, :, :m] = k[b * ps:b * ps + m].transpose(0, 1)
            vals[page, :, :m] = v[b * ps:b * ps + m].transpose(0, 1)
        s = torch.einsum("ihgd,jgd->hij", rows, k) if talks else torch.einsum("ihd,jhd->hij", rows, k[:, of])
        mask = P.chunk_mask(n, size) if chunked else P.window_mask(n, size)
        o = torch.einsum("hij,jhe->ihe", P.masked_softmax(s * scale, mask), v[:, of])
        wants.append((o * gate[:, :, None] if gated else o)[first:])
        qs.append(rows.reshape(n, -1)[first:])
        gates.append(gate[first:])
    pages = torch.stack([keys, vals], 1) if vd == hd else torch.cat([keys.reshape(n_pages, -1), vals.reshape(n_pages, -1)], 1)
    ctx = _Ctx(lens, ctxs, table.to(dev()))
    out = torch.full((ctx.T, nh * vd), float("nan"), dtype=dtype, device=dev())
    paged_attention(ctx, _Kv(pages.to(dtype).to(dev())), torch.cat(qs).to(dtype).to(dev()), out, nh=nh, nkv=nkv, hd=hd, vd=vd, scale=scale,
                    window=size, chunked=chunked, wide=talks, out_gate=f32(torch.cat(gates)) if gated else None)
    assert int(ctx.status.item()) == 0
    return out.double().cpu().view(-1, nh, vd), torch.cat(wants)


ATTN_TOL = {torch.float32: dict(atol=3e-5, rtol=3e-5), torch.bfloat16: dict(atol=3e-2, rtol=2e-2)}
MIXED_LENS = [1, 1, 1, 7, 40, 1, 130, 2]
MIXED_CTXS = [1, 17, 700, 7, 95, 64, 200, 50]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd,size,chunked,talks,gated", [
    (4, 2, 8, 6, 10, True, True, True), (6, 3, 80, 80, 50, True, True, False), (2, 1, 64, 64, 33, True, True, True),
    (8, 4, 64, 64, 0, True, True, True), (4, 4, 128, 128, 48, True, True, True), (8, 4, 128, 128, 200, True, True, True),
    (6, 2, 128, 128, 1, True, True, True), (12, 6, 64, 64, 37, True, True, False), (10, 5, 128, 128, 90, True, True, True),
    (16, 8, 128, 128, 64, True, True, True), (11, 11, 128, 128, 70, True, True, True), (24, 24, 64, 64, 60, True, True, True),
    (4, 2, 64, 64, 50, True, False, True), (4, 2, 128, 128, 40, True, False, False), (4, 2, 64, 64, 40, False, True, True),
    (4, 2, 64, 64, 40, False, False, True), (2, 1, 300, 290, 20, False, False, True), (3, 3, 16, 16, 7, True, False, True)])
def test_attention_on_a_mixed_batch(dtype, nh, nkv, hd, vd, size, chunked, talks, gated):
    """First tokens, single tokens behind short and long contexts, portions that cross borders of pages and chunks: rows wide
    enough for each of the kernels, and for none but the plain one."""
    got, want = attention_by_hand(nh, nkv, hd, dtype, size, chunked, MIXED_CTXS, MIXED_LENS, talks=talks, gated=gated, vd=vd,
                                  scale=0.5 * hd ** -0.5)
    torch.testing.assert_close(got, want, **ATTN_TOL[dtype])


@gpu
@pytest.mark.parametrize("nh,nkv,hd", [(8, 4, 128), (32, 8, 128), (20, 5, 64), (64, 16, 64), (48, 3, 128), (14, 7, 128)])
def test_single_tokens_of_many_lengths(nh, nkv, hd):
    """One to four tiles of heads; many tokens (one slice each) and few (sliced keys, merged); contexts that end at the first
    key of a page, of a tile and of a chunk."""
    for ctxs in ([1, 2, 16, 17, 64, 65, 128, 129, 300, 301, 500, 600, 601, 899], [900], [899, 601, 640]):
        got, want = attention_by_hand(nh, nkv, hd, torch.bfloat16, 300, True, ctxs, [1] * len(ctxs), scale=0.5 * hd ** -0.5)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])
    ctxs = list(range(5, 5 + 160))          # more tokens than SMs
    got, want = attention_by_hand(nh, nkv, hd, torch.bfloat16, 0, True, ctxs, [1] * len(ctxs), scale=0.5 * hd ** -0.5)
    torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("ps", [8, 12, 32, 64])
def test_attention_on_other_page_sizes(ps):
    """Pages that the tensor cores' loaders bring in whole, and one size (12) that they do not."""
    for nkv, hd, size in ((2, 64, 45), (4, 128, 100)):
        got, want = attention_by_hand(2 * nkv, nkv, hd, torch.bfloat16, size, True, MIXED_CTXS, MIXED_LENS, ps=ps, scale=0.5 * hd ** -0.5)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("env", [{"TCGEN05_SPANS": False}, {"WIDE_DECODE": False}, {"MMA_ATTENTION": False}])
def test_portions_and_single_tokens_agree_on_every_kernel(env, monkeypatch):
    """The kernels that serve what the tcgen05 kernel and the one for single tokens do not: forced onto sizes they do take."""
    import vllm_cpp_b200.parts.window_attention as wa
    for k, v in env.items():
        monkeypatch.setattr(wa, k, v)
    for nh, nkv, hd in ((4, 2, 64), (8, 4, 128), (10, 5, 128), (16, 8, 128)):
        got, want = attention_by_hand(nh, nkv, hd, torch.bfloat16, 60, True, MIXED_CTXS, MIXED_LENS, scale=0.5 * hd ** -0.5)
        torch.testing.assert_close(got, want, **ATTN_TOL[torch.bfloat16])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd,nkv", [(16, 2), (64, 2), (128, 4)])
def test_one_key_decides_the_row(dtype, hd, nkv):
    """A key whose score stands out, placed just inside and just outside the query's chunk or window and far back among
    hundreds, in a prompt portion and behind a single token -- in a head that reads it through another head's score only."""
    nh = 2 * nkv
    for chunked in (True, False):
        size, length = 70, 300          # the last query, 299, lies in the chunk [280, 350), or sees keys from 230 on
        edge = 280 if chunked else 230
        for n_new in (1, 60):
            for at, window in ((299, size), (edge, size), (edge - 1, size), (3, size), (3, 0)):
                def hot(e, q, k, v, talk, at=at):
                    # head 0's own score with the key is nothing; it reads head nh - 1's, whose keys are the last KV head's
                    talk.zero_()
                    talk.fill_diagonal_(0.3)
                    talk[0] = 0.0
                    talk[0, nh - 1] = 1.0
                    q *= 0.05
                    q[-1, 0] = 0.0
                    q[-1, nh - 1] = torch.ones(hd, dtype=F64)
                    k[at, nkv - 1] = 400.0 / hd
                    v[at, 0] = 5.0
                got, want = attention_by_hand(nh, nkv, hd, dtype, window, chunked, [length], [n_new], make_hot=hot, gated=False)
                torch.testing.assert_close(got, want, **ATTN_TOL[dtype])
                seen = at >= edge or window == 0
                assert (abs(float(want[-1, 0, 0]) - 5.0) < 0.5) == seen, (chunked, at, want[-1, 0, 0])


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
def test_replay(name, dtype, mode, nufetar_dirs, oracle, tmp_path):
    """Whole prompts; the last 32 tokens one by one; portions of changing size down to two tokens; up to four live
    requests with pages and slots used again -- the last two also as serving asks (logits of an entry's last token
    only: captured steps), all over a NaN-filled cache."""
    requests = requests_of(name)
    trace = MODES[mode](requests)
    out = R.run_trace(nufetar_dirs[name], dtype, trace, tmp_path / "out", configs()[name][1], extra_args=["--poison"])
    worst = compare(name, dtype, trace, out, requests, oracle)
    print(f"{name} {dtype} {mode}: worst relative error {worst:.3e}, pool {trace.max_tokens} tokens, {len(trace.steps)} steps")


@gpu
def test_replay_modes_agree_with_each_other(nufetar_dirs, tmp_path):
    """Cutting and batching change the logits by rounding only."""
    for name in ("A", "B"):
        requests = requests_of(name)
        vocab = configs()[name][0].vocab
        rows = {}
        for mode in ("whole", "mixed"):
            trace = MODES[mode](requests)
            out = R.run_trace(nufetar_dirs[name], "float32", trace, tmp_path / (name + mode), configs()[name][1])
            for step, want in enumerate(trace.wanted):
                got = R.read_step(out, step, vocab)
                for i, key in enumerate(want):
                    rows.setdefault(key, {})[mode] = got[i]
        worst = max(np.abs(v["whole"] - v[m]).max() / np.abs(v["whole"]).max() for v in rows.values() for m in ("mixed",))
        assert worst < 2e-5, (name, worst)


@gpu
def test_long_decoding(nufetar_dirs, oracle, tmp_path):
    """A short prompt, then 250 tokens one by one: the states carried through 250 steps, windows and chunks passing over
    decoded tokens and pages' borders, pages given back as they pass."""
    for name, dtype in (("A", "float32"), ("B", "float32"), ("D", "bfloat16")):
        toks = random_tokens(configs()[name][0].vocab, 260, 99)
        trace = R.tail_one_by_one({"long": toks}, tail=250)
        out = R.run_trace(nufetar_dirs[name], dtype, trace, tmp_path / name, configs()[name][1], extra_args=["--poison"])
        compare(name, dtype, trace, out, {"long": toks}, oracle)


# -------------------------------------------------------------------------- generation through the engine's entry point


@gpu
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(name, nufetar_dirs):
    """Several prompts at once through LLM.generate (scheduler, portions under a small token budget, captured decoding
    steps, device-side sampling at temperature 0) against the plain implementation's greedy continuation."""
    from vllm_cpp_b200 import LLM
    cfg, w = P.read_model(nufetar_dirs[name])
    vocab, page = configs()[name][0].vocab, configs()[name][1]
    prompts = [random_tokens(vocab, n, 3 + n) for n in (5, 41, 18, 70, 2)]
    llm = LLM(str(nufetar_dirs[name]), dtype="float32", page_size=page, max_tokens=page * 64, max_num_seqs=3, max_step_tokens=32,
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
