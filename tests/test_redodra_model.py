"""Sandwich layer-by-layer decoders through the registry, the engine, its cache and its scheduler, against the plain
statement of the whole model in redodra_oracle.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import redodra_oracle as O  # noqa: E402

from nkipy_b200.models import config as C  # noqa: E402
from nkipy_b200.models import registry, runner  # noqa: E402
from nkipy_b200.models.engine import GenerationEngine, Sampling, StepEntry  # noqa: E402
from nkipy_b200.models.hybrid import HybridLM  # noqa: E402
from nkipy_b200.models.kv_cache import KVLayer, StateLayer  # noqa: E402
from nkipy_b200.models.weights import hybrid_random_weights, hybrid_weight_shapes  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
on_devices = pytest.mark.parametrize("device", DEVICES)
in_dtypes = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
TOL = {torch.float32: 1e-4, torch.bfloat16: 8e-2}


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


# name -> small_config arguments; sizes, orders and branches differ between them
MODELS = {
    "mixed": dict(),
    "attention-first": dict(layers="akpd", mlps="dd-d", width=128, heads=6, kv_heads=2, dim=64, vdim=64, rot=64, lheads=3, lkv=3,
                            ldim=64, lvdim=40, window=7, first=2, rheads=2, groups=1, state=128, rvdim=64, rconv=2, parts=1,
                            dheads=2, dkv=1, ddim=64, dvdim=128, dconv=4),
    "no-ff": dict(layers="dD", mlps="--", width=64, dheads=3, dkv=3, ddim=24, dvdim=20, dconv=1, vocab=96),
    "parallel-only": dict(layers="pp", mlps="d-", lheads=4, lkv=1, ldim=32, lvdim=72, window=33, first=40, rheads=4, groups=4, state=40,
                          rvdim=8, rconv=5, parts=4, eps=1e-3),
    "wide-heads": dict(layers="apd", mlps="-dd", heads=2, kv_heads=1, dim=136, vdim=144, rot=96, lheads=2, lkv=1, ldim=160, lvdim=20,
                       window=40, first=1, rheads=3, groups=1, state=136, rvdim=136, parts=3, dheads=2, dkv=2, ddim=136, dvdim=24),
    "one-token": dict(layers="pad", mlps="ddd", window=1, first=0, heads=6, kv_heads=3, dim=16, vdim=24, rot=2, parts=6, cap=2.0,
                      lcap=1.5),
    "odd": dict(layers="dapk", mlps="dd-d", width=54, heads=2, kv_heads=1, dim=7, vdim=11, rot=6, dheads=3, dkv=1, ddim=5, dvdim=7,
                lheads=3, lkv=1, ldim=9, lvdim=5, window=9, first=3, rheads=3, groups=1, state=7, rvdim=3, rconv=3, parts=3, ff=33,
                vocab=61),
    "many-heads": dict(layers="ap", mlps="dd", heads=34, kv_heads=2, dim=8, vdim=8, rot=8, lheads=34, lkv=1, ldim=8, lvdim=8,
                       window=40, first=4, rheads=32, groups=2, state=8, rvdim=4, parts=2),
}


class Case:
    def __init__(self, name, device, dtype, max_batch=3, blocks=16, seed=1, graph=None, sharing=True, **changes):
        self.raw = O.small_config(**{**MODELS[name], **changes})
        self.cfg = registry.architecture_of(self.raw).config(self.raw)
        self.weights = O.small_weights(self.raw, hybrid_weight_shapes(self.cfg), seed)
        self.device, self.dtype = device, dtype
        self.model = HybridLM(self.cfg, self.weights, device=device, dtype=dtype)
        self.engine = GenerationEngine(self.model, max_batch=max_batch, max_seq_len=32 * blocks, num_blocks=blocks,
                                       use_cuda_graph=graph, enable_prefix_sharing=sharing)

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def want(self, ids):
        return O.forward(self.raw, self.weights, ids)[0]

    def feed(self, ids, cuts):
        """Logits at every position of ids, brought in portions."""
        seq = self.engine.open_request()
        out, lo = [], 0
        for n in cuts:
            out.append(self.engine.run_step([StepEntry(seq, ids[lo:lo + n], range(n))]))
            lo += n
        assert lo == len(ids)
        self.engine.release([seq])
        return torch.cat(out)

    def close(self, got, want, what=""):
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = (d.pow(2).mean(-1).sqrt() / want.std())
        worst = err.max().item()
        assert worst < TOL[self.dtype], f"{what}: error {worst} of the logits' spread"


@on_devices
@in_dtypes
@pytest.mark.parametrize("name", MODELS)
def test_whole_prompts_portions_and_single_tokens(name, device, dtype):
    c = Case(name, device, dtype)
    n = 75
    ids = c.tokens(n, 3)
    want = c.want(ids)
    c.close(c.feed(ids, [n]), want, "whole")
    c.close(c.feed(ids, [2, 2, 31, 1, 1, 28, 10]), want, "portions")
    c.close(c.feed(ids, [40] + [1] * 35), want, "prompt, then single tokens")
    if name in ("mixed", "attention-first"):
        c.close(c.feed(ids, [1] * n), want, "single tokens")
        c.close(c.feed(ids, [2] * 37 + [1]), want, "portions of two")


@on_devices
@pytest.mark.parametrize("name", ["mixed", "attention-first", "no-ff", "odd", "wide-heads"])
def test_residual_after_every_layer(name, device):
    c = Case(name, device, torch.float32)
    ids = c.tokens(21, 5)
    taps = O.forward(c.raw, c.weights, ids)[1]
    s = c.engine.cache.add_sequence(ids)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    _, got = c.model.prefill(t(ids), t(list(range(21))), c.engine.cache.slots_for(s, 0, 21).to(device), c.engine.cache,
                             c.engine.cache.block_table[s.slot:s.slot + 1], t([0]), t([21]), t([21]), 21,
                             return_hidden=True, rows=t([s.slot]))
    assert len(got) == len(taps) == len(c.raw["layers"])
    for i, (a, b) in enumerate(zip(got, taps)):
        assert ((a.double().cpu() - b).abs().max() / b.abs().max()) < 1e-5, f"layer {i}"


@on_devices
@in_dtypes
@pytest.mark.parametrize("name,window,first", [("mixed", 64, 3), ("mixed", 130, 131), ("attention-first", 200, 64), ("wide-heads", 70, 129)])
def test_long_prompt_and_long_decoding(name, device, dtype, window, first):
    """Hundreds of tokens: attention tiles, pages, windows and kept tokens end inside and between portions."""
    c = Case(name, device, dtype, window=window, first=first)
    n = 420
    ids = c.tokens(n, 8)
    want = c.want(ids)
    c.close(c.feed(ids, [n]), want, "whole")
    c.close(c.feed(ids, [127, 2, 126, 1, 33, 31, 100]), want, "portions")
    c.close(c.feed(ids, [130, 290]), want, "large portions")
    c.close(c.feed(ids, [250] + [1] * 170), want, "long decoding")


@on_devices
@in_dtypes
@pytest.mark.parametrize("size", [1, 2, 31, 32, 33])
def test_edges_of_the_window_and_of_the_kept_tokens_in_the_whole_model(device, dtype, size):
    """Scores of a size at which a window, or the number of kept first tokens, that is one off changes most logits."""
    sharp = dict(window=size, first=4, lscale=1.0, lcap=30.0)
    c = Case("attention-first", device, dtype, **sharp)
    ids = c.tokens(70, 11)
    want = c.want(ids)
    for key in ("window", "first"):
        other = O.small_config(**{**MODELS["attention-first"], **sharp, key: sharp[key] + 1})
        off = O.forward(other, c.weights, ids)[0]
        assert ((off - want)[size + 6:].pow(2).mean(-1).sqrt() / want.std()).median() > 3 * TOL[torch.float32]
    c.close(c.feed(ids, [70]), want, "whole")
    c.close(c.feed(ids, [2, size, 68 - size]), want, "portions")
    c.close(c.feed(ids, [1] * 70), want, "single tokens")


@on_devices
@in_dtypes
def test_unequal_requests_in_one_batch_match_each_alone(device, dtype):
    c = Case("mixed", device, dtype, max_batch=4, blocks=24)
    lens = [210, 3, 64, 41]
    ids = [c.tokens(n, 20 + i) for i, n in enumerate(lens)]
    want = [c.want(x) for x in ids]
    # portions of some beside single tokens of others; requests pause and go on; steps of more and of less than 128 tokens
    plan = [{0: 60, 1: 1}, {0: 1, 1: 1, 2: 33}, {2: 1, 3: 2}, {0: 1, 2: 1, 3: 1}, {1: 1}, {0: 120, 2: 20, 3: 1},
            {0: 1, 3: 1}, {0: 27, 2: 9, 3: 36}]
    at, seqs = {}, {}
    got = {i: [] for i in range(4)}
    for step in plan:
        entries = []
        for i, k in step.items():
            if i not in seqs:
                seqs[i] = c.engine.open_request()
            lo = at.get(i, 0)
            entries.append(StepEntry(seqs[i], ids[i][lo:lo + k], range(k)))
            at[i] = lo + k
        out = c.engine.run_step(entries)
        o = 0
        for i, k in step.items():
            got[i].append(out[o:o + k])
            o += k
    for i in range(4):
        assert at[i] == lens[i]
        c.close(torch.cat(got[i]), want[i], f"request {i}")
    c.engine.release(list(seqs.values()))


@on_devices
@in_dtypes
def test_freed_blocks_and_rows_are_used_again(device, dtype):
    """A pool that holds one and a half requests: every request after the first runs on recycled blocks and rows."""
    c = Case("attention-first", device, dtype, max_batch=2, blocks=6)
    for r in range(4):
        a, b = c.tokens(70 + 11 * r, 30 + r), c.tokens(40 + r, 60 + r)
        sa, sb = c.engine.open_request(), c.engine.open_request()
        la = c.engine.run_step([StepEntry(sa, a[:50], range(50)), StepEntry(sb, b[:-5], [0])])
        c.close(la[:50], c.want(a)[:50], f"turn {r}")
        outs = []
        for t in range(5):
            lo = len(b) - 5 + t
            outs.append(c.engine.run_step([StepEntry(sb, b[lo:lo + 1], [0]), StepEntry(sa, a[50 + t:51 + t], [])]))
        c.close(torch.cat(outs), c.want(b)[-5:], f"turn {r} decoded")
        c.engine.release([sb])
        c.close(c.engine.run_step([StepEntry(sa, a[55:], [len(a) - 56])]), c.want(a)[-1:], f"turn {r} rest")
        c.engine.release([sa])
    assert c.engine.cache.allocator.num_free() == 6


@on_devices
def test_nothing_of_what_blocks_and_slots_held_is_seen(device):
    """Short prompts on blocks and slots whose former tokens left large keys, values, states and convolution inputs."""
    c = Case("mixed", device, torch.float32, max_batch=1, blocks=4)
    c.feed(c.tokens(90, 1), [90])
    for t in (*c.engine.cache.k, *c.engine.cache.v, *c.engine.cache.state):
        if t is not None:
            t.mul_(100.0)
    for n, cuts in ((1, [1]), (2, [2]), (2, [1, 1]), (5, [1, 2, 2]), (40, [33, 7])):
        ids = c.tokens(n, 40 + n)
        c.close(c.feed(ids, cuts), c.want(ids), f"{cuts}")


def test_cache_entries_of_every_kind_of_layer():
    c = Case("mixed", "cpu", torch.float32)
    delta = [StateLayer((4, 24, 16)), StateLayer((3, 2 * 2 * 16 + 4 * 24))]
    parallel = [KVLayer(2, 20, 28), StateLayer((6, 20, 12)), StateLayer((4, 6 * 20 + 2 * 3 * 12))]
    assert c.engine.cache.layers == [*delta, *parallel, KVLayer(2, 24, 40), *parallel]
    assert c.model.entry == [0, 2, 5, 5, 6]              # the fourth layer reads the third one's keys and values
    assert not c.engine.cache.allocator.enable_prefix_sharing


# --------------------------------------------------------------------------- generation, loading, command lines
def greedy_oracle(c, ids, n):
    ids, margins = list(ids), []
    for _ in range(n):
        last = c.want(ids)[-1]
        top = last.topk(2).values
        margins.append(((top[0] - top[1]) / last.std()).item())
        ids.append(int(last.argmax()))
    return ids[-n:], margins


def agrees(got, want, margins, tol):
    for g, w, m in zip(got, want, margins):
        if g != w:
            assert m < tol, f"token {g} instead of {w} at a margin of {m}"
            return                                  # a near tie: the continuations differ from here on


@on_devices
@in_dtypes
@pytest.mark.parametrize("budget", [4096, 16])
def test_greedy_generation_through_the_scheduler(device, dtype, budget):
    c = Case("mixed", device, dtype, max_batch=3, blocks=12)
    c.engine.prefill_chunk_tokens = budget          # 16: every prompt runs in portions
    prompts = [c.tokens(n, 70 + n) for n in (45, 7, 1)]
    for _ in range(2):                              # the second time on recycled rows
        outs = c.engine.generate(prompts, 9)
        for p, o in zip(prompts, outs):
            agrees(o, *greedy_oracle(c, p, 9), 4 * TOL[dtype])
    assert not c.engine.active and c.engine.cache.allocator.num_free() == 12


@on_devices
def test_sampling_follows_the_logits(device):
    c = Case("attention-first", device, torch.float32, max_batch=2, blocks=8)
    prompts = [c.tokens(12, 1), c.tokens(30, 2)]
    greedy = c.engine.generate(prompts, 6)
    assert c.engine.generate(prompts, 6, sampling=Sampling(1.0, top_k=1)) == greedy
    a = c.engine.generate(prompts, 12, sampling=Sampling(300.0, seed=1))
    assert a != c.engine.generate(prompts, 12, sampling=Sampling(300.0, seed=2))


def write_model(folder, name="mixed", seed=4):
    from safetensors.torch import save_file

    raw = O.small_config(**MODELS[name])
    cfg = registry.architecture_of(raw).config(raw)
    w = O.small_weights(raw, hybrid_weight_shapes(cfg), seed)
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(raw))
    save_file(w, str(folder / "model.safetensors"))
    return raw, w


@on_devices
@pytest.mark.parametrize("name", ["mixed", "no-ff"])
def test_model_folder_loads_by_its_architecture(device, tmp_path, name):
    raw, w = write_model(tmp_path / "m", name)
    model = registry.load_model(str(tmp_path / "m"), device=device, dtype=torch.float32)
    assert isinstance(model, HybridLM)
    assert model.cfg.param_count() == sum(t.numel() for t in w.values())
    eng = GenerationEngine(model, max_batch=1, max_seq_len=64)
    ids = list(range(40))
    got = eng.run_step([StepEntry(eng.open_request(), ids, range(40))])
    want = O.forward(raw, w, ids)[0]
    assert ((got.double().cpu() - want).abs().max() / want.std()) < 1e-3


def test_config_reader():
    raw = O.small_config()
    cfg = registry.architecture_of(raw).config(raw)
    delta, parallel, full, shared, last = cfg.layers
    assert {l.block for l in cfg.layers} == {"sandwich"} and [l.ff for l in cfg.layers] == [104, 104, 0, 104, 104]
    assert delta.mixer == C.DeltaSpec(4, 2, 16, 24, 3)
    assert parallel.mixer.left == C.GroupedAttentionSpec(6, 2, 20, 28, 1.5 * 20 ** -0.5, 7.0, None, 19, 5, distance=True, bias=True)
    assert parallel.mixer.right == C.StateSpaceSpec(6, 3, 12, 20, 4, 2) and last.mixer == parallel.mixer
    assert full.mixer == C.GroupedAttentionSpec(4, 2, 24, 40, 1.5 * 24 ** -0.5, 9.0, C.RopeSpec(900.0, 16), sink=True, gate=True)
    assert shared.mixer.kv_from == 2
    assert cfg.tanh_norm and cfg.depth_average and not cfg.tie_embeddings and (cfg.rms_eps, cfg.vocab_size) == (1e-4, 150)
    uncapped = json.loads(json.dumps(raw))
    del uncapped["layers"][2]["mixer"]["softcap"]
    assert registry.architecture_of(raw).config(uncapped).layers[2].mixer.softcap == 0.0
    for change in (lambda r: r["layers"][0].update(type="other"),
                   lambda r: r["layers"][0].update(mlp={"kind": "other", "ff": 8}),
                   lambda r: r["layers"][3]["mixer"].update(kv_from=0),
                   lambda r: r["layers"][2]["mixer"].update(kv_from=3)):
        bad = json.loads(json.dumps(raw))
        change(bad)
        with pytest.raises(ValueError):
            registry.architecture_of(bad).config(bad)


@on_devices
def test_regular_shapes_and_random_weights_run(device):
    cfg = C.redodra_shape(128, layers=11, heads=4, kv_heads=2, ff=256, vocab=300, dim=32, window=40, state=16, groups=2, share_every=2)
    assert registry.for_config(cfg) is registry.ARCHITECTURES["Redodra"]
    assert [l.mixer.kind for l in cfg.layers[:5]] == ["delta", "blend", "delta", "blend", "grouped"]
    assert [cfg.layers[i].mixer.kv_from for i in (4, 9)] == [None, 4]
    cfg = runner.shrink(cfg) if device == "cpu" else cfg
    assert cfg.name == "redodra"
    model = HybridLM(cfg, hybrid_random_weights(cfg, device=device), device=device)
    out = GenerationEngine(model, max_batch=2, max_seq_len=128).generate([list(range(50)), [1, 2, 3]], 5)
    assert [len(o) for o in out] == [5, 5]


@on_devices
def test_trace_command_replays_steps(device, tmp_path):
    raw, w = write_model(tmp_path / "m", "attention-first")
    out = tmp_path / "out"
    out.mkdir()
    g = torch.Generator().manual_seed(5)
    a, b = (torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for n in (50, 9))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:45], "want": [3, 44]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:4], "want": []}, {"id": "a", "tokens": a[45:46], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:5], "want": [0]}, {"id": "a", "tokens": a[46:47], "want": [0]}],
              "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[5:], "want": [3]}, {"id": "a", "tokens": a[:20], "want": [19]}],
              "end": ["a", "b"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                          "--out", str(out), "--max-tokens", "128", "--device", device],
                         input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=900)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = O.forward(raw, w, a)[0], O.forward(raw, w, b)[0]
    for n, want in ((0, wa[[3, 44]]), (2, torch.stack([wb[4], wa[46]])), (3, torch.stack([wb[8], wa[19]]))):
        got = torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, raw["vocab"])
        assert ((got.double() - want).abs().max() / want.std()) < 1e-3


@on_devices
def test_generation_command_line(device, tmp_path):
    write_model(tmp_path / "m")
    env = dict(os.environ, PYTHONPATH=ROOT)
    if device == "cpu":
        env["CUDA_VISIBLE_DEVICES"] = ""
    cmd = [sys.executable, "-m", "nkipy_b200.models.runner", "--model", str(tmp_path / "m"), "--batch", "2",
           "--prompt-len", "12", "-n", "4", "--max-seq-len", "96", "--dtype", "float32", "--temperature", "0.8", "--top-k", "5"]
    res = subprocess.run(cmd, capture_output=True, text=True, timeout=600, env=env, cwd=ROOT)
    assert res.returncode == 0 and "Decode tokens/sec" in res.stdout, res.stderr[-2000:]
