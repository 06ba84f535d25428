"""Helpers of the architecture tests: device tensors from numpy, row errors, random page assignments, checkpoints on disk, and
replaying schedules of prompt portions and single tokens through an engine."""
import json

import numpy as np
import torch


def dev_t(a, dev, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).to(dev).to(dtype)


def dev_i(a, dev, dtype=torch.int32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dev).to(dtype)


def f32r(x):
    return np.asarray(x, np.float32).astype(np.float64)


def npf(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def rel_err(got, ref):
    """Per row: rms of the centred difference over the rms of the centred reference."""
    d = np.asarray(got, np.float64) - ref
    d = d - d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((r ** 2).mean(-1))


def paged(rng, ctxs, bs, spare=3):
    """Random page assignment: tables [seqs, cap], the cache slot of every (sequence, position), rows of the cache."""
    need = [(c + bs - 1) // bs for c in ctxs]
    perm = rng.permutation(sum(need) + spare)
    tables = -np.ones((len(ctxs), max(need) + 1), np.int32)
    k = 0
    for s, nb in enumerate(need):
        tables[s, :nb] = perm[k:k + nb]; k += nb
    return tables, (lambda s, p: int(tables[s, p // bs]) * bs + p % bs), (sum(need) + spare) * bs


def write_checkpoint(path, cfg, w, to_bits):
    from nano_vllm_rs_b200.loader import write_safetensors
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(path / "model.safetensors"), {k: to_bits(v) for k, v in w.items()})
    return str(path)


def engine_on(model_dir, dtype, bs=16, blocks=24, max_seqs=4, eager=1):
    from nano_vllm_rs_b200.engine import LLMEngine
    return LLMEngine.from_pretrained(model_dir, dtype=dtype, kvcache_block_size=bs, num_kvcache_blocks=blocks, max_num_seqs=max_seqs,
                                     max_num_batched_tokens=blocks * bs, max_model_len=blocks * bs, enforce_eager=eager)


def replay(eng, requests, schedule):
    """schedule: list of steps, each a list of (request index, token count).  Returns every position's logits per request."""
    from nano_vllm_rs_b200.engine import SamplingParams
    sp = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)
    sid, at, out = {}, {}, {i: [] for i in range(len(requests))}
    for step in schedule:
        ids, counts = [], []
        for i, c in step:
            toks = requests[i][at.get(i, 0):at.get(i, 0) + c]
            if i in sid:
                eng.scheduler.extend_sequence(sid[i], toks)
            else:
                sid[i] = eng.scheduler.add_sequence(toks, sp)
            ids.append(sid[i]); counts.append(c)
        lg = eng.step_chunks(ids, counts, list(range(sum(counts))))
        k = 0
        for i, c in step:
            out[i].append(lg[k:k + c]); k += c
            at[i] = at.get(i, 0) + c
            if at[i] == len(requests[i]):
                eng.scheduler.finish_sequence(sid[i]); eng.scheduler.release_sequence(sid[i])
                del sid[i]
    return {i: np.concatenate(v) for i, v in out.items() if v}


def cut(n, sizes):
    out, k = [], 0
    while n > 0:
        c = min(n, sizes[k % len(sizes)]); out.append(c); n -= c; k += 1
    return out
