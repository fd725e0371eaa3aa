"""torchrun worker of the layered multi-rank tests: rank 0 drives, the others follow."""
import random
import sys

import torch
import torch.distributed as dist

import xfastertransformer_b200 as xft

path, out = sys.argv[1], sys.argv[2]
model = xft.AutoModel.from_pretrained(path, dtype="fp32")
m = model.model
r = random.Random(8)
V = m.cfg.vocab_size
prompts = [[r.randrange(V) for _ in range(50)], [r.randrange(V) for _ in range(21)]]
if model.rank == 0:
    sid = model.set_input_cb(prompts, None, 64, rows=[[3, 49], [20]])
    rows = model.forward_cb()
    model.free_seqs(sid)
    tokens = model.generate(torch.tensor(prompts[:1]), max_length=60)
else:
    model.set_input_cb()
    model.forward_cb()
    model.free_seqs()
    model.generate()
heads = [None] * dist.get_world_size()
dist.all_gather_object(heads, [L.hq for L in m.decoder.layers][:2])
if model.rank == 0:
    torch.save({"rows": rows, "tokens": tokens, "prompts": prompts, "heads": heads}, out)
m._closed = True
dist.barrier()
dist.destroy_process_group()
