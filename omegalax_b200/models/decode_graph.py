"""Single-token steps as recorded CUDA graphs.

A decode step launches a few small kernels per layer, so its time is launch overhead unless it is
recorded once and replayed.  A step's shapes depend on the cache only (one row per sequence, idle rows
marked), so the recording lives on the cache: the first single-token step runs eagerly, the second one
records, later ones copy their token batch into the recorded buffers and replay.
"""
from __future__ import annotations

import os

import torch

from ..ops import kernels as K


class DecodeGraph:
    def __init__(self, model, cache, batch):
        self.batch = batch            # the recorded step reads these tensors
        before = K.launch_count()
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph):
            self.out = model.run_layers(batch, cache)
        self.launches = K.launch_count() - before
        self.model = model

    @staticmethod
    def enabled() -> bool:
        return os.environ.get("OMEGALAX_B200_DECODE_GRAPH", "1") == "1"

    @staticmethod
    def step(model, cache, batch):
        """fp32 residual rows of a single-token batch; the tensor is reused by the next step."""
        state = cache.decode_graph
        if not DecodeGraph.enabled():
            return model.run_layers(batch, cache)
        if state is None or state[0] is not model:
            cache.decode_graph = (model, None)
            return model.run_layers(batch, cache)
        graph = state[1]
        if graph is None:
            graph = DecodeGraph(model, cache, batch)
            cache.decode_graph = (model, graph)
        else:
            graph.batch.flat.copy_(batch.flat)
            K.add_launches(graph.launches)
        graph.graph.replay()
        return graph.out
