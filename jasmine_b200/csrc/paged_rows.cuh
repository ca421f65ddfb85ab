// Host bookkeeping of a paged cache shared by the active batch rows of a model: pages are handed out on demand from one
// pool, the active sequences occupy the rows 0 .. n_active-1, and a retiring row is refilled with the last one (its
// block-table row moves, its pages stay where they are).  The device holds only the block table; the host is the
// authority on context lengths and free pages.
#pragma once
#include "common.cuh"
#include <utility>
#include <vector>

namespace jsm {

struct PagedRows {
    int n_pool_pages = 0, pages_per_row = 0, max_context = 0, n_active = 0;
    int32_t* block_table = nullptr;  // device, [rows][pages_per_row]
    std::vector<int32_t> free_pages;
    std::vector<std::vector<int32_t>> row_pages;  // page of every 64 positions of a row; -1: given back (release_before)
    std::vector<int32_t> h_ctx;                   // cached positions per row

    void init(int rows, int pool_pages, int per_row, int context, int32_t* d_block_table) {
        n_pool_pages = pool_pages; pages_per_row = per_row; max_context = context; block_table = d_block_table;
        free_pages.clear();
        for (int p = pool_pages - 1; p >= 0; --p) free_pages.push_back(p);  // page 0 is handed out first
        row_pages.assign(rows, {});
        h_ctx.assign(rows, 0);
        n_active = 0;
    }
    // pages for `positions` cached positions of row `row`; uploads the part of the row's block table that changed
    jsm_status provision(int row, int positions, cudaStream_t st) {
        std::vector<int32_t>& pages = row_pages[row];
        const int have = (int)pages.size(), need = (positions + JSM_PAGE_SIZE - 1) / JSM_PAGE_SIZE;
        if (need <= have) return JSM_OK;
        if (need > pages_per_row) JSM_FAIL(JSM_SHAPE, "context overflow: %d positions, the model was created for %d", positions, max_context);
        if (need - have > (int)free_pages.size())
            JSM_FAIL(JSM_OOM, "page pool exhausted: %d pages needed, %zu free of %d", need - have, free_pages.size(), n_pool_pages);
        for (int i = have; i < need; ++i) {
            pages.push_back(free_pages.back());
            free_pages.pop_back();
        }
        JSM_CUDA_CHECK(cudaMemcpyAsync(block_table + (size_t)row * pages_per_row + have, pages.data() + have, sizeof(int32_t) * (need - have),
                                       cudaMemcpyHostToDevice, st));
        JSM_CUDA_CHECK(cudaStreamSynchronize(st));  // the host vector may be reallocated by the next call
        return JSM_OK;
    }
    // gives back the pages of `row` that lie wholly before `position` (no later token of the row reads them; the block
    // table keeps their stale entries)
    void release_before(int row, int position) {
        std::vector<int32_t>& pages = row_pages[row];
        for (int i = position / JSM_PAGE_SIZE - 1; i >= 0 && i < (int)pages.size() && pages[i] >= 0; --i) {
            free_pages.push_back(pages[i]);
            pages[i] = -1;
        }
    }
    // returns the row's pages to the pool; the last active row then takes its place (*moved_from, or -1)
    jsm_status retire(int row, int* moved_from, int32_t* d_ctx, cudaStream_t st) {
        for (int32_t p : row_pages[row])
            if (p >= 0) free_pages.push_back(p);
        row_pages[row].clear();
        const int last = n_active - 1;
        if (moved_from) *moved_from = -1;
        if (row != last) {
            // the last active row takes the freed place: its block-table row and context length move, its pages do not
            row_pages[row] = std::move(row_pages[last]);
            row_pages[last].clear();
            h_ctx[row] = h_ctx[last];
            JSM_CUDA_CHECK(cudaMemcpyAsync(block_table + (size_t)row * pages_per_row, row_pages[row].data(),
                                           sizeof(int32_t) * row_pages[row].size(), cudaMemcpyHostToDevice, st));
            if (d_ctx) JSM_CUDA_CHECK(cudaMemcpyAsync(d_ctx + row, &h_ctx[row], sizeof(int32_t), cudaMemcpyHostToDevice, st));
            JSM_CUDA_CHECK(cudaStreamSynchronize(st));
            if (moved_from) *moved_from = last;
        }
        h_ctx[last] = 0;
        n_active = last;
        return JSM_OK;
    }
};

}  // namespace jsm
